"""Mechanisms of the Fubelorn decoder one by one against the plain restatement: streams with the convolution ahead of a sublayer, the three
recurrences in portions of any size, attention with kept positions and pooled blocks in its three forms, norms and rotations around it."""
import math
import random

import pytest
import torch

import fubelorn_oracle as O

BF16, F32, F64 = torch.bfloat16, torch.float32, torch.float64
gpu = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def _rel(got, want):
    d = (got.double().cpu() - want.double().cpu()).abs()
    return float(d.max() / want.double().abs().max())


def _lim(dtype, f32=5e-6, bf16=2e-2):
    return f32 if dtype == F32 else bf16


def _pad(n):
    return (n + 7) // 8 * 8


def batches(rnd, lens, sizes, most=4):
    """Steps of (sequence, first, count): up to ``most`` sequences live, some left out, slots used again. Yields also the slots."""
    waiting, live, free = list(lens), {}, list(range(most))
    while waiting or live:
        while waiting and free:
            live[waiting.pop(0)] = [free.pop(rnd.randrange(len(free))), 0]
        step = []
        for k in list(live):
            if rnd.random() < 0.2:
                continue
            slot, at = live[k]
            c = min(lens[k] - at, rnd.choice(sizes))
            step.append((k, slot, at, c))
            live[k][1] += c
            if live[k][1] == lens[k]:
                free.append(slot)
                del live[k]
        if step:
            yield step


# ---------------------------------------------------------------------------------------------------------------------------
# CPU
# ---------------------------------------------------------------------------------------------------------------------------
def test_stretched_frequencies():
    from ironpangu_b200.ops.linear_attn import RotaryScaling, rotary_frequencies

    for dims, base, (factor, low, high, ctx) in ((64, 5e5, (8.0, 1.0, 4.0, 8192)), (10, 1e4, (3.0, 0.5, 2.0, 50)), (2, 1e4, (2.0, 1.0, 2.0, 3)), (128, 1e3, (32.0, 1.0, 4.0, 128))):
        want = O.frequencies(dims, base, {"factor": factor, "low": low, "high": high, "original": ctx})
        got = rotary_frequencies(dims, base, "cpu", RotaryScaling(factor, low, high, ctx))
        assert torch.allclose(got, want, rtol=1e-13, atol=0)
        assert torch.allclose(rotary_frequencies(dims, base, "cpu"), O.frequencies(dims, base, None), rtol=1e-13, atol=0)
    f, plain = O.frequencies(128, 5e5, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}), O.frequencies(128, 5e5, None)
    assert torch.equal(f[:20], plain[:20]) and torch.allclose(f[-20:], plain[-20:] / 8) and ((f < plain) & (f > plain / 8)).sum() > 3
    for bad in (RotaryScaling(0.0, 1.0, 4.0, 64), RotaryScaling(2.0, 4.0, 4.0, 64), RotaryScaling(2.0, 1.0, 4.0, 0)):
        with pytest.raises(ValueError):
            bad.check()


def test_entries_ahead_of_a_window():
    """How many kept positions and blocks a query counts, and that no block's entry shares its place in a page with another."""
    from ironpangu_b200.ops.window_attn import Ahead, GroupedShape

    n = 400
    for size, keep, pool in ((7, 3, 0), (1, 40, 0), (64, 64, 0), (12, 0, 1), (12, 0, 5), (40, 0, 16), (3, 0, 33)):
        a, d = Ahead(keep, pool), O._distance(n)
        if keep:
            want = ((torch.arange(n)[None] < keep) & (d >= size)).sum(1)
        else:
            want = O.block_seen(n, size, pool).sum(1)
        assert [a.count(max(0, i - size + 1)) for i in range(n)] == want.tolist()
    for pt in (16, 8):
        for pool in (1, 2, 3, 5, 7, 8, 15, 16, 17, 40):
            room = GroupedShape(1, 1, 8, 8, 1.0, 4, pool=pool).entries(pt)
            ends = [b * pool + pool - 1 for b in range(200)]
            places = [(e // pt, b - e // pt * pt // pool) for b, e in enumerate(ends)]
            assert len(set(places)) == 200 and all(0 <= r < room for _, r in places)


# ---------------------------------------------------------------------------------------------------------------------------
# streams
# ---------------------------------------------------------------------------------------------------------------------------
@gpu
@DTYPES
@pytest.mark.parametrize("S,taps,width", [(1, 1, 20), (2, 4, 64), (3, 2, 53), (4, 3, 136), (5, 7, 24), (2, 0, 40), (16, 16, 8), (1, 4, 1000)])
def test_streams_and_convolution(dtype, S, taps, width):
    """The end of a sublayer and the front of the next over steps of several sequences: the restatement over whole sequences."""
    from ironpangu_b200.ops import hyper_streams as HS

    g = torch.Generator().manual_seed(width + S)
    rn = lambda *s: torch.randn(s, generator=g)
    W = {"hc1.mix": rn(S, S), "hc1.in": rn(S), "hc1.out": rn(S), "norm1": rn(), "canon1": rn(width, taps)}
    a = HS.Sublayer(W, "", 1, S, 0.7, taps, width, "cuda")
    a.make_history(4, width, "cuda")
    assert (a.history is None) == (taps < 2)
    if taps > 1:
        a.history.fill_(float("nan"))                 # what no sequence has written is never read
    eps, rnd = 1e-2, random.Random(S)
    lens = {"a": 150, "b": 3, "c": 41, "d": 70, "e": 1, "f": 290, "g": 5}
    X, Y = {k: rn(n, S, width) for k, n in lens.items()}, {k: rn(n, width) for k, n in lens.items()}
    new = {k: torch.einsum("st,nsw->ntw", W["hc1.mix"].double(), X[k].double()) + 0.7 * W["hc1.out"].double()[:, None] * Y[k].double()[:, None] for k in lens}
    u = {k: torch.einsum("s,nsw->nw", W["hc1.in"].double(), new[k]) for k in lens}
    h = {k: O.unit_rms(u[k], eps) * W["norm1"].double() for k in lens}
    want = {k: h[k] + O.short_conv(h[k], W["canon1"].double()) for k in lens}
    epoch = torch.zeros(4, dtype=torch.int32, device="cuda")
    pad = _pad(width)
    for step in batches(rnd, lens, [1, 1, 2, 3, 5, 8, 9, 33, 200]):
        cat = lambda src: torch.cat([src[k][lo:lo + c] for k, _, lo, c in step])
        n = sum(c for *_, c in step)
        pos = torch.cat([torch.arange(lo, lo + c) for _, _, lo, c in step]).to(torch.int32).cuda()
        slots = torch.cat([torch.full((c,), s) for _, s, _, c in step]).to(torch.int32).cuda()
        x_in, x_out, y = torch.zeros(n, S, pad, device="cuda"), torch.full((n, S, pad), 7.0, device="cuda"), torch.zeros(3, n, pad, device="cuda")
        x_in[:, :, :width], yc = cat(X).cuda(), cat(Y)
        y[0, :, :width], y[1, :, :width], y[2, :, :width] = (yc - 1.0).cuda(), 0.25, 0.75      # parts of a sum
        xa, total = torch.zeros(n, pad, dtype=dtype, device="cuda"), torch.zeros(n, pad, device="cuda")
        HS.step_epoch(slots, epoch)
        HS.streams_rows(x_in[:, :, :width], x_out[:, :, :width], y, a, a, a.gain, eps, epoch, pos, slots, xa, total[:, :width])
        assert _rel(x_out[:, :, :width], cat(new)) < 2e-6 and (x_out[:, :, width:] == 7).all()
        assert _rel(total[:, :width], cat(u)) < 2e-6 and not xa[:, width:].any()
        assert _rel(xa[:, :width], cat(want)) < _lim(dtype, 3e-6, 5e-3)
        HS.streams_rows(x_in[:, :1, :width].expand(-1, S, -1), None, None, None, None, a.gain, eps, epoch, pos, slots, xa, total[:, :width])      # one row repeated
        s1 = S * cat(X)[:, 0].double()
        assert _rel(total[:, :width], s1) < 2e-6 and _rel(xa[:, :width], O.unit_rms(s1, eps) * W["norm1"].double()) < _lim(dtype, 3e-6, 5e-3)


@gpu
@pytest.mark.parametrize("S,taps,width,N", [(1, 4, 64, 40), (2, 4, 264, 2400), (3, 2, 136, 9), (4, 7, 1032, 5000), (2, 0, 40, 33), (1, 1, 24, 100), (4, 3, 2048, 300)])
def test_linear_behind_the_streams(S, taps, width, N):
    """Decode rows: the fused launch against streams, norm, convolution and a linear of the restatement, over sequences from their first token on, alone, two sequences
    together, and two rows of one sequence."""
    from ironpangu_b200.ops import hyper_streams as HS

    g = torch.Generator().manual_seed(width + S)
    rn = lambda *s: torch.randn(s, generator=g)
    W = {"hc1.mix": rn(S, S), "hc1.in": rn(S), "hc1.out": rn(S), "norm1": rn(), "canon1": rn(width, taps)}
    a = HS.Sublayer(W, "", 1, S, 0.7, taps, width, "cuda")
    a.make_history(3, width, "cuda")
    if taps > 1:
        a.history.fill_(float("nan"))
    eps, n = 1e-2, 24
    w = (rn(N, width) * width ** -0.5).to(BF16)
    X, Y = {k: rn(n, S, width) for k in "ab"}, {k: rn(n, width) for k in "ab"}
    new = {k: torch.einsum("st,nsw->ntw", W["hc1.mix"].double(), X[k].double()) + 0.7 * W["hc1.out"].double()[:, None] * Y[k].double()[:, None] for k in "ab"}
    h = {k: O.unit_rms(torch.einsum("s,nsw->nw", W["hc1.in"].double(), new[k]), eps) * W["norm1"].double() for k in "ab"}
    z = {k: torch.nn.functional.gelu((h[k] + O.short_conv(h[k], W["canon1"].double())) @ w.double().T) for k in "ab"}
    epoch = torch.zeros(3, dtype=torch.int32, device="cuda")
    at, slot = {"a": 0, "b": 0}, {"a": 2, "b": 0}
    for step in ("a", "a", "b", "ab", "aa", "ba", "bb", "a", "aa", "aa", "ab", "b", "bb", "ab"):
        rows = []
        for k in step:
            rows.append((k, at[k]))
            at[k] += 1
        cat = lambda src: torch.stack([src[k][i] for k, i in rows])
        m = len(rows)
        pos, slots = torch.tensor([i for _, i in rows], dtype=torch.int32, device="cuda"), torch.tensor([slot[k] for k, _ in rows], dtype=torch.int32, device="cuda")
        x_out, out = torch.zeros(m, S, width, device="cuda"), torch.full((m, N + 3), 5.0, device="cuda")
        HS.step_epoch(slots, epoch)
        HS.gemv_streams(cat(X).cuda(), x_out, cat(Y).cuda(), a, a, eps, epoch, pos, slots, w.cuda(), out[:, :N], "gelu_erf")
        assert _rel(x_out, cat(new)) < 2e-6 and (out[:, N:] == 5).all()
        assert _rel(out[:, :N], cat(z)) < 8e-3, step
    first = torch.zeros(1, N, device="cuda")                # a sequence's first token ahead of the first layer: one row for every stream, nothing to add
    HS.step_epoch(torch.tensor([1], dtype=torch.int32, device="cuda"), epoch)
    x = rn(1, 1, width)
    HS.gemv_streams(x.cuda().expand(1, S, width), None, None, None, a, eps, epoch, torch.zeros(1, dtype=torch.int32, device="cuda"), torch.ones(1, dtype=torch.int32, device="cuda"),
                    w.cuda(), first)
    h = O.unit_rms(x[0].double() * W["hc1.in"].double().sum(), eps) * W["norm1"].double()
    assert _rel(first, (h + O.short_conv(h, W["canon1"].double())) @ w.double().T) < 8e-3


@gpu
@DTYPES
def test_embedding_norm_and_plain_residual(dtype):
    from ironpangu_b200.ops import hyper_streams as HS

    g = torch.Generator().manual_seed(1)
    table, gain = torch.randn(50, 72, generator=g).to(dtype), torch.tensor([1.7])
    ids = torch.tensor([3, 49, 0, 3], dtype=torch.int32)
    x, st = torch.zeros(4, 72, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    HS.embed_norm(ids.cuda(), table.cuda(), gain.cuda(), 1e-3, x, st.data_ptr())
    assert _rel(x, O.unit_rms(table.double()[ids.long()], 1e-3) * 1.7) < 1e-6 and int(st) == 0
    HS.embed_norm(torch.tensor([50, -1], dtype=torch.int32, device="cuda"), table.cuda(), gain.cuda(), 1e-3, x[:2], st.data_ptr())
    assert int(st) != 0                                                                      # ids outside the table are reported
    plain = HS.Sublayer({"norm1": torch.tensor(0.5)}, "", 1, 0, 0.3, 0, 72, "cuda")          # no stream tensors: x + 0.3 y
    pos = torch.arange(4, dtype=torch.int32, device="cuda")
    y, out, xa = torch.randn(4, 72, generator=g).cuda(), torch.zeros(4, 1, 72, device="cuda"), torch.zeros(4, 72, dtype=dtype, device="cuda")
    HS.streams_rows(x[:, None], out, y, plain, plain, plain.gain, 1e-3, torch.zeros(1, dtype=torch.int32, device="cuda"), pos, torch.zeros_like(pos), xa)
    want = (x + 0.3 * y).double().cpu()
    assert _rel(out[:, 0], want) < 1e-6 and _rel(xa, O.unit_rms(want, 1e-3) * 0.5) < _lim(dtype, 2e-6, 5e-3)


@gpu
def test_turning_epochs():
    from ironpangu_b200.ops import hyper_streams as HS

    epoch = torch.tensor([0, 1, 1, 0, 0], dtype=torch.int32, device="cuda")
    HS.step_epoch(torch.tensor([2] * 200 + [0] + [4] * 30 + [1], dtype=torch.int32, device="cuda"), epoch)
    assert epoch.tolist() == [1, 0, 0, 0, 1]


@gpu
@DTYPES
@pytest.mark.parametrize("rows", [1, 5, 130, 300])
def test_exact_gelu(dtype, rows):
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(rows)
    x, w = torch.randn(rows, 64, generator=g).to(dtype), (torch.randn(96, 64, generator=g) * 0.4).to(dtype)
    out = torch.zeros(rows, 96, dtype=F32 if dtype == F32 else BF16, device="cuda")
    N.linear(x.cuda(), w.cuda(), out, "gelu_erf")
    z = x.double() @ w.double().T
    assert _rel(out, torch.nn.functional.gelu(z)) < _lim(dtype, 3e-6, 5e-3)
    if dtype == F32:
        lo, exact = (z < -2.5) & (z > -8), 0.5 * z * torch.special.erfc(-z / 2 ** 0.5)          # the far tail keeps its relative precision
        assert not lo.any() or ((out.cpu().double() - exact).abs() / exact.abs())[lo].max() < 1e-3


# ---------------------------------------------------------------------------------------------------------------------------
# recurrences
# ---------------------------------------------------------------------------------------------------------------------------
SHAPES = {"delta": [("delta", 2, 2, 16, 16, 4), ("delta", 6, 2, 32, 24, 3), ("delta", 3, 1, 7, 11, 5), ("delta", 1, 1, 1, 1, 1), ("delta", 2, 1, 136, 72, 2), ("delta", 4, 4, 64, 128, 4),
                    ("delta", 1, 1, 264, 20, 3)],
          "ssd": [("ssd", 4, 2, 16, 24, 4, 2), ("ssd", 6, 1, 32, 16, 2, 1), ("ssd", 3, 3, 5, 7, 3, 7), ("ssd", 1, 1, 1, 1, 1, 1), ("ssd", 2, 1, 128, 64, 4, 2), ("ssd", 2, 2, 300, 136, 4, 1)],
          "memory": [("memory", 2, 2, 16, 16), ("memory", 3, 3, 32, 24), ("memory", 5, 5, 7, 11), ("memory", 1, 1, 1, 1), ("memory", 2, 2, 136, 72), ("memory", 2, 2, 64, 128)]}
MIXERS = {"delta": O.delta_mixer, "ssd": O.ssd_mixer, "memory": O.memory_mixer}


class Recurrence:
    """Random weights of one recurrence whose projections and output matrix are identities (the inputs are the projections, exact in 16 bits), inputs of
    several sequences, and the restatement's results."""

    def __init__(self, shape, dtype, lens, seed=0, strong=1.0):
        from ironpangu_b200.ops import gated_recurrence as GR

        kind, heads, kv, dim, vdim = shape[:5]
        cap = 5.0
        self.shape = GR.RecurrenceShape(kind, heads, kv, dim, vdim, *shape[5:], **({"gate_cap": cap} if kind == "memory" else {}))
        self.shape.check()
        s, g, self.dtype = self.shape, torch.Generator().manual_seed(seed), dtype
        rn = lambda *a: torch.randn(a, generator=g)
        qk, v, width = kv * dim, heads * vdim, s.in_cols
        one, at = torch.eye(width), 0
        w, gain = {"norm": 1 + 0.3 * rn(vdim if kind == "delta" else v), "o": torch.eye(v)}, torch.ones(width)
        for n, c in s.columns.items():
            w[n] = one[at:at + c]
            gain[at:at + c] = {"i": 3.0 * strong, "f": 2.0, "b": 2.0}.get(n, 1.0)
            at += c
        if kind == "ssd":
            w = {"norm": w["norm"], "o": w["o"], "in": one, "conv": rn(s.channels, s.taps) * s.taps ** -0.5, "conv.b": 0.3 * rn(s.channels), "D": rn(heads)}
        if kind == "delta":
            w.update({"q.conv": rn(qk, s.taps), "k.conv": rn(qk, s.taps), "v.conv": rn(v, s.taps)})
        if kind == "memory":
            w.update({"i.b": rn(heads), "f.b": 2.0 + rn(heads) - 3.0 * (strong - 1.0)})
        else:
            w.update({"A_log": math.log(strong) - 0.5 + 0.8 * rn(heads), "dt_bias": -1.5 + rn(heads)})
        m = {"heads": heads, "kv_heads": kv, "groups": kv, "dim": dim, "state": dim, "vdim": vdim, "norm_groups": s.norm_groups, "gate_cap": cap}
        self.w = {k: t.to(BF16).float() for k, t in w.items()}
        h = {k: (rn(n, width) * gain).to(BF16) for k, n in lens.items()}
        self.mixer, self.eps, self.GR = GR.GatedRecurrence(s, self.w, "", "cuda", dtype, at=3, factor=0.75), 1e-2, GR
        self.proj = {k: torch.nn.functional.pad(x, (3, 0)).to(dtype) for k, x in h.items()}
        wd = {k: t.double() for k, t in self.w.items()}
        self.want = {k: 0.75 * MIXERS[kind](x.double(), m, wd, "", self.eps) for k, x in h.items()}
        self.state = self.mixer.make_state(4, "cuda", dtype)
        for t in (self.state.s, self.state.m, self.state.history):
            if t is not None:
                t.fill_(float("nan"))
        self.epoch = torch.zeros(4, dtype=torch.int32, device="cuda")

    def step(self, step, short=4):
        """Rows of one packed step; returns each entry's result."""
        from ironpangu_b200.ops import hyper_streams as HS
        from ironpangu_b200.ops.linear_attn import StepPlan

        n, v = sum(c for *_, c in step), self.shape.inner
        pos = [p for _, _, lo, c in step for p in range(lo, lo + c)]
        slots = [s for _, s, _, c in step for _ in range(c)]
        chunk = self.GR.TILE if self.dtype == BF16 and self.shape.tiles else self.GR.CHUNK
        plan = StepPlan(slots, pos, short=short, chunk=chunk)
        dp, ds = torch.tensor(pos, dtype=torch.int32, device="cuda"), torch.tensor(slots, dtype=torch.int32, device="cuda")
        B = self.GR.RecurrenceBuffers([self.shape], n, self.dtype, "cuda", chunk=chunk, slots=4)
        out = torch.full((n, _pad(v) + 8), 5.0, dtype=self.dtype, device="cuda")
        HS.step_epoch(ds, self.epoch)
        proj = torch.cat([self.proj[k][lo:lo + c] for k, _, lo, c in step]).cuda()
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        self.mixer.mix(B, self.state, proj, dp, ds, plan.bind(plan.control.cuda(), dp), self.epoch, self.eps, out[:, 4:], st.data_ptr())
        assert int(st) == 0
        assert (out[:, :4] == 5).all() and (out[:, 4 + v:] == 5).all()
        return torch.split(out[:, 4:4 + v].cpu(), [c for *_, c in step])

    def error(self, steps):
        worst = 0.0
        for step in steps:
            for (k, _, lo, c), got in zip(step, self.step(step)):
                worst = max(worst, float((got.double() - self.want[k][lo:lo + c]).abs().max() / self.want[k].abs().max()))
        return worst


def _cuts(n, c):
    return [[("a", 1, lo, min(c, n - lo))] for lo in range(0, n, c)]


@gpu
@DTYPES
@pytest.mark.parametrize("shape", [s for v in SHAPES.values() for s in v], ids=str)
def test_recurrence_in_portions(shape, dtype):
    """Whole, in portions around the chunk size, in pairs, and token by token; then several sequences over slots that are used again."""
    lens = {"a": 200, "b": 3, "c": 70, "d": 129, "e": 1, "f": 64, "g": 21}
    r = Recurrence(shape, dtype, lens)
    lim = _lim(dtype, 2e-5, 8e-2)          # in 16 bits the convolved rows are rounded
    for cuts in (_cuts(200, 200), _cuts(200, 128), _cuts(200, 129), _cuts(200, 64), _cuts(200, 65), _cuts(200, 63), _cuts(200, 7), _cuts(60, 2), _cuts(60, 1), [[("a", 1, 0, 130)]] + [[("a", 1, i, 1)] for i in range(130, 160)]):
        assert r.error(cuts) < lim, cuts[0]
    assert r.error(batches(random.Random(3), lens, [1, 1, 2, 4, 5, 17, 64, 66, 130])) < lim


@gpu
@pytest.mark.parametrize("shape,dtype", [(SHAPES["delta"][1], F32), (SHAPES["ssd"][0], F32), (SHAPES["memory"][1], F32), (("delta", 2, 1, 128, 128, 4), BF16), (("delta", 1, 1, 40, 72, 2), BF16),
                                         (("ssd", 2, 1, 128, 64, 4, 1), BF16), (("memory", 2, 2, 64, 128), BF16), (("memory", 1, 1, 128, 96), BF16)], ids=str)
def test_recurrence_of_long_and_short_memory(shape, dtype):
    """Decays so strong that a chunk's logs sum to hundreds, and gates so large that the running maximum jumps; a state that hardly decays
    over a thousand rows."""
    for strong, n in ((30.0, 300), (0.002, 1000)):
        r = Recurrence(shape, dtype, {"a": n}, strong=strong, seed=4)
        lim = 5e-5 if dtype == F32 else 2e-2
        assert r.error(_cuts(n, n)) < lim and r.error(_cuts(n, 100)) < lim


@gpu
@pytest.mark.parametrize("shape", [("delta", 6, 2, 32, 24, 3), ("delta", 2, 1, 136, 72, 2), ("delta", 4, 4, 64, 128, 4), ("delta", 1, 1, 4, 4, 1), ("ssd", 4, 2, 16, 24, 4, 2),
                                   ("ssd", 6, 1, 32, 16, 2, 1), ("ssd", 2, 1, 128, 64, 4, 2), ("ssd", 2, 2, 200, 136, 4, 1), ("memory", 3, 3, 32, 24), ("memory", 2, 2, 136, 72),
                                   ("memory", 2, 2, 64, 128)], ids=str)
@pytest.mark.parametrize("K1", [0, 24])
def test_fused_decode_of_recurrences(shape, K1):
    """Step and output projection in two launches: one or two rows, of one sequence or two, behind a prompt and from the first token on."""
    from ironpangu_b200.ops import hyper_streams as HS

    r = Recurrence(shape, BF16, {"a": 40, "b": 40}, seed=2)
    g = torch.Generator().manual_seed(9)
    v, N = r.shape.inner, 72
    w = torch.zeros(N, K1 + _pad(v))
    w[:, :K1 + v] = torch.randn(N, K1 + v, generator=g) * (K1 + v) ** -0.5
    w = w.to(BF16)
    r.error([[("a", 1, 0, 20)]])
    at, slot = {"a": 20, "b": 0}, {"a": 1, "b": 3}
    proj0 = {k: torch.nn.functional.pad(x, (1, 0)) for k, x in r.proj.items()}          # columns from 4 on: whole loads
    mixer = r.GR.GatedRecurrence(r.shape, r.w, "", "cuda", BF16, at=4, factor=0.75)
    assert mixer.fusable
    for step in ("a", "b", "ab", "aa", "bb", "ba", "b", "a", "bb", "aa"):
        rows = []
        for k in step:
            rows.append((k, at[k]))
            at[k] += 1
        m = len(rows)
        pos, slots = torch.tensor([i for _, i in rows], dtype=torch.int32, device="cuda"), torch.tensor([slot[k] for k, _ in rows], dtype=torch.int32, device="cuda")
        proj = torch.stack([proj0[k][i] for k, i in rows])
        proj = torch.nn.functional.pad(proj, (0, -proj.shape[1] % 8)).cuda()
        B = r.GR.RecurrenceBuffers([r.shape], m, BF16, "cuda", chunk=0, slots=4)
        x, y = torch.randn(m, K1 + 8, generator=g).to(BF16), torch.full((m, N), 5.0, device="cuda")
        HS.step_epoch(slots, r.epoch)
        mixer.decode(B, r.state, proj, pos, slots, r.epoch)
        mixer.gemv_mixed(B, proj, r.eps, x.cuda(), K1, w.cuda(), y)
        want = torch.cat([x[:, :K1].double(), torch.stack([r.want[k][i] for k, i in rows])], 1) @ w[:, :K1 + v].double().T
        assert _rel(y, want) < 5e-2, step


def test_restated_recurrences_by_hand():
    """Two steps of every recurrence, written out."""
    q, k, v = torch.tensor([[[1.0, 2.0]], [[0.5, -1.0]]]), torch.tensor([[[0.6, 0.8]], [[1.0, 0.0]]]), torch.tensor([[[3.0]], [[-2.0]]])
    a, b = torch.tensor([[0.5], [0.25]]), torch.tensor([[0.5], [1.0]])
    S1 = torch.tensor([0.6, 0.8]) * 1.5
    S2 = 0.25 * S1
    S2 = S2 + torch.tensor([1.0, 0.0]) * (-2.0 - S2[0])
    assert torch.allclose(O.delta_rule(q, k, v, a, b).flatten(), torch.stack([q[0, 0] @ S1, q[1, 0] @ S2]))
    S1, S2 = 0.5 * 3 * k[0, 0], 0.25 * 0.5 * 3 * k[0, 0] - 2.0 * k[1, 0]
    assert torch.allclose(O.ssd_scan(v, k, q, b, a.log()).flatten(), torch.stack([q[0, 0] @ S1, q[1, 0] @ S2]))
    # log gates: the input gate below, then above the running maximum
    li, lf = torch.tensor([[-1.0], [2.0]]), torch.tensor([[-0.5], [-0.25]])
    m1 = -0.5
    n1 = math.exp(-1.0 - m1) * k[0, 0]
    o1 = (q[0, 0] @ n1) * 3.0 / (max(abs(float(q[0, 0] @ n1)), math.exp(-m1)) + 1e-6)
    n2, S2 = math.exp(-0.25 + m1 - 2.0) * n1 + k[1, 0], math.exp(-0.25 + m1 - 2.0) * 3.0 * n1 - 2.0 * k[1, 0]
    o2 = (q[1, 0] @ S2) / (max(abs(float(q[1, 0] @ n2)), math.exp(-2.0)) + 1e-6)
    assert torch.allclose(O.matrix_memory(q, k, v, li, lf).flatten(), torch.stack([torch.as_tensor(o1), o2]), rtol=1e-5)
    x, w = torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[10.0, 100.0]])
    assert O.short_conv(x, w, torch.tensor([0.5])).flatten().tolist() == [100.5, 210.5, 420.5]


# ---------------------------------------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------------------------------------
@gpu
@DTYPES
@pytest.mark.parametrize("H,G,d,e,rot,norm", [(4, 2, 16, 24, 16, False), (5, 1, 14, 6, 6, False), (3, 3, 40, 40, 0, True), (16, 4, 128, 128, 128, False), (8, 2, 64, 64, 0, True), (2, 1, 144, 100, 100, False),
                                              (1, 1, 8, 8, 2, False), (7, 7, 9, 5, 0, True)])
def test_head_norm_halves_rotation_and_pages(dtype, H, G, d, e, rot, norm):
    """Every head of q and k by its rms without a gain, or turned in halves by stretched frequencies; keys and values land in their pages."""
    from ironpangu_b200.ops import window_attn as WA
    from ironpangu_b200.ops.linear_attn import RotaryScaling, RotaryTables

    g = torch.Generator().manual_seed(d)
    n, eps = 21, 1e-2
    stride = WA.tile_width(d) or d
    proj = (torch.randn(n, (H + G) * d + G * e, generator=g) * torch.rand(n, 1, generator=g)).to(dtype)
    pos = (torch.randperm(4000, generator=g)[:n].sort().values).to(torch.int32)
    table = torch.randperm(250, generator=g).to(torch.int32).view(1, 250).cuda()
    kc, vc = torch.zeros(250, 16, G, d, dtype=dtype, device="cuda"), torch.zeros(250, 16, G, e, dtype=dtype, device="cuda")
    sc = RotaryScaling(4.0, 1.0, 4.0, 512.0)
    tables = RotaryTables([(rot, 7e4, sc), (rot, 7e4)], n, "cuda")
    tables.fill(pos.cuda())
    q, ones = torch.zeros(n, H * stride, dtype=dtype, device="cuda"), torch.ones(d, device="cuda") if norm else None
    WA.qk_norm_rope_write(proj.cuda(), (0, H * d, (H + G) * d), ones, ones, eps, heads=H, kv_heads=G, dim=d, vdim=e, rot=rot, interleaved=False, rope=tables.get(rot, 7e4, sc),
                          positions=pos.cuda(), slots=torch.zeros(n, dtype=torch.int32, device="cuda"), page_table=table, q_out=q, k_cache=kc, v_cache=vc)
    p = proj.double()
    f = O.frequencies(rot, 7e4, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 512.0})
    do = lambda x: O.turn_halves(O.unit_rms(x, eps) if norm else x, pos, f)
    got = q.view(n, H, stride)
    assert _rel(got[..., :d], do(p[:, :H * d].view(n, H, d))) < _lim(dtype, 3e-6, 5e-3) and not got[..., d:].any()
    at = table[0, (pos // 16).long().cuda()].long(), (pos % 16).long().cuda()
    assert _rel(kc[at], do(p[:, H * d:(H + G) * d].view(n, G, d))) < _lim(dtype, 3e-6, 5e-3)
    assert torch.equal(vc[at].cpu(), proj[:, (H + G) * d:].view(n, G, e))


class Keys:
    """Random queries, keys and values of one sequence over pages in random order, and the restatement's result."""

    def __init__(self, H, G, d, e, dtype, n=420, seed=0, slots=3, gain=1.0):
        from ironpangu_b200.ops import window_attn as WA

        g = torch.Generator().manual_seed(seed)
        rn = lambda *s: torch.randn(s, generator=g)
        self.H, self.G, self.d, self.e, self.dtype, self.n, self.WA = H, G, d, e, dtype, n, WA
        self.q, self.k, self.v, self.gate = (gain * rn(n, H, d)).to(dtype), rn(n, G, d).to(dtype), rn(n, G, e).to(dtype), rn(n, H).to(dtype)
        self.pages = (n + 15) // 16
        self.table = torch.randperm(slots * self.pages, generator=g).to(torch.int32).view(slots, self.pages).cuda()
        self.slot = slots - 1

    def want(self, size, keep, pool, scale, gated, lo, hi):
        """Of rows lo .. hi - 1."""
        q, k, v, n = self.q[lo:hi].double(), self.k.double(), self.v.double(), self.n
        if pool:
            mk, mv = (O.block_means(x, pool).to(self.dtype).double() for x in (k, v))
            o = O.softmax_over(q, k, v, mk, mv, O.window_seen(n, size)[lo:hi], O.block_seen(n, size, pool)[lo:hi], scale)
        else:
            o = O.softmax_over(q, k, v, k[:0], v[:0], O.window_seen(n, size, keep)[lo:hi], torch.zeros(hi - lo, 0, dtype=torch.bool), scale)
        return 0.7 * (o * torch.sigmoid(self.gate[lo:hi].double())[..., None] if gated else o)

    def run(self, form, lo, hi, size, keep, pool, scale, gated):
        """Rows lo .. hi - 1. Pages hold what these rows may see and nothing else; the blocks are written as their last positions arrive."""
        WA, H, G, d, e, n, t = self.WA, self.H, self.G, self.d, self.e, self.n, self.dtype
        z = lambda m, w: torch.full((self.table.numel(), m, G, w), float("nan"), dtype=t, device="cuda")
        kc, vc = z(16, d), z(16, e)
        first = max(0, lo - size + 1)
        put = lambda pos: self.table[self.slot, (pos // 16).cuda()].long(), lambda pos: (pos % 16).cuda()
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        ahead = WA.Ahead(keep, 0)
        whole = torch.arange(hi)
        if pool:
            per = (15 + pool) // pool
            ahead = WA.Ahead(0, pool, (z(per, d), z(per, e)))
            kc[put[0](whole), put[1](whole)], vc[put[0](whole), put[1](whole)] = self.k[:hi].cuda(), self.v[:hi].cuda()
            p = whole.to(torch.int32).cuda()
            for a, b in ((0, hi // 3), (hi // 3, hi)):
                if a < b:
                    WA.pool_write(kc, vc, p[a:b].contiguous(), torch.full((b - a,), self.slot, dtype=torch.int32, device="cuda"), self.table, ahead, st.data_ptr())
            kc.fill_(float("nan"))
            vc.fill_(float("nan"))
        pos = torch.cat([torch.arange(min(keep, first)), torch.arange(first, hi)])
        kc[put[0](pos), put[1](pos)], vc[put[0](pos), put[1](pos)] = self.k[pos].cuda(), self.v[pos].cuda()
        stride = (WA.tile_width(d) or d) if form == "tiles" else d
        q = torch.zeros(hi - lo, H, stride, dtype=t, device="cuda")
        q[..., :d] = self.q[lo:hi].cuda()
        q = q.view(hi - lo, H * stride)
        out = torch.zeros(hi - lo, _pad(H * e), dtype=t, device="cuda")
        how = dict(heads=H, window=size, scale=scale, out=out, gate=self.gate[lo:hi].cuda() if gated else None, gate_act="sigmoid" if gated else None, gate_head=gated, ahead=ahead,
                   factor=0.7, status_ptr=st.data_ptr())
        p, s = torch.arange(lo, hi, dtype=torch.int32, device="cuda"), torch.full((hi - lo,), self.slot, dtype=torch.int32, device="cuda")
        most = ahead.count(max(0, n - size))
        if form == "general":
            WA.window_attn(q, kc, vc, p, s, self.table, **how)
        elif form == "split":
            sp = WA.split_form(H, G, d, e, size, most)
            for r in range(0, hi - lo, 64):
                part = dict(how, out=out[r:r + 64], gate=how["gate"][r:r + 64] if gated else None)
                m = len(p[r:r + 64])
                WA.gqa_window(q[r:r + 64], kc, vc, p[r:r + 64], s[r:r + 64], self.table, splits=sp, most_ahead=most, scratch=torch.empty(m * H * sp * (e + 2), device="cuda"), **part)
        else:
            rows = (hi - first + 31) // 32 * 32 + WA.ahead_rows(most)
            nan = lambda *a: torch.full(a, float("nan"), dtype=t, device="cuda")
            WA.fa_window(q, kc, vc, self.table, slot=self.slot, pos0=lo, ctx_k=nan(rows, G * stride), ctx_vt=nan(G * 128, rows), **how)
        assert int(st) == 0
        return out[:, :H * e].view(hi - lo, H, e).cpu()


FORMS = [("general", F32, (5, 1, 14, 9)), ("general", F32, (4, 2, 200, 136)), ("general", BF16, (6, 3, 40, 56)), ("split", BF16, (4, 4, 64, 64)), ("split", BF16, (4, 2, 128, 128)),
         ("split", BF16, (8, 2, 64, 64)), ("split", BF16, (8, 1, 128, 128)), ("split", BF16, (4, 1, 256, 256)), ("tiles", BF16, (4, 2, 64, 64)), ("tiles", BF16, (8, 2, 128, 128)),
         ("tiles", BF16, (3, 1, 40, 24)), ("tiles", BF16, (2, 2, 72, 128))]
RULES = [(16, 5, 0), (1, 1, 0), (65, 130, 0), (150, 64, 0), (16, 0, 5), (1, 0, 1), (65, 0, 16), (150, 0, 33), (40, 0, 2), (20, 0, 300)]
forms = pytest.mark.parametrize("form,dtype,shape", FORMS, ids=lambda v: str(v).replace("torch.", ""))


@gpu
@forms
@pytest.mark.parametrize("rule", RULES, ids=str)
def test_attention_with_entries_ahead(form, dtype, shape, rule):
    """Windows, kept positions and blocks around pages, tiles and portions; rows from the first positions and from the middle on."""
    K = Keys(*shape, dtype, gain=2.0)
    scale = shape[2] ** -0.5
    for gated, (lo, hi) in enumerate(((0, 420), (130, 131), (149, 152), (7, 199))):
        want = K.want(*rule, scale, gated % 2 == 1, lo, hi)
        got = K.run(form, lo, hi, *rule, scale, gated % 2 == 1)
        assert _rel(got, want) < _lim(dtype, 5e-6, 8e-3), (lo, hi)


@gpu
@forms
def test_a_single_entry_at_the_edges(form, dtype, shape):
    """A key, or the keys of a block, that take most of a query's weight: the last kept position and the one behind it, the window's oldest and the one
    before it, a block that is just seen and one that is not yet, the first tokens."""
    size, keep, pool, scale = 88, 5, 11, shape[2] ** -0.5
    for query in (299, 196, 195, 99, 98, 94):
        old, seen = query - size, (query - size + 1) // pool * pool          # the position just outside the window, the first position of no seen block
        for rule, keys in (((size, keep, 0), ([0], [keep - 1], [keep], [old + 1], [old], [query])),
                           ((size, 0, pool), ([old + 1], [old], range(pool), range(seen - pool, seen), range(seen, seen + pool)))):
            for some in keys:
                some = [k for k in some if k >= 0]
                K = Keys(*shape, dtype, n=300, seed=query)
                if some:
                    K.k[some] = (K.q[query].float().view(K.G, -1, K.d).mean(1) * 6.0 * (K.H // K.G) ** 0.5).to(dtype)
                lo = query - 2
                want = K.want(*rule, scale, False, lo, query + 1)
                assert _rel(K.run(form, lo, query + 1, *rule, scale, False), want) < _lim(dtype, 5e-6, 1e-2), (query, rule, some)
