"""Mechanisms of the Ponenex decoder one by one on the device against the plain restatement: latent attention in its three forms, routed
experts in both, the norms and the router around them."""
import random

import pytest
import torch

import ponenex_oracle as O

BF16, F32, F64 = torch.bfloat16, torch.float32, torch.float64
pytestmark = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def _rel(got, want):
    d = (got.double().cpu() - want.double().cpu()).abs()
    return float(d.max() / want.double().abs().max())


def _lim(dtype, f32=5e-6, bf16=2e-2):
    return f32 if dtype == F32 else bf16


# ---------------------------------------------------------------------------------------------------------------------------
# row operators
# ---------------------------------------------------------------------------------------------------------------------------
@DTYPES
@pytest.mark.parametrize("width", [36, 64, 1000])
def test_scaled_embedding_with_norm(dtype, width):
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(1)
    table, w = torch.randn(50, width, generator=g).to(dtype), 0.3 * torch.randn(width, generator=g)
    ids = torch.tensor([3, 49, 0, 3, 17], dtype=torch.int32)
    pad = (width + 7) // 8 * 8
    t = torch.zeros(50, pad, dtype=dtype)
    t[:, :width] = table
    x, xa = torch.zeros(5, pad, device="cuda"), torch.zeros(5, pad, dtype=dtype, device="cuda")
    N.embed_rows(ids.cuda(), t.cuda(), x[:, :width], xa, scale=0.37, gain=(1 + w).cuda(), eps=1e-3)
    want = table.double()[ids.long()] * 0.37
    assert _rel(x[:, :width], want) < 1e-6
    assert _rel(xa[:, :width], O.centred_norm(want, w.double(), 1e-3)) < _lim(dtype, bf16=5e-3) and not xa[:, width:].any()


@pytest.mark.parametrize("rows", [1, 2, 5, 8])
@pytest.mark.parametrize("width,cols", [(64, 40), (1032, 300), (4096, 2500)])
def test_linear_behind_two_norms(rows, width, cols):
    """x' = x + rms(y) g; z = bf16(rms(x') g2) W^T in one launch."""
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(rows)
    y, x = torch.randn(rows, width, generator=g) * 3, torch.randn(rows, width, generator=g)
    g1, g2 = torch.randn(width, generator=g), torch.randn(width, generator=g)
    w = (torch.randn(cols, width, generator=g) * width ** -0.5).to(BF16)
    x2, z = torch.zeros(rows, width, device="cuda"), torch.zeros(rows, cols, device="cuda")
    N.gemv_post_norm(y.cuda(), g1.cuda(), 1e-4, x.cuda(), x2, w.cuda(), z, next_norm=g2.cuda())
    wx = x.double() + O.rms(y.double(), 1e-4, g1.double())
    assert _rel(x2, wx) < 1e-6
    assert _rel(z, O.rms(wx, 1e-4, g2.double()).float().to(BF16).double() @ w.double().T) < 2e-3


@pytest.mark.parametrize("experts,top", [(1, 1), (5, 2), (33, 16), (256, 8)])
def test_router_selection_from_logits(experts, top):
    """Extreme logits, negative ones, ties (the lower index first), a bias that changes the choice, the shared expert's column."""
    from ironpangu_b200.ops import _lib
    from ironpangu_b200.ops.stream_norm import _s

    g = torch.Generator().manual_seed(experts)
    M = 37
    z = torch.randn(M, experts + 1, generator=g) * 5
    z[0], z[1], z[2] = -300.0 + z[0], 0.25, z[2] * 40           # far below zero, all equal, far apart
    b = torch.randn(experts, generator=g)
    b[: experts // 3] = 0.0
    z[1, :experts] -= b
    zd, bd = z.cuda(), b.cuda()
    ids, wts, sw = (torch.zeros(M, top, dtype=t, device="cuda") for t in (torch.int32, F32, F32))
    sw = torch.zeros(M, device="cuda")
    rc = _lib.load().ifab_moe_route(zd.data_ptr(), experts + 1, bd.data_ptr(), M, experts, top, 2, 1, 1.0, 1, 1, ids.data_ptr(), wts.data_ptr(), sw.data_ptr(), _s())
    assert rc == 0
    best, want = (z[:, :experts] + b).sort(dim=-1, descending=True, stable=True)
    assert torch.equal(ids.cpu().long(), want[:, :top])
    assert (wts.cpu() - torch.softmax(best[:, :top].double(), -1)).abs().max() < 1e-6
    assert (sw.cpu() - torch.sigmoid(z[:, experts])).abs().max() < 1e-6


@DTYPES
@pytest.mark.parametrize("heads,k,n,rows", [(1, 8, 8, 1), (5, 13, 40, 9), (3, 96, 512, 64), (4, 512, 129, 65), (2, 72, 33, 300)])
def test_one_product_per_head(dtype, heads, k, n, rows):
    from ironpangu_b200.ops.latent_attn import heads_product

    g = torch.Generator().manual_seed(k)
    sa, sc, kp = (k + 7) // 8 * 8 + 16, n + 3, (k + 7) // 8 * 8
    a = torch.randn(rows, heads * sa, generator=g).to(dtype)
    b = torch.zeros(heads, n, kp, dtype=dtype)
    b[:, :, :k] = (torch.randn(heads, n, k, generator=g) * k ** -0.5).to(dtype)
    want = torch.einsum("thk,hnk->thn", a.double().view(rows, heads, sa)[:, :, :k], b.double()[:, :, :k])
    for out in (F32, dtype):
        c = torch.full((rows, heads * sc), 7.0, dtype=out, device="cuda")
        heads_product(a.cuda(), sa, b.cuda(), c, sc, heads, k)
        got = c.view(rows, heads, sc)
        assert _rel(got[:, :, :n], want) < (5e-6 if dtype == F32 else 1e-5 if out == F32 else 5e-3)
        assert (got[:, :, n:] == 7).all()                      # what lies between the heads is not touched


# ---------------------------------------------------------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------------------------------------------------------
SHAPES = {          # heads, dim, rot_dim, vdim, kv_rank, q_rank, rot dims
    "small": (4, 16, 16, 24, 40, 32, 16),
    "odd": (3, 13, 6, 9, 21, 11, 6),
    "padded": (8, 40, 32, 72, 96, 64, 20),
    "full": (4, 128, 64, 128, 512, 128, 64),
    "half": (2, 64, 64, 64, 264, 64, 64),
    "wide": (2, 136, 80, 132, 600, 40, 80),
    "one head": (1, 8, 8, 8, 8, 8, 8),
}


class Layer:
    """One latent-attention layer with random weights over pages in random order; ``needle``: scores so sharp that one key takes most of
    the weight."""

    def __init__(self, shape, dtype, *, window, width=96, context=256, slots=3, seed=0, sharp=2.0, eps=1e-5):
        from ironpangu_b200.ops.latent_attn import LatentMixer, LatentShape

        H, d, r, e, L, R, rot = shape
        g = torch.Generator().manual_seed(seed)
        rn = lambda *s: torch.randn(*s, generator=g)
        self.m = {"heads": H, "dim": d, "rot_dim": r, "vdim": e, "kv_rank": L, "q_rank": R, "rot": {"dims": rot, "base": 3e4}, "mask": {"size": window},
                  "scale": 0.9 * (d + r) ** -0.5}
        mat = lambda o, i: rn(o, i) * i ** -0.5
        self.w = {"dq": mat(R, width), "dq.norm": 1 + 0.2 * rn(R), "uq": sharp * mat(H * (d + r), R), "dkv": mat(L + r, width), "dkv.norm": 1 + 0.2 * rn(L),
                  "uk": mat(H * d, L), "uv": mat(H * e, L), "g": mat(H, width), "o": mat(width, H * e)}
        self.w = {k: v.to(BF16) for k, v in self.w.items()}
        self.eps, self.dtype, self.width, self.context = eps, dtype, width, context
        self.shape = LatentShape(H, d, r, e, L, R, rot, 3e4, window, self.m["scale"])
        self.mix = LatentMixer(self.shape, self.w, "", "cuda", dtype, max_context=context)
        pages = context // 16
        self.table = torch.randperm(slots * pages, generator=g).to(torch.int32).view(slots, pages).cuda()
        self.mix.make_pages(slots * pages, 16)
        self.wd = {k: v.double() for k, v in self.w.items()}

    def buffers(self, rows, chunked):
        from ironpangu_b200.ops.latent_attn import LatentBuffers
        from ironpangu_b200.ops.linear_attn import RotaryTables

        B = LatentBuffers([self.shape], rows, self.dtype, "cuda", chunked=chunked, max_context=self.context, group=64)
        return B, RotaryTables([(self.shape.rot_dims, 3e4)], rows, "cuda")

    def step(self, B, rotary, h, positions, slots, *, form):
        """Output rows ``[m, width]`` of the layer. form: "plan" (packed step), "rows", "decode"."""
        from ironpangu_b200.ops import stream_norm as N
        from ironpangu_b200.ops.linear_attn import StepPlan

        m, s = h.shape[0], self.shape
        pos, sl = torch.tensor(positions, dtype=torch.int32, device="cuda"), torch.tensor(slots, dtype=torch.int32, device="cuda")
        rotary.fill(pos)
        xa = h.to(self.dtype).cuda().contiguous()
        N.linear(xa, self.mix.w_in, B.proj[:m, :s.in_cols])
        rope = rotary.get(s.rot_dims, 3e4)
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        if form == "decode":
            self.mix.decode(B, m, rope, pos, sl, self.table, self.eps, st.data_ptr())
        else:
            plan = None
            if form == "plan":
                p = StepPlan(slots, positions, chunk=128)
                plan = p.bind(p.control.cuda(), pos)
            self.mix.mix(B, m, rope, pos, sl, plan, self.table, self.eps, st.data_ptr())
        y = torch.zeros(m, self.width, device="cuda")
        N.linear(B.mixed[s.heads * s.vdim][:m], self.mix.w_o, y)
        assert int(st) == 0
        return y.cpu()

    def want(self, h, faults=()):
        return O.latent_attention(h.to(self.dtype).double(), self.m, self.wd, "", self.eps, faults)


def _decodes(shape, dtype):
    return dtype == BF16 and all(SHAPES[shape][i] % 8 == 0 for i in (5,)) and SHAPES[shape][0] * SHAPES[shape][3] % 8 == 0


@DTYPES
@pytest.mark.parametrize("shape", list(SHAPES))
@pytest.mark.parametrize("window", [0, 1, 30, 130])
def test_latent_attention_of_prompts_and_decoded_rows(shape, window, dtype):
    n = 200
    L = Layer(SHAPES[shape], dtype, window=window)
    h = torch.randn(n, L.width, generator=torch.Generator().manual_seed(5))
    want = L.want(h)
    lim = _lim(dtype, bf16=3e-2)
    B, rot = L.buffers(n, True)
    for form in ("plan", "rows"):
        assert _rel(L.step(B, rot, h, list(range(n)), [1] * n, form=form), want) < lim, form
        L.mix.cache.zero_()                                    # what a form has not written itself must not be there
    B8, rot8 = L.buffers(8, False)
    got, i, rnd = [], 0, random.Random(3)
    while i < 120:
        k = min(120 - i, rnd.choice([1, 2]) if _decodes(shape, dtype) else rnd.choice([1, 3, 8]))
        got.append(L.step(B8, rot8, h[i:i + k], list(range(i, i + k)), [2] * k, form="decode" if _decodes(shape, dtype) else "rows"))
        i += k
    assert _rel(torch.cat(got), want[:120]) < lim


@pytest.mark.parametrize("fault", ["window_plus_one", "window_minus_one", "no_gate", "no_rotation", "latent_not_normed"])
def test_the_comparison_would_notice(fault):
    """The restatement with a mistake planted in it is far outside every tolerance used here."""
    L = Layer(SHAPES["small"], BF16, window=30)
    h = torch.randn(120, L.width, generator=torch.Generator().manual_seed(5))
    assert _rel(L.want(h, (fault,)), L.want(h)) > 0.15


@DTYPES
@pytest.mark.parametrize("shape", ["small", "full", "wide"])
def test_one_key_among_hundreds_at_every_border(shape, dtype):
    """A row whose query all but picks one key (its score stands out): at the far end of the window, one past it, at page borders, as the first
    token, for prompts and decoding. What is outside must have no effect, what is inside nearly all of it."""
    n, window = 250, 100
    L = Layer(SHAPES[shape], dtype, window=window, sharp=1.0)
    s = L.shape
    H, d = s.heads, s.dim
    g = torch.Generator().manual_seed(9)
    base = 0.2 * torch.randn(n, L.width, generator=g)
    form = "decode" if dtype == BF16 else "rows"
    for query, key in ((249, 150), (249, 149), (249, 240), (249, 239), (160, 61), (160, 60), (99, 0), (100, 0), (100, 1), (175, 80), (175, 75)):
        h = base.clone()
        # make the key's row the one the query likes: the input direction whose latent key points along the query's latent query
        h[query] = 3.0 * torch.randn(L.width, generator=g)
        cq = O.rms(h[query].double() @ L.wd["dq"].T, L.eps, L.wd["dq.norm"])
        q = (cq @ L.wd["uq"].T).view(H, -1)[:, :d]
        lat = torch.einsum("hd,hdl->l", q, L.wd["uk"].view(H, d, -1)) * L.wd["dkv.norm"]
        h[key] = 30.0 * torch.linalg.lstsq(L.wd["dkv"][: s.kv_rank], lat[:, None] / lat.norm()).solution[:, 0].float()
        want = L.want(h)[query]
        without = h.clone()
        without[key] = base[key]
        effect = _rel(L.want(without)[query], want)
        inside = query - key < window
        assert (effect > 0.08) if inside else effect < 1e-9, (query, key, effect)
        B, rot = L.buffers(n, True)
        got = L.step(B, rot, h, list(range(n)), [0] * n, form="plan")[query]
        assert _rel(got, want) < _lim(dtype, bf16=3e-2), (query, key)
        B8, rot8 = L.buffers(8, False)
        got = L.step(B8, rot8, h[query:query + 1], [query], [0], form=form)[0]
        assert _rel(got, want) < _lim(dtype, bf16=3e-2), (query, key, form)


@DTYPES
def test_unequal_sequences_in_one_step(dtype):
    """Portions and single rows of three sequences in one packed step equal each alone, on pages in any order; a negative position is skipped."""
    L = Layer(SHAPES["padded"], dtype, window=40)
    g = torch.Generator().manual_seed(11)
    seqs = [torch.randn(n, L.width, generator=g) for n in (150, 70, 33)]
    want = [L.want(h) for h in seqs]
    B, rot = L.buffers(256, True)
    done = [0, 0, 0]
    rnd = random.Random(2)
    while any(done[i] < len(seqs[i]) for i in range(3)):
        h, pos, sl = [], [], []
        for i in rnd.sample(range(3), 3):
            k = min(len(seqs[i]) - done[i], rnd.choice([0, 1, 1, 2, 5, 31, 64]))
            h.append(seqs[i][done[i]:done[i] + k])
            pos += range(done[i], done[i] + k)
            sl += [i] * k
            done[i] += k
        if not pos:
            continue
        y = L.step(B, rot, torch.cat(h), pos, sl, form="plan")
        for r, (p, i) in enumerate(zip(pos, sl)):
            assert _rel(y[r], want[i][p]) < _lim(dtype, bf16=4e-2), (i, p)


def test_pages_that_are_gone_are_reported():
    L = Layer(SHAPES["small"], BF16, window=0)
    B, rot = L.buffers(64, True)
    L.table[1, 0] = -1
    with pytest.raises(AssertionError):
        L.step(B, rot, torch.randn(20, L.width), list(range(20)), [1] * 20, form="rows")


# ---------------------------------------------------------------------------------------------------------------------------
# routed experts
# ---------------------------------------------------------------------------------------------------------------------------
class Unit:
    def __init__(self, dtype, width, experts, top, ff, shared, seed=0):
        from ironpangu_b200.ops.routed_experts import ExpertsShape, RoutedExperts

        g = torch.Generator().manual_seed(seed)
        mat = lambda o, i: (torch.randn(o, i, generator=g) * i ** -0.5).to(BF16)
        self.w = {"router": (3.0 * mat(experts, width).float()).to(BF16), "router.b": (0.5 * torch.randn(experts, generator=g)).to(BF16)}
        for name, f in [(f"e{e}.", ff) for e in range(experts)] + ([("shared.", shared)] if shared else []):
            self.w.update({name + "gate": mat(f, width), name + "up": mat(f, width), name + "down": mat(width, f)})
        if shared:
            self.w["shared.sg"] = mat(1, width)
        self.m = {"router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}
        self.shape = ExpertsShape(width, experts, top, ff, shared)
        self.ff = RoutedExperts(self.shape, self.w, "", "cuda", dtype)
        self.dtype, self.width = dtype, width
        self.gain, self.next = torch.randn(width, generator=g), torch.randn(width, generator=g)

    def inputs(self, rows, seed):
        """Operands rounded to the activation type, without close calls of the router."""
        g = torch.Generator().manual_seed(seed)
        h = torch.randn(40 * rows, self.width, generator=g).to(self.dtype).double()
        z = (h @ self.w["router"].double().T + self.w["router.b"].double()).sort(dim=-1, descending=True).values
        t = self.shape.top
        if t < self.shape.experts:
            h = h[z[:, t - 1] - z[:, t] > 0.02]
        return h[:rows], torch.randn(rows, self.width, generator=g)

    def want(self, h, x, faults=()):
        y = O.experts(h, self.m, {k: v.double() for k, v in self.w.items()}, "", faults)
        x = x.double() + O.rms(y, 1e-5, self.gain.double())
        return y, x, O.rms(x, 1e-5, self.next.double())


UNITS = [(64, 4, 2, 24, 16), (52, 7, 3, 19, 35), (136, 3, 3, 40, 0), (64, 1, 1, 8, 72), (256, 40, 8, 96, 288), (1032, 5, 1, 136, 32)]


@DTYPES
@pytest.mark.parametrize("width,experts,top,ff,shared", UNITS)
@pytest.mark.parametrize("rows", [1, 3, 65, 300])
def test_experts_of_a_packed_step(dtype, width, experts, top, ff, shared, rows):
    from ironpangu_b200.ops.routed_experts import ExpertBuffers

    U = Unit(dtype, width, experts, top, ff, shared)
    h, x = U.inputs(rows, rows)
    B = ExpertBuffers([U.shape], 320, dtype, "cuda")
    B.start(rows)
    pad = (width + 7) // 8 * 8
    xa, xd = torch.zeros(rows, pad, dtype=dtype, device="cuda"), torch.zeros(rows, pad, device="cuda")
    xa[:, :width], xd[:, :width] = h.to(dtype), x
    U.ff.rows(B, rows, xa, U.gain.cuda(), U.next.cuda(), 1e-5, xd, None)
    _, wx, wn = U.want(h, x)
    assert _rel(xd[:, :width], wx) < _lim(dtype) and _rel(xa[:, :width], wn) < _lim(dtype)
    assert not xd[:, width:].any() and not xa[:, width:].any()


@pytest.mark.parametrize("width,experts,top,ff,shared", [u for u in UNITS if u[0] % 8 == 0])
@pytest.mark.parametrize("rows", [1, 2, 8])
def test_experts_of_decode_rows(width, experts, top, ff, shared, rows):
    """The residual update and norm ahead, router, experts and shared expert as three launches."""
    from ironpangu_b200.ops.routed_experts import ExpertBuffers

    U = Unit(BF16, width, experts, top, ff, shared)
    g = torch.Generator().manual_seed(3)
    rn = lambda *s: torch.randn(*s, generator=g)
    owed, gain, eps = rn(width), 1 + 0.2 * rn(width), 1e-5
    prev, x = rn(80 * rows, width) * 4, rn(80 * rows, width)
    wx = x.double() + O.rms(prev.double(), eps, owed.double())
    h = O.rms(wx, eps, gain.double()).float().to(BF16).double()
    z = (h @ U.w["router"].double().T + U.w["router.b"].double()).sort(dim=-1, descending=True).values
    keep = (z[:, top - 1] - z[:, top] > 0.1 if top < experts else torch.ones(len(z), dtype=torch.bool)).nonzero()[:rows, 0]
    prev, x, wx, h = prev[keep], x[keep], wx[keep], h[keep]
    B = ExpertBuffers([U.shape], 8, BF16, "cuda")
    y, x2, xn = prev.cuda().contiguous(), torch.zeros(rows, width, device="cuda"), torch.zeros(rows, width, dtype=BF16, device="cuda")
    ticket = torch.zeros(1, dtype=torch.int32, device="cuda")
    for _ in range(2):                                          # the second run finds the ticket as the first one left it
        y.copy_(prev)
        U.ff.decode(B, rows, y, owed.cuda(), gain.cuda(), eps, x.cuda().contiguous(), x2, xn, ticket.data_ptr())
        want = O.experts(h, U.m, {k: v.double() for k, v in U.w.items()}, "")
        assert _rel(x2, wx) < 1e-6 and _rel(xn, h) < 5e-3 and _rel(y, want) < 2e-2 and int(ticket) == 0


@pytest.mark.parametrize("fault", ["no_bias", "no_shared", "shared_not_gated"])
def test_the_comparison_would_notice_in_experts(fault):
    U = Unit(BF16, 64, 4, 2, 24, 16)
    h, x = U.inputs(65, 65)
    assert _rel(U.want(h, x, (fault,))[1], U.want(h, x)[1]) > 0.1
