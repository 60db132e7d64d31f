"""Each mechanism of the Falinex decoder on the GPU against the plain restatement: recurrences by steps, f32 chunks and tensor-core
tiles, windowed attention in its three forms, output norms, gated head norms, linears with fused prologues."""
import math

import pytest
import torch

import falinex_oracle as O

pytestmark = pytest.mark.gpu
BF16, F32 = torch.bfloat16, torch.float32


def _cuda(*ts):
    return [t.cuda() for t in ts]


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def _fabric():
    from ironpangu_b200.parallel.fabric import Fabric

    return Fabric(0, 1)


# ---------------------------------------------------------------------------------------------------------------------------
# recurrences
# ---------------------------------------------------------------------------------------------------------------------------
def _recurrence_case(kind, H, d, e, T, seed=0, rot=None):
    """(mixer options, packed projection [T, ...] bf16 values, reference (o, S), positions) of one sequence."""
    g = torch.Generator().manual_seed(seed)
    decay = [0.6, 0.97, 0.9995, 1.0, 0.0][:H] if H <= 5 else [1 - 2.0 ** -(1 + h) for h in range(H)]
    cols = [H * d, H * d, H * e]
    proj = torch.randn(T, sum(cols) + 3, generator=g).to(BF16)
    x = proj.double()
    q, k, v = x[:, :cols[0]].view(T, H, d), x[:, cols[0]:2 * cols[0]].view(T, H, d), x[:, 2 * cols[0]:sum(cols)].view(T, H, e)
    if kind == "rotated":
        rot = rot or d
        pos = torch.arange(T)
        q, k = O.rotate(q, pos, rot, 1e4, False), O.rotate(k, pos, rot, 1e4, False) * d ** -0.5
        opts = dict(rot_dims=rot, k_scale=d ** -0.5)
    elif kind == "interleaved":
        rot = rot or d
        pos = torch.arange(T)
        q, k = O.rotate(q, pos, rot, 1e4, True), O.rotate(k, pos, rot, 1e4, True)
        opts = dict(rot_dims=rot, interleaved=True)
    else:
        q, k, v = O.silu(q), O.silu(k), O.silu(v)
        opts = dict(act="silu")
        rot = 0
    ref = O.decayed_state(q, k, v, torch.tensor(decay, dtype=torch.float64))
    return dict(heads=H, dim=d, vdim=e, decay=decay, offsets=(0, cols[0], 2 * cols[0]), **opts), proj, ref, rot


SHAPES = [("rotated", 2, 16, 24, 200, None), ("activated", 3, 32, 16, 200, None), ("rotated", 5, 128, 128, 300, None), ("activated", 2, 128, 96, 270, None),
          ("rotated", 1, 20, 9, 131, 12), ("interleaved", 2, 40, 64, 140, 24), ("activated", 1, 9, 5, 133, None), ("rotated", 2, 64, 128, 140, 32)]


@pytest.mark.parametrize("kind,H,d,e,T,rot", SHAPES)
def test_recurrence_forms_match_the_restatement(kind, H, d, e, T, rot):
    from ironpangu_b200.ops import linear_attn as LA

    opts, proj, (want, S), rot = _recurrence_case(kind, H, d, e, T, rot=rot)
    mx = LA.DecayedMixer(device="cuda", **opts)
    tabs = LA.RotaryTables([(rot, 1e4)], T, "cuda")
    pos, slot = _i32(list(range(T))), torch.full((T,), 1, dtype=torch.int32, device="cuda")
    tabs.fill(pos)
    rope = tabs.get(rot, 1e4)
    rms = float(want.pow(2).mean().sqrt())

    def compare(o, st, tol):
        assert float((o.cpu().double() - want).abs().max()) < tol * rms * 8, "outputs"
        assert float((st[1].cpu().double().transpose(1, 2) - S).abs().max()) < tol * float(S.abs().max()) * 2, "state"

    for dt in (F32, BF16):
        p = proj.cuda().to(dt)
        act_round = 4e-3 if dt == BF16 and kind == "activated" else 2e-5      # activations are bf16 values in bf16 mode
        # one row at a time (a used slot: garbage before), then runs of up to three rows
        for width in (1, 3):
            st = mx.state(3, "cuda").fill_(7.0)
            o = torch.zeros(T, H * e, dtype=F32, device="cuda")
            for t in range(0, T, width):
                n = min(width, T - t)
                sub = rope[t:t + n] if rope is not None else None
                mx.step(p[t:t + n], st, pos[t:t + n], slot[t:t + n], sub, o[t:t + n])
            compare(o.view(T, H, e), st, act_round)
            assert bool((st[0] == 7.0).all() and (st[2] == 7.0).all())
        # portions of several sizes through the chunk forms
        for cuts in ([T], [65, T - 65], [2, 63, 64, T - 129]):
            for tiles in ([False, True] if dt == BF16 and max(d, e) <= 128 else [False]):
                chunk = LA.TILE if tiles else LA.CHUNK
                st = mx.state(3, "cuda").fill_(7.0)
                o = torch.zeros(T, H * e, dtype=F32, device="cuda")
                cs = torch.empty((T // chunk + 2) * H * d * e, dtype=F32, device="cuda")
                buf = [torch.empty(T * H * w, dtype=F32, device="cuda") for w in (d, d, e)]
                r = 0
                for n in cuts:
                    plan = LA.StepPlan([1] * n, list(range(r, r + n)), short=0, chunk=chunk)
                    dp = plan.bind(plan.control.cuda(), pos[r:r + n])
                    sub = rope[r:r + n] if rope is not None else None
                    if tiles:
                        mx.tiles(p[r:r + n], st, pos[r:r + n], dp.table, sub, cs, out=o[r:r + n])
                    else:
                        mx.chunks(p[r:r + n], st, pos[r:r + n], dp.table, sub, o[r:r + n], (*buf, cs))
                    r += n
                compare(o.view(T, H, e), st, max(act_round, 1e-4 if tiles else 2e-5))


def test_tiles_with_head_norm_and_gate_and_many_sequences():
    """Several sequences in one launch, normed and gated in the epilogue, equal each sequence alone."""
    from ironpangu_b200.ops import linear_attn as LA

    H, d, e, eps = 3, 64, 48, 1e-5
    lens = [130, 1, 5, 128, 257]
    opts, proj, _, rot = _recurrence_case("rotated", H, d, e, sum(lens), seed=4)
    g = torch.Generator().manual_seed(5)
    gate = torch.randn(sum(lens), H * e, generator=g).to(BF16)
    mx = LA.DecayedMixer(device="cuda", **opts)
    slots = [s for s, n in enumerate(lens) for _ in range(n)]
    positions = [i for n in lens for i in range(n)]
    plan = LA.StepPlan(slots, positions, short=0, chunk=LA.TILE)
    T = sum(lens)
    pos = _i32(positions)
    tabs = LA.RotaryTables([(rot, 1e4)], T, "cuda")
    tabs.fill(pos)
    st = mx.state(5, "cuda").fill_(3.0)
    y = torch.zeros(T, H * e, dtype=BF16, device="cuda")
    cs = torch.empty(len(plan.chunks) * H * d * e, dtype=F32, device="cuda")
    mx.tiles(proj.cuda(), st, pos, plan.bind(plan.control.cuda(), pos).table, tabs.get(rot, 1e4), cs, gated=y, gate=gate.cuda(), gate_act="silu", eps=eps)
    at = 0
    for s, n in enumerate(lens):
        x = proj[at:at + n].double()
        q, k = x[:, :H * d].view(n, H, d), x[:, H * d:2 * H * d].view(n, H, d)
        q, k = O.rotate(q, torch.arange(n), rot, 1e4, False), O.rotate(k, torch.arange(n), rot, 1e4, False) * d ** -0.5
        o, S = O.decayed_state(q, k, x[:, 2 * H * d:2 * H * d + H * e].view(n, H, e), torch.tensor(opts["decay"], dtype=torch.float64))
        want = O.rms(o, eps).reshape(n, -1) * O.silu(gate[at:at + n].double())
        torch.testing.assert_close(y[at:at + n].cpu().double(), want, rtol=1e-2, atol=1e-2)
        torch.testing.assert_close(st[s].cpu().double().transpose(1, 2), S, rtol=1e-3, atol=1e-3)
        at += n


# ---------------------------------------------------------------------------------------------------------------------------
# windowed attention
# ---------------------------------------------------------------------------------------------------------------------------
def _pages(k, v, page_tokens=16, spare=3, seed=0):
    """Paged caches that hold k [T, G, d], v [T, G, e] of one sequence in shuffled pages; the rest of the pool is garbage."""
    T, G, d = k.shape
    n = (T + page_tokens - 1) // page_tokens
    perm = torch.randperm(n + spare, generator=torch.Generator().manual_seed(seed))
    table = torch.full((2, n + 2), -1, dtype=torch.int32)
    table[1, :n] = perm[:n].int()
    kc, vc = (torch.full((n + spare, page_tokens, G, x.shape[2]), 50.0, dtype=x.dtype) for x in (k, v))
    for i in range(T):
        kc[perm[i // page_tokens], i % page_tokens], vc[perm[i // page_tokens], i % page_tokens] = k[i], v[i]
    return kc.cuda(), vc.cuda(), table.cuda()


ATT = [(4, 2, 16, 16), (6, 2, 40, 24), (5, 5, 20, 9), (4, 1, 128, 128), (2, 2, 64, 64), (8, 1, 64, 64), (3, 1, 200, 72), (4, 2, 96, 128)]


@pytest.mark.parametrize("H,G,d,e", ATT)
@pytest.mark.parametrize("window", [1, 16, 33, 150])
def test_windowed_attention_forms(H, G, d, e, window):
    """Random keys, then one key that stands out just inside and one just outside the window of every row, at page borders too."""
    from ironpangu_b200.ops import window_attn as WA

    T = 180
    g = torch.Generator().manual_seed(H * 100 + d)
    q, k, v = torch.randn(T, H, d, generator=g), torch.randn(T, G, d, generator=g), torch.randn(T, G, e, generator=g)
    # keys 0, 15, 16, 47, 48, 100: twelve times longer, so that a softmax which sees one of them is ruled by it
    for j in (0, 15, 16, 47, 48, 100):
        k[j] *= 12.0
    sink = torch.randn(H, generator=g) * 2
    gate = torch.randn(T, H * e, generator=g)
    scale = 0.7 * d ** -0.5
    fab = _fabric()
    st = fab.desc.status
    for dt in (F32, BF16):
        qq, kk, vv, gg = (x.to(dt) for x in (q, k, v, gate))
        want = O.windowed_softmax(qq.double(), kk.double(), vv.double(), scale, window, sink.double()).reshape(T, -1) * torch.sigmoid(gg.double())
        kc, vc, table = _pages(kk, vv, seed=d)
        pos, slot = _i32(list(range(T))), torch.ones(T, dtype=torch.int32, device="cuda")
        sg = dict(sink=sink.cuda(), gate_act="sigmoid", status_ptr=st)
        tol = dict(rtol=2e-5, atol=2e-5) if dt == F32 else dict(rtol=1e-2, atol=1e-2)
        out = torch.zeros(T, H * e, dtype=dt, device="cuda")
        qd, gd = qq.reshape(T, -1).cuda(), gg.cuda()
        WA.window_attn(qd, kc, vc, pos, slot, table, heads=H, window=window, scale=scale, out=out, gate=gd, **sg)
        torch.testing.assert_close(out.cpu().double(), want, **tol)
        if dt == F32:
            continue
        splits = WA.split_form(H, G, d, e, window)
        if splits:
            out.zero_()
            scratch = torch.empty(T * H * splits * (d + 2), dtype=F32, device="cuda")
            WA.gqa_window(qd, kc, vc, pos, slot, table, heads=H, window=window, scale=scale, splits=splits, scratch=scratch, out=out, gate=gd, **sg)
            torch.testing.assert_close(out.cpu().double(), want, **tol)
        dp = WA.tile_width(d)
        if dp and e <= 128:
            qp = torch.zeros(T, H, dp, dtype=BF16)
            qp[..., :d] = qq
            qp = qp.reshape(T, -1).cuda()
            for cuts in ([T], [2, 31, 128, T - 161]):
                out.zero_()
                r = 0
                for n in cuts:
                    rows = WA.context_rows(n, window)
                    ck = torch.full((rows, G * dp), 9.0, dtype=BF16, device="cuda")
                    cv = torch.full((G * 128, rows), 9.0, dtype=BF16, device="cuda")
                    WA.fa_window(qp[r:r + n], kc, vc, table, slot=1, pos0=r, heads=H, window=window, scale=scale, ctx_k=ck, ctx_vt=cv, out=out[r:r + n],
                                 gate=gd[r:r + n], **sg)
                    r += n
                torch.testing.assert_close(out.cpu().double(), want, **tol)
    assert fab.status() == 0
    fab.close()


def test_softmax_weights_keep_more_than_bf16_on_the_tensor_cores():
    """Many equal keys with large values of both signs: weights rounded to 8 bits would not cancel."""
    from ironpangu_b200.ops import window_attn as WA

    T, d = 128, 64
    g = torch.Generator().manual_seed(3)
    k = torch.randn(T, 1, d, generator=g).to(BF16) * 0.3
    q = torch.randn(T, 1, d, generator=g).to(BF16) * 0.3
    v = torch.zeros(T, 1, d)
    v[0::2], v[1::2] = 96.0, -96.0
    v = v.to(BF16)
    sink = torch.full((1,), -30.0)
    want = O.windowed_softmax(q.double(), k.double(), v.double(), 0.125, T, sink.double()).reshape(T, -1)
    kc, vc, table = _pages(k, v)
    out = torch.zeros(T, d, dtype=BF16, device="cuda")
    rows = WA.context_rows(T, T)
    WA.fa_window(q.reshape(T, -1).cuda(), kc, vc, table, slot=1, pos0=0, heads=1, window=T, scale=0.125, ctx_k=torch.zeros(rows, 64, dtype=BF16, device="cuda"),
                 ctx_vt=torch.zeros(128, rows, dtype=BF16, device="cuda"), out=out, sink=sink.cuda())
    err = (out.cpu().double() - want)[64:].abs()
    assert float((err - want[64:].abs() * 2.0 ** -8).max()) < 4e-3       # beyond the rounding of the result itself


@pytest.mark.parametrize("sink", [-40.0, 0.0, 40.0])
def test_a_sink_takes_its_share(sink):
    from ironpangu_b200.ops import window_attn as WA

    T, d = 40, 64
    q, k = torch.zeros(T, 1, d).to(BF16), torch.ones(T, 1, d).to(BF16)
    v = torch.ones(T, 1, d).to(BF16)
    kc, vc, table = _pages(k, v)
    s = torch.full((1,), sink, device="cuda")
    pos, slot = _i32(list(range(T))), torch.ones(T, dtype=torch.int32, device="cuda")
    for form in ("general", "split", "tile"):
        out = torch.zeros(T, d, dtype=BF16, device="cuda")
        how = dict(heads=1, window=8, scale=1.0, out=out, sink=s)
        qd = q.reshape(T, -1).cuda()
        if form == "general":
            WA.window_attn(qd, kc, vc, pos, slot, table, **how)
        elif form == "split":
            WA.gqa_window(qd, kc, vc, pos, slot, table, splits=1, scratch=torch.empty(T * (d + 2), device="cuda"), **how)
        else:
            rows = WA.context_rows(T, 8)
            WA.fa_window(qd, kc, vc, table, slot=1, pos0=0, ctx_k=torch.zeros(rows, 64, dtype=BF16, device="cuda"),
                         ctx_vt=torch.zeros(128, rows, dtype=BF16, device="cuda"), **how)
        n = torch.arange(1, T + 1).clamp(max=8).double()
        want = n / (n + math.exp(sink))
        torch.testing.assert_close(out[:, 0].cpu().double(), want, rtol=1e-2, atol=1e-6)


def test_query_key_norm_rotation_and_cache_write():
    from ironpangu_b200.ops import linear_attn as LA
    from ironpangu_b200.ops import window_attn as WA

    T, H, G, d, e, rot, eps = 21, 3, 1, 20, 12, 14, 1e-3
    g = torch.Generator().manual_seed(9)
    cols = [H * d, G * d, G * e]
    proj = torch.randn(T, sum(cols), generator=g)
    qg, kg = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) + 0.5
    p0 = 100000                                     # positions far out: angles need more than float products
    pos_host = torch.arange(p0, p0 + T)
    for interleaved in (True, False):
        tabs = LA.RotaryTables([(rot, 5e5)], T, "cuda")
        pos = pos_host.int().cuda()
        tabs.fill(pos)
        table = torch.full((1, (p0 + T) // 16 + 1), -1, dtype=torch.int32)
        first = p0 // 16
        table[0, first:] = torch.arange(table.shape[1] - first).int().flip(0)
        n = table.shape[1] - first
        kc, vc = torch.zeros(n, 16, G, d, device="cuda"), torch.zeros(n, 16, G, e, device="cuda")
        q = torch.zeros(T, H * 32, device="cuda")
        WA.qk_norm_rope_write(proj.cuda(), (0, cols[0], cols[0] + cols[1]), qg.cuda(), kg.cuda(), eps, heads=H, kv_heads=G, dim=d, vdim=e, rot=rot,
                              interleaved=interleaved, rope=tabs.get(rot, 5e5), positions=pos, slots=torch.zeros(T, dtype=torch.int32, device="cuda"),
                              page_table=table.cuda(), q_out=q, k_cache=kc, v_cache=vc)
        x = proj.double()
        wq = O.rotate(O.rms(x[:, :cols[0]].view(T, H, d), eps, qg.double()), pos_host, rot, 5e5, interleaved)
        wk = O.rotate(O.rms(x[:, cols[0]:cols[0] + cols[1]].view(T, G, d), eps, kg.double()), pos_host, rot, 5e5, interleaved)
        q = q.view(T, H, 32).cpu()
        assert bool((q[..., d:] == 0).all())
        torch.testing.assert_close(q[..., :d].double(), wq, rtol=1e-5, atol=2e-6)
        for i in range(T):
            pg = int(table[0, (p0 + i) // 16])
            torch.testing.assert_close(kc[pg, (p0 + i) % 16].cpu().double(), wk[i], rtol=1e-5, atol=2e-6)
            assert torch.equal(vc[pg, (p0 + i) % 16].cpu(), proj[i, cols[0] + cols[1]:].view(G, e))


# ---------------------------------------------------------------------------------------------------------------------------
# norms, gates, linears
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("D", [64, 52, 97, 2048, 5000])
def test_output_norm_residual_and_final_norm(D):
    from ironpangu_b200.ops import stream_norm as N

    T, eps = 5, 1e-2                                   # an eps that matters
    g = torch.Generator().manual_seed(D)
    y, x, w, w2 = torch.randn(T, D, generator=g) * 0.2, torch.randn(T, D, generator=g), torch.rand(D, generator=g) + 0.5, torch.rand(D, generator=g) + 0.5
    want = x.double() + O.rms(y.double(), eps, w.double())
    for dt, tol in ((F32, 2e-6), (BF16, 1e-2)):
        for final in (None, w2):
            xd, xa = x.cuda().clone(), torch.zeros(T, D, dtype=dt, device="cuda")
            N.post_norm_add(y.cuda(), w.cuda(), eps, xd, xa, None if final is None else final.cuda())
            torch.testing.assert_close(xd.cpu().double(), want, rtol=1e-5, atol=2e-6)
            torch.testing.assert_close(xa.cpu().double(), want if final is None else O.rms(want, eps, w2.double()), rtol=tol, atol=tol)
        out = torch.zeros(2, D, dtype=dt, device="cuda")
        N.rms_rows(x.cuda(), w2.cuda(), eps, out, _i32([3, 0]))
        torch.testing.assert_close(out.cpu().double(), O.rms(x[[3, 0]].double(), eps, w2.double()), rtol=tol, atol=tol)


@pytest.mark.parametrize("groups,n,act,gain", [(4, 16, "silu", False), (1, 192, "sigmoid", True), (1, 2048, "sigmoid", True), (3, 7, "silu", False)])
def test_gated_head_norm(groups, n, act, gain):
    from ironpangu_b200.ops import stream_norm as N

    T, eps = 6, 1e-3
    g = torch.Generator().manual_seed(n)
    o, gate, w = torch.randn(T, groups * n, generator=g), torch.randn(T, groups * n, generator=g) * 3, torch.rand(groups * n, generator=g) + 0.5
    f = O.silu if act == "silu" else torch.sigmoid
    for dt, tol in ((F32, 1e-5), (BF16, 1e-2)):
        gt = gate.to(dt)
        want = O.rms(o.double().view(T, groups, n), eps).reshape(T, -1) * (w.double() if gain else 1.0) * f(gt.double())
        out = torch.zeros(T, groups * n, dtype=dt, device="cuda")
        N.group_norm_gate(o.cuda(), gt.cuda(), act, eps, out, groups, w.cuda() if gain else None)
        torch.testing.assert_close(out.cpu().double(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("T,N_,K", [(1, 96, 64), (3, 200, 72), (40, 131, 52), (300, 256, 128), (300, 512, 64)])
def test_linears_with_activation(T, N_, K):
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(T)
    x, w = torch.randn(T, K, generator=g).to(BF16), (torch.randn(N_, K, generator=g) * K ** -0.5).to(BF16)
    for act, f in ((None, lambda z: z), ("gelu_tanh", O.gelu_tanh), ("silu", O.silu), ("sigmoid", torch.sigmoid)):
        want = f(x.double() @ w.double().T)
        out = torch.zeros(T, N_, device="cuda")
        N.linear(x.float().cuda(), w.float().cuda(), out, act)
        torch.testing.assert_close(out.cpu().double(), want, rtol=1e-5, atol=5e-6)
        if K % 8 == 0:
            for dt, tol in ((F32, 1e-4), (BF16, 1e-2)):
                out = torch.zeros(T, N_, dtype=dt, device="cuda")
                N.linear(x.cuda(), w.cuda(), out, act)
                torch.testing.assert_close(out.cpu().double(), want, rtol=tol, atol=tol)


def test_gelu_far_from_zero():
    from ironpangu_b200.ops import stream_norm as N

    z = torch.tensor([[-200.0, -30.0, -6.0, -0.5, 0.0, 0.5, 6.0, 200.0]])
    for dt in (F32, BF16):
        out = torch.zeros(8, 8, dtype=F32, device="cuda")
        x = torch.diag(z[0]).to(dt).cuda()
        N.linear(x, torch.eye(8).to(dt).cuda(), out, "gelu_tanh")
        got = out.diagonal().cpu().double()
        torch.testing.assert_close(got, O.gelu_tanh(z[0].double()), rtol=1e-4, atol=1e-4)


@pytest.mark.parametrize("T", [1, 2, 3, 8])
def test_fused_decode_linears(T):
    from ironpangu_b200.ops import stream_norm as N

    K, N_, eps = 192, 328, 1e-3
    g = torch.Generator().manual_seed(T)
    w = (torch.randn(N_, K, generator=g) * K ** -0.5).to(BF16)
    y, x, nw = torch.randn(T, K, generator=g), torch.randn(T, K, generator=g) * 4, torch.rand(K, generator=g) + 0.5
    x_out, z = torch.zeros(T, K, device="cuda"), torch.zeros(T, N_, device="cuda")
    N.gemv_post_norm(y.cuda(), nw.cuda(), eps, x.cuda(), x_out, w.cuda(), z, "gelu_tanh")
    want_x = x.double() + O.rms(y.double(), eps, nw.double())
    torch.testing.assert_close(x_out.cpu().double(), want_x, rtol=1e-5, atol=2e-6)
    torch.testing.assert_close(z.cpu().double(), O.gelu_tanh(want_x.to(BF16).double() @ w.double().T), rtol=5e-3, atol=5e-3)
    for groups, act, gain in ((6, "silu", None), (1, "sigmoid", nw)):
        gate = (torch.randn(T, K, generator=g) * 2).to(BF16)
        N.gemv_group_norm(y.cuda(), gate.cuda(), act, eps, w.cuda(), z, groups, None if gain is None else gain.cuda())
        f = O.silu if act == "silu" else torch.sigmoid
        op = O.rms(y.double().view(T, groups, -1), eps).reshape(T, K) * (1.0 if gain is None else gain.double()) * f(gate.double())
        torch.testing.assert_close(z.cpu().double(), op.to(BF16).double() @ w.double().T, rtol=2e-2, atol=2e-2)
    xb, zb = x.to(BF16), torch.zeros(T, N_, dtype=BF16, device="cuda")
    N.gemv_act(xb.cuda(), w.cuda(), zb)
    torch.testing.assert_close(zb.cpu().double(), xb.double() @ w.double().T, rtol=1e-2, atol=2e-2)
