"""Mechanisms of the Mikutar decoder one by one on the device against the plain restatement: attention over windows and chunks in its three
forms, norms and rotation around it, gated units, the grouped router, experts, and the two ends of a parallel layer."""

import pytest
import torch

import mikutar_oracle as O

BF16, F32, F64 = torch.bfloat16, torch.float32, torch.float64
pytestmark = pytest.mark.gpu
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def _rel(got, want):
    d = (got.double().cpu() - want.double().cpu()).abs()
    return float(d.max() / want.double().abs().max())


def _lim(dtype, f32=5e-6, bf16=2e-2):
    return f32 if dtype == F32 else bf16


def _pad(n):
    return (n + 7) // 8 * 8


# ---------------------------------------------------------------------------------------------------------------------------
# linears, units, row operators
# ---------------------------------------------------------------------------------------------------------------------------
@DTYPES
@pytest.mark.parametrize("rows,cols,width", [(1, 40, 24), (7, 131, 56), (64, 300, 136), (200, 96, 64), (300, 320, 512), (515, 2080, 128)])
def test_linear_with_bias_and_soft_limit(dtype, rows, cols, width):
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(rows)
    x, w = torch.randn(rows, width, generator=g).to(dtype), (torch.randn(cols, width, generator=g) * width ** -0.5 * 3).to(dtype)
    b = torch.randn(cols, generator=g)
    z = x.double() @ w.double().T + b.double()
    for cap in (0.0, 4.0, 0.5):
        out = torch.zeros(rows, cols, device="cuda")
        N.linear(x.cuda(), w.cuda(), out, bias=b.cuda(), cap=cap)
        d = out.cpu().double() - (O.soft_limit(z, cap) if cap else z)
        assert d.abs().max() / z.abs().max() < (3e-6 if dtype == F32 else 1e-5), cap
    if dtype == BF16 and rows <= 8:
        out, add = torch.zeros(rows, cols, device="cuda"), torch.randn(rows, cols, generator=g)
        N.gemv_act(x.cuda(), w.cuda(), out, bias=b.cuda(), addend=add.cuda())
        assert _rel(out, z + add.double()) < 1e-5
        out = add.cuda()
        N.gemv_act(x.cuda(), w.cuda(), out, addend=out)
        assert _rel(out, z - b.double() + add.double()) < 1e-5


@pytest.mark.parametrize("rows,cols,width,parts", [(1, 40, 64, 1), (3, 33, 512, 8), (8, 131, 1000, 3), (64, 1024, 5120, 8), (128, 96, 328, 6), (70, 10000, 256, 2)])
def test_product_in_parts(rows, cols, width, parts):
    """Parts along K, the ragged last one included; the row operators add them up."""
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(cols)
    x, w, b = torch.randn(rows, width, generator=g).to(BF16), (torch.randn(cols, width, generator=g) * width ** -0.5).to(BF16), torch.randn(cols, generator=g)
    out = torch.full((parts, rows, _pad(cols)), 5.0, device="cuda")
    N.split_linear(x.cuda(), w.cuda(), out[:, :, :cols], b.cuda())
    want = x.double() @ w.double().T + b.double()
    assert _rel(out.sum(0)[:, :cols], want) < 2e-5 and (out[:, :, cols:] == 5).all()
    r = torch.randn(rows, _pad(cols), generator=g)
    xd, xa = r.cuda(), torch.zeros(rows, _pad(cols), device="cuda")
    N.post_norm_add(out[:, :, :cols], None, 1e-3, xd[:, :cols], xa)
    assert _rel(xd[:, :cols], r[:, :cols].double() + want) < 2e-5
    assert N.split_count(rows, cols, width) >= 1 and N.split_count(200, cols, width) == 1


UNITS = [("relu", 0.0, 1.0), ("limited", 0.7, 1.702), ("limited", 7.0, 0.9), ("silu", 0.0, 1.0)]


def _unit(kind, limit, alpha, g, u):
    if kind == "relu":
        return torch.relu(g) * u
    if kind == "silu":
        return g * torch.sigmoid(g) * u
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(alpha * g) * (u + 1.0)


@DTYPES
@pytest.mark.parametrize("unit", UNITS, ids=lambda u: f"{u[0]}{u[1]}")
@pytest.mark.parametrize("rows,ff,width", [(1, 8, 24), (5, 72, 40), (64, 336, 136), (100, 4800, 64), (130, 200, 72), (256, 96, 64), (300, 416, 512)])
def test_gated_linear(dtype, unit, rows, ff, width):
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(ff)
    x = torch.randn(rows, width, generator=g).to(dtype)
    w = (torch.randn(2 * ff, width, generator=g) * width ** -0.5 * 2).to(dtype)
    z = x.double() @ w.double().T
    wide = torch.full((rows, ff + 16), 3.0, dtype=dtype, device="cuda")
    N.gated_linear(x.cuda(), w.cuda(), N.GatedUnit(*unit), wide[:, 8:8 + ff], torch.zeros(rows, 2 * ff, dtype=dtype, device="cuda"))
    assert _rel(wide[:, 8:8 + ff], _unit(*unit, z[:, :ff], z[:, ff:])) < _lim(dtype, 1e-5, 1.2e-2)
    assert (wide[:, :8] == 3).all() and (wide[:, 8 + ff:] == 3).all()


@DTYPES
@pytest.mark.parametrize("width", [20, 53, 64, 1000])
def test_residual_update_without_a_norm(dtype, width):
    from ironpangu_b200.ops import stream_norm as N

    g = torch.Generator().manual_seed(width)
    rn = lambda *s: torch.randn(*s, generator=g)
    y, x, e, w = rn(5, _pad(width)), rn(5, _pad(width)), rn(5, _pad(width)), rn(width)
    for yy, ee, ww in ((y, None, w), (y, e, w), (None, e, w), (y, e, None), (None, None, w)):
        xd, xa = x.cuda(), torch.zeros(5, _pad(width), dtype=dtype, device="cuda")
        cut = lambda t: None if t is None else t.cuda()[:, :width]
        N.post_norm_add(cut(yy), None, 1e-3, xd[:, :width], xa, None if ww is None else ww.cuda(), cut(ee))
        want = x[:, :width].double() + (0 if yy is None else yy[:, :width].double()) + (0 if ee is None else ee[:, :width].double())
        assert _rel(xd[:, :width], want) < 1e-6
        assert _rel(xa[:, :width], want if ww is None else O.rms(want, 1e-3, ww.double())) < _lim(dtype, 2e-6, 5e-3) and not xa[:, width:].any()


@DTYPES
@pytest.mark.parametrize("H,G,d,rot,e", [(4, 2, 16, 16, 16), (5, 1, 14, 6, 14), (3, 3, 40, 0, 40), (16, 4, 128, 128, 128), (2, 1, 144, 100, 144), (1, 1, 8, 2, 8)])
def test_norm_over_whole_projections_rotation_and_pages(dtype, H, G, d, rot, e):
    """q and k normed over all their heads, turned in neighbouring pairs; the pages get the keys and, as values, the keys as projected."""
    from ironpangu_b200.ops import window_attn as WA
    from ironpangu_b200.ops.linear_attn import RotaryTables

    g = torch.Generator().manual_seed(d)
    n, eps = 21, 1e-2
    stride = WA.tile_width(d) or d
    proj = (torch.randn(n, (H + G) * d, generator=g) * torch.rand(n, 1, generator=g)).to(dtype)
    gq, gk = torch.randn(H * d, generator=g), torch.randn(G * d, generator=g)
    pos = torch.randint(0, 4000, (n,), generator=g).sort().values.to(torch.int32)
    slots = torch.zeros(n, dtype=torch.int32)
    table = torch.randperm(250, generator=g).to(torch.int32).view(1, 250).cuda()
    pages = torch.zeros(250, 16, G, d, dtype=dtype, device="cuda"), torch.zeros(250, 16, G, d, dtype=dtype, device="cuda")
    rot_tables = RotaryTables([(rot, 7e4)], n, "cuda")
    rot_tables.fill(pos.cuda())
    q = torch.zeros(n, H * stride, dtype=dtype, device="cuda")
    WA.qk_norm_rope_write(proj.cuda(), (0, H * d, H * d), gq.cuda(), gk.cuda(), eps, heads=H, kv_heads=G, dim=d, vdim=d, rot=rot, interleaved=True,
                          rope=rot_tables.get(rot, 7e4), positions=pos.cuda(), slots=slots.cuda(), page_table=table, q_out=q, k_cache=pages[0], v_cache=pages[1], whole=True)
    p = proj.double()
    turn = lambda x: O.turn_neighbours(x, pos, rot, 7e4) if rot else x
    wq = turn(O.rms(p[:, :H * d], eps, gq.double()).view(n, H, d))
    wk = turn(O.rms(p[:, H * d:], eps, gk.double()).view(n, G, d))
    got = q.view(n, H, stride)
    assert _rel(got[..., :d], wq) < _lim(dtype, 2e-6, 5e-3) and not got[..., d:].any()
    last = {int(x): i for i, x in enumerate(pos)}                          # rows at the same position overwrite one another
    rows = [i for i in range(n) if last[int(pos[i])] == i and (pos == pos[i]).sum() == 1]
    at = table[0, (pos[rows] // 16).long().cuda()].long(), (pos[rows] % 16).long().cuda()
    assert _rel(pages[0][at], wk[rows]) < _lim(dtype, 2e-6, 5e-3)
    assert torch.equal(pages[1][at].cpu(), proj[rows][:, H * d:].view(-1, G, d))


# ---------------------------------------------------------------------------------------------------------------------------
# attention
# ---------------------------------------------------------------------------------------------------------------------------
class Keys:
    """Random queries, keys and values of one sequence over pages in random order, and the restatement's result."""

    def __init__(self, H, G, d, e, dtype, n=300, seed=0, slots=3, gain=1.0):
        from ironpangu_b200.ops import window_attn as WA

        g = torch.Generator().manual_seed(seed)
        rn = lambda *s: torch.randn(*s, generator=g)
        self.H, self.G, self.d, self.e, self.dtype, self.n, self.WA = H, G, d, e, dtype, n, WA
        self.q, self.k, self.v, self.gate = (gain * rn(n, H, d)).to(dtype), rn(n, G, d).to(dtype), rn(n, G, e).to(dtype), rn(n, H).to(dtype)
        self.pages = (n + 15) // 16
        self.table = torch.randperm(slots * self.pages, generator=g).to(torch.int32).view(slots, self.pages).cuda()
        self.slot = slots - 1
        self.slopes = O.bias_slopes(H).float().cuda()

    def want(self, size, chunked, scale, cap, biased, rows=None):
        seen = (O.chunk_seen if chunked else O.window_seen)(self.n, size or self.n)
        o = O.attend(self.q.double(), self.k.double(), self.v.double(), seen, scale, cap, O.bias_slopes(self.H) if biased else None)
        return o * torch.sigmoid(self.gate.double())[..., None]

    def run(self, form, lo, hi, size, chunked, scale, cap, biased):
        WA, H, G, d, e, n, t = self.WA, self.H, self.G, self.d, self.e, self.n, self.dtype
        kc = torch.full((self.table.numel(), 16, G, d), float("nan"), dtype=t, device="cuda")
        vc = torch.full((self.table.numel(), 16, G, e), float("nan"), dtype=t, device="cuda")
        first = (lo // size * size if chunked else max(0, lo - size + 1)) if size else 0
        pos = torch.arange(first, hi)                                     # only what the rows may see is there
        at = self.table[self.slot, (pos // 16).cuda()].long(), (pos % 16).cuda()
        kc[at], vc[at] = self.k[first:hi].cuda(), self.v[first:hi].cuda()
        table = self.table.clone()
        table[self.slot, :first // 16] = -1                               # pages behind it are gone
        stride = (WA.tile_width(d) or d) if form == "tiles" else d
        q = torch.zeros(hi - lo, H, stride, dtype=t, device="cuda")
        q[..., :d] = self.q[lo:hi].cuda()
        q = q.view(hi - lo, H * stride)
        out = torch.zeros(hi - lo, _pad(H * e), dtype=t, device="cuda")
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        how = dict(heads=H, window=size, scale=scale, out=out, gate=self.gate[lo:hi].cuda(), gate_act="sigmoid", gate_head=True, chunked=chunked, cap=cap,
                   slopes=self.slopes if biased else None, status_ptr=st.data_ptr())
        p, s = torch.arange(lo, hi, dtype=torch.int32, device="cuda"), torch.full((hi - lo,), self.slot, dtype=torch.int32, device="cuda")
        if form == "general":
            WA.window_attn(q, kc, vc, p, s, table, **how)
        elif form == "split":
            sp = WA.split_form(H, G, d, e, size)
            for r in range(0, hi - lo, 64):
                part = dict(how, out=out[r:r + 64], gate=how["gate"][r:r + 64])
                m = len(p[r:r + 64])
                WA.gqa_window(q[r:r + 64], kc, vc, p[r:r + 64], s[r:r + 64], table, splits=sp, scratch=torch.empty(m * H * sp * (e + 2), device="cuda"), **part)
        else:
            rows = (hi - first + 31) // 32 * 32
            WA.fa_window(q, kc, vc, table, slot=self.slot, pos0=lo, ctx_k=torch.zeros(rows, G * stride, dtype=t, device="cuda"),
                         ctx_vt=torch.zeros(G * 128, rows, dtype=t, device="cuda"), **how)
        assert int(st) == 0
        return out[:, :H * e].view(hi - lo, H, e).cpu()


FORMS = [("general", F32, (5, 1, 14, 9)), ("general", F32, (4, 2, 200, 136)), ("general", BF16, (6, 3, 40, 56)), ("split", BF16, (4, 4, 64, 64)), ("split", BF16, (4, 2, 128, 128)),
         ("split", BF16, (8, 2, 64, 64)), ("split", BF16, (8, 1, 128, 128)), ("split", BF16, (4, 1, 256, 256)), ("tiles", BF16, (4, 2, 64, 64)), ("tiles", BF16, (8, 2, 128, 128)),
         ("tiles", BF16, (3, 1, 40, 24)), ("tiles", BF16, (2, 2, 72, 128))]
RULES = {"window": (False, 0.0, False), "chunk": (True, 0.0, False), "capped": (True, 3.0, False), "biased": (False, 0.0, True), "capped and biased chunk": (True, 5.0, True)}


@pytest.mark.parametrize("form,dtype,shape", FORMS, ids=lambda v: str(v).replace("torch.", ""))
@pytest.mark.parametrize("rule", list(RULES))
def test_attention_forms(form, dtype, shape, rule):
    """Sizes around pages, tiles and portions; rows from the middle of a stretch on."""
    chunked, cap, biased = RULES[rule]
    K = Keys(*shape, dtype, gain=2.0)
    scale = shape[2] ** -0.5
    for size in ((16, 65, 150) if form == "split" or chunked else (0, 16, 65, 150)):
        want = K.want(size, chunked, scale, cap, biased)
        for lo, hi in ((0, 300), (130, 131), (149, 152), (7, 199)):
            got = K.run(form, lo, hi, size, chunked, scale, cap, biased)
            assert _rel(got, want[lo:hi]) < _lim(dtype, 5e-6, 8e-3), (size, lo, hi)


@pytest.mark.parametrize("form,dtype,shape", FORMS, ids=lambda v: str(v).replace("torch.", ""))
@pytest.mark.parametrize("chunked", [False, True], ids=["window", "chunk"])
def test_a_single_key_at_the_edges(form, dtype, shape, chunked):
    """One key that takes most of a query's weight: just inside and just outside a window or a chunk, at page borders, at the first token."""
    size, scale = 96, shape[2] ** -0.5
    for query, key in ((299, 204), (299, 203), (299, 288), (299, 287), (287, 192), (192, 191), (192, 192), (95, 0), (96, 0), (191, 96), (191, 95), (160, 144), (160, 143), (0, 0)):
        K = Keys(*shape, dtype, seed=query)
        K.k[key] = (K.q[query].float().view(K.G, -1, K.d).mean(1) * 6.0 * (K.H // K.G) ** 0.5).to(dtype)
        for cap, biased in ((0.0, False), (30.0, False), (0.0, True)):
            want = K.want(size, chunked, scale, cap, biased)
            got = K.run(form, max(0, query - 2), query + 1, size, chunked, scale, cap, biased)
            assert _rel(got, want[max(0, query - 2):query + 1]) < _lim(dtype, 5e-6, 1e-2), (query, key, cap)


def test_scores_far_beyond_the_cap():
    """Scores that saturate in either direction: every key at the cap counts the same."""
    for form, dtype, shape in (FORMS[0], FORMS[2], FORMS[4], FORMS[9]):
        K = Keys(*shape, dtype, gain=500.0)
        want = K.want(80, True, shape[2] ** -0.5, 2.0, True)
        assert _rel(K.run(form, 0, 300, 80, True, shape[2] ** -0.5, 2.0, True), want) < _lim(dtype, 5e-6, 8e-3)


# ---------------------------------------------------------------------------------------------------------------------------
# router and experts
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("experts,top,groups,keep", [(1, 1, 1, 1), (12, 3, 3, 2), (8, 2, 8, 3), (9, 3, 3, 1), (64, 8, 8, 4), (66, 6, 2, 1), (256, 8, 8, 4), (256, 16, 64, 9), (40, 16, 1, 1),
                                                     (200, 5, 200, 5)])
def test_grouped_selection(experts, top, groups, keep):
    """Negative choice scores, ties (the lower index first), extreme logits, a correction that overrules the scores, more groups than lanes."""
    from ironpangu_b200.ops import _lib
    from ironpangu_b200.ops.stream_norm import _s

    g = torch.Generator().manual_seed(experts)
    M = 37
    z = torch.randn(M, experts, generator=g) * 2
    z[0], z[1], z[2] = -60.0, 0.25, z[2] * 30                   # scores of zero, all equal, saturated
    b = torch.randn(experts, generator=g) - 1.0
    b[: experts // 3] = -0.5
    for renorm in (0, 1):
        ids, wts = torch.zeros(M, top, dtype=torch.int32, device="cuda"), torch.zeros(M, top, device="cuda")
        zd, bd = z.cuda(), b.cuda()
        assert _lib.load().ifab_moe_route(zd.data_ptr(), experts, bd.data_ptr(), M, experts, top, 3, renorm, 1.0, groups, keep, ids.data_ptr(), wts.data_ptr(), None, _s()) == 0
        s = torch.sigmoid(z.double()).float()                   # f32 scores: what is equal there is a tie
        wid, ww = O.choose(s, b, top, groups, keep, ("weights_renormed",) if renorm else ())
        live = torch.tensor([r for r in range(M) if r not in (0, 2)])
        assert torch.equal(ids.cpu().long()[live], wid[live]) and (wts.cpu()[live] - ww[live]).abs().max() < 1e-6
        for r in (0, 2):                                         # saturated: ties may turn on the last bit of a score
            got = ids[r].cpu().long()
            assert len(set(got.tolist())) == top and len({int(i) // (experts // groups) for i in got}) <= keep
            assert ((s[r] + b)[got] - (s[r] + b)[wid[r]]).abs().max() < 1e-6
    for bad in ((experts, top, 3, groups, groups + 1), (experts, top, 4, groups, keep), (experts, top, 3, 0, 0)):
        assert _lib.load().ifab_moe_route(zd.data_ptr(), experts, bd.data_ptr(), M, *bad[:3], 0, 1.0, *bad[3:], ids.data_ptr(), wts.data_ptr(), None, _s()) != 0


def _expert_weights(width, shape, g, dtype):
    rn = lambda *s: torch.randn(*s, generator=g)
    w = {"router": 3 * rn(shape.experts, width) * width ** -0.5, "correction": 0.3 * rn(shape.experts) - 0.8}
    for e in range(shape.experts):
        w.update({f"e{e}.gate": rn(shape.ff, width) * width ** -0.5, f"e{e}.up": rn(shape.ff, width) * width ** -0.5, f"e{e}.down": rn(width, shape.ff) * shape.ff ** -0.5})
    return {k: v.to(BF16) for k, v in w.items()}


@DTYPES
@pytest.mark.parametrize("width,experts,top,groups,keep,ff,rows", [(64, 12, 3, 3, 2, 40, 1), (53, 9, 2, 3, 1, 19, 37), (136, 16, 5, 4, 2, 64, 300), (72, 1, 1, 1, 1, 8, 9), (256, 64, 8, 8, 4, 136, 70)])
def test_routed_experts_beside_another_sublayer(dtype, width, experts, top, groups, keep, ff, rows):
    """x + base + extra + experts(h) and the norm of it, in any number of rows; decode rows: the experts alone."""
    from ironpangu_b200.ops import stream_norm as N
    from ironpangu_b200.ops.routed_experts import ExpertBuffers, ExpertsShape, RoutedExperts

    g = torch.Generator().manual_seed(rows)
    sh = ExpertsShape(width, experts, top, ff, scoring="sigmoid", renorm=False, groups=groups, keep=keep, unit=N.GatedUnit("limited", 0.9, 1.702))
    w = _expert_weights(width, sh, g, dtype)
    ex = RoutedExperts(sh, w, "", "cuda", dtype, bias="correction")
    B = ExpertBuffers([sh], rows, dtype, "cuda")
    h = torch.randn(rows, width, generator=g).to(BF16)                    # equal operands in both types: no close call can go two ways
    pad = lambda t, dt: torch.nn.functional.pad(t, (0, _pad(width) - width)).to(dt).cuda()
    cfg = {"router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}, "expert": {"limit": 0.9}}
    y = O.experts(h.double(), cfg, {k: v.double() for k, v in w.items()}, "")
    x, base, extra = (torch.randn(rows, width, generator=g) for _ in range(3))
    gain = 1 + 0.2 * torch.randn(width, generator=g)
    xd, xa = pad(x, F32), pad(h, dtype)
    B.start(rows)
    part = pad(0.25 * base, F32), pad(0.75 * base, F32)                   # what ran beside the experts, as one piece and as parts of a sum
    ex.rows(B, rows, xa, None, gain.cuda(), 1e-4, xd, None, base=pad(base, F32) if rows == 9 else torch.stack(part), extra=pad(extra, F32))
    want = x.double() + base.double() + extra.double() + y
    assert _rel(xd[:, :width], want) < _lim(dtype, 3e-6, 8e-3)
    assert _rel(xa[:, :width], O.rms(want, 1e-4, gain.double())) < _lim(dtype, 3e-6, 1.2e-2) and not xd[:, width:].any() and not xa[:, width:].any()
    if dtype == BF16 and width % 8 == 0:
        n = min(rows, 2)
        out = torch.zeros(n, width, device="cuda")
        ex.decode_chosen(B, n, pad(h, dtype)[:n], out)                    # the choice of the rows above
        assert _rel(out, y[:n]) < 1e-2


# ---------------------------------------------------------------------------------------------------------------------------
# the ends of a parallel layer
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows", [1, 2])
@pytest.mark.parametrize("width,heads,ff,experts", [(64, 4, 0, 0), (72, 3, 51, 0), (136, 6, 200, 12), (2048, 16, 6144, 0), (1024, 8, 768, 64)])
def test_front_and_end_of_a_parallel_layer(rows, width, heads, ff, experts):
    from ironpangu_b200.ops import parallel_layer as PL
    from ironpangu_b200.ops import stream_norm as N
    from ironpangu_b200.ops.routed_experts import ExpertBuffers, ExpertsShape, RoutedExperts
    from ironpangu_b200.ops.window_attn import GroupedAttention, GroupedShape

    g = torch.Generator().manual_seed(width)
    rn = lambda *s: torch.randn(*s, generator=g)
    sh = GroupedShape(heads, heads, 24, 24, 0.2, 16, norm=True, keys_are_values=True, bias=True)
    w = {"q": rn(heads * 24, width), "k": rn(heads * 24, width), "g": rn(heads, width), "o": rn(width, heads * 24), "gate": rn(ff, width), "up": rn(ff, width), "down": rn(width, ff)}
    w = {k: (v * v.shape[1] ** -0.5 if v.numel() else v).to(BF16) for k, v in w.items()}
    w.update({"q.b": rn(heads * 24).to(BF16), "k.b": rn(heads * 24).to(BF16), "o.b": rn(width).to(BF16), "q.norm": rn(heads * 24), "k.norm": rn(heads * 24)})
    mix = GroupedAttention(sh, w, "", "cuda", BF16)
    unit = PL.UnitWeights(w, "", ff, N.GatedUnit("limited", 1.5, 1.702) if experts else N.GatedUnit("relu"), "cuda", BF16) if ff else None
    join = PL.Join(w["o"], w["o.b"], unit, "cuda", BF16)
    JB = PL.JoinBuffers([join], 2, BF16, "cuda")
    ex = EB = None
    if experts:
        es = ExpertsShape(width, experts, 3, 16, scoring="sigmoid", renorm=False, groups=4, keep=2, unit=N.GatedUnit("limited", 0.9, 1.702))
        ew = _expert_weights(width, es, g, BF16)
        ex, EB = RoutedExperts(es, ew, "", "cuda", BF16, bias="correction"), ExpertBuffers([es], 2, BF16, "cuda")
    ticket = torch.zeros(1, dtype=torch.int32, device="cuda")
    gain, x, y, extra = 1 + 0.2 * rn(width), rn(rows, width), rn(rows, width), rn(rows, width)
    for yy, ee in ((None, None), (y, None), (y, extra)):
        x2, xn, proj = torch.zeros(rows, width, device="cuda"), torch.zeros(rows, width, dtype=BF16, device="cuda"), torch.zeros(rows, sh.in_cols, dtype=BF16, device="cuda")
        dev = lambda t: None if t is None else t.cuda()
        PL.parallel_in(dev(yy), dev(ee), gain.cuda(), 1e-4, x.cuda(), x2, xn, mix, proj, join, JB, ex, EB, ticket.data_ptr())
        want = x.double() + (0 if yy is None else yy.double()) + (0 if ee is None else ee.double())
        h = O.rms(want, 1e-4, gain.double())
        assert _rel(x2, want) < 1e-6 and _rel(xn, h) < 5e-3
        h = xn.cpu().double()                                             # the rounded operand is the kernel's
        d = lambda n: w[n].double()
        z = torch.cat([h @ d("q").T + d("q.b"), h @ d("k").T + d("k.b"), h @ d("g").T], 1)
        assert _rel(proj[:, :z.shape[1]], z) < 5e-3 and not proj[:, z.shape[1]:].any()
        op = join.operand(JB, rows)
        act = torch.zeros(rows, 0, dtype=F64)
        if ff:
            act = _unit("limited" if experts else "relu", 1.5, 1.702, h @ d("gate").T, h @ d("up").T)
            assert _rel(op[:, join.at:join.at + ff], act) < 1e-2 and not op[:, join.at + ff:].any()
        if experts:
            ids, wts = O.route(h, ew["router"].double(), ew["correction"].double(), 3, 4, 2)
            assert torch.equal(EB.ids[3][:rows].cpu().long(), ids) and (EB.wts[3][:rows].cpu().double() - wts).abs().max() < 1e-5 and int(ticket) == 0
        mixed = rn(rows, heads * 24).to(BF16)
        op[:, :heads * 24] = mixed.cuda()
        act = op[:, join.at:join.at + ff].cpu().double()
        out = rn(rows, width)
        want = mixed.double() @ d("o").T + d("o.b") + (act @ d("down").T if ff else 0)
        got, got2 = out.cuda(), torch.zeros(rows, width, device="cuda")
        join.decode(JB, rows, got, got)
        got2 = join.rows(JB, rows, got2, None)
        got2 = got2.sum(0) if got2.dim() == 3 else got2
        assert _rel(got, want + out.double()) < 1e-5 and _rel(got2, want) < 4e-5
