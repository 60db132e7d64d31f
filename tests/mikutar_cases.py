"""Small Mikutar configurations and weights for the tests: sizes that stress one thing each, weights that make attention sharp (so that a key
at the edge of a window or a chunk, or far away, shows in the logits) and, on request, routers without close calls."""
import torch


def window(heads=4, kv_heads=2, dim=16, rot=None, base=1e4, size=12, scale=None, **mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "rot": {"dims": dim if rot is None else rot, "base": base}, "mask": {"size": size},
         "scale": 2.0 * dim ** -0.5 if scale is None else scale}
    return {"type": "attention", "mixer": m, "mlp": feed_forward(**mlp)}


def chunk(heads=4, kv_heads=2, dim=16, vdim=None, size=12, cap=7.0, scale=None, **mlp):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim or dim, "mask": {"size": size}, "softcap": cap, "scale": dim ** -0.5 if scale is None else scale}
    return {"type": "attention_2", "mixer": m, "mlp": feed_forward(**mlp)}


def feed_forward(ff=0, experts=0, top=1, groups=(1, 1), expert_ff=24, limit=1.1, shared=0, shared_limit=0.8):
    if not experts:
        return {"kind": "dense", "ff": ff} if ff else None
    f = {"kind": "moe", "expert": {"ff": expert_ff, "limit": limit}, "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}}}
    if shared:
        f["shared"] = {"ff": shared, "limit": shared_limit}
    return f


def config(layers, *, width=64, vocab=96, eps=1e-5, cap=9.0, loop=(0, 0, 1)):
    return {"architecture": "Mikutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers,
            "loop": dict(zip(("start", "stop", "times"), loop))}


CASES = {
    # both mixers in unequal sizes, every kind of feed-forward, none, a loop
    "mixed": config([window(6, 2, 40, rot=24, size=24, ff=200), chunk(3, 3, 24, 56, size=20, experts=12, top=3, groups=(3, 2), expert_ff=40, shared=72),
                     window(6, 3, 24, size=33), chunk(3, 1, 24, 16, size=27, experts=5, top=2), window(2, 1, 32, rot=8, size=50, experts=8, top=3, groups=(2, 1), shared=24)],
                    width=72, loop=(1, 3, 2)),
    # nothing is a multiple of eight, or of four
    "odd": config([window(5, 1, 14, rot=6, size=7, ff=51), chunk(7, 7, 9, 5, size=33, experts=9, top=2, groups=(3, 1), expert_ff=19, limit=0.6, shared=35, shared_limit=2.0),
                   window(3, 3, 22, rot=22, size=21, experts=4, top=4, groups=(4, 4), expert_ff=7)], width=53, vocab=131, eps=1e-3, cap=30.0, loop=(0, 1, 3)),
    # the sizes of the tensor-core and split kernels: windows and chunks over several key tiles, of one token, groups of 1, 2, 4 and 8 heads
    "tiles": config([window(4, 1, 128, size=150, base=5e5, ff=96), chunk(8, 1, 64, size=130, experts=16, top=3, groups=(4, 2), shared=64), window(2, 2, 64, size=1, ff=40),
                     chunk(4, 2, 128, size=64, ff=136), window(8, 4, 128, rot=64, size=64)], width=128, vocab=200, loop=(3, 5, 2)),
    # heads wider than the tiles
    "wide": config([window(2, 1, 144, rot=100, size=33, ff=24), chunk(3, 1, 40, 200, size=21), chunk(2, 2, 136, 48, size=40, experts=3, top=1, groups=(3, 2))]),
    # single heads, single experts, a chunk of one token, the whole model looped
    "single": config([window(1, 1, 8, size=9, experts=1, top=1, shared=8), chunk(1, 1, 8, size=1, ff=8), chunk(1, 1, 16, 8, size=16, experts=2, top=1, groups=(2, 1))],
                     loop=(0, 3, 2)),
}

MARK = 4           # columns of the residual that keep a token's mark when routers are separated


def weights(cfg, seed=0, separated=False):
    """``separated``: every token carries a pattern of signs in the first MARK columns, which no sublayer changes and the routers read, chosen so
    that the groups and experts chosen are well ahead of the next (a 16-bit rounding never turns a choice)."""
    from ironpangu_b200.models.mikutar import MikutarConfig, weight_shapes

    c = MikutarConfig.from_dict(cfg)
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g)
    out = {}
    for name, shape in weight_shapes(c).items():
        layer = c.layers[int(name[1:name.index(".")])] if name[0] == "l" else None
        if name == "embed":
            t = rn(*shape)
            if separated:
                bits = torch.arange(shape[0])[:, None] * 7 >> torch.arange(MARK) & 1
                t[:, :MARK] = (2.0 * bits - 1.0) * 2.0
        elif "norm" in name:
            t = 1.0 + 0.2 * rn(*shape)
            if separated and name.endswith("norm1"):
                t[:MARK] = 1.0
        elif name.endswith(".b"):
            t = 0.5 * rn(*shape)
        elif name.endswith("correction"):
            t = out.pop("correction", None)
            t = 0.3 * rn(*shape) - 0.8 if t is None else t
        elif name.endswith("router"):
            if separated:
                t, out["correction"] = _separated_router(shape, layer.experts, g)
            else:
                t = 2.0 * rn(*shape) * shape[-1] ** -0.5
        else:
            t = rn(*shape) * shape[-1] ** -0.5
            if name.endswith("mix.q") and layer.kind == "attention_2":
                t = t * 5.0                                    # scores of a few units, some at the cap: single keys stand out
            if name.endswith(("mix.q", "mix.k")) and layer.kind == "attention":
                t = t * torch.exp(0.6 * rn(shape[0] // layer.mixer.dim)).repeat_interleave(layer.mixer.dim)[:, None]      # heads of unequal size
            if name.endswith(("gate", "up")):
                t = t * 1.5
        if separated and name.endswith(("mix.o", "mix.o.b", ".down")):
            t[:MARK] = 0.0
        out[name] = t.to(torch.bfloat16)
    return out


def choice_gap(s, c, x):
    """How far choice scores ``[T, E]`` are from another choice of groups or experts."""
    T, E = c.shape
    v = c.view(T, x.groups, E // x.groups).sort(dim=-1, descending=True).values[..., :2].sum(-1).sort(dim=-1, descending=True)
    gap = torch.full((T,), 9.0)
    if x.keep < x.groups:
        gap = v.values[:, x.keep - 1] - v.values[:, x.keep]
    closed = torch.ones(T, x.groups, dtype=torch.bool).scatter(1, v.indices[:, :x.keep], False)
    best = c.view(T, x.groups, -1).masked_fill(closed[..., None], -99.0).view(T, E).sort(dim=-1, descending=True).values
    return gap if x.top == E else torch.minimum(gap, best[:, x.top - 1] - best[:, x.top])


def _separated_router(shape, x, g):
    E = shape[0]
    signs = 2.0 * (torch.arange(2 ** MARK)[:, None] >> torch.arange(MARK) & 1) - 1.0
    marks = torch.cat([signs * f for f in (0.4, 0.5, 0.6, 0.75, 0.9, 1.1, 1.3, 1.5, 1.8, 2.1)])
    best, best_gap = None, -1.0
    for _ in range(6000):
        a, b = torch.randn(E, MARK, generator=g) * 0.8, 0.5 * torch.randn(E, generator=g) - 0.8
        a, b = a.to(torch.bfloat16).float(), b.to(torch.bfloat16).float()
        s = torch.sigmoid(marks @ a.T)
        gap = float(choice_gap(s, s + b, x).min())
        if gap > best_gap:
            best, best_gap = (a, b), gap
        if best_gap > 0.05:
            break
    t = 0.002 * torch.randn(*shape, generator=g)
    t[:, :MARK] = best[0]
    return t, best[1]


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
