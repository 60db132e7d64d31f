"""Small Ponenex configurations and weights for the tests: sizes that stress one thing each, weights that make attention sharp (so that
a key at a window's edge or far away shows in the logits) and, on request, routers without close calls."""
import torch


def layer(heads=4, dim=16, rot_dim=16, vdim=16, kv_rank=32, q_rank=24, rot=None, base=1e4, window=12, scale=None, experts=4, top=2, ff=24, shared=16, mlp=True):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"dims": rot_dim if rot is None else rot, "base": base},
         "mask": {"size": window}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    f = None
    if mlp:
        f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
        if shared:
            f["shared"] = {"ff": shared}
    return {"type": "latent_attention", "mixer": m, "mlp": f}


def config(layers, *, width=64, vocab=96, eps=1e-5, mult=0.7, scale=1.3):
    return {"architecture": "Ponenex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "embedding": {"scale": scale}, "layers": layers}


CASES = {
    # layers of unequal sizes, one without a shared expert, one without a feed-forward; one expert of several, all experts
    "mixed": config([layer(6, 40, 24, 56, 72, 48, window=24, experts=6, top=1, ff=40, shared=72), layer(3, 20, 16, 24, 104, 40, rot=12, window=50, mlp=False),
                     layer(3, 20, 16, 24, 104, 40, rot=12, window=50, shared=0, experts=5, top=5), layer(1, 8, 8, 8, 16, 8, window=9, experts=1, top=1)], width=72),
    # nothing is a multiple of eight
    "odd": config([layer(5, 13, 6, 9, 21, 11, window=7, experts=3, top=2, ff=19, shared=35), layer(7, 9, 14, 5, 43, 30, rot=10, window=33, experts=7, top=4, ff=51, shared=3)],
                  width=52, vocab=131, eps=1e-3, mult=1.0, scale=0.6),
    # the tiles of the tensor-core prompt kernel: full heads, wide latents, a window over several key tiles, one of one token, none
    "tiles": config([layer(4, 128, 64, 128, 512, 96, window=150, base=5e5, experts=8, top=3, ff=64, shared=32), layer(2, 64, 64, 64, 256, 64, window=1),
                     layer(8, 64, 32, 128, 264, 64, window=0, experts=16, top=7, ff=40, shared=200)], width=128, vocab=200, mult=0.5, scale=1.0),
    # wider than the tiles: the general forms in bf16 as well
    "wide": config([layer(2, 144, 32, 48, 640, 40, window=33), layer(3, 24, 96, 136, 48, 40, window=21, rot=90), layer(4, 32, 200, 16, 520, 16, window=64)], width=64),
}

MARK = 5           # columns of the residual that keep a token's mark when routers are separated


def weights(cfg, seed=0, separated=False):
    """``separated``: every token carries a pattern of signs in the first MARK columns, which no sublayer changes and the routers read, chosen so
    that the last chosen expert is well ahead of the next (a 16-bit rounding never turns a choice)."""
    from ironpangu_b200.models.ponenex import PonenexConfig, weight_shapes

    c = PonenexConfig.from_dict(cfg)
    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(*s, generator=g)
    out = {}
    for name, shape in weight_shapes(c).items():
        if name == "embed":
            t = rn(*shape)
            if separated:
                bits = torch.arange(shape[0])[:, None] * 7 >> torch.arange(MARK) & 1
                t[:, :MARK] = (2.0 * bits - 1.0) * 2.0
        elif name.endswith(("dq.norm", "dkv.norm")):
            t = 1.0 + 0.2 * rn(*shape)
        elif "norm" in name:
            t = 0.2 * rn(*shape)
            if separated and name.endswith("norm2"):
                t[:MARK] = 0.0
        elif name.endswith("router.b"):
            t = 0.3 * rn(*shape)
        elif name.endswith("router"):
            t = _separated_router(shape, c.layers[int(name[1:name.index(".")])].mlp.top, g) if separated else 2.0 * rn(*shape) * shape[-1] ** -0.5
        else:
            t = rn(*shape) * shape[-1] ** -0.5
            if name.endswith("uq"):
                t = t * 2.5                                    # scores of a few units: single keys stand out
            if separated and name.endswith(("mix.o", ".down")):
                t[:MARK] = 0.0
        out[name] = t.to(torch.bfloat16)
    return out


def _separated_router(shape, top, g):
    E = shape[0]
    signs = 2.0 * (torch.arange(2 ** MARK)[:, None] >> torch.arange(MARK) & 1) - 1.0
    best, best_gap = None, -1.0
    for _ in range(300):
        a = torch.randn(E, MARK, generator=g)
        z = (signs @ a.T).sort(-1, descending=True).values
        gap = float((z[:, top - 1] - z[:, top]).min()) if top < E else 1.0
        if gap > best_gap:
            best, best_gap = a, gap
    t = 0.02 * torch.randn(*shape, generator=g)
    t[:, :MARK] = best * (4.0 / max(best_gap, 0.05)) ** 0.5
    return t


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
