"""Small Falinex configurations and weights for the tests: sizes that stress one thing each, weights that make attention sharp (so that
a key at a window's edge, a sink or a lost state shows in the logits)."""
import torch


def config(layers, *, width=64, vocab=96, eps=1e-5):
    return {"architecture": "Falinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def retention(heads=2, dim=16, vdim=16, decay=None, rot=None, base=1e4, ff=96, **kw):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1 - 2.0 ** -(2 + 2 * h) for h in range(heads)], "rot": {"dims": rot or dim, "base": base}}
    return {"type": "retention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None, **kw}


def lightning(heads=2, dim=16, vdim=16, decay=None, ff=96, **kw):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.5 + 0.49 * h / heads for h in range(heads)]}
    return {"type": "lightning", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None, **kw}


def attention(heads=4, kv_heads=2, dim=16, vdim=16, rot=None, base=1e4, window=12, scale=None, ff=96, **kw):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot or dim, "base": base}, "mask": {"size": window},
         "scale": dim ** -0.5 if scale is None else scale}
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None, **kw}


CASES = {
    # every mixer, different head sizes for keys and values, a layer without a feed-forward, shared layers in another order
    "mixed": config([attention(6, 2, 40, 24, rot=24, window=24, scale=0.21), retention(3, 24, 40, rot=16, ff=0), lightning(2, 32, 24),
                     retention(3, 24, 40, rot=16, ff=0, weights_of=1), attention(6, 2, 40, 24, rot=24, window=24, scale=0.21, weights_of=0)], width=72),
    # widths that are no multiple of eight, five heads, one value head per query head
    "odd": config([lightning(5, 12, 9, ff=51), attention(5, 5, 20, 9, rot=6, window=7, ff=51), retention(3, 10, 7, rot=4, ff=51)], width=52, vocab=131, eps=1e-4),
    # heads of 128 and 64: the split-KV and tensor-core forms without padding; windows of one token and of one page
    "tiles": config([attention(4, 1, 128, 128, window=150, base=5e5), lightning(2, 128, 128), retention(2, 128, 64), attention(4, 2, 64, 64, window=16),
                     attention(2, 2, 64, 64, window=1)], width=128, vocab=200),
    # heads wider than a tile: the general kernels in bf16 as well
    "wide": config([retention(1, 160, 136), attention(2, 1, 144, 136, window=33), lightning(1, 64, 160)], width=64),
}


def weights(cfg, seed=0):
    from ironpangu_b200.models.falinex import FalinexConfig, weight_shapes

    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in weight_shapes(FalinexConfig.from_dict(cfg)).items():
        if name == "embed":
            t = torch.randn(shape, generator=g)
        elif name.endswith("sink"):
            t = torch.randn(shape, generator=g) * 1.5
        elif name.endswith(("q.norm", "k.norm")):
            t = 1.6 + 0.2 * torch.randn(shape, generator=g)      # scores of a few units: single keys stand out
        elif "norm" in name:
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * shape[-1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()

