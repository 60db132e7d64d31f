"""Small Fubelorn configurations and weights for the tests: sizes that stress one thing each, weights that make attention sharp (so that a key
at the edge of a window, a kept position, a block or a far key shows in the logits) and states that remember for unequal times."""
import torch


def _mlp(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def delta(heads=2, kv_heads=None, dim=12, vdim=None, conv=3):
    return {"heads": heads, "kv_heads": kv_heads or heads, "dim": dim, "vdim": vdim or dim, "conv": conv}


def memory(heads=2, dim=12, vdim=None, cap=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim or dim, "gate_cap": cap}


def kept(heads=4, kv_heads=2, dim=16, vdim=None, size=12, keep=3, scale=None, right=None, scales=(0.9, 0.8), ff=0):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim or dim, "mask": {"size": size, "keep_first": keep}, "scale": 2.5 * dim ** -0.5 if scale is None else scale}
    return {"type": "parallel", "mixer": {"left": left, "right": right or delta(), "left_scale": scales[0], "right_scale": scales[1]}, "mlp": _mlp(ff)}


def pooled(heads=4, kv_heads=2, dim=16, vdim=None, size=12, pool=4, rot=None, base=1e4, scaling=(4.0, 1.0, 4.0, 64), scale=None, right=None, scales=(1.1, 0.7), ff=0):
    r = {"dims": dim if rot is None else rot, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim or dim, "mask": {"size": size, "pool": pool}, "rot": r, "scale": 2.0 * dim ** -0.5 if scale is None else scale}
    return {"type": "parallel_2", "mixer": {"left": left, "right": right or memory(), "left_scale": scales[0], "right_scale": scales[1]}, "mlp": _mlp(ff)}


def ssd(heads=4, groups=2, state=12, vdim=8, conv=4, norm_groups=2, ff=0):
    return {"type": "mamba2", "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": norm_groups}, "mlp": _mlp(ff)}


def config(layers, *, width=64, vocab=96, eps=1e-5, streams=2, mult=0.8, taps=3):
    return {"architecture": "Fubelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "residual_mult": mult, "canon": {"taps": taps}, "layers": layers}


CASES = {
    # every mixer in unequal sizes, with and without a feed-forward
    "mixed": config([kept(6, 2, 40, 24, size=24, keep=5, right=delta(6, 3, 16, 24, 4), ff=200), ssd(6, 3, 20, 16, norm_groups=3, ff=72),
                     pooled(3, 3, 24, 56, size=6, pool=2, rot=16, scale=0.6, right=memory(3, 16, 40), scales=(1.2, 0.7)), ssd(4, 1, 16, 24, 2, 1),
                     kept(2, 1, 32, size=33, keep=17, right=delta(2, 1, 24, 40, 2), ff=64), pooled(4, 1, 32, size=16, pool=3, scale=0.5, scaling=None, right=memory(1, 32, 32, 3.0), ff=40)],
                    width=72, streams=3, taps=4),
    # nothing is a multiple of eight, or of four
    "odd": config([pooled(5, 1, 14, 9, size=7, pool=3, rot=6, right=memory(3, 9, 13), ff=51), ssd(3, 3, 11, 7, 3, 1, ff=19), kept(7, 7, 9, 5, size=33, keep=1, right=delta(3, 1, 7, 11, 5)),
                   ssd(2, 1, 5, 9, 2, 6), kept(3, 3, 22, size=5, keep=29, right=delta(5, 5, 13, 6, 2), ff=35)], width=53, vocab=131, eps=1e-3, streams=3, mult=1.3, taps=2),
    # the sizes of the tensor-core and split kernels: windows over several key tiles, more kept positions and blocks than a tile holds, groups of 1, 2, 4 and 8 heads
    "tiles": config([kept(4, 1, 128, size=70, keep=130, right=delta(2, 2, 64, 64, 4), ff=96), pooled(8, 1, 64, size=40, pool=1, right=memory(2, 64, 64)), ssd(4, 1, 64, 32, 4, 4, ff=64),
                     pooled(4, 2, 128, size=64, pool=8, rot=64, right=memory(1, 128, 64), ff=136), kept(2, 2, 64, size=1, keep=16, right=delta(4, 2, 32, 64))],
                    width=128, vocab=200, streams=4, taps=4),
    # heads wider than the tiles, in attention and in the states
    "wide": config([kept(2, 1, 144, 40, size=33, keep=4, right=delta(2, 1, 136, 72, 3), ff=24), pooled(3, 1, 40, 200, size=21, pool=6, right=memory(1, 144, 200)),
                    ssd(2, 1, 264, 136, 4, 1)], streams=2, taps=3),
    # one of everything: single heads, streams, taps, blocks and windows of one token
    "single": config([kept(1, 1, 8, size=1, keep=0, right=delta(1, 1, 1, 1, 1), ff=8), pooled(1, 1, 8, size=1, pool=1, rot=0, right=memory(1, 1, 1), ff=8), ssd(1, 1, 1, 1, 1, 1, ff=1),
                      kept(1, 1, 16, 8, size=9, keep=9, right=delta(1, 1, 8, 8, 2)), pooled(1, 1, 16, 8, size=16, pool=50, rot=2, right=memory(1, 8, 16))], streams=1, mult=1.0, taps=1),
}


def weights(cfg, seed=0):
    from ironpangu_b200.models.fubelorn import FubelornConfig, weight_shapes

    g = torch.Generator().manual_seed(seed)
    rn = lambda *s: torch.randn(s, generator=g)
    out = {}
    for name, shape in weight_shapes(FubelornConfig.from_dict(cfg)).items():
        last = name.split(".")[-1]
        if name == "embed":
            t = rn(*shape)
        elif "norm" in name or last == "D":
            t = 1.0 + 0.2 * rn(*shape)
        elif "canon" in name:
            t = 0.4 * rn(*shape)
        elif last == "mix":
            t = torch.eye(shape[0]) + 0.25 * rn(*shape)
        elif last == "in" and ".hc" in name:
            t = shape[0] ** -0.5 * (1.0 + 0.4 * rn(*shape))
        elif last == "out":
            t = 1.0 + 0.4 * rn(*shape)
        elif last == "conv":
            t = rn(*shape) * shape[1] ** -0.5
        elif last == "A_log":
            t = -0.5 + 0.8 * rn(*shape)
        elif last == "dt_bias":
            t = -2.0 + rn(*shape)
        elif name.endswith("f.b"):
            t = 3.0 + rn(*shape)
        elif last == "b" and len(shape) == 1:
            t = 0.5 * rn(*shape)
        else:
            t = rn(*shape) * shape[-1] ** -0.5
            if name.endswith((".i", ".f", "right.a", "right.b")):
                t = 1.5 * t
        out[name] = t.to(torch.bfloat16)
    return out


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
