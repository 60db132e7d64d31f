"""Checkpoint directories of the families in ``registry.py``: ``config.json`` beside one or more safetensors files. A family brings its
configuration class (``from_dict`` / ``to_dict``) and the names and shapes of its tensors; reading and writing is the same for all."""
from __future__ import annotations

import json
import struct
from pathlib import Path
from typing import Callable, Dict

import torch

DTYPES = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16}


def pad8(n: int) -> int:
    """Elements of a row whose 16-bit form is a whole number of 16-byte chunks."""
    return (n + 7) // 8 * 8


def save(path, cfg, weights: Dict[str, torch.Tensor]) -> None:
    """Write ``config.json`` and ``model.safetensors`` (bf16)."""
    d = Path(path)
    d.mkdir(parents=True, exist_ok=True)
    (d / "config.json").write_text(json.dumps(cfg.to_dict(), indent=1))
    hdr, blobs, at = {}, [], 0
    for n, t in weights.items():
        raw = t.detach().to(torch.bfloat16).cpu().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        hdr[n] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(hdr).encode()
    head += b" " * (-len(head) % 8)
    (d / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))


def load(path, config_of: Callable[[dict], object], shapes_of: Callable[[object], Dict[str, tuple]]) -> tuple:
    """``(config, weights on the host)`` of a checkpoint directory; every expected tensor must be there with its shape."""
    from ..runtime.plan_engine import SafetensorsDir

    c = config_of(json.loads((Path(path) / "config.json").read_text()))
    src = SafetensorsDir(str(path))
    out = {}
    for name, shape in shapes_of(c).items():
        if name not in src.tensors:
            raise ValueError(f"the checkpoint has no tensor {name}")
        _, _, _, dt, have = src.tensors[name]
        if tuple(have) != tuple(shape) or dt not in DTYPES:
            raise ValueError(f"{name}: {dt} {list(have)} in the checkpoint, {list(shape)} expected")
        out[name] = torch.from_numpy(src.bytes_of(name).copy()).view(DTYPES[dt]).view(tuple(shape))
    return c, out


def param_count(shapes: Dict[str, tuple]) -> int:
    n = 0
    for shape in shapes.values():
        k = 1
        for d in shape:
            k *= d
        n += k
    return n
