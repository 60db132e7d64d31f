"""Plain restatement of the Ponenex decoder in PyTorch on the CPU: one function per mechanism, whole sequences at once, no cache, no
batching, no absorbed products, double precision unless the caller asks for another type. It shares no code with the package; the
tests compare the product path with it.

A configuration is the dictionary of a ``config.json``, weights are a dictionary of tensors under the checkpoint names. ``faults``
plants deliberate mistakes in the restatement, for tests that check that the comparison would notice them."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float, gain: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if gain is None else y * gain


def centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The norm whose stored weight is the gain's distance from one."""
    return rms(x, eps, 1.0 + w)


def turn_halves(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x ``[T, ..., d]``: column i < dims / 2 and column i + dims / 2 turn together by position * base^(-2i / dims)."""
    h = dims // 2
    ang = positions.to(F64)[:, None] * base ** (-2.0 * torch.arange(h, dtype=F64) / dims)
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (h,)
    c, s = torch.cos(ang).to(x.dtype).view(shape), torch.sin(ang).to(x.dtype).view(shape)
    u, v = x[..., :h], x[..., h:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def window_mask(n: int, size: int) -> torch.Tensor:
    """``[n, n]``: query i sees keys i - size + 1 .. i (all earlier keys without a size)."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None]
    return (j <= i) & ((i - j < size) if size else torch.ones(n, n, dtype=torch.bool))


def softmax_rows(scores: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    return torch.softmax(scores.masked_fill(~seen, -math.inf), -1)


def latent_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, faults=()) -> torch.Tensor:
    T, H, d, r, e, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    turn = (lambda x: x) if "no_rotation" in faults else (lambda x: turn_halves(x, pos, m["rot"]["dims"], m["rot"]["base"]))
    cq = rms(h @ w[p + "dq"].T, eps, w[p + "dq.norm"])
    q = (cq @ w[p + "uq"].T).view(T, H, d + r)
    q1, q2 = q[..., :d], turn(q[..., d:])
    kv = h @ w[p + "dkv"].T
    c = kv[:, :L] if "latent_not_normed" in faults else rms(kv[:, :L], eps, w[p + "dkv.norm"])
    k2 = turn(kv[:, L:])
    k1 = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, e)
    score = (torch.einsum("thd,shd->hts", q1, k1) + torch.einsum("thr,sr->hts", q2, k2)) * m["scale"]
    size = (m.get("mask") or {}).get("size", 0)
    size += ("window_plus_one" in faults) - ("window_minus_one" in faults)
    o = torch.einsum("hts,she->the", softmax_rows(score, window_mask(T, size)), v)
    if "no_gate" not in faults:
        o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * e) @ w[p + "o"].T


def gated_unit(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    g = h @ w[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h: torch.Tensor, w_router: torch.Tensor, bias: torch.Tensor, top: int):
    """(ids, weights) ``[T, top]``: the largest biased logits, weighted by the softmax over just these."""
    z = h @ w_router.T + bias
    best, ids = z.sort(dim=-1, descending=True, stable=True)
    return ids[:, :top], torch.softmax(best[:, :top], -1)


def experts(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, faults=()) -> torch.Tensor:
    E, top = m["router"]["experts"], m["router"]["top"]
    bias = w[p + "router.b"] * (0.0 if "no_bias" in faults else 1.0)
    ids, wts = route(h, w[p + "router"], bias, top)
    y = torch.zeros_like(h)
    for e in range(E):
        share = (wts * (ids == e)).sum(-1, keepdim=True)
        y = y + share * gated_unit(h, w, f"{p}e{e}.")
    if m.get("shared") and "no_shared" not in faults:
        s = gated_unit(h, w, p + "shared.")
        y = y + (s if "shared_not_gated" in faults else s * torch.sigmoid(h @ w[p + "shared.sg"].T))
    return y


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None, dtype=F64, faults=()) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``residuals`` (a list) receives the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = latent_attention(centred_norm(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.", eps, faults)
        x = x + mult * centred_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = experts(centred_norm(x, w[p + "norm2"], eps), layer["mlp"], w, p + "mlp.", faults)
            x = x + mult * centred_norm(y, w[p + "norm2b"], eps)
        if residuals is not None:
            residuals.append(x.clone())
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T
