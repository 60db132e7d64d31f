"""Plain restatement of the Mikutar decoder in PyTorch on the CPU: one function per mechanism, whole sequences at once, no cache, no
batching, double precision unless the caller asks for another type. It shares no code with the package; the tests compare the product
path with it.

A configuration is the dictionary of a ``config.json``, weights are a dictionary of tensors under the checkpoint names. ``faults``
plants deliberate mistakes in the restatement, for tests that check that the comparison would notice them."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float, gain: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def soft_limit(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def turn_neighbours(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x ``[T, heads, d]``: columns 2 i and 2 i + 1 below ``dims`` turn together by position * base^(-2 i / dims)."""
    ang = positions.to(F64)[:, None] * base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims)
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


def distances(n: int) -> torch.Tensor:
    return torch.arange(n)[:, None] - torch.arange(n)[None]


def window_seen(n: int, size: int) -> torch.Tensor:
    """``[n, n]``: query i sees keys i - size + 1 .. i."""
    d = distances(n)
    return (d >= 0) & (d < size)


def chunk_seen(n: int, size: int) -> torch.Tensor:
    """``[n, n]``: query i sees the keys up to i of its own stretch of ``size`` positions."""
    part = torch.arange(n) // size
    return (distances(n) >= 0) & (part[:, None] == part[None])


def bias_slopes(heads: int) -> torch.Tensor:
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=F64)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, seen: torch.Tensor, scale: float, cap: float = 0.0, slopes: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q ``[T, H, d]``, k ``[T, G, d]``, v ``[T, G, e]`` -> ``[T, H, e]``."""
    H, G = q.shape[1], k.shape[1]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    score = torch.einsum("thd,shd->hts", q, k) * scale
    if cap:
        score = soft_limit(score, cap)
    if slopes is not None:
        score = score - slopes.to(q.dtype)[:, None, None] * distances(q.shape[0]).to(q.dtype)
    return torch.einsum("hts,she->the", torch.softmax(score.masked_fill(~seen, -math.inf), -1), v)


def _size(m: dict, faults) -> int:
    return m["mask"]["size"] + ("mask_plus_one" in faults) - ("mask_minus_one" in faults)


def _finish(o, h, w, p, bias, faults):
    if "no_gate" not in faults:
        o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    y = o.reshape(o.shape[0], -1) @ w[p + "o"].T
    return y + w[p + "o.b"] if bias and "no_output_bias" not in faults else y


def windowed_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, faults=()) -> torch.Tensor:
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    b = 0.0 if "no_projection_bias" in faults else 1.0
    q, k = h @ w[p + "q"].T + b * w[p + "q.b"], h @ w[p + "k"].T + b * w[p + "k.b"]
    pos = torch.arange(T)
    turn = lambda x: turn_neighbours(x, pos, m["rot"]["dims"], m["rot"]["base"])
    if "norm_per_head" in faults:
        norm = lambda x, n, g: rms(x.view(T, n, d), eps, w[p + g].view(n, d)).reshape(T, -1)
    else:
        norm = lambda x, n, g: rms(x, eps, w[p + g])
    keys = turn(norm(k, G, "k.norm").view(T, G, d))
    values = k.view(T, G, d)
    if "values_after_norm" in faults:
        values = norm(k, G, "k.norm").view(T, G, d)
    if "values_are_turned" in faults:
        values = turn(values)
    o = attend(turn(norm(q, H, "q.norm").view(T, H, d)), keys, values, window_seen(T, _size(m, faults)), m["scale"])
    return _finish(o, h, w, p, True, faults)


def chunked_attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, faults=()) -> torch.Tensor:
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, G, d), (h @ w[p + "v"].T).view(T, G, e)
    seen = window_seen(T, _size(m, faults)) if "chunk_is_a_window" in faults else chunk_seen(T, _size(m, faults))
    o = attend(q, k, v, seen, m["scale"], 0.0 if "no_score_cap" in faults else m["softcap"], None if "no_slopes" in faults else bias_slopes(H))
    return _finish(o, h, w, p, False, faults)


MIXERS = {"attention": windowed_attention, "attention_2": chunked_attention}


def relu_unit(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (torch.relu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def limited_unit(h: torch.Tensor, w: Dict[str, torch.Tensor], p: str, limit: float, faults=()) -> torch.Tensor:
    g, u = h @ w[p + "gate"].T, h @ w[p + "up"].T
    if "no_limit" not in faults:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + (0.0 if "up_without_one" in faults else 1.0))) @ w[p + "down"].T


def choose(s: torch.Tensor, correction: torch.Tensor, top: int, count: int, keep: int, faults=()):
    """``(ids, weights)`` ``[T, top]``: experts chosen by score + correction among the ``keep`` best of ``count`` groups (a group is as good as its
    two best together), weighted by the score alone."""
    c = s if "no_correction" in faults else s + correction
    if "all_groups" not in faults:
        T, E = c.shape
        g = c.view(T, count, E // count)
        value = g.sort(dim=-1, descending=True).values[..., :1 if "group_by_best" in faults else 2].sum(-1)
        best = value.sort(dim=-1, descending=True, stable=True).indices[:, :keep]
        closed = torch.ones(T, count, dtype=torch.bool).scatter(1, best, False)
        c = g.masked_fill(closed[..., None], 0.0 if "closed_groups_score_zero" in faults else -math.inf).view(T, E)
    ids = c.sort(dim=-1, descending=True, stable=True).indices[:, :top]
    wts = (c if "weights_with_correction" in faults else s).gather(1, ids)
    return ids, wts / wts.sum(-1, keepdim=True) if "weights_renormed" in faults else wts


def route(h: torch.Tensor, w_router: torch.Tensor, correction: torch.Tensor, top: int, count: int, keep: int, faults=()):
    return choose(torch.sigmoid(h @ w_router.T), correction, top, count, keep, faults)


def experts(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, faults=()) -> torch.Tensor:
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    ids, wts = route(h, w[p + "router"], w[p + "correction"], r["top"], groups["count"], groups["keep"], faults)
    y = torch.zeros_like(h)
    for e in range(r["experts"]):
        y = y + (wts * (ids == e)).sum(-1, keepdim=True) * limited_unit(h, w, f"{p}e{e}.", m["expert"]["limit"], faults)
    if m.get("shared") and "no_shared" not in faults:
        y = y + limited_unit(h, w, p + "shared.", m["shared"]["limit"], faults)
    return y


def run_order(cfg: dict) -> list:
    """``[(layer, whether the embedding is added first)]`` in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    body = range(loop["start"], loop["stop"])
    order = [(i, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t > 0 and i == loop["start"]) for i in body]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None, dtype=F64, faults=()) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``residuals`` (a list) receives the residual stream after every layer run."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    first = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = first
    for i, add in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if add and "embedding_added_once" not in faults:
            x = x + first
        h = rms(x, eps, w[p + "norm1"])
        y = MIXERS[layer["type"]](h, layer["mixer"], w, p + "mix.", eps, faults)
        m = layer.get("mlp")
        if m and "serial" in faults:
            x, y = x + y, 0.0
            h = rms(x, eps, w[p + "norm1"])
        if m:
            y = y + (relu_unit(h, w, p + "mlp.") if m["kind"] == "dense" else experts(h, m, w, p + "mlp.", faults))
        x = x + y
        if residuals is not None:
            residuals.append(x.clone())
    logits = rms(x, eps, w["final.norm"]) @ w["embed"].T
    return logits if "no_logit_cap" in faults else soft_limit(logits, cfg["logit_softcap"])
