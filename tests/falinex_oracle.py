"""Plain restatement of the Falinex decoder in PyTorch on the CPU: one function per mechanism, whole sequences at once, no cache,
no chunking, double precision unless the caller passes float tensors. It shares no code with the package; the tests compare the
product path with it.

A configuration is the dictionary of a ``config.json`` (``layers``, ``norm.eps``, ``vocab``, ``width``), weights are a dictionary
of tensors under the checkpoint names. ``faults`` plants one deliberate mistake in the restatement, for tests that check that
the comparison would notice it."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms(x: torch.Tensor, eps: float, w: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rotate(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, interleaved: bool) -> torch.Tensor:
    """x ``[T, heads, d]``; the first ``dims`` columns of every head turn by position * base^(-2i / dims)."""
    i = torch.arange(dims // 2, dtype=F64)
    ang = positions.to(F64)[:, None] * base ** (-2.0 * i / dims)
    c, s = torch.cos(ang)[:, None].to(x.dtype), torch.sin(ang)[:, None].to(x.dtype)
    out = x.clone()
    if interleaved:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    else:
        h = dims // 2
        u, v = x[..., :h], x[..., h:dims]
        out[..., :h], out[..., h:dims] = u * c - v * s, v * c + u * s
    return out


def decayed_state(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: Optional[torch.Tensor] = None):
    """q, k ``[T, H, d]``, v ``[T, H, e]``: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t. Returns (o ``[T, H, e]``, S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hd,hde->he", q[t], S))
    return torch.stack(out), S


def retention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rotate((h @ w[p + "q"].T).view(T, H, d), pos, m["rot"]["dims"], m["rot"]["base"], False)
    k = rotate((h @ w[p + "k"].T).view(T, H, d), pos, m["rot"]["dims"], m["rot"]["base"], False) * d ** -0.5
    v = (h @ w[p + "v"].T).view(T, H, e)
    o, _ = decayed_state(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o, eps).reshape(T, H * e) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def lightning(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(h @ w[p + n].T).view(T, H, d) for n in "qk")
    v = silu(h @ w[p + "v"].T).view(T, H, e)
    o, _ = decayed_state(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (rms(o.reshape(T, H * e), eps, w[p + "norm"]) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def windowed_softmax(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int, sink: torch.Tensor) -> torch.Tensor:
    """q ``[T, H, d]``, k ``[T, G, d]``, v ``[T, G, e]``; row i sees keys j with 0 <= i - j < window; exp(sink_h) joins the
    denominator of head h."""
    T, H, _ = q.shape
    r = H // k.shape[1]
    s = torch.einsum("thd,shd->hts", q, k.repeat_interleave(r, 1)) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    s = s.masked_fill(~((j <= i) & (i - j < window)), -math.inf)
    full = torch.cat([s, sink[:, None, None].expand(H, T, 1)], -1)
    a = torch.softmax(full, -1)[..., :T]
    return torch.einsum("hts,shd->thd", a, v.repeat_interleave(r, 1))


def attention(h: torch.Tensor, m: dict, w: Dict[str, torch.Tensor], p: str, eps: float, faults=()) -> torch.Tensor:
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    rot = lambda x: rotate(x, pos, m["rot"]["dims"], m["rot"]["base"], True)
    q = rot(rms((h @ w[p + "q"].T).view(T, H, d), eps, w[p + "q.norm"]))
    k = rot(rms((h @ w[p + "k"].T).view(T, G, d), eps, w[p + "k.norm"]))
    v = (h @ w[p + "v"].T).view(T, G, e)
    sink = w[p + "sink"]
    if "no_sink" in faults:
        sink = torch.full_like(sink, -math.inf)
    size = m["mask"]["size"] + (1 if "window_plus_one" in faults else 0) - (1 if "window_minus_one" in faults else 0)
    o = windowed_softmax(q, k, v, m["scale"], size, sink).reshape(T, H * e)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"retention": retention, "lightning": lightning, "attention": attention}


def owner(cfg: dict, i: int) -> int:
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None, dtype=F64, faults=()) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``residuals`` (a list) receives the residual stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        mix = MIXERS[layer["type"]]
        args = (x, layer["mixer"], w, p + "mix.", eps)
        y = mix(*args, faults) if layer["type"] == "attention" else mix(*args)
        x = x + rms(y, eps, w[p + "norm1"])
        if layer.get("mlp"):
            x = x + rms(gelu_tanh(x @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T, eps, w[p + "norm2"])
        if residuals is not None:
            residuals.append(x.clone())
    return rms(x, eps, w["final.norm"]) @ w["head"].T
