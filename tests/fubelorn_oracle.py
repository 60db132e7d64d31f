"""Plain restatement of the Fubelorn decoder in PyTorch on the CPU: one function per mechanism, whole sequences at once, recurrences token by
token, no cache, no batching, double precision unless the caller asks for another type. It shares no code with the package; the tests compare
the product path with it.

A configuration is the dictionary of a ``config.json``, weights are a dictionary of tensors under the checkpoint names. ``faults``
plants deliberate mistakes in the restatement, for tests that check that the comparison would notice them."""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F

F64 = torch.float64


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def short_conv(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, reversed_taps: bool = False) -> torch.Tensor:
    """x ``[T, C]``, w ``[C, taps]``: out[t] = sum over k of w[:, taps - 1 - k] x[t - k], nothing ahead of the start."""
    taps, out = w.shape[1], torch.zeros_like(x)
    for k in range(min(taps, x.shape[0])):
        out[k:] += x[:x.shape[0] - k] * w[:, k if reversed_taps else taps - 1 - k]
    return out if bias is None else out + bias


def frequencies(dims: int, base: float, scaling: Optional[dict]) -> torch.Tensor:
    """Radians per position of every pair; long wavelengths are stretched by ``factor``, those in between by a mixture."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave, ctx = 2.0 * math.pi / f, scaling["original"]
            if wave > ctx / scaling["low"]:
                f /= scaling["factor"]
            elif wave >= ctx / scaling["high"]:
                s = (ctx / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def turn_halves(x: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor) -> torch.Tensor:
    """x ``[T, heads, d]``: columns i and i + n (n = len(freq)) turn together by position * freq[i]."""
    n, ang = freq.numel(), positions.to(F64)[:, None] * freq
    c, s = torch.cos(ang).to(x.dtype)[:, None], torch.sin(ang).to(x.dtype)[:, None]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def softmax_over(q, k, v, extra_k, extra_v, seen, seen_extra, scale):
    """q ``[T, H, d]``, k / v ``[T, G, .]`` and further keys ``[B, G, .]`` -> ``[T, H, e]`` with one softmax over both."""
    r = q.shape[1] // k.shape[1]
    k, v = torch.cat([extra_k, k]).repeat_interleave(r, 1), torch.cat([extra_v, v]).repeat_interleave(r, 1)
    score = torch.einsum("thd,shd->hts", q, k) * scale
    return torch.einsum("hts,she->the", torch.softmax(score.masked_fill(~torch.cat([seen_extra, seen], 1), -math.inf), -1), v)


def _distance(n: int) -> torch.Tensor:
    return torch.arange(n)[:, None] - torch.arange(n)[None]


def window_seen(n: int, size: int, keep: int = 0) -> torch.Tensor:
    """``[n, n]``: query i sees keys i - size + 1 .. i, and the first ``keep`` keys."""
    d = _distance(n)
    return (d >= 0) & ((d < size) | (torch.arange(n)[None] < keep))


def block_seen(n: int, size: int, pool: int) -> torch.Tensor:
    """``[n, n // pool]``: query i sees the blocks that end at i - size or before."""
    return torch.arange(n // pool)[None] * pool + pool - 1 <= torch.arange(n)[:, None] - size


def block_means(x: torch.Tensor, pool: int) -> torch.Tensor:
    b = x.shape[0] // pool
    return x[:b * pool].view(b, pool, *x.shape[1:]).mean(1)


def _shifted(size: int, faults) -> int:
    return size + ("mask_plus_one" in faults) - ("mask_minus_one" in faults)


def kept_attention(h, m, w, p, eps, faults=()):
    """Window with kept first tokens; q and k by their rms, no rotation."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, G, d), (h @ w[p + "v"].T).view(T, G, e)
    if "no_qk_norm" not in faults:
        q, k = unit_rms(q, eps), unit_rms(k, eps)
    keep = m["mask"]["keep_first"] + ("keep_plus_one" in faults) - ("keep_minus_one" in faults)
    none = torch.zeros(T, 0, dtype=torch.bool)
    o = softmax_over(q, k, v, k[:0], v[:0], window_seen(T, _shifted(m["mask"]["size"], faults), 0 if "no_kept" in faults else keep), none, m["scale"])
    return o.reshape(T, -1) @ w[p + "o"].T


def pooled_attention(h, m, w, p, eps, faults=()):
    """Window beside pooled blocks; rotated halves, a gate per head."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    freq = frequencies(rot["dims"], rot["base"], None if "no_scaling" in faults else rot.get("scaling"))
    q, k, v = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, G, d), (h @ w[p + "v"].T).view(T, G, e)
    pos, plain = torch.arange(T), k
    q, k = turn_halves(q, pos, freq), turn_halves(k, pos, freq)
    size, P = _shifted(m["mask"]["size"], faults), m["mask"]["pool"]
    extra = block_seen(T, size + ("pool_late" in faults) - ("pool_early" in faults), P)
    if "no_pool" in faults:
        extra = torch.zeros_like(extra)
    o = softmax_over(q, k, v, block_means(plain if "pool_before_rotation" in faults else k, P), block_means(v, P), window_seen(T, size), extra, m["scale"])
    if "no_gate" not in faults:
        o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T


def delta_rule(q, k, v, decay, beta, faults=()):
    """q, k ``[T, H, d]``, v ``[T, H, e]``, decay and beta ``[T, H]`` -> ``[T, H, e]``: the state forgets, corrects what it holds for the key, is read."""
    T, H, d = q.shape
    S, out = torch.zeros(H, d, v.shape[2], dtype=q.dtype), []
    for t in range(T):
        before = S
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", before if "correct_before_decay" in faults else S, k[t]))
        if "no_correction" in faults:
            u = beta[t][:, None] * v[t]
        read = S
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hde,hd->he", read if "read_before_write" in faults else S, q[t]))
    return torch.stack(out)


def delta_mixer(h, m, w, p, eps, faults=()):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rev = "taps_reversed" in faults
    conv = lambda n: F.silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"], None, rev))
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q, k = (unit(conv(n).view(T, G, d)).repeat_interleave(H // G, 1) for n in "qk")
    v = conv("v").view(T, H, e)
    if "no_q_factor" not in faults:
        q = q * d ** -0.5
    beta = torch.sigmoid(h @ w[p + "b"].T)
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * F.softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = unit_rms(delta_rule(q, k, v, decay, beta, faults), eps) * w[p + "norm"] * F.silu(h @ w[p + "g"].T).view(T, H, e)
    return o.reshape(T, -1) @ w[p + "o"].T


def ssd_scan(x, B, C, dt, log_decay):
    """x ``[T, H, e]``, B and C ``[T, H, N]``, dt and log_decay ``[T, H]`` -> ``[T, H, e]``."""
    S, out = torch.zeros(x.shape[1], B.shape[2], x.shape[2], dtype=x.dtype), []
    for t in range(x.shape[0]):
        S = torch.exp(log_decay[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hne,hn->he", S, C[t]))
    return torch.stack(out)


def ssd_mixer(h, m, w, p, eps, faults=()):
    T, H, e, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = F.silu(short_conv(xbc, w[p + "conv"], None if "no_conv_bias" in faults else w[p + "conv.b"], "taps_reversed" in faults))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    if "swap_bc" in faults:
        B, C = C, B
    x = x.view(T, H, e)
    B, C = (t.view(T, G, N).repeat_interleave(H // G, 1) for t in (B, C))
    dt = F.softplus(dt + w[p + "dt_bias"])
    y = ssd_scan(x, B, C, dt, -torch.exp(w[p + "A_log"]) * dt)
    if "no_skip" not in faults:
        y = y + w[p + "D"][:, None] * x
    y, gate, ng = y.reshape(T, inner), F.silu(z), m["norm_groups"]
    norm = lambda t: unit_rms(t.view(T, ng, inner // ng), eps).reshape(T, inner) * w[p + "norm"]
    y = norm(y) * gate if "gate_after_norm" in faults else norm(y * gate)
    return y @ w[p + "o"].T


def matrix_memory(q, k, v, log_in, log_forget, faults=()):
    """q, k ``[T, H, d]``, v ``[T, H, e]``, log gates ``[T, H]`` -> ``[T, H, e]``."""
    T, H, d = q.shape
    S, n = torch.zeros(H, d, v.shape[2], dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype)
    m = torch.full((H,), -math.inf if "maximum_from_minus_infinity" in faults else 0.0, dtype=q.dtype)
    out = []
    for t in range(T):
        new = torch.maximum(log_forget[t] + m, log_in[t])
        a, b = torch.exp(log_forget[t] + m - new), torch.exp(log_in[t] - new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n, m = a[:, None] * n + b[:, None] * k[t], new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        if "no_floor" in faults:
            den = (n * q[t]).sum(-1).abs() + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
    return torch.stack(out)


def memory_mixer(h, m, w, p, eps, faults=()):
    T, H, d, e, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q, k, v = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5, (h @ w[p + "k"].T).view(T, H, d), (h @ w[p + "v"].T).view(T, H, e)
    soft = (lambda z: z) if "no_gate_cap" in faults else (lambda z: cap * torch.tanh(z / cap))
    log_in, log_forget = soft(h @ w[p + "i"].T + w[p + "i.b"]), F.logsigmoid(soft(h @ w[p + "f"].T + w[p + "f.b"]))
    o = unit_rms(matrix_memory(q, k, v, log_in, log_forget, faults), eps).reshape(T, H * e)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(left, right):
    def mixer(h, m, w, p, eps, faults=()):
        l = m["left_scale"] * left(h, m["left"], w, p + "left.", eps, faults)
        return l if "no_right" in faults else l + m["right_scale"] * right(h, m["right"], w, p + "right.", eps, faults)
    return mixer


MIXERS = {"parallel": side_by_side(kept_attention, delta_mixer), "mamba2": ssd_mixer, "parallel_2": side_by_side(pooled_attention, memory_mixer)}


def dense(h, w, p, faults=()):
    return F.gelu(h @ w[p + "up"].T, approximate="tanh" if "gelu_tanh" in faults else "none") @ w[p + "down"].T


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None, dtype=F64, faults=()) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``residuals`` (a list) receives the sum of the streams after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    first = unit_rms(w["embed"][torch.as_tensor(tokens, dtype=torch.long)], eps) * w["embed.norm"]
    X = [first.clone() for _ in range(cfg["streams"])]
    S = range(len(X))

    def sublayer(q: int, p: str, fn) -> None:
        a, b, M = w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"], w[f"{p}hc{q}.mix"]
        h = unit_rms(sum(a[s] * X[s] for s in S), eps) * w[f"{p}norm{q}"]
        if "no_canon" not in faults:
            h = h + short_conv(h, w[f"{p}canon{q}"], None, "canon_reversed" in faults)
        y = mult * fn(h)
        if "mix_transposed" in faults:
            M = M.T
        X[:] = [sum(M[s, t] * X[s] for s in S) + b[t] * y for t in S]

    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        sublayer(1, p, lambda h: MIXERS[layer["type"]](h, layer["mixer"], w, p + "mix.", eps, faults))
        if layer.get("mlp"):
            sublayer(2, p, lambda h: dense(h, w, p + "mlp.", faults))
        if residuals is not None:
            residuals.append(sum(X))
    return (unit_rms(sum(X), eps) * w["final.norm"]) @ w["head"].T
