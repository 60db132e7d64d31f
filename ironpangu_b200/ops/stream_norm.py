"""Operators of decoders with an f32 residual stream and norms on sublayer outputs (``csrc/kernels/post_norm.cu``,
``decode_post_norm.cu``, ``linear_f32.cu``). Activations are bf16 (serving) or f32 (exact mode); the dtype of the tensors picks the
kernel. Thin wrappers: current stream, no allocation when outputs are given, no fallback."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from ._lib import check

BF16 = torch.bfloat16
ACTIVATIONS = {None: 0, "silu": 1, "sigmoid": 2, "gelu_tanh": 3, "gelu_erf": 4}


UNITS = {"silu": 0, "relu": 1, "limited": 2}


@dataclass(frozen=True)
class GatedUnit:
    """What a gated feed-forward makes of its two projections g and u: ``silu`` silu(g) u; ``relu`` relu(g) u; ``limited`` g' sigmoid(alpha g')
    (u' + 1) with g' = min(g, limit) and u' = u within [-limit, limit]."""

    kind: str = "silu"
    limit: float = 0.0
    alpha: float = 1.0

    def check(self) -> None:
        if self.kind not in UNITS or (self.kind == "limited" and self.limit <= 0):
            raise ValueError(f"gated unit {self} is not supported")

    @property
    def args(self) -> tuple:
        return UNITS[self.kind], self.limit, self.alpha


SILU = GatedUnit()


def _s() -> int:
    return torch.cuda.current_stream().cuda_stream


def _p(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def _f32(t: torch.Tensor) -> int:
    assert t.dtype in (BF16, torch.float32)
    return int(t.dtype == torch.float32)


def embed_rows(ids: torch.Tensor, table: torch.Tensor, x: torch.Tensor, xa: torch.Tensor, *, scale: float = 1.0, gain: Optional[torch.Tensor] = None,
               eps: float = 0.0, copy: Optional[torch.Tensor] = None, status_ptr: Optional[int] = None) -> None:
    """``x`` (f32 residual) = rows ``ids`` of ``table`` times ``scale``; ``xa`` (activation type) = x, or ``rms(x) * gain``. ``copy``: a second
    place for x."""
    T, D = x.shape
    assert copy is None or copy.stride(0) == x.stride(0)
    assert ids.dtype == torch.int32 and x.dtype == torch.float32 and table.dtype == xa.dtype
    check(_lib.load().ifab_embed_rows(ids.data_ptr(), table.data_ptr(), table.stride(0), scale, _p(gain), eps, x.data_ptr(), x.stride(0), _p(copy), xa.data_ptr(),
                                      xa.stride(0), _f32(xa), T, D, table.shape[0], status_ptr, _s()), "embed_rows")


def _parts(y: Optional[torch.Tensor]) -> tuple:
    """Row stride, parts and their distance of rows ``[T, D]`` or of parts of a sum ``[parts, T, D]``."""
    if y is None:
        return 0, 1, 0
    return (y.stride(1), y.shape[0], y.stride(0)) if y.dim() == 3 else (y.stride(0), 1, 0)


def post_norm_add(y: Optional[torch.Tensor], w: Optional[torch.Tensor], eps: float, x: torch.Tensor, xa: torch.Tensor, final: Optional[torch.Tensor] = None,
                  extra: Optional[torch.Tensor] = None) -> None:
    """``x += rms(y) * w [+ extra]`` in f32 (``y`` as it is without ``w``, nothing without ``y``); ``xa`` = x, or ``rms(x) * final`` (the norm
    ahead of the next linears). ``y`` may be the parts of a sum, ``[parts, T, D]``."""
    T, D = x.shape
    assert all(t is None or t.dtype == torch.float32 for t in (y, w, x, extra))
    check(_lib.load().ifab_post_norm_add(_p(y), *_parts(y), _p(w), _p(final), eps, x.data_ptr(), x.stride(0), _p(extra),
                                         0 if extra is None else extra.stride(0), xa.data_ptr(), xa.stride(0), _f32(xa), T, D, _s()), "post_norm_add")


def gated_rows(gu: torch.Tensor, unit: GatedUnit, out: torch.Tensor) -> None:
    """``out`` ``[T, F]`` = the gated unit of the halves of ``gu`` ``[T, 2 * n]`` (their first F columns)."""
    T, F = out.shape
    assert gu.dtype == out.dtype
    check(_lib.load().ifab_gated_rows(gu.data_ptr(), gu.stride(0), gu.shape[1] // 2, *unit.args, out.data_ptr(), out.stride(0), _f32(out), T, F, _s()), "gated_rows")


def rms_rows(x: torch.Tensor, w: torch.Tensor, eps: float, out: torch.Tensor, rows: Optional[torch.Tensor] = None) -> None:
    """``out[i] = rms(x[rows[i]]) * w`` (all rows in order without ``rows``)."""
    T = out.shape[0]
    assert x.dtype == w.dtype == torch.float32 and (rows is None or (rows.dtype == torch.int32 and rows.numel() == T))
    check(_lib.load().ifab_rms_rows(x.data_ptr(), x.stride(0), _p(rows), w.data_ptr(), eps, out.data_ptr(), out.stride(0), _f32(out), T, w.numel(), _s()),
          "rms_rows")


def group_norm_gate(o: torch.Tensor, gate: torch.Tensor, act: str, eps: float, out: torch.Tensor, groups: int, gain: Optional[torch.Tensor] = None) -> None:
    """``out = (o / rms of each of the groups [* gain]) * act(gate)`` for f32 ``o`` ``[T, groups * n]``."""
    T, K = o.shape
    assert o.dtype == torch.float32 and gate.dtype == out.dtype and K % groups == 0
    check(_lib.load().ifab_group_norm_gate(o.data_ptr(), o.stride(0), _p(gain), eps, gate.data_ptr(), gate.stride(0), ACTIVATIONS[act], out.data_ptr(),
                                           out.stride(0), _f32(out), T, groups, K // groups, _s()), "group_norm_gate")


def gate_rows(o: torch.Tensor, head_stride: int, gate: torch.Tensor, act: str, out: torch.Tensor, heads: int, n: int) -> None:
    """``out[t, h * n + j] = o[t, h * head_stride + j] * act(gate[t, h * n + j])``."""
    check(_lib.load().ifab_gate_rows(o.data_ptr(), o.stride(0), head_stride, gate.data_ptr(), gate.stride(0), ACTIVATIONS[act], out.data_ptr(),
                                     out.stride(0), _f32(out), out.shape[0], heads, n, _s()), "gate_rows")


def gemv_post_norm(y: torch.Tensor, norm_w: torch.Tensor, eps: float, x_in: torch.Tensor, x_out: torch.Tensor, w: torch.Tensor, out: torch.Tensor,
                   act: Optional[str] = None, next_norm: Optional[torch.Tensor] = None) -> None:
    """``x_out = x_in + rms(y) * norm_w``; ``out = act(bf16(x_out) @ w.T)``, or of ``bf16(rms(x_out) * next_norm)``, in one launch (decode
    rows)."""
    T, K = y.shape
    N = w.shape[0]
    assert w.shape[1] == K and w.is_contiguous() and x_in.stride(0) == x_out.stride(0)
    check(_lib.load().ifab_gemv_post_norm(y.data_ptr(), y.stride(0), norm_w.data_ptr(), _p(next_norm), eps, x_in.data_ptr(), x_out.data_ptr(), x_in.stride(0), w.data_ptr(),
                                          out.data_ptr(), out.stride(0), _f32(out), ACTIVATIONS[act], T, N, K, _s()), "gemv_post_norm")


def gemv_group_norm(o: torch.Tensor, gate: torch.Tensor, gate_act: str, eps: float, w: torch.Tensor, out: torch.Tensor, groups: int,
                    gain: Optional[torch.Tensor] = None) -> None:
    """``out = bf16((o / rms per group [* gain]) * gate_act(gate)) @ w.T`` in one launch (decode rows)."""
    T, K = o.shape
    N = w.shape[0]
    assert w.shape[1] == K and w.is_contiguous() and gate.dtype == BF16
    check(_lib.load().ifab_gemv_group_norm(o.data_ptr(), o.stride(0), _p(gain), eps, groups, gate.data_ptr(), gate.stride(0), ACTIVATIONS[gate_act],
                                           w.data_ptr(), out.data_ptr(), out.stride(0), _f32(out), 0, T, N, K, _s()), "gemv_group_norm")


def gemv_act(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: Optional[str] = None, bias: Optional[torch.Tensor] = None,
             addend: Optional[torch.Tensor] = None) -> None:
    """``out = act(x @ w.T + bias + addend)`` for decode rows; ``bias`` f32 ``[N]``, ``addend`` f32 rows (may be ``out``)."""
    T, K = x.shape
    assert w.shape[1] == K and w.is_contiguous() and x.dtype == BF16
    check(_lib.load().ifab_gemv_act(x.data_ptr(), x.stride(0), w.data_ptr(), _p(bias), _p(addend), 0 if addend is None else addend.stride(0), out.data_ptr(),
                                    out.stride(0), _f32(out), ACTIVATIONS[act], T, w.shape[0], K, _s()), "gemv_act")


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: Optional[str] = None, status_ptr: Optional[int] = None,
           bias: Optional[torch.Tensor] = None, cap: float = 0.0) -> None:
    """``out = act(x @ w.T + bias)`` for any number of rows: the tensor-core GEMM for bf16 operands (bf16 or f32 result), true f32 otherwise.
    ``bias``: f32 ``[N]``; ``cap`` > 0: ``cap * tanh(out / cap)`` at the end."""
    T, K = x.shape
    N = w.shape[0]
    assert w.shape[1] == K and x.dtype == w.dtype and x.stride(1) == 1 and w.stride(1) == 1 and out.stride(1) == 1
    assert bias is None or (bias.dtype == torch.float32 and bias.numel() >= N)
    if x.dtype == torch.float32:
        check(_lib.load().ifab_linear_f32(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), _p(bias), cap, T, N, K,
                                          ACTIVATIONS[act], _s()), "linear_f32")
    else:
        check(_lib.load().ifab_gemm_epilogue_bf16(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), _f32(out), None, 0,
                                                  _p(bias), ACTIVATIONS[act], cap, T, N, K, status_ptr, _s()), "gemm_epilogue")


def split_count(rows: int, n: int, k: int) -> int:
    """Parts along K that give a product of one tile row (128) about two CTAs an SM; 1 when it has enough columns or is too short."""
    if rows > 128:
        return 1
    blocks = (k + 63) // 64
    want = max(1, min(8, 296 // ((n + 31) // 32), blocks // 4))
    per = (blocks + want - 1) // want
    return (blocks + per - 1) // per


def split_linear(x: torch.Tensor, w: torch.Tensor, parts: torch.Tensor, bias: Optional[torch.Tensor] = None, status_ptr: Optional[int] = None) -> None:
    """``parts`` (f32 ``[parts, T, N]``, T <= 128): their sum is ``x @ w.T + bias``."""
    T, K = x.shape
    S, _, N = parts.shape
    assert parts.shape[1] == T and w.shape == (N, K) and x.dtype == w.dtype == BF16 and parts.stride(2) == 1
    check(_lib.load().ifab_gemm_split_bf16(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), parts.data_ptr(), parts.stride(1), parts.stride(0), S, _p(bias), T, N, K,
                                           status_ptr, _s()), "gemm_split")


def gated_linear(x: torch.Tensor, w: torch.Tensor, unit: GatedUnit, out: torch.Tensor, pair: Optional[torch.Tensor] = None, status_ptr: Optional[int] = None) -> None:
    """``out`` ``[T, F]`` = the gated unit of ``x @ gate.T`` and ``x @ up.T`` with ``w`` = [gate | up] ``[2 F, K]``: one launch for bf16; in f32 the
    two projections go through ``pair`` ``[T, 2 F]``."""
    T, K = x.shape
    F = w.shape[0] // 2
    assert w.shape == (2 * F, K) and out.shape == (T, F) and x.dtype == w.dtype == out.dtype and out.stride(1) == 1 and x.stride(1) == 1
    if x.dtype == torch.float32:
        linear(x, w, pair)
        gated_rows(pair, unit, out)
    else:
        check(_lib.load().ifab_gemm_gated_bf16(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), *unit.args, T, F, K, status_ptr,
                                               _s()), "gemm_gated")
