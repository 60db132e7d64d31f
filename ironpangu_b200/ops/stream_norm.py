"""Operators of decoders with an f32 residual stream and norms on sublayer outputs (``csrc/kernels/post_norm.cu``,
``decode_post_norm.cu``, ``linear_f32.cu``). Activations are bf16 (serving) or f32 (exact mode); the dtype of the tensors picks the
kernel. Thin wrappers: current stream, no allocation when outputs are given, no fallback."""
from __future__ import annotations

from typing import Optional

import torch

from . import _lib
from ._lib import check

BF16 = torch.bfloat16
ACTIVATIONS = {None: 0, "silu": 1, "sigmoid": 2, "gelu_tanh": 3}


def _s() -> int:
    return torch.cuda.current_stream().cuda_stream


def _p(t: Optional[torch.Tensor]) -> Optional[int]:
    return None if t is None else t.data_ptr()


def _f32(t: torch.Tensor) -> int:
    assert t.dtype in (BF16, torch.float32)
    return int(t.dtype == torch.float32)


def embed_rows(ids: torch.Tensor, table: torch.Tensor, x: torch.Tensor, xa: torch.Tensor, *, scale: float = 1.0, gain: Optional[torch.Tensor] = None,
               eps: float = 0.0, status_ptr: Optional[int] = None) -> None:
    """``x`` (f32 residual) = rows ``ids`` of ``table`` times ``scale``; ``xa`` (activation type) = x, or ``rms(x) * gain``."""
    T, D = x.shape
    assert ids.dtype == torch.int32 and x.dtype == torch.float32 and table.dtype == xa.dtype
    check(_lib.load().ifab_embed_rows(ids.data_ptr(), table.data_ptr(), table.stride(0), scale, _p(gain), eps, x.data_ptr(), x.stride(0), xa.data_ptr(),
                                      xa.stride(0), _f32(xa), T, D, table.shape[0], status_ptr, _s()), "embed_rows")


def post_norm_add(y: torch.Tensor, w: torch.Tensor, eps: float, x: torch.Tensor, xa: torch.Tensor, final: Optional[torch.Tensor] = None) -> None:
    """``x += rms(y) * w`` in f32; ``xa`` = x, or ``rms(x) * final`` (the norm ahead of the output matrix)."""
    T, D = x.shape
    assert y.dtype == x.dtype == w.dtype == torch.float32
    check(_lib.load().ifab_post_norm_add(y.data_ptr(), y.stride(0), w.data_ptr(), _p(final), eps, x.data_ptr(), x.stride(0), xa.data_ptr(), xa.stride(0),
                                         _f32(xa), T, D, _s()), "post_norm_add")


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


def gemv_act(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: Optional[str] = None) -> None:
    """``out = act(x @ w.T)`` for decode rows."""
    T, K = x.shape
    assert w.shape[1] == K and w.is_contiguous() and x.dtype == BF16
    check(_lib.load().ifab_gemv_act(x.data_ptr(), x.stride(0), w.data_ptr(), out.data_ptr(), out.stride(0), _f32(out), ACTIVATIONS[act], T, w.shape[0], K,
                                    _s()), "gemv_act")


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: Optional[str] = None, status_ptr: Optional[int] = None) -> None:
    """``out = act(x @ w.T)`` for any number of rows: the tensor-core GEMM for bf16 operands (bf16 or f32 result), true f32 otherwise."""
    T, K = x.shape
    N = w.shape[0]
    assert w.shape[1] == K and x.dtype == w.dtype and x.stride(1) == 1 and w.stride(1) == 1 and out.stride(1) == 1
    if x.dtype == torch.float32:
        check(_lib.load().ifab_linear_f32(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), T, N, K, ACTIVATIONS[act], _s()),
              "linear_f32")
    else:
        check(_lib.load().ifab_gemm_act_bf16(x.data_ptr(), x.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), _f32(out), None, 0,
                                             ACTIVATIONS[act], T, N, K, status_ptr, _s()), "gemm_act")
