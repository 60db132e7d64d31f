"""Sliding-window softmax attention with sinks over paged keys / values (``csrc/kernels/window_attn.cu``)."""
from __future__ import annotations

from typing import Optional

import torch

from . import _lib
from ._lib import check
from .stream_norm import ACTIVATIONS, _f32, _p, _s


def qk_norm_rope_write(proj: torch.Tensor, offsets, q_gain: Optional[torch.Tensor], k_gain: Optional[torch.Tensor], eps: float, *, heads: int, kv_heads: int,
                       dim: int, vdim: int, rot: int, interleaved: bool, freq: Optional[torch.Tensor], positions: torch.Tensor, slots: torch.Tensor,
                       page_table: torch.Tensor, q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, status_ptr=None) -> None:
    """Packed projection rows -> normalised, rotated queries in ``q_out`` and normalised, rotated keys / plain values in the pages
    (``k_cache`` ``[pages, page_tokens, kv_heads, dim]``, ``v_cache`` ``[..., vdim]``)."""
    pages, pt = k_cache.shape[:2]
    check(_lib.load().ifab_qk_norm_rope_write(proj.data_ptr(), proj.stride(0), _f32(proj), *offsets, _p(q_gain), _p(k_gain), eps, heads, kv_heads, dim, vdim, rot,
                                              int(interleaved), _p(freq), positions.data_ptr(), slots.data_ptr(), page_table.data_ptr(), page_table.shape[1],
                                              pt, pages, q_out.data_ptr(), q_out.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), proj.shape[0], status_ptr,
                                              _s()), "qk_norm_rope_write")


def window_attn(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, page_table: torch.Tensor, *,
                heads: int, window: int, scale: float, out: torch.Tensor, sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None,
                gate_act: Optional[str] = None, status_ptr=None) -> None:
    """Rows of any sequences: row at position i attends keys j with 0 <= i - j < window (0: all), exp(sink) joins the denominator,
    the result is multiplied by ``gate_act(gate)``."""
    pages, pt, G, d = k_cache.shape
    check(_lib.load().ifab_window_attn(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), _f32(q), positions.data_ptr(), slots.data_ptr(),
                                       page_table.data_ptr(), page_table.shape[1], pt, pages, heads, G, d, v_cache.shape[3], window, scale, _p(sink), _p(gate),
                                       0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], out.data_ptr(), out.stride(0), q.shape[0], status_ptr,
                                       _s()), "window_attn")
