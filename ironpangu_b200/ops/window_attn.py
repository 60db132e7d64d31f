"""Sliding-window softmax attention with sinks over paged keys / values (``csrc/kernels/window_attn.cu``)."""
from __future__ import annotations

from typing import Optional

import torch

from . import _lib
from ._lib import check
from .stream_norm import ACTIVATIONS, _f32, _p, _s


def qk_norm_rope_write(proj: torch.Tensor, offsets, q_gain: Optional[torch.Tensor], k_gain: Optional[torch.Tensor], eps: float, *, heads: int, kv_heads: int,
                       dim: int, vdim: int, rot: int, interleaved: bool, rope: Optional[torch.Tensor], positions: torch.Tensor, slots: torch.Tensor,
                       page_table: torch.Tensor, q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, status_ptr=None) -> None:
    """Packed projection rows -> normalised, rotated queries in ``q_out`` (``[T, heads * stride]``, stride >= dim) and normalised, rotated keys / plain values in the pages
    (``k_cache`` ``[pages, page_tokens, kv_heads, dim]``, ``v_cache`` ``[..., vdim]``). ``rope``: (cos, sin) of the rows, ``[T, rot / 2, 2]``
    (``linear_attn.RotaryTables``)."""
    pages, pt = k_cache.shape[:2]
    check(_lib.load().ifab_qk_norm_rope_write(proj.data_ptr(), proj.stride(0), _f32(proj), *offsets, _p(q_gain), _p(k_gain), eps, heads, kv_heads, dim, vdim, rot,
                                              int(interleaved), _p(rope), positions.data_ptr(), slots.data_ptr(), page_table.data_ptr(), page_table.shape[1],
                                              pt, pages, q_out.data_ptr(), q_out.stride(0), q_out.shape[1] // heads, k_cache.data_ptr(), v_cache.data_ptr(), proj.shape[0], status_ptr,
                                              _s()), "qk_norm_rope_write")


def window_attn(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, page_table: torch.Tensor, *,
                heads: int, window: int, scale: float, out: torch.Tensor, sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None,
                gate_act: Optional[str] = None, status_ptr=None) -> None:
    """Rows of any sequences: row at position i attends keys j with 0 <= i - j < window (0: all), exp(sink) joins the denominator,
    the result is multiplied by ``gate_act(gate)``."""
    pages, pt, G, d = k_cache.shape
    check(_lib.load().ifab_window_attn(q.data_ptr(), q.stride(0), q.shape[1] // heads, k_cache.data_ptr(), v_cache.data_ptr(), _f32(q), positions.data_ptr(), slots.data_ptr(),
                                       page_table.data_ptr(), page_table.shape[1], pt, pages, heads, G, d, v_cache.shape[3], window, scale, _p(sink), _p(gate),
                                       0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], out.data_ptr(), out.stride(0), q.shape[0], status_ptr,
                                       _s()), "window_attn")


SPLIT_KEYS = 64            # fewest keys per split of the split-KV decode form
SPLIT_CTAS = 600           # CTAs the splits of a launch aim at: more rows, longer splits


def split_form(heads: int, kv_heads: int, dim: int, vdim: int, window: int) -> int:
    """Most splits the split-KV decode kernels take for this shape, 0 when it needs the general kernel."""
    if dim != vdim or dim not in (64, 128, 256) or heads // kv_heads not in (1, 2, 4, 8) or (dim == 256 and heads // kv_heads == 8) or not window:
        return 0
    return max(1, min(64, (window + SPLIT_KEYS - 1) // SPLIT_KEYS))


def gqa_window(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, page_table: torch.Tensor, *,
               heads: int, window: int, scale: float, splits: int, scratch: torch.Tensor, out: torch.Tensor, sink: Optional[torch.Tensor] = None,
               gate: Optional[torch.Tensor] = None, gate_act: Optional[str] = None, status_ptr=None) -> None:
    """:func:`window_attn` by splits of the window (query heads of a group share the key loads), bf16, shapes of :func:`split_form`.
    ``splits``: the most to use; launches of many rows use fewer, longer ones."""
    pages, pt, G, d = k_cache.shape
    splits = max(1, min(splits, SPLIT_CTAS // (q.shape[0] * G)))
    kps = ((window + splits - 1) // splits + 31) // 32 * 32
    check(_lib.load().ifab_gqa_window_attention(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), positions.data_ptr(), slots.data_ptr(),
                                                page_table.data_ptr(), page_table.shape[1], pt, pages, scale, window, _p(sink), _p(gate),
                                                0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], q.shape[0], heads, G, d, kps, splits,
                                                scratch.data_ptr(), scratch.numel() * 4, out.data_ptr(), out.stride(0), status_ptr, _s()), "gqa_window")


def tile_width(dim: int) -> int:
    """Columns a query / key head takes as an operand of the tensor-core attention (0: too wide)."""
    return 64 if dim <= 64 else 128 if dim <= 128 else 0


def context_rows(count: int, window: int) -> int:
    """Rows of the gathered context of ``count`` consecutive queries, a whole number of gather tiles (upper bound)."""
    return (count + window - 1 + 31) // 32 * 32


def fa_window(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, page_table: torch.Tensor, *, slot: int, pos0: int, heads: int, window: int,
              scale: float, ctx_k: torch.Tensor, ctx_vt: torch.Tensor, out: torch.Tensor, sink: Optional[torch.Tensor] = None,
              gate: Optional[torch.Tensor] = None, gate_act: Optional[str] = None, status_ptr=None) -> None:
    """Prompt attention of consecutive positions ``pos0 ..`` of one sequence (keys already in its pages) on the tensor cores: the keys
    and values the rows can see are gathered out of the pages into ``ctx_k`` ``[rows, kv_heads * tile]`` / ``ctx_vt`` ``[kv_heads * 128,
    rows]``. ``q``: ``[m, heads * tile]``, columns past the head width zero; ``window`` 0: the whole context."""
    pages, pt, G, d = k_cache.shape
    m, e = q.shape[0], v_cache.shape[3]
    dp = q.shape[1] // heads
    first = max(0, pos0 - window + 1) if window else 0
    n = pos0 + m - first
    rows = (n + 31) // 32 * 32
    assert dp == tile_width(d) and e <= 128 and ctx_k.shape[0] >= rows and ctx_vt.shape[1] >= rows and ctx_k.shape[1] == G * dp
    lib = _lib.load()
    check(lib.ifab_ctx_gather_pad(k_cache.data_ptr(), v_cache.data_ptr(), page_table.data_ptr(), slot, page_table.shape[1], pt, pages, first, n, rows, G, d,
                                  dp, e, ctx_k.data_ptr(), ctx_vt.data_ptr(), ctx_vt.stride(0), status_ptr, _s()), "ctx_gather_pad")
    check(lib.ifab_fa_window_bf16(q.data_ptr(), q.stride(0), ctx_k.data_ptr(), ctx_k.stride(0), None, 0, 0, ctx_vt.data_ptr(), ctx_vt.stride(0), out.data_ptr(),
                                  out.stride(0), m, n, heads, heads // G, dp, e, pos0 - first, window, scale, _p(sink), _p(gate),
                                  0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], 0, status_ptr, _s()), "fa_window")
