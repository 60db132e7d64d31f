"""Residual streams side by side with fixed mixing weights and a short causal convolution ahead of every sublayer
(``csrc/kernels/hyper_streams.cu``, for decode rows ``decode_hyper.cu``)."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from . import _lib
from ._lib import check
from .stream_norm import ACTIVATIONS, _f32, _p, _parts, _s

F32 = torch.float32
MOST_STREAMS, MOST_TAPS = 16, 16
FUSED_STREAMS = 4        # most streams of the fused decode form
BLOCK = 8                # rows of a CTA in steps of many rows


def embed_norm(ids: torch.Tensor, table: torch.Tensor, gain: torch.Tensor, eps: float, x: torch.Tensor, status_ptr: Optional[int] = None) -> None:
    """``x`` (f32 ``[T, D]``) = rows ``ids`` of ``table`` divided by their rms, times ``gain`` (one number on the device)."""
    T, D = x.shape
    assert ids.dtype == torch.int32 and x.dtype == F32 and x.stride(1) == 1
    check(_lib.load().ifab_embed_norm(ids.data_ptr(), table.data_ptr(), table.stride(0), gain.data_ptr(), eps, x.data_ptr(), x.stride(0), _f32(table), T, D,
                                      table.shape[0], status_ptr, _s()), "embed_norm")


def step_epoch(slots: torch.Tensor, epoch: torch.Tensor) -> None:
    """Turns over the epoch of every sequence of a step: histories are read on the side it names and written on the other."""
    check(_lib.load().ifab_step_epoch(slots.data_ptr(), epoch.data_ptr(), slots.numel(), _s()), "step_epoch")


class Sublayer:
    """What one sublayer needs of the streams: weights of its input (``in``), of its output (``out``, with the residual factor) and between the
    streams (``mix``), the number its norm multiplies by, the taps of the convolution and its history. Without ``hc`` tensors a plain residual."""

    def __init__(self, W: Dict[str, torch.Tensor], p: str, q: int, streams: int, mult: float, taps: int, width: int, device):
        f = lambda n: W[n].to(device).float()
        if streams:
            self.mix, self.inp, self.out = f(f"{p}hc{q}.mix").contiguous(), f(f"{p}hc{q}.in").contiguous(), (f(f"{p}hc{q}.out") * mult).contiguous()
        else:
            one = torch.ones(1, dtype=F32, device=device)
            self.mix, self.inp, self.out = one.view(1, 1), one, one * mult
        self.gain = f(f"{p}norm{q}").reshape(1).contiguous()
        self.taps, self.taps_w = taps, None
        if taps:
            self.taps_w = f(f"{p}canon{q}").t().contiguous()
        self.history: Optional[torch.Tensor] = None

    def make_history(self, slots: int, width: int, device) -> None:
        self.history = torch.zeros(slots, 2, self.taps - 1, width, dtype=F32, device=device) if self.taps > 1 else None


def streams_rows(x_in: torch.Tensor, x_out: Optional[torch.Tensor], y: Optional[torch.Tensor], before: Optional[Sublayer], after: Optional[Sublayer], gain: torch.Tensor,
                 eps: float, epoch: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, xa: Optional[torch.Tensor], total: Optional[torch.Tensor] = None) -> None:
    """The end of sublayer ``before`` (its result ``y``, f32 rows or parts of a sum; None: nothing is added and ``x_out`` stays as it is) and the
    front of ``after``, whose operand goes to ``xa``; without ``after`` the streams are summed and ``xa`` = ``rms(sum) * gain``. ``total`` (f32
    ``[T, D]``): the weighted sum ahead of the norm. Streams ``[T, S, D]``; ``x_in`` may repeat one row (stream stride 0)."""
    T, S, D = x_in.shape
    assert x_in.stride(2) == 1 and (x_out is None or x_out.stride(2) == 1) and (y is None or before is not None)
    a = after
    some = xa if xa is not None else total
    check(_lib.load().ifab_streams_rows(
        x_in.data_ptr(), x_in.stride(0), x_in.stride(1), _p(x_out), 0 if x_out is None else x_out.stride(0), 0 if x_out is None else x_out.stride(1), _p(y), *_parts(y),
        None if y is None else before.mix.data_ptr(), None if y is None else before.out.data_ptr(), None if a is None else a.inp.data_ptr(),
        (a.gain if a else gain).data_ptr(), eps, _p(a.taps_w) if a else None, a.taps if a else 0, _p(a.history) if a else None, epoch.data_ptr(), positions.data_ptr(),
        slots.data_ptr(), _p(total), 0 if total is None else total.stride(0), _p(xa), 0 if xa is None else xa.stride(0), _f32(some), T, S, D,
        1 if T <= 256 else BLOCK, _s()), "streams_rows")


def gemv_streams(x_in: torch.Tensor, x_out: Optional[torch.Tensor], y: Optional[torch.Tensor], before: Optional[Sublayer], after: Sublayer, eps: float, epoch: torch.Tensor,
                 positions: torch.Tensor, slots: torch.Tensor, w: torch.Tensor, out: torch.Tensor, act: Optional[str] = None) -> None:
    """:func:`streams_rows` and a linear over its operand (bf16 ``w`` ``[N, D]``, ``out = act(operand @ w.T)``) in one launch, for one or two rows of up to
    four streams."""
    T, S, D = x_in.shape
    N, a = w.shape[0], after
    assert w.shape[1] == D and w.is_contiguous() and (y is None or y.dim() == 2)
    check(_lib.load().ifab_gemv_streams(
        x_in.data_ptr(), x_in.stride(0), x_in.stride(1), _p(x_out), 0 if x_out is None else x_out.stride(0), 0 if x_out is None else x_out.stride(1), _p(y),
        0 if y is None else y.stride(0), None if y is None else before.mix.data_ptr(), None if y is None else before.out.data_ptr(), a.inp.data_ptr(), a.gain.data_ptr(), eps,
        _p(a.taps_w), a.taps, _p(a.history), epoch.data_ptr(), positions.data_ptr(), slots.data_ptr(), S, w.data_ptr(), out.data_ptr(), out.stride(0), _f32(out),
        ACTIVATIONS[act], T, N, D, _s()), "gemv_streams")
