"""Layers whose mixer and feed-forward read the same norm and are added together. The two ends of such a layer are shared: the front
(residual update, norm, the mixer's projection, the gated unit every row takes, the router) is one launch for decode rows
(``csrc/kernels/decode_post_norm.cu``), and the output projection of the mixer and of the unit are one product, their operands side by side
in a row."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from . import _lib
from . import stream_norm as N
from ._lib import check
from .stream_norm import _p, _s

F32 = torch.float32


def _pad(n: int) -> int:
    return (n + 7) // 8 * 8


class UnitWeights:
    """A gated feed-forward of ``ff`` columns: gate and up packed as [gate | up] with padded halves, down as it comes."""

    def __init__(self, W: Dict[str, torch.Tensor], p: str, ff: int, unit: N.GatedUnit, device, dtype: torch.dtype):
        gate, up, self.down = (W[p + n].to(device).to(dtype) for n in ("gate", "up", "down"))
        self.ff, self.unit = ff, unit
        F, width = _pad(ff), gate.shape[1]
        self.gate_up = torch.zeros(2 * F, _pad(width), dtype=dtype, device=device)
        self.gate_up[:ff, :width] = gate
        self.gate_up[F:F + ff, :width] = up


class Join:
    """The end of a parallel layer: [W_o | W_down] over rows [mixer result | unit result], each part padded to 8 columns."""

    def __init__(self, w_o: torch.Tensor, bias: Optional[torch.Tensor], unit: Optional[UnitWeights], device, dtype: torch.dtype):
        width, mixed = w_o.shape
        self.mixed, self.at = mixed, _pad(mixed)                  # columns of the mixer, where the unit's begin
        self.F = _pad(unit.ff) if unit else 0
        self.gate_up, self.unit = (unit.gate_up, unit.unit) if unit else (None, N.SILU)
        self.w = torch.zeros(width, self.at + self.F, dtype=dtype, device=device)
        self.w[:, :mixed] = w_o.to(device).to(dtype)
        if unit:
            self.w[:, self.at:self.at + unit.ff] = unit.down
        self.bias = None if bias is None else bias.to(device).float().contiguous()

    @property
    def key(self) -> tuple:
        return self.mixed, self.F

    def operand(self, B: "JoinBuffers", m: int) -> torch.Tensor:
        return B.rows[self.key][:m]

    def unit_rows(self, B: "JoinBuffers", xa: torch.Tensor, status_ptr) -> None:
        """The unit's part of the operand for any number of rows."""
        m = xa.shape[0]
        if self.F:
            N.gated_linear(xa, self.gate_up, self.unit, self.operand(B, m)[:, self.at:], None if B.pair is None else B.pair[:m, :2 * self.F], status_ptr)

    def rows(self, B: "JoinBuffers", m: int, y: torch.Tensor, status_ptr) -> torch.Tensor:
        """The product and its bias in f32: in ``y``, or for few rows as parts of a sum ``[parts, m, padded width]``; returns which."""
        width, k = self.w.shape
        n = 1 if B.parts is None else N.split_count(m, width, k)
        if n == 1:
            N.linear(self.operand(B, m), self.w, y[:, :width], bias=self.bias, status_ptr=status_ptr)
            return y
        parts = B.parts[:n, :m]
        N.split_linear(self.operand(B, m), self.w, parts[:, :, :width], self.bias, status_ptr)
        return parts

    def decode(self, B: "JoinBuffers", n: int, y: torch.Tensor, addend: Optional[torch.Tensor]) -> None:
        """The same for decode rows; ``addend`` (f32 rows, may be ``y``) is added."""
        N.gemv_act(self.operand(B, n), self.w, y, bias=self.bias, addend=addend)


class JoinBuffers:
    """Operand rows of every kind of :class:`Join` (columns that fill up a part stay zero)."""

    def __init__(self, joins, rows: int, dtype: torch.dtype, device):
        self.rows = {j.key: torch.zeros(rows, j.at + j.F, dtype=dtype, device=device) for j in joins}
        widest = max(j.F for j in joins)
        self.parts = torch.zeros(8, min(rows, 128), _pad(joins[0].w.shape[0]), dtype=F32, device=device) if dtype != F32 else None
        self.pair = torch.zeros(rows, 2 * widest, dtype=dtype, device=device) if widest and dtype == F32 else None


def parallel_in(y: Optional[torch.Tensor], extra: Optional[torch.Tensor], gain: torch.Tensor, eps: float, x_in: torch.Tensor, x_out: torch.Tensor, xn: torch.Tensor,
                mix, proj: torch.Tensor, join: Join, join_buffers: JoinBuffers, experts, expert_buffers, ticket_ptr: int) -> None:
    """Front of a parallel layer for one or two decode rows: ``x_out = x_in (+ y) (+ extra)``, ``xn = rms(x_out) * gain``, ``proj`` = the
    projection of ``mix`` (``w_in``, ``b_in``), the unit's part of the operand of ``join``, and the choice of ``experts`` into
    ``expert_buffers`` (both may be None)."""
    n, K = x_in.shape
    assert n <= 2 and x_in.stride(0) == x_out.stride(0) and mix.w_in.shape[1] == K
    cols = mix.shape.in_cols
    unit = (join.gate_up.data_ptr(), join.F, *join.unit.args, join.operand(join_buffers, n)[:, join.at:].data_ptr(), join.w.shape[1]) if join.F else (None, 0, 0, 0.0, 0.0, None, 0)
    router = (None, None, 0, None, 0, 0, 0, 0, 0.0, 1, 1, None, None)
    if experts is not None:
        s, B = experts.shape, expert_buffers
        router = (experts.w_router.data_ptr(), B.logits.data_ptr(), B.logits.stride(0), experts.bias.data_ptr(), s.experts, s.top, *s.rule, B.ids[s.top].data_ptr(),
                  B.wts[s.top].data_ptr())
    check(_lib.load().ifab_parallel_in_decode(_p(y), 0 if y is None else y.stride(0), _p(extra), 0 if extra is None else extra.stride(0), gain.data_ptr(), eps,
                                              x_in.data_ptr(), x_out.data_ptr(), x_in.stride(0), xn.data_ptr(), xn.stride(0), mix.w_in.data_ptr(), _p(mix.b_in),
                                              proj.data_ptr(), proj.stride(0), cols, *unit, *router, ticket_ptr, n, K, _s()), "parallel_in")
