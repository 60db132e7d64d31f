"""Routed experts (gated units) with an optional gated shared expert for decoders with an f32 residual stream: router in 32-bit, dispatch on
the device, grouped products, and one kernel that sums the chosen experts, applies the output norm (or adds what ran beside the experts),
updates the residual and norms the next operand (``csrc/kernels/moe_rows.cu``, ``moe_prefill.cu``, ``tc_grouped.cu``,
``linear_f32.cu``; decode rows: ``decode_post_norm.cu``, ``decode_moe.cu``)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch

from . import _lib
from . import decode as K
from . import prefill as P
from . import stream_norm as N
from ._lib import check
from .stream_norm import _f32, _p, _s

BF16, F32 = torch.bfloat16, torch.float32
SCORING = {"softmax": 0, "sigmoid_bias": 1, "biased_logits": 2, "sigmoid": 3}


def _pad(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class ExpertsShape:
    width: int
    experts: int
    top: int
    ff: int
    shared_ff: int = 0     # 0: no shared expert
    scoring: str = "biased_logits"
    renorm: bool = True
    groups: int = 1        # groups of neighbours, of which the best ``keep`` are open
    keep: int = 1
    unit: N.GatedUnit = N.SILU

    def check(self) -> None:
        if min(self.width, self.experts, self.top, self.ff) < 1 or self.shared_ff < 0:
            raise ValueError("routed experts: sizes must be positive")
        if self.top > self.experts or self.top > 16 or self.experts > 256:
            raise ValueError(f"routed experts: {self.top} of {self.experts} experts are not supported")
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep <= self.groups or self.top > self.keep * (self.experts // self.groups):
            raise ValueError(f"routed experts: {self.top} of {self.experts} experts in {self.keep} of {self.groups} groups are not supported")
        self.unit.check()

    @property
    def rule(self) -> tuple:
        """How the selection kernels choose: scoring, renormalisation, factor, groups, open groups."""
        return SCORING[self.scoring], int(self.renorm), 1.0, self.groups, self.keep

    @property
    def slot_cols(self) -> int:
        return max(_pad(self.ff), _pad(self.shared_ff))


class ExpertBuffers:
    """Work buffers of the expert layers of a model for up to ``rows`` rows."""

    def __init__(self, shapes, rows: int, dtype: torch.dtype, device):
        z = lambda *s, dt=dtype: torch.zeros(*s, dtype=dt, device=device)
        self.logits = z(rows, max(s.experts for s in shapes) + 1, dt=F32)
        self.shared_w = z(rows, dt=F32)
        self.ids = {t: z(rows, t, dt=torch.int32) for t in {s.top for s in shapes}}
        self.wts = {t: z(rows, t, dt=F32) for t in self.ids}
        self.route = {(s.top, s.experts): P.DispatchBuffers(rows, s.top, s.experts, device) for s in shapes}
        self.slots = {(s.top, s.slot_cols): z(min(rows, 8), s.top + 1, s.slot_cols) for s in shapes} if dtype == BF16 else {}
        width, routes = _pad(shapes[0].width), rows * max(s.top for s in shapes)
        mpad = (rows + 127) // 128 * 128
        f = 1 if dtype == BF16 else 2                                     # f32: gate | up pairs stay apart until the down product
        self.xp = z(routes, width) if dtype == BF16 else None
        self.act = {s.ff: z(routes, f * _pad(s.ff)) for s in shapes}
        self.y = z(routes, width)
        self.sact = {s.shared_ff: z(mpad, f * _pad(s.shared_ff)) for s in shapes if s.shared_ff}
        self.sy = z(mpad, width) if self.sact else None
        # the shared expert as a one-expert group over the rows of a step: its tile table never changes but for the count
        self.row_tiles = torch.tensor([[0, i * 128, 128, 0] for i in range(mpad // 128)], dtype=torch.int32, device=device)
        self.row_ntiles = z(1, dt=torch.int32)

    def start(self, m: int) -> None:
        """Once per step, before any layer."""
        self.row_ntiles.fill_((m + 127) // 128)


class RoutedExperts:
    """One layer's router, experts and shared expert in the layouts the kernels take."""

    def __init__(self, shape: ExpertsShape, W: Dict[str, torch.Tensor], p: str, device, dtype: torch.dtype, bias: str = "router.b"):
        """``W[p + name]`` for router, its ``bias``, e<i>.{gate, up, down} and, with a shared expert, shared.{gate, up, down, sg}."""
        s = shape
        self.shape, self.dtype = s, dtype
        D, F, Fs = _pad(s.width), _pad(s.ff), _pad(s.shared_ff)
        get = lambda n: W[p + n].to(device).to(dtype)
        self.bias = W[p + bias].to(device).float().contiguous()
        rows = [get("router")] + ([get("shared.sg")] if s.shared_ff else [])
        self.w_router = torch.zeros(s.experts + len(rows) - 1, D, dtype=dtype, device=device)
        self.w_router[:, :s.width] = torch.cat(rows, 0)
        self.gate_up = torch.zeros(s.experts, 2 * F, D, dtype=dtype, device=device)
        self.down = torch.zeros(s.experts, D, F, dtype=dtype, device=device)
        for e in range(s.experts):
            self._unit(self.gate_up[e], self.down[e], get, f"e{e}.", s.width, s.ff, F)
        self.shared_gate_up = self.shared_down = None
        if s.shared_ff:
            self.shared_gate_up = torch.zeros(2 * Fs, D, dtype=dtype, device=device)
            self.shared_down = torch.zeros(D, Fs, dtype=dtype, device=device)
            self._unit(self.shared_gate_up, self.shared_down, get, "shared.", s.width, s.shared_ff, Fs)

    @staticmethod
    def _unit(gate_up, down, get, name, width, ff, padded) -> None:
        gate_up[:ff, :width] = get(name + "gate")
        gate_up[padded:padded + ff, :width] = get(name + "up")
        down[:width, :ff] = get(name + "down")

    @property
    def fits_decode(self) -> bool:
        """Sizes the streaming decode kernels take without padding (a norm over a padded row would count the padding)."""
        return self.dtype == BF16 and self.shape.width % 8 == 0

    def rows(self, B: ExpertBuffers, m: int, xa: torch.Tensor, gain: Optional[torch.Tensor], next_gain: Optional[torch.Tensor], eps: float, x: torch.Tensor,
             status_ptr, base: Optional[torch.Tensor] = None, extra: Optional[torch.Tensor] = None) -> None:
        """``x += rms(experts(xa)) * gain``, or without a gain ``x += experts(xa) + base`` (f32 rows, or parts of their sum); ``extra`` (f32 rows) joins either. ``xa`` =
        ``rms(x) * next_gain`` (x without one). ``xa``: ``[m, padded width]``."""
        s, lib = self.shape, _lib.load()
        D = self.gate_up.shape[2]
        n = self.w_router.shape[0]
        logits, ids, wts, route = B.logits[:m, :n], B.ids[s.top][:m], B.wts[s.top][:m], B.route[s.top, s.experts]
        N.linear(xa, self.w_router, logits, status_ptr=status_ptr)
        check(lib.ifab_moe_route(logits.data_ptr(), logits.stride(0), self.bias.data_ptr(), m, s.experts, s.top, *s.rule, ids.data_ptr(),
                                 wts.data_ptr(), B.shared_w.data_ptr() if s.shared_ff else None, _s()), "moe_route")
        P.moe_dispatch(ids, 0, s.experts, route)
        act, y, tiles = B.act[s.ff], B.y, route.tiles[:(m * s.top + 127) // 128 + s.experts]
        sh = None
        if self.dtype == F32:
            self._grouped_f32(xa, route.perm_token, self.gate_up, self.down, tiles, route.num_tiles, act, y, m * s.top)
            if s.shared_ff:
                sh = B.sy
                self._grouped_f32(xa, None, self.shared_gate_up[None], self.shared_down[None], B.row_tiles[:(m + 127) // 128], B.row_ntiles,
                                  B.sact[s.shared_ff], sh, m)
        else:
            P.moe_gather(xa, route, B.xp)
            P.grouped_gemm(B.xp, self.gate_up, tiles, route.num_tiles, act, unit=s.unit, status_ptr=status_ptr)
            P.grouped_gemm(act, self.down, tiles, route.num_tiles, y, status_ptr=status_ptr)
            if s.shared_ff:
                sact, sh = B.sact[s.shared_ff], B.sy
                if m >= 256 and sact.shape[1] % 32 == 0:
                    N.gated_linear(xa, self.shared_gate_up, s.unit, sact[:m], status_ptr=status_ptr)
                else:
                    P.grouped_gemm(xa, self.shared_gate_up[None], B.row_tiles, B.row_ntiles, sact, unit=s.unit, status_ptr=status_ptr)
                N.linear(sact[:m], self.shared_down, sh[:m], status_ptr=status_ptr)
        check(lib.ifab_moe_combine_norm(y.data_ptr(), y.stride(0), route.route_row.data_ptr(), wts.data_ptr(), s.top, _p(sh), 0 if sh is None else sh.stride(0),
                                        B.shared_w.data_ptr() if s.shared_ff else None, _p(gain), _p(next_gain), eps, _p(base), *N._parts(base),
                                        _p(extra), 0 if extra is None else extra.stride(0), x.data_ptr(), x.stride(0), xa.data_ptr(), xa.stride(0), _f32(xa), m, s.width, _s()), "moe_combine_norm")

    def _grouped_f32(self, xa, index, gate_up, down, tiles, ntiles, act, y, rows: int) -> None:
        lib = _lib.load()
        E, F2, D = gate_up.shape
        most = tiles.shape[0]
        check(lib.ifab_grouped_linear_f32(xa.data_ptr(), xa.stride(0), _p(index), 0, 0, 0.0, 0.0, gate_up.data_ptr(), F2, D, tiles.data_ptr(), ntiles.data_ptr(), most, rows, act.data_ptr(),
                                          act.stride(0), _s()), "grouped_linear_f32")
        check(lib.ifab_grouped_linear_f32(act.data_ptr(), act.stride(0), None, 1, *self.shape.unit.args, down.data_ptr(), D, F2 // 2, tiles.data_ptr(), ntiles.data_ptr(), most, rows, y.data_ptr(),
                                          y.stride(0), _s()), "grouped_linear_f32")

    def decode(self, B: ExpertBuffers, n: int, y: torch.Tensor, owed: torch.Tensor, gain: torch.Tensor, eps: float, x_in: torch.Tensor, x_out: torch.Tensor,
               xn: torch.Tensor, ticket_ptr: int) -> None:
        """Decode rows in three launches. ``x_out = x_in + rms(y) * owed`` (the sublayer before), ``xn = rms(x_out) * gain``, then ``y`` = the
        experts' output of ``xn`` in f32."""
        s, lib = self.shape, _lib.load()
        N_ = self.w_router.shape[0]
        ids, wts = B.ids[s.top][:n], B.wts[s.top][:n]
        shared_w = B.shared_w.data_ptr() if s.shared_ff else None
        assert s.scoring == "biased_logits" and s.groups == 1
        check(lib.ifab_router_post_norm(y.data_ptr(), y.stride(0), owed.data_ptr(), gain.data_ptr(), eps, x_in.data_ptr(), x_out.data_ptr(), x_in.stride(0),
                                        xn.data_ptr(), xn.stride(0), self.w_router.data_ptr(), B.logits.data_ptr(), B.logits.stride(0), self.bias.data_ptr(),
                                        s.experts, s.top, SCORING["biased_logits"], 1, 1.0, ids.data_ptr(), wts.data_ptr(), shared_w, ticket_ptr, n, N_, s.width,
                                        _s()), "router_post_norm")
        self.decode_chosen(B, n, xn, y)

    def decode_chosen(self, B: ExpertBuffers, n: int, xn: torch.Tensor, y: torch.Tensor) -> None:
        """Decode rows whose choice is in ``B.ids`` / ``B.wts``: ``y`` (f32) = the experts' output of ``xn``, in two launches."""
        s, lib = self.shape, _lib.load()
        ids, wts, act = B.ids[s.top][:n], B.wts[s.top][:n], B.slots[s.top, s.slot_cols][:n]
        shared_w = B.shared_w.data_ptr() if s.shared_ff else None
        K.moe_gate_up(xn, ids, self.gate_up, 0, w_shared_gu=self.shared_gate_up, act=act, unit=s.unit)
        check(lib.ifab_moe_down_f32_decode(act.data_ptr(), act.shape[2], ids.data_ptr(), wts.data_ptr(), shared_w, n, s.width, self.down.shape[2], s.top, s.experts,
                                           self.down.data_ptr(), _p(self.shared_down), _pad(s.shared_ff), y.data_ptr(), y.stride(0), _s()), "moe_down_f32")
