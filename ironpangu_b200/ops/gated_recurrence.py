"""Recurrences over a matrix state per head with a decay per token - state-space duality, gated delta rule, matrix memory with exponential
gates - between a packed input projection and the operand of the output projection (``csrc/kernels/gated_recurrence.cu``, ``gated_delta.cu``, ``gated_tiles.cu``, for
decode rows ``decode_hyper.cu``)."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Dict, Optional

import torch

from . import _lib
from ._lib import check
from .linear_attn import DevicePlan
from .stream_norm import ACTIVATIONS, _f32, _p, _s

F32 = torch.float32
CHUNK = 64               # rows of a chunk of the f32 form
TILE = 128               # of the tensor-core form (bf16, heads up to 128 columns)
KINDS = {"ssd": 0, "delta": 1, "memory": 2}


@dataclass(frozen=True)
class RecurrenceShape:
    """``kv_heads``: heads of q and k (the groups of ``ssd``). ``taps``: of the short convolution (0: none). ``norm_groups``: equal parts of the
    result that are normed (0: one per head)."""

    kind: str
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int = 0
    norm_groups: int = 0
    gate_cap: float = 0.0

    def check(self) -> None:
        if self.kind not in KINDS:
            raise ValueError(f"unknown recurrence {self.kind!r}")
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads or max(self.dim, self.E) > 1024:
            raise ValueError(f"recurrence: {self.heads} heads over {self.kv_heads} of {self.dim} / {self.vdim} columns are not supported")
        if not 0 <= self.taps <= 64 or (self.taps > 0) != (self.kind != "memory"):
            raise ValueError(f"recurrence: a convolution of {self.taps} taps is not supported")
        if self.inner % self.groups or self.heads > 2048:
            raise ValueError(f"recurrence: {self.inner} columns in {self.groups} norm groups")
        if self.kind == "memory" and (self.gate_cap <= 0 or self.kv_heads != self.heads):
            raise ValueError("recurrence: a matrix memory needs a gate cap above 0 and as many key heads as heads")

    @property
    def E(self) -> int:
        """Value columns of a head in the state: the memory keeps the sum of its keys in one more."""
        return self.vdim + (self.kind == "memory")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def groups(self) -> int:
        return self.norm_groups or self.heads

    @property
    def columns(self) -> Dict[str, int]:
        """Widths of the packed projection's parts, in their order."""
        qk, v, h = self.kv_heads * self.dim, self.inner, self.heads
        if self.kind == "ssd":
            return {"z": v, "v": v, "k": qk, "q": qk, "a": h}
        return {"q": qk, "k": qk, "v": v, "g": v, **({"b": h, "a": h} if self.kind == "delta" else {"i": h, "f": h})}

    @property
    def in_cols(self) -> int:
        return sum(self.columns.values())

    @property
    def channels(self) -> int:
        """Of the convolution."""
        return 2 * self.kv_heads * self.dim + self.inner if self.taps else 0

    @property
    def tiles(self) -> bool:
        """Fits the tensor-core form."""
        return max(self.dim, self.vdim) <= 128

    @property
    def image_bytes(self) -> int:
        """Of the delta rule's operands of a chunk and head."""
        return (4 if self.dim <= 64 else 6) * 16384

    @property
    def slot_floats(self) -> int:
        """32-bit words a sequence holds besides the convolution's history."""
        return self.heads * self.E * self.dim + (2 * self.heads if self.kind == "memory" else 0)


class RecurrenceBuffers:
    """Work buffers of the recurrences of a model for up to ``rows`` rows; ``chunk`` > 0: for packed steps over ``slots`` sequences with chunks of so many
    rows (TILE: all recurrences take the tensor-core form)."""

    def __init__(self, shapes, rows: int, dtype: torch.dtype, device, *, chunk: int, slots: int):
        f = lambda n, dt=F32: torch.empty(max(n, 1), dtype=dt, device=device)
        most = lambda fn: max([fn(s) for s in shapes] or [1])
        self.q, self.k = f(rows * most(lambda s: s.kv_heads * s.dim), dtype), f(rows * most(lambda s: s.kv_heads * s.dim), dtype)
        self.v, self.o = f(rows * most(lambda s: s.inner), dtype), f(rows * most(lambda s: s.heads * s.E))
        self.qs, self.ks = f(rows * most(lambda s: s.kv_heads)), f(rows * most(lambda s: s.kv_heads))
        self.log_decay, self.weight, self.m = (f(rows * most(lambda s: s.heads)) for _ in range(3))
        self.chunk = chunk
        self.cstate = self.cdecay = self.w_rows = self.u_rows = self.images = None
        if chunk and shapes:
            assert chunk == CHUNK or (chunk == TILE and dtype == torch.bfloat16 and all(s.tiles for s in shapes))
            n = rows // chunk + slots + 1                    # chunks of a step: whole ones and one ragged end per sequence
            self.cstate, self.cdecay = f(n * most(lambda s: s.heads * s.dim * s.E)), f(n * most(lambda s: s.heads))
            delta = [s for s in shapes if s.kind == "delta"]
            if delta:
                self.u_rows = f(rows * max(s.inner for s in delta))
                if chunk == TILE:
                    self.images = f(n * max(s.heads * s.image_bytes for s in delta), torch.uint8)
                else:
                    self.w_rows = f(rows * max(s.heads * s.dim for s in delta))


class GatedRecurrence:
    """One recurrent mixer: its weights in the layouts the kernels take, its states, and the launches between the packed projection (its part
    starts at column ``at``) and the operand of the output projection. The output matrix (``W[p + "o"]``) is the caller's. ``factor``
    multiplies the result."""

    def __init__(self, shape: RecurrenceShape, W: Dict[str, torch.Tensor], p: str, device, dtype: torch.dtype, *, at: int = 0, factor: float = 1.0):
        s = shape
        self.shape, self.kind, self.at = s, KINDS[s.kind], at
        get = lambda n: W[p + n].to(device)
        vec = lambda n: get(n).float().contiguous()
        names = ("in",) if s.kind == "ssd" else tuple(s.columns)
        self.w_in = torch.cat([get(n).to(dtype) for n in names], 0)
        self.col, c = {}, at
        for n, w in s.columns.items():
            self.col[n] = c
            c += w
        qk = s.kv_heads * s.dim
        channel = {"v": 0, "k": s.inner, "q": s.inner + qk} if s.kind == "ssd" else {"q": 0, "k": qk, "v": 2 * qk}
        if not s.taps:
            channel = dict.fromkeys("qkv", -1)
        sec = []
        for n, heads, w in (("q", s.kv_heads, s.dim), ("k", s.kv_heads, s.dim), ("v", s.heads, s.vdim)):
            sec += [self.col[n], heads, w, channel[n]]
        self.sections = (ctypes.c_int32 * 12)(*sec)
        self.cols, self.channels = (ctypes.c_int32 * 3)(*(self.col[n] for n in "qkv")), (ctypes.c_int32 * 3)(*(channel[n] for n in "qkv"))
        self.q_factor = s.dim ** -0.5 if s.kind != "ssd" else 1.0
        self.taps_w = self.bias = self.a_log = self.decay_bias = self.weight_bias = self.skip = None
        if s.taps:
            conv = [get("conv")] if s.kind == "ssd" else [get(n + ".conv") for n in "qkv"]
            self.taps_w = torch.cat(conv, 0).float().t().contiguous()
            self.a_log, self.decay_bias = vec("A_log"), vec("dt_bias")
        if s.kind == "ssd":
            self.bias, self.skip = vec("conv.b"), vec("D")
        if s.kind == "memory":
            self.decay_bias, self.weight_bias = vec("f.b"), vec("i.b")
        gain = vec("norm")
        self.gain = (gain.repeat(s.heads) if s.kind == "delta" else gain).mul(factor).contiguous()
        self.gate, self.gate_act = ("z" if s.kind == "ssd" else "g"), ACTIVATIONS["sigmoid" if s.kind == "memory" else "silu"]
        self.decay_col, self.weight_col = (self.col["f"], self.col["i"]) if s.kind == "memory" else (self.col["a"], self.col.get("b", self.col["a"]))

    def make_state(self, slots: int, device, dtype: torch.dtype) -> "RecurrenceState":
        return RecurrenceState(self.shape, slots, device, dtype)

    def mix(self, B: RecurrenceBuffers, state: "RecurrenceState", proj: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, plan: Optional[DevicePlan], epoch: torch.Tensor,
            eps: float, out: torch.Tensor, status_ptr=None) -> None:
        """Rows of a packed step (``plan``), or decode rows (None), from ``proj`` to ``out`` ``[m, >= heads * vdim]``."""
        self.prepare(B, state, proj, pos, slot, epoch)
        # norm and gate belong to the tensor-core form when every row is one of its and the norm is per head
        whole = plan is not None and plan.table is not None and not plan.groups and B.chunk == TILE and self.shape.kind != "ssd"
        self.run(B, state, pos, slot, plan, epoch, (proj[:, self.col[self.gate]:], out, eps) if whole else None, status_ptr)
        if not whole:
            self.finish(B, proj, eps, out)

    def prepare(self, B, state, proj, pos, slot, epoch) -> None:
        s = self.shape
        unit = s.kind == "delta"
        check(_lib.load().ifab_gr_prepare(proj.data_ptr(), proj.stride(0), _f32(proj), self.sections, B.q.data_ptr(), B.k.data_ptr(), B.v.data_ptr(),
                                          B.qs.data_ptr() if unit else None, B.ks.data_ptr() if unit else None, self.q_factor, _p(self.taps_w), _p(self.bias), s.taps,
                                          s.channels, _p(state.history), epoch.data_ptr(), self.kind, s.heads, self.decay_col, self.weight_col, _p(self.a_log),
                                          _p(self.decay_bias), _p(self.weight_bias), s.gate_cap, B.log_decay.data_ptr(), B.weight.data_ptr(), pos.data_ptr(),
                                          slot.data_ptr(), proj.shape[0], _s()), "gr_prepare")

    def run(self, B, state, pos, slot, plan: Optional[DevicePlan], epoch, finish=None, status_ptr=None) -> None:
        """The prepared rows through the states, into ``B.o`` - or with ``finish`` (gate rows, result, eps) through norm and gate too."""
        s, m = self.shape, pos.numel()
        unit = s.kind == "delta"
        qkv = B.q.data_ptr(), B.k.data_ptr(), B.v.data_ptr()
        rows = (B.qs.data_ptr() if unit else None, B.ks.data_ptr() if unit else None, self.q_factor, B.log_decay.data_ptr(), B.weight.data_ptr(), self.kind, s.heads, s.kv_heads,
                s.dim, s.vdim)
        ldo = s.heads * s.E
        long = plan is not None and plan.table is not None
        if long:
            chunks = plan.table.data_ptr(), plan.table.shape[0], pos.data_ptr(), B.cstate.data_ptr(), B.cstate.numel() * 4, B.cdecay.data_ptr()
            states = state.s.data_ptr(), _p(state.m), epoch.data_ptr(), B.m.data_ptr()
            if B.chunk == TILE:
                gate, out, eps = finish or (None, None, 0.0)
                check(_lib.load().ifab_gr_tiles(*qkv, *rows, *chunks, _p(B.u_rows), _p(B.images), 0 if B.images is None else B.images.numel(), *states, B.o.data_ptr(), ldo,
                                                _p(gate), 0 if gate is None else gate.stride(0), self.gate_act, self.gain.data_ptr(), eps, _p(out),
                                                0 if out is None else out.stride(0), status_ptr, _s()), "gr_tiles")
            else:
                check(_lib.load().ifab_gr_chunks(*qkv, _f32(B.q), *rows, *chunks, _p(B.w_rows), _p(B.u_rows), *states, B.o.data_ptr(), ldo, _s()), "gr_chunks")
        if not long or plan.groups:
            check(_lib.load().ifab_gr_step(*qkv, _f32(B.q), *rows, state.s.data_ptr(), _p(state.m), epoch.data_ptr(), B.m.data_ptr(),
                                           (pos if plan is None else plan.step_positions).data_ptr(), slot.data_ptr(), B.o.data_ptr(), ldo, m, _s()), "gr_step")

    @property
    def fusable(self) -> bool:
        """The fused decode form takes this shape (bf16)."""
        s = self.shape
        return s.dim % 4 == 0 and s.dim <= 256 and s.vdim % 4 == 0 and s.inner // s.groups % 4 == 0 and self.col[self.gate] % 4 == 0

    def decode(self, B, state, proj, pos, slot, epoch) -> None:
        """:meth:`prepare` and :meth:`run` of decode rows in one launch."""
        s = self.shape
        check(_lib.load().ifab_gr_decode(proj.data_ptr(), proj.stride(0), self.cols, self.channels, int(s.kind == "delta"), self.q_factor, _p(self.taps_w), _p(self.bias), s.taps,
                                         s.channels, _p(state.history), self.kind, s.heads, s.kv_heads, s.dim, s.vdim, self.decay_col, self.weight_col, _p(self.a_log),
                                         _p(self.decay_bias), _p(self.weight_bias), s.gate_cap, state.s.data_ptr(), _p(state.m), epoch.data_ptr(),
                                         B.v.data_ptr() if s.kind == "ssd" else None, B.m.data_ptr(), pos.data_ptr(), slot.data_ptr(), B.o.data_ptr(), s.heads * s.E,
                                         proj.shape[0], _s()), "gr_decode")

    def gemv_mixed(self, B, proj, eps: float, x: torch.Tensor, K1: int, w: torch.Tensor, out: torch.Tensor) -> None:
        """``out`` (f32) = ``[first K1 columns of x | finished recurrence] @ w.T`` for one or two rows (:meth:`finish` and the output projection in one launch)."""
        s = self.shape
        gate = proj[:, self.col[self.gate]:]
        assert w.is_contiguous() and x.dtype == torch.bfloat16
        check(_lib.load().ifab_gemv_mixed(x.data_ptr(), x.stride(0), K1, B.o.data_ptr(), s.heads * s.E, s.heads, s.vdim, s.E, B.m.data_ptr() if s.kind == "memory" else None,
                                          B.v.data_ptr(), _p(self.skip), gate.data_ptr(), proj.stride(0), self.gate_act, int(s.kind == "ssd"), s.groups, eps,
                                          self.gain.data_ptr(), w.data_ptr(), out.data_ptr(), out.stride(0), proj.shape[0], w.shape[0], w.shape[1], _s()), "gemv_mixed")

    def finish(self, B, proj, eps: float, out: torch.Tensor) -> None:
        s = self.shape
        gate = proj[:, self.col[self.gate]:]
        check(_lib.load().ifab_gr_finish(B.o.data_ptr(), s.heads * s.E, s.heads, s.vdim, s.E, B.m.data_ptr() if s.kind == "memory" else None, B.v.data_ptr(),
                                         _p(self.skip), gate.data_ptr(), proj.stride(0), self.gate_act, int(s.kind == "ssd"), s.groups, eps, self.gain.data_ptr(),
                                         out.data_ptr(), out.stride(0), _f32(out), proj.shape[0], _s()), "gr_finish")


class RecurrenceState:
    """Per sequence slot: the f32 state ``[slots, heads, E, dim]``, the memory's running maximum and the convolution's last inputs."""

    def __init__(self, s: RecurrenceShape, slots: int, device, dtype: torch.dtype):
        self.s = torch.zeros(slots, s.heads, s.E, s.dim, dtype=F32, device=device)
        self.m = torch.zeros(slots, 2, s.heads, dtype=F32, device=device) if s.kind == "memory" else None
        self.history = torch.zeros(slots, 2, s.taps - 1, s.channels, dtype=dtype, device=device) if s.taps > 1 else None
