"""Linear attention with a fixed decay per head (``csrc/kernels/linear_attn.cu``): S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t over
per-sequence f32 states, for any head sizes."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from . import _lib
from ._lib import check
from .stream_norm import ACTIVATIONS, _f32, _p, _s

CHUNK = 64            # rows of a chunk of the f32 form
TILE = 128            # rows of a chunk of the tensor-core form


@dataclass(frozen=True)
class RotaryScaling:
    """Stretching of long wavelengths: a frequency whose wavelength is above ``original / low`` is divided by ``factor``, one below ``original /
    high`` stays, between them the two are mixed in proportion to ``original / wavelength``."""

    factor: float
    low: float
    high: float
    original: float

    def check(self) -> None:
        if self.factor <= 0 or self.original <= 0 or not 0 < self.low < self.high:
            raise ValueError(f"rotation scaling {self} is not supported")

    def apply(self, f: float) -> float:
        turns = self.original * f / (2.0 * math.pi)          # of the pair over the original context
        if turns > self.high:
            return f
        if turns < self.low:
            return f / self.factor
        s = (turns - self.low) / (self.high - self.low)
        return (1.0 - s) * f / self.factor + s * f


def rotary_frequencies(dims: int, base: float, device, scaling: Optional[RotaryScaling] = None) -> torch.Tensor:
    """``base^(-2 i / dims)`` for i < dims / 2, scaled, in double."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    return torch.tensor([scaling.apply(v) for v in f] if scaling else f, dtype=torch.float64, device=device)


class RotaryTables:
    """(cos, sin) of every rotation a model uses, for the rows of a step: one table f32 ``[rows, dims / 2, 2]`` per (dims, base[, scaling]), filled by
    one launch each per step and read by all layers."""

    def __init__(self, rotations, rows: int, device):
        self.freq = {r: rotary_frequencies(r[0], r[1], device, r[2]) for r in {(*r, None)[:3] for r in rotations} if r[0]}
        self.table = {r: torch.zeros(rows, r[0] // 2, 2, dtype=torch.float32, device=device) for r in self.freq}

    def fill(self, positions: torch.Tensor) -> None:
        for r, f in self.freq.items():
            check(_lib.load().ifab_rope_table(positions.data_ptr(), f.data_ptr(), self.table[r].data_ptr(), positions.numel(), f.numel(), _s()), "rope_table")

    def get(self, dims: int, base: float, scaling: Optional[RotaryScaling] = None) -> Optional[torch.Tensor]:
        return self.table[(dims, base, scaling)] if dims else None


def decay_powers(decay: Sequence[float], device) -> torch.Tensor:
    """f32 ``[heads, TILE + 1]``: decay^n, formed in double."""
    return torch.tensor([[float(d) ** n for n in range(TILE + 1)] for d in decay], dtype=torch.float64).float().to(device)


class StepPlan:
    """How the rows of a packed step are run: runs of equal consecutive slots (one sequence's rows, in position order) of more than
    ``short`` rows go by chunks, the others through the decode kernels.

    ``chunks``: ``[first row, rows, slot, 2 * chunks of the run + 1]`` (last entry 0 at all but the first chunk of a run); ``runs``: ``(first row, rows, slot, first
    position)`` of the long runs; ``groups``: row ranges ``[lo, hi)`` of at most ``group`` rows that hold every short row. ``control`` is what
    the device needs of it (int32, host): the chunk table, then - when there are short rows beside long runs - the positions with
    those of the long runs replaced by -1, so that the decode kernels skip them."""

    def __init__(self, slots: Sequence[int], positions: Sequence[int], short: int = 4, group: int = 64, chunk: int = CHUNK):
        n = len(slots)
        self.rows, self.chunks, self.runs, self.groups = n, [], [], []
        step = list(positions)
        i = 0
        while i < n:
            j = i
            while j < n and slots[j] == slots[i]:
                j += 1
            if j - i > short:
                self.runs.append((i, j - i, slots[i], positions[i]))
                for r in range(i, j, chunk):
                    self.chunks.append([r, min(chunk, j - r), slots[i], 2 * ((j - i + chunk - 1) // chunk) + 1 if r == i else 0])
                step[i:j] = [-1] * (j - i)
            i = j
        i = 0
        while i < n:
            if step[i] < 0:
                i += 1
                continue
            hi = min(n, i + group)
            last = max(r for r in range(i, hi) if step[r] >= 0)
            self.groups.append((i, last + 1))
            i = last + 1
        flat = [v for c in self.chunks for v in c]
        self.masked = bool(self.runs) and bool(self.groups)
        self.control = torch.tensor(flat + (step if self.masked else []) or [0], dtype=torch.int32)

    def bind(self, control: torch.Tensor, positions: torch.Tensor) -> "DevicePlan":
        """The plan over its control words on the device."""
        k = 4 * len(self.chunks)
        return DevicePlan(self, control[:k].view(-1, 4) if k else None, control[k:k + self.rows] if self.masked else positions)


class DevicePlan:
    def __init__(self, plan: StepPlan, table: Optional[torch.Tensor], step_positions: torch.Tensor):
        self.table, self.step_positions, self.runs, self.groups = table, step_positions, plan.runs, plan.groups


class DecayedMixer:
    """What one mixer does between its packed input projection and its gated norm: where q, k and v start in the projection row,
    head sizes, decay, and what happens to q / k / v first (rotation or activation, factor on k). ``rope``: the table of
    :class:`RotaryTables` for the step's rows (None without rotation)."""

    def __init__(self, *, heads: int, dim: int, vdim: int, decay: Sequence[float], offsets, device, rot_dims: int = 0, interleaved: bool = False,
                 act: Optional[str] = None, k_scale: float = 1.0):
        if len(decay) != heads:
            raise ValueError(f"{heads} heads but {len(decay)} decay factors")
        self.H, self.d, self.e, self.offsets = heads, dim, vdim, tuple(offsets)
        self.rot, self.interleaved, self.act, self.k_scale = rot_dims, int(interleaved), ACTIVATIONS[act], k_scale
        self.powers = decay_powers(decay, device)

    def state(self, slots: int, device) -> torch.Tensor:
        """f32 ``[slots, heads, vdim, dim]``."""
        return torch.zeros(slots, self.H, self.e, self.d, dtype=torch.float32, device=device)

    def _front(self, proj, rope):
        assert self.rot == 0 or rope.shape[0] >= proj.shape[0] and rope.shape[1] == self.rot // 2
        return (*self.offsets, self.H, self.d, self.e, self.rot, self.interleaved, _p(rope) if self.rot else None, self.act, self.k_scale)

    def step(self, proj: torch.Tensor, state: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, rope, out: torch.Tensor) -> None:
        """Decode: rows of one slot (consecutive, in position order) walk their state one after the other; rows at negative positions
        are skipped."""
        check(_lib.load().ifab_la_step(proj.data_ptr(), proj.stride(0), _f32(proj), *self._front(proj, rope), self.powers.data_ptr(), state.data_ptr(),
                                       positions.data_ptr(), slots.data_ptr(), out.data_ptr(), out.stride(0), proj.shape[0], _s()), "la_step")

    def chunks(self, proj: torch.Tensor, state: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, rope, out: torch.Tensor, scratch) -> None:
        """Prompts, f32 products: the chunks of ``table`` (``StepPlan.chunks`` of at most CHUNK rows, on the device). ``scratch``: ``(q, k, v,
        cstate)`` f32 buffers of at least ``rows * H * d``, the same, ``rows * H * e`` and ``chunks * H * d * e`` elements."""
        T = proj.shape[0]
        q, k, v, cs = scratch
        assert q.numel() >= T * self.H * self.d and v.numel() >= T * self.H * self.e
        check(_lib.load().ifab_la_prepare(proj.data_ptr(), proj.stride(0), _f32(proj), *self._front(proj, rope), q.data_ptr(), k.data_ptr(), v.data_ptr(), T,
                                          _s()), "la_prepare")
        check(_lib.load().ifab_la_chunks(q.data_ptr(), k.data_ptr(), v.data_ptr(), table.data_ptr(), table.shape[0], positions.data_ptr(), self.H, self.d,
                                         self.e, self.powers.data_ptr(), cs.data_ptr(), cs.numel() * 4, state.data_ptr(), out.data_ptr(), out.stride(0),
                                         _s()), "la_chunks")

    def tiles(self, proj: torch.Tensor, state: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, rope, cstate: torch.Tensor, *,
              out: Optional[torch.Tensor] = None, gated: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, gate_act: Optional[str] = None,
              eps: float = 0.0, status_ptr=None) -> None:
        """Prompts on the tensor cores (bf16 projections, heads up to 128 columns, chunks of at most TILE rows): f32 heads into ``out``, or
        heads divided by their rms and multiplied by ``gate_act(gate)`` into ``gated`` (bf16)."""
        assert proj.dtype == torch.bfloat16 and (out is None) != (gated is None)
        check(_lib.load().ifab_la_tiles(proj.data_ptr(), proj.stride(0), *self._front(proj, rope), self.powers.data_ptr(), table.data_ptr(), table.shape[0],
                                        positions.data_ptr(), cstate.data_ptr(), cstate.numel() * 4, state.data_ptr(), _p(out),
                                        0 if out is None else out.stride(0), _p(gate), 0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], _p(gated),
                                        0 if gated is None else gated.stride(0), eps, status_ptr, _s()), "la_tiles")
