"""Linear attention with a fixed decay per head (``csrc/kernels/linear_attn.cu``): S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t over
per-sequence f32 states, for any head sizes."""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from . import _lib
from ._lib import check
from .stream_norm import ACTIVATIONS, _f32, _p, _s

CHUNK = 64


def rotary_frequencies(dims: int, base: float, device) -> torch.Tensor:
    """``base^(-2 i / dims)`` for i < dims / 2, in double."""
    return torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=device)


def decay_powers(decay: Sequence[float], device) -> torch.Tensor:
    """f32 ``[heads, CHUNK + 1]``: decay^n, formed in double."""
    return torch.tensor([[float(d) ** n for n in range(CHUNK + 1)] for d in decay], dtype=torch.float64).float().to(device)


class StepPlan:
    """How the rows of a packed step are run: runs of equal consecutive slots (one sequence's rows, in position order) of more than
    ``short`` rows go by chunks, the others through the decode kernels.

    ``chunks``: ``[first row, rows, slot, flags]`` (1: first chunk of its run, 2: last); ``runs``: ``(first row, rows, slot, first
    position)`` of the long runs; ``groups``: row ranges ``[lo, hi)`` of at most ``group`` rows that hold every short row. ``control`` is what
    the device needs of it (int32, host): the chunk table, then - when there are short rows beside long runs - the positions with
    those of the long runs replaced by -1, so that the decode kernels skip them."""

    def __init__(self, slots: Sequence[int], positions: Sequence[int], short: int = 4, group: int = 64):
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
                for r in range(i, j, CHUNK):
                    self.chunks.append([r, min(CHUNK, j - r), slots[i], (1 if r == i else 0) | (2 if r + CHUNK >= j else 0)])
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
    head sizes, decay, and what happens to q / k / v first (rotation or activation, factor on k)."""

    def __init__(self, *, heads: int, dim: int, vdim: int, decay: Sequence[float], offsets, device, rot_dims: int = 0, rot_base: float = 0.0,
                 interleaved: bool = False, act: Optional[str] = None, k_scale: float = 1.0):
        if len(decay) != heads:
            raise ValueError(f"{heads} heads but {len(decay)} decay factors")
        self.H, self.d, self.e, self.offsets = heads, dim, vdim, tuple(offsets)
        self.rot, self.interleaved, self.act, self.k_scale = rot_dims, int(interleaved), ACTIVATIONS[act], k_scale
        self.freq = rotary_frequencies(rot_dims, rot_base, device) if rot_dims else None
        self.powers = decay_powers(decay, device)

    def state(self, slots: int, device) -> torch.Tensor:
        return torch.zeros(slots, self.H, self.d, self.e, dtype=torch.float32, device=device)

    def step(self, proj: torch.Tensor, state: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, out: torch.Tensor) -> None:
        """Decode: rows of one slot (consecutive, in position order) walk their state one after the other."""
        check(_lib.load().ifab_la_step(proj.data_ptr(), proj.stride(0), _f32(proj), *self.offsets, self.H, self.d, self.e, self.rot, self.interleaved,
                                       _p(self.freq), self.act, self.k_scale, self.powers.data_ptr(), state.data_ptr(), positions.data_ptr(),
                                       slots.data_ptr(), out.data_ptr(), out.stride(0), proj.shape[0], _s()), "la_step")

    def chunks(self, proj: torch.Tensor, state: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, out: torch.Tensor, scratch) -> None:
        """Prompts: the chunks of ``table`` (``StepPlan.chunks``, on the device). ``scratch``: ``(q, k, v, cstate)`` f32 buffers of at
        least ``rows * H * d``, the same, ``rows * H * e`` and ``chunks * H * d * e`` elements."""
        T = proj.shape[0]
        q, k, v, cs = scratch
        assert q.numel() >= T * self.H * self.d and v.numel() >= T * self.H * self.e
        check(_lib.load().ifab_la_prepare(proj.data_ptr(), proj.stride(0), _f32(proj), *self.offsets, self.H, self.d, self.e, self.rot, self.interleaved,
                                          _p(self.freq), self.act, self.k_scale, positions.data_ptr(), q.data_ptr(), k.data_ptr(), v.data_ptr(), T, _s()),
              "la_prepare")
        check(_lib.load().ifab_la_chunks(q.data_ptr(), k.data_ptr(), v.data_ptr(), table.data_ptr(), table.shape[0], positions.data_ptr(), self.H, self.d,
                                         self.e, self.powers.data_ptr(), cs.data_ptr(), cs.numel() * 4, state.data_ptr(), out.data_ptr(), out.stride(0),
                                         _s()), "la_chunks")
