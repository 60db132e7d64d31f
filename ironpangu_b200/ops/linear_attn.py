"""Linear attention with a fixed decay per head (``csrc/kernels/linear_attn.cu``): S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t over
per-sequence f32 states, for any head sizes."""
from __future__ import annotations

from typing import List, Optional, Sequence

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


def chunk_table(slots: Sequence[int]) -> torch.Tensor:
    """Chunks of a packed step: runs of equal consecutive slots (one sequence's rows in position order), cut every CHUNK rows.
    int32 ``[n, 4]`` on the host: first row, rows, slot, flags (1: first chunk of the run, 2: last)."""
    out: List[List[int]] = []
    i, n = 0, len(slots)
    while i < n:
        j = i
        while j < n and slots[j] == slots[i]:
            j += 1
        for r in range(i, j, CHUNK):
            out.append([r, min(CHUNK, j - r), slots[i], (1 if r == i else 0) | (2 if r + CHUNK >= j else 0)])
        i = j
    return torch.tensor(out, dtype=torch.int32)


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
        """Prompts: the chunks of ``table`` (see :func:`chunk_table`, on the device). ``scratch``: ``(q, k, v, cstate)`` f32 buffers of at
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
