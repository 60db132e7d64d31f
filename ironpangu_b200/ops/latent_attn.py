"""Latent attention with a query latent, a rotated key part shared by all heads, an optional sliding window and an optional gate per head,
over pages that hold one row [latent | rotated key part] per token (``csrc/kernels/latent_attn.cu``, ``tc_heads.cu``, the tensor-core prompt
kernel of ``fa_prefill.cu``). Any sizes within :meth:`LatentShape.check`; bf16, or f32 throughout.

Three forms of the same attention:

  decode     a few rows: absorb, split, merge + value up-projection, all as streams of the weights and the pages
  rows       any rows: the per-head projections as one tensor-core launch each (``tc_heads``), splits in between
  run        consecutive positions of one sequence: keys and values of what they can see are up-projected once and attended on the tensor
             cores (``fa_prefill``); needs head sizes that fit its tiles and bf16"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch

from . import _lib
from ._lib import check
from . import stream_norm as N
from .stream_norm import ACTIVATIONS, _f32, _p, _s
from .window_attn import context_rows, tile_width

BF16, F32 = torch.bfloat16, torch.float32
SPLIT_KEYS = 32            # fewest keys of a split (one batch of every warp)
SPLIT_CTAS = 600           # CTAs the splits of a launch aim at: more rows, longer splits
MAX_SPLITS = 64
BATCH_ROWS = 8             # rows from which the warps of a CTA split the heads instead of the keys
BATCH_CTAS = 148
V_TILE = 128               # value columns per head of the tensor-core prompt kernel


def _pad(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class LatentShape:
    heads: int
    dim: int               # unrotated query / key columns of a head
    rot_dim: int           # columns of the rotated part
    vdim: int
    kv_rank: int
    q_rank: int
    rot_dims: int          # of these, how many turn
    rot_base: float
    window: int            # 0: the whole context
    scale: float

    def check(self) -> None:
        if min(self.heads, self.dim, self.vdim, self.kv_rank, self.q_rank) < 1 or self.rot_dim < 0:
            raise ValueError("latent attention: sizes must be positive")
        if self.kv_rank > 1024 or self.rot_dim > 256:
            raise ValueError(f"latent attention: a latent of {self.kv_rank} and a rotated part of {self.rot_dim} columns are not supported")
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.rot_dim or self.window < 0:
            raise ValueError(f"latent attention: rotation of {self.rot_dims} columns of {self.rot_dim}, window {self.window}")

    @property
    def latent_cols(self) -> int:
        return _pad(self.kv_rank)

    @property
    def rot_cols(self) -> int:
        return _pad(self.rot_dim)

    @property
    def row(self) -> int:
        """Elements of a cached row."""
        return self.latent_cols + self.rot_cols

    @property
    def tiles(self) -> bool:
        """Heads fit the tiles of the tensor-core prompt kernel."""
        return self.dim <= 128 and self.rot_dim <= 64 and self.vdim <= V_TILE

    def q_parts(self, dtype: torch.dtype) -> tuple:
        """Columns of the unrotated and of the rotated part of a query head as the kernels take it."""
        return (tile_width(self.dim), 64) if self.tiles and dtype == BF16 else (_pad(self.dim), self.rot_cols)

    def batched(self, rows: int) -> bool:
        """A launch of ``rows`` rows takes the kernel whose warps split the heads."""
        return rows >= BATCH_ROWS and self.heads >= 4 and self.latent_cols <= 512 and self.rot_cols <= 64

    def batch_splitting(self, rows: int, max_context: int) -> tuple:
        """(splits, keys per split, partials per split) of that kernel: about one CTA per SM."""
        keys = min(self.window, max_context) if self.window else max_context
        sub = 8
        while sub > 1 and self.heads * sub > 32:
            sub //= 2
        n = max(1, min(MAX_SPLITS // sub, (keys + 63) // 64, BATCH_CTAS // (rows * ((self.heads + 31) // 32))))
        kps = ((keys + n - 1) // n + 31) // 32 * 32
        return (keys + kps - 1) // kps, kps, sub

    @property
    def in_cols(self) -> int:
        """Columns of the packed input projection: query latent, key / value latent, rotated key part, head gates; the key part starts at a
        multiple of eight."""
        return self.kv_off + _pad(self.kv_rank + self.rot_dim) + self.heads

    @property
    def kv_off(self) -> int:
        return _pad(self.q_rank)

    @property
    def gate_off(self) -> int:
        return self.kv_off + _pad(self.kv_rank + self.rot_dim)


class LatentBuffers:
    """Work buffers of the latent layers of a model for up to ``rows`` rows; ``chunked``: with the context of prompt runs."""

    def __init__(self, shapes, rows: int, dtype: torch.dtype, device, *, chunked: bool, max_context: int, group: int):
        z = lambda *s, dt=dtype: torch.zeros(*s, dtype=dt, device=device)
        self.group = min(rows, group)
        self.proj = z(rows, max(_pad(s.in_cols) for s in shapes))
        self.cq = {s.q_rank: z(rows, _pad(s.q_rank)) for s in shapes}                    # padding columns stay zero: one per width
        self.q = {}
        for s in shapes:
            n1, n2 = s.q_parts(dtype)
            self.q[s.heads, n1, n2] = z(rows, s.heads * (n1 + n2))
        self.q_lat = z(self.group * max(s.heads * s.latent_cols for s in shapes), dt=F32)
        self.o_lat = z(self.group * max(s.heads * s.latent_cols for s in shapes))
        self.mixed = {s.heads * s.vdim: z(rows, _pad(s.heads * s.vdim)) for s in shapes}
        partials = lambda s, n: max(most_splits(s, n, max_context), s.batch_splitting(n, max_context)[0] * s.batch_splitting(n, max_context)[2])
        self.scratch = torch.empty(max(partials(s, n) * n * s.heads * (s.latent_cols + 2) for s in shapes for n in range(1, self.group + 1)), dtype=F32, device=device)
        self.lat, self.k, self.vt, self.rot, self.cap = {}, None, None, None, 0
        tiled = [s for s in shapes if s.tiles]
        if chunked and dtype == BF16 and tiled:
            most = (max_context + 63) // 64 * 64
            self.cap = max(min(most, (context_rows(rows, s.window) + 63) // 64 * 64) if s.window else most for s in tiled)
            self.lat = {s.latent_cols: z(self.cap, s.latent_cols) for s in tiled}
            self.rot = z(self.cap, 64)
            self.k = {w: z(self.cap, w) for w in {s.heads * tile_width(s.dim) for s in tiled}}
            self.vt = {s.heads: z(s.heads * V_TILE, self.cap) for s in tiled}


def most_splits(s: LatentShape, rows: int, max_context: int) -> int:
    keys = min(s.window, max_context) if s.window else max_context
    return max(1, min(MAX_SPLITS, (keys + SPLIT_KEYS - 1) // SPLIT_KEYS, SPLIT_CTAS // max(1, rows * ((s.heads + 3) // 4))))


class LatentMixer:
    """One latent-attention layer: its weights in the layouts the kernels take, its pages and the launches between the packed input
    projection (``B.proj``) and the operand of the output projection (``B.mixed``)."""

    def __init__(self, shape: LatentShape, W: Dict[str, torch.Tensor], p: str, device, dtype: torch.dtype, *, max_context: int):
        """``W[p + name]`` for dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o."""
        s = shape
        self.shape, self.dtype, self.max_context = s, dtype, max_context
        H, Lp = s.heads, s.latent_cols
        get = lambda n: W[p + n].to(device).to(dtype)
        pad = lambda t, *size: _padded(t, *size)
        self.q_gain, self.kv_gain = W[p + "dq.norm"].to(device).float().contiguous(), W[p + "dkv.norm"].to(device).float().contiguous()
        self.q_gain_act = self.q_gain.to(dtype)
        width = W[p + "dq"].shape[1]
        self.w_in = pad(torch.cat([pad(get("dq"), s.kv_off, width), pad(get("dkv"), s.gate_off - s.kv_off, width), get("g")], 0), s.in_cols, _pad(width))
        n1, n2 = self.q_parts = s.q_parts(dtype)
        uq = get("uq").view(H, s.dim + s.rot_dim, s.q_rank)
        q = torch.zeros(H, n1 + n2, _pad(s.q_rank), dtype=dtype, device=device)
        q[:, :s.dim, :s.q_rank] = uq[:, :s.dim]
        q[:, n1:n1 + s.rot_dim, :s.q_rank] = uq[:, s.dim:]
        self.w_uq = q.view(H * (n1 + n2), _pad(s.q_rank))
        uk = get("uk").view(H, s.dim, s.kv_rank)
        self.w_uk = pad(uk, H, s.dim, Lp)                                            # query row -> latent row by rows (decode)
        self.w_uk_t = pad(uk.transpose(1, 2), H, Lp, _pad(s.dim))                    # the same as a [N, K] operand
        self.w_uv = pad(get("uv").view(H, s.vdim, s.kv_rank), H, s.vdim, Lp)
        self.w_o = pad(get("o"), width, _pad(H * s.vdim))
        self.tiles = s.tiles and dtype == BF16
        if self.tiles:                                                               # operands of the prompt up-projections: heads padded to tiles
            self.w_k = pad(uk, H, n1, Lp).view(H * n1, Lp)
            self.w_v = pad(get("uv").view(H, s.vdim, s.kv_rank), H, V_TILE, Lp).view(H * V_TILE, Lp)
        self.cache: Optional[torch.Tensor] = None

    def make_pages(self, pages: int, page_tokens: int) -> None:
        self.cache = torch.zeros(pages, page_tokens, self.shape.row, dtype=self.dtype, device=self.w_in.device)

    # -- steps ---------------------------------------------------------------------------------------------------------------
    def _paging(self, pos, slot, table):
        pages, pt, _ = self.cache.shape
        return pos.data_ptr(), slot.data_ptr(), table.data_ptr(), table.shape[1], pt, pages

    def _q(self, B: LatentBuffers) -> torch.Tensor:
        return B.q[self.shape.heads, self.q_parts[0], self.q_parts[1]]

    def prepare(self, B: LatentBuffers, m: int, rope, pos, slot, table, eps: float, status_ptr) -> None:
        """Projection rows -> normed query latent in ``B.cq``, pages of the rows written."""
        s = self.shape
        cq = B.cq[s.q_rank]
        check(_lib.load().ifab_latent_prepare(B.proj.data_ptr(), B.proj.stride(0), _f32(B.proj), 0, s.q_rank, s.kv_off, s.kv_rank, s.rot_dim, self.q_gain.data_ptr(),
                                              self.kv_gain.data_ptr(), eps, _p(rope), s.rot_dims, *self._paging(pos, slot, table), cq.data_ptr(),
                                              cq.stride(0), self.cache.data_ptr(), s.latent_cols, s.rot_cols, m, status_ptr, _s()),
              "latent_prepare")

    def rotate(self, q: torch.Tensor, rope) -> None:
        s, (n1, n2) = self.shape, self.q_parts
        if s.rot_dims:
            check(_lib.load().ifab_rotate_heads(q.data_ptr(), q.stride(0), _f32(q), n1 + n2, n1, s.heads, s.rot_dims, _p(rope), q.shape[0], _s()), "rotate_heads")

    def splitting(self, rows: int) -> tuple:
        """(splits, keys per split) of a launch of ``rows`` rows."""
        s = self.shape
        keys = min(s.window, self.max_context) if s.window else self.max_context
        n = most_splits(s, rows, self.max_context)
        kps = ((keys + n - 1) // n + SPLIT_KEYS - 1) // SPLIT_KEYS * SPLIT_KEYS
        return (keys + kps - 1) // kps, kps

    def _split(self, B: LatentBuffers, q, q_lat, pos, slot, table, how, status_ptr) -> None:
        s, n1 = self.shape, self.q_parts[0]
        check(_lib.load().ifab_latent_split(q_lat.data_ptr(), q[:, n1:].data_ptr(), q.stride(0), sum(self.q_parts), self.cache.data_ptr(), _f32(self.cache),
                                            s.latent_cols, s.rot_cols, *self._paging(pos, slot, table), s.window, s.scale, q.shape[0], s.heads, how[1], how[0],
                                            B.scratch.data_ptr(), B.scratch.numel() * 4, status_ptr, _s()), "latent_split")

    def decode(self, B: LatentBuffers, m: int, rope, pos, slot, table, eps: float, status_ptr) -> None:
        """A few bf16 rows (at most 8) from ``B.proj`` to ``B.mixed``: query projection (pages written beside it), absorb, split, merge + values."""
        s, (n1, n2) = self.shape, self.q_parts
        q, lib, H, Lp = self._q(B)[:m], _lib.load(), s.heads, s.latent_cols
        check(lib.ifab_latent_query(B.proj.data_ptr(), B.proj.stride(0), 0, s.q_rank, s.kv_off, s.kv_rank, s.rot_dim, self.q_gain_act.data_ptr(),
                                    self.kv_gain.data_ptr(), eps, _p(rope), s.rot_dims, *self._paging(pos, slot, table), self.cache.data_ptr(), Lp, s.rot_cols,
                                    self.w_uq.data_ptr(), q.shape[1], q.data_ptr(), q.stride(0), m, status_ptr, _s()), "latent_query")
        check(lib.ifab_latent_absorb(q.data_ptr(), q.stride(0), n1 + n2, n1, self.w_uk.data_ptr(), _p(rope), s.rot_dims, B.q_lat.data_ptr(), m, H, s.dim, Lp, _s()),
              "latent_absorb")
        how = self.splitting(m)
        self._split(B, q, B.q_lat, pos, slot, table, how, status_ptr)
        out, gate = B.mixed[H * s.vdim], B.proj[:, s.gate_off:]
        check(lib.ifab_latent_merge_vup(B.scratch.data_ptr(), pos.data_ptr(), s.window, how[1], how[0], gate.data_ptr(), gate.stride(0), m, H, Lp,
                                        self.w_uv.data_ptr(), s.vdim, out.data_ptr(), out.stride(0), _s()), "latent_merge_vup")

    def rows(self, B: LatentBuffers, lo: int, hi: int, pos, slot, table, status_ptr) -> None:
        """Rows lo .. hi - 1 (queries rotated, pages written; rows at negative positions give zeros) into ``B.mixed``."""
        s, (n1, n2), lib = self.shape, self.q_parts, _lib.load()
        q, n, H, Lp = self._q(B)[lo:hi], hi - lo, s.heads, s.latent_cols
        out = B.mixed[H * s.vdim][lo:hi]
        q_lat, o_lat = B.q_lat[:n * H * Lp].view(n, H * Lp), B.o_lat[:n * H * Lp].view(n, H * Lp)
        heads_product(q, n1 + n2, self.w_uk_t, q_lat, Lp, H, s.dim, status_ptr)
        pos, slot, sub = pos[lo:hi], slot[lo:hi], 1
        if self.dtype == BF16 and s.batched(n):
            splits, kps, sub = s.batch_splitting(n, self.max_context)
            check(lib.ifab_latent_batch(q_lat.data_ptr(), q[:, n1:].data_ptr(), q.stride(0), n1 + n2, self.cache.data_ptr(), Lp, s.rot_cols,
                                        *self._paging(pos, slot, table), s.window, s.scale, n, H, kps, splits, sub, B.scratch.data_ptr(), B.scratch.numel() * 4,
                                        status_ptr, _s()), "latent_batch")
        else:
            splits, kps = self.splitting(n)
            self._split(B, q, q_lat, pos, slot, table, (splits, kps), status_ptr)
        gate = B.proj[lo:hi, s.gate_off:]
        check(lib.ifab_latent_merge(B.scratch.data_ptr(), pos.data_ptr(), s.window, kps, splits, sub, gate.data_ptr(), gate.stride(0), _f32(o_lat), n, H, Lp,
                                    o_lat.data_ptr(), o_lat.stride(0), _s()), "latent_merge")
        heads_product(o_lat, Lp, self.w_uv, out, s.vdim, H, Lp, status_ptr)

    def run(self, B: LatentBuffers, lo: int, n: int, slot: int, pos0: int, table, status_ptr) -> None:
        """Rows lo .. lo + n - 1 = positions pos0 .. of one sequence (queries rotated, pages written) into ``B.mixed``, on the tensor cores."""
        s, (n1, n2), lib, H = self.shape, self.q_parts, _lib.load(), self.shape.heads
        first = max(0, pos0 - s.window + 1) if s.window else 0
        ctx = pos0 + n - first
        rows = (ctx + 63) // 64 * 64
        pages, pt, _ = self.cache.shape
        lat, rot, k, vt = B.lat[s.latent_cols][:rows], B.rot[:rows], B.k[H * n1][:rows], B.vt[H]
        check(lib.ifab_latent_gather(self.cache.data_ptr(), table.data_ptr(), slot, table.shape[1], pt, pages, first, ctx, rows, s.latent_cols, s.rot_cols, 64,
                                     lat.data_ptr(), rot.data_ptr(), status_ptr, _s()), "latent_gather")
        N.linear(lat, self.w_k, k, status_ptr=status_ptr)
        N.linear(self.w_v, lat, vt[:, :rows], status_ptr=status_ptr)
        q, out, gate = self._q(B)[lo:lo + n], B.mixed[H * s.vdim][lo:lo + n], B.proj[lo:lo + n, s.gate_off:]
        check(lib.ifab_fa_window_bf16(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), rot.data_ptr(), rot.stride(0), 64, vt.data_ptr(), vt.stride(0),
                                      out.data_ptr(), out.stride(0), n, ctx, H, 1, n1, s.vdim, pos0 - first, s.window, s.scale, 0.0, None, 0, None, gate.data_ptr(),
                                      gate.stride(0), ACTIVATIONS["sigmoid"], 1, 0, 0, 0, 0, 1.0, status_ptr, _s()), "fa_window")

    def mix(self, B: LatentBuffers, m: int, rope, pos, slot, plan, table, eps: float, status_ptr) -> None:
        """``m`` rows of a packed step (``plan``), or decode rows (None), from ``B.proj`` to ``B.mixed`` as matrix products and row kernels."""
        s = self.shape
        q = self._q(B)[:m]
        self.prepare(B, m, rope, pos, slot, table, eps, status_ptr)
        N.linear(B.cq[s.q_rank][:m], self.w_uq, q, status_ptr=status_ptr)
        self.rotate(q, rope)
        runs = plan.runs if plan is not None and self.tiles else []
        step = plan.step_positions if runs else pos
        for lo, hi in plan.groups if runs else [(r, min(m, r + B.group)) for r in range(0, m, B.group)]:
            self.rows(B, lo, hi, step, slot, table, status_ptr)
        for lo, n, sl, p0 in runs:                   # after the groups, which may reach over rows of a run
            self.run(B, lo, n, sl, p0, table, status_ptr)


def _padded(t: torch.Tensor, *size: int) -> torch.Tensor:
    out = torch.zeros(*size, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def heads_product(a: torch.Tensor, a_stride: int, b: torch.Tensor, c: torch.Tensor, c_stride: int, heads: int, k: int, status_ptr=None) -> None:
    """``c[t, h * c_stride + n] = sum_k a[t, h * a_stride + k] * b[h, n, k]``: on the tensor cores for bf16 operands (bf16 or f32 result), f32
    products otherwise."""
    H, n, kb = b.shape
    assert H == heads and kb >= k and a.dtype == b.dtype and b.is_contiguous()
    if a.dtype == F32:
        check(_lib.load().ifab_linear_f32_batched(a.data_ptr(), a.stride(0), a_stride, b.data_ptr(), kb, n * kb, c.data_ptr(), c.stride(0), c_stride, H, a.shape[0], n,
                                                  k, _s()), "linear_f32_batched")
    else:
        check(_lib.load().ifab_gemm_heads_bf16(a.data_ptr(), a.stride(0), a_stride, b.data_ptr(), kb, c.data_ptr(), c.stride(0), c_stride, _f32(c), H, a.shape[0], n, k,
                                               status_ptr, _s()), "gemm_heads")
