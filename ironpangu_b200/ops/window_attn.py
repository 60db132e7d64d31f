"""Softmax attention over a window or a chunk of paged keys / values, with sinks, score caps, distance biases and output gates
(``csrc/kernels/window_attn.cu``, ``decode_gqa.cu``, ``fa_prefill.cu``), and a grouped-query attention layer over them.

The mask: the last ``window`` positions (0: all), or with ``chunked`` the positions of the query's own stretch of ``window``, counted from
position 0 of the sequence. A score is ``q k scale``, with ``cap`` > 0 ``cap * tanh(score / cap)``, and with ``slopes`` (f32 ``[heads]``) less
``slope * (distance of the key)``. A gate has a value per column of the result, or one per head (``gate_head``).

Beside its window a query may see entries ahead of it, in the same softmax (:class:`Ahead`): the first ``keep`` positions, or one mean key and
value per block of ``pool`` positions that lies wholly before the window."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch

from . import _lib
from . import stream_norm as N
from ._lib import check
from .linear_attn import RotaryScaling
from .stream_norm import ACTIVATIONS, _f32, _p, _s


@dataclass(frozen=True)
class Ahead:
    """``pages``: the blocks' keys and values ``[pages, entries, kv_heads, .]`` (an entry lives in the page of its block's last position)."""

    keep: int = 0
    pool: int = 0
    pages: Optional[tuple] = None

    @property
    def args(self) -> tuple:
        k, v = self.pages or (None, None)
        return self.keep, self.pool, _p(k), _p(v)

    def count(self, first: int) -> int:
        """Entries that a query sees whose window starts at position ``first`` (at most)."""
        return min(self.keep, first) if self.keep else first // self.pool if self.pool else 0


NOTHING_AHEAD = Ahead()


def pool_write(k_cache: torch.Tensor, v_cache: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, page_table: torch.Tensor, ahead: Ahead, status_ptr=None) -> None:
    """The means of the blocks that end with a row of the step, out of the pages into ``ahead.pages``."""
    pages, pt, G, d = k_cache.shape
    check(_lib.load().ifab_pool_write(k_cache.data_ptr(), v_cache.data_ptr(), _f32(k_cache), positions.data_ptr(), slots.data_ptr(), page_table.data_ptr(),
                                      page_table.shape[1], pt, pages, G, d, v_cache.shape[3], ahead.pool, ahead.pages[0].data_ptr(), ahead.pages[1].data_ptr(),
                                      positions.numel(), status_ptr, _s()), "pool_write")


def qk_norm_rope_write(proj: torch.Tensor, offsets, q_gain: Optional[torch.Tensor], k_gain: Optional[torch.Tensor], eps: float, *, heads: int, kv_heads: int,
                       dim: int, vdim: int, rot: int, interleaved: bool, rope: Optional[torch.Tensor], positions: torch.Tensor, slots: torch.Tensor,
                       page_table: torch.Tensor, q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, whole: bool = False, status_ptr=None) -> None:
    """Packed projection rows -> normalised, rotated queries in ``q_out`` (``[T, heads * stride]``, stride >= dim) and normalised, rotated keys / plain values in the pages
    (``k_cache`` ``[pages, page_tokens, kv_heads, dim]``, ``v_cache`` ``[..., vdim]``). ``rope``: (cos, sin) of the rows, ``[T, rot / 2, 2]``
    (``linear_attn.RotaryTables``). The norm is per head with one gain of ``dim`` columns, or with ``whole`` over all columns of q and all of k,
    with a gain for each. ``offsets``: where q, k and v start in a row (v may be k)."""
    pages, pt = k_cache.shape[:2]
    check(_lib.load().ifab_qk_norm_rope_write(proj.data_ptr(), proj.stride(0), _f32(proj), *offsets, _p(q_gain), _p(k_gain), eps, heads, kv_heads, dim, vdim, rot,
                                              int(interleaved), _p(rope), positions.data_ptr(), slots.data_ptr(), page_table.data_ptr(), page_table.shape[1],
                                              pt, pages, q_out.data_ptr(), q_out.stride(0), q_out.shape[1] // heads, k_cache.data_ptr(), v_cache.data_ptr(), int(whole), proj.shape[0], status_ptr,
                                              _s()), "qk_norm_rope_write")


def window_attn(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, page_table: torch.Tensor, *,
                heads: int, window: int, scale: float, out: torch.Tensor, sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None,
                gate_act: Optional[str] = None, gate_head: bool = False, chunked: bool = False, cap: float = 0.0, slopes: Optional[torch.Tensor] = None,
                ahead: Ahead = NOTHING_AHEAD, factor: float = 1.0, status_ptr=None) -> None:
    """Rows of any sequences, any head sizes: exp(sink) joins the denominator, the result is multiplied by ``gate_act(gate)`` and ``factor``."""
    pages, pt, G, d = k_cache.shape
    check(_lib.load().ifab_window_attn(q.data_ptr(), q.stride(0), q.shape[1] // heads, k_cache.data_ptr(), v_cache.data_ptr(), _f32(q), positions.data_ptr(), slots.data_ptr(),
                                       page_table.data_ptr(), page_table.shape[1], pt, pages, heads, G, d, v_cache.shape[3], window, scale, cap, _p(slopes), int(chunked), _p(sink), _p(gate),
                                       0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], int(gate_head), *ahead.args, factor, out.data_ptr(), out.stride(0), q.shape[0],
                                       status_ptr, _s()), "window_attn")


SPLIT_KEYS = 64            # fewest keys per split of the split-KV decode form
SPLIT_CTAS = 600           # CTAs the splits of a launch aim at: more rows, longer splits


def split_form(heads: int, kv_heads: int, dim: int, vdim: int, window: int, ahead: int = 0) -> int:
    """Most splits the split-KV decode kernels take for this shape (``ahead``: most entries ahead of a window), 0 when it needs the general kernel."""
    if dim != vdim or dim not in (64, 128, 256) or heads // kv_heads not in (1, 2, 4, 8) or (dim == 256 and heads // kv_heads == 8) or not window:
        return 0
    return max(1, min(64, (window + ahead + SPLIT_KEYS - 1) // SPLIT_KEYS))


def gqa_window(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, page_table: torch.Tensor, *,
               heads: int, window: int, scale: float, splits: int, scratch: torch.Tensor, out: torch.Tensor, sink: Optional[torch.Tensor] = None,
               gate: Optional[torch.Tensor] = None, gate_act: Optional[str] = None, gate_head: bool = False, chunked: bool = False, cap: float = 0.0,
               slopes: Optional[torch.Tensor] = None, ahead: Ahead = NOTHING_AHEAD, most_ahead: int = 0, factor: float = 1.0, status_ptr=None) -> None:
    """:func:`window_attn` by splits of what a row sees (query heads of a group share the key loads), bf16, shapes of :func:`split_form`.
    ``splits``: the most to use; launches of many rows use fewer, longer ones. ``most_ahead``: how many entries ahead of its window a row may see."""
    pages, pt, G, d = k_cache.shape
    splits = max(1, min(splits, SPLIT_CTAS // (q.shape[0] * G)))
    kps = ((window + most_ahead + splits - 1) // splits + 31) // 32 * 32
    check(_lib.load().ifab_gqa_window_attention(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), positions.data_ptr(), slots.data_ptr(),
                                                page_table.data_ptr(), page_table.shape[1], pt, pages, scale, window, cap, _p(slopes), int(chunked), _p(sink), _p(gate),
                                                0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], int(gate_head), *ahead.args, factor, q.shape[0], heads, G, d,
                                                kps, splits,
                                                scratch.data_ptr(), scratch.numel() * 4, out.data_ptr(), out.stride(0), status_ptr, _s()), "gqa_window")


def tile_width(dim: int) -> int:
    """Columns a query / key head takes as an operand of the tensor-core attention (0: too wide)."""
    return 64 if dim <= 64 else 128 if dim <= 128 else 0


def context_rows(count: int, window: int) -> int:
    """Rows of the gathered context of ``count`` consecutive queries, a whole number of gather tiles (upper bound)."""
    return (count + window - 1 + 31) // 32 * 32


def ahead_rows(count: int) -> int:
    """Context rows that ``count`` entries ahead of the windows take: whole key tiles."""
    return (count + 127) // 128 * 128


def fa_window(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, page_table: torch.Tensor, *, slot: int, pos0: int, heads: int, window: int,
              scale: float, ctx_k: torch.Tensor, ctx_vt: torch.Tensor, out: torch.Tensor, sink: Optional[torch.Tensor] = None,
              gate: Optional[torch.Tensor] = None, gate_act: Optional[str] = None, gate_head: bool = False, chunked: bool = False, cap: float = 0.0,
              slopes: Optional[torch.Tensor] = None, ahead: Ahead = NOTHING_AHEAD, factor: float = 1.0, status_ptr=None) -> None:
    """Prompt attention of consecutive positions ``pos0 ..`` of one sequence (keys already in its pages) on the tensor cores: the keys
    and values the rows can see are gathered out of the pages into ``ctx_k`` ``[rows, kv_heads * tile]`` / ``ctx_vt`` ``[kv_heads * 128,
    rows]``, entries ahead of the windows first. ``q``: ``[m, heads * tile]``, columns past the head width zero; ``window`` 0: the whole context."""
    pages, pt, G, d = k_cache.shape
    m, e = q.shape[0], v_cache.shape[3]
    dp = q.shape[1] // heads
    first = 0 if not window else pos0 // window * window if chunked else max(0, pos0 - window + 1)
    n = pos0 + m - first
    rows = (n + 31) // 32 * 32
    seen = ahead.count(max(0, pos0 + m - window)) if window else 0         # by the last row
    front = ahead_rows(seen)
    assert dp == tile_width(d) and e <= 128 and ctx_k.shape[0] >= front + rows and ctx_vt.shape[1] >= front + rows and ctx_k.shape[1] == G * dp
    lib = _lib.load()
    check(lib.ifab_ctx_gather_pad(k_cache.data_ptr(), v_cache.data_ptr(), page_table.data_ptr(), slot, page_table.shape[1], pt, pages, first, n, rows, *ahead.args,
                                  seen, front, G, d, dp, e, ctx_k.data_ptr(), ctx_vt.data_ptr(), ctx_vt.stride(0), status_ptr, _s()), "ctx_gather_pad")
    check(lib.ifab_fa_window_bf16(q.data_ptr(), q.stride(0), ctx_k.data_ptr(), ctx_k.stride(0), None, 0, 0, ctx_vt.data_ptr(), ctx_vt.stride(0), out.data_ptr(),
                                  out.stride(0), m, n, heads, heads // G, dp, e, pos0 - first, window, scale, cap, _p(slopes), int(chunked), _p(sink), _p(gate),
                                  0 if gate is None else gate.stride(0), ACTIVATIONS[gate_act], int(gate_head), ahead.keep, ahead.pool, front, first, factor, status_ptr, _s()),
          "fa_window")


# ---------------------------------------------------------------------------------------------------------------------------
# a grouped-query attention layer
# ---------------------------------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class GroupedShape:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0                # 0: no mask but the causal one
    chunked: bool = False
    cap: float = 0.0               # soft limit of the scores
    biased: bool = False           # distance bias with slope 2^(-8 (h + 1) / heads)
    rot_dims: int = 0              # rotated columns of a head
    rot_base: float = 10000.0
    rot_scaling: Optional[RotaryScaling] = None
    rot_halves: bool = False       # pairs (i, i + rot_dims / 2) instead of neighbours
    norm: bool = False             # rms of all of q and of all of k before the rotation
    head_norm: bool = False        # rms of every head of q and k instead, without a gain
    keys_are_values: bool = False  # values = keys as projected
    bias: bool = False             # of the q, k and output projections
    gated: bool = True             # a gate per head
    keep: int = 0                  # first positions seen beside the window
    pool: int = 0                  # positions of a block seen beside the window
    factor: float = 1.0            # of the result

    def check(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or self.heads % self.kv_heads:
            raise ValueError(f"attention: {self.heads} heads over {self.kv_heads} key / value heads are not supported")
        if max(self.dim, self.vdim) > 256 or (self.keys_are_values and self.dim != self.vdim):
            raise ValueError(f"attention: heads of {self.dim} / {self.vdim} columns are not supported")
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.dim:
            raise ValueError(f"attention: rotation of {self.rot_dims} columns in heads of {self.dim}")
        if self.window < 0 or self.cap < 0:
            raise ValueError("attention: window and cap must not be negative")
        if min(self.keep, self.pool) < 0 or (self.keep and self.pool) or ((self.keep or self.pool) and (self.chunked or self.cap or self.biased or not self.window)):
            raise ValueError(f"attention: {self.keep} kept positions, blocks of {self.pool} beside a window of {self.window} are not supported")
        if self.rot_scaling:
            self.rot_scaling.check()
        if self.norm and self.head_norm:
            raise ValueError("attention: one norm of q and k at most")

    @property
    def offsets(self) -> tuple:
        """Where q, k, v and the head gates start in a projection row, and where it ends."""
        q, k = self.heads * self.dim, self.kv_heads * self.dim
        v = 0 if self.keys_are_values else self.kv_heads * self.vdim
        return 0, q, q if self.keys_are_values else q + k, q + k + v, q + k + v + self.heads * self.gated

    @property
    def in_cols(self) -> int:
        """Columns of the packed projection, filled up to whole stores of the GEMMs."""
        return (self.offsets[4] + 31) // 32 * 32

    @property
    def tiles(self) -> bool:
        return max(self.dim, self.vdim) <= 128

    @property
    def q_stride(self) -> int:
        return tile_width(self.dim) if self.tiles else self.dim

    def most_ahead(self, context: int) -> int:
        """Most entries a row sees ahead of its window in sequences of ``context`` positions."""
        return Ahead(self.keep, self.pool).count(max(0, context - self.window)) if self.window else 0

    def splits(self, context: int) -> int:
        return split_form(self.heads, self.kv_heads, self.dim, self.vdim, self.window, self.most_ahead(context)) if self.q_stride == self.dim else 0

    @property
    def row(self) -> int:
        """Elements a token holds in the pages."""
        return self.kv_heads * (self.dim + self.vdim)

    def page(self, page_tokens: int) -> int:
        """Elements of a page, with the entries of the blocks that may end in it."""
        return self.row * (page_tokens + self.entries(page_tokens))

    def entries(self, page_tokens: int) -> int:
        return (page_tokens + self.pool - 1) // self.pool if self.pool else 0

    @property
    def rotation(self) -> tuple:
        return self.rot_dims, self.rot_base, self.rot_scaling


class GroupedBuffers:
    """Work buffers of the grouped attention layers of a model for up to ``rows`` rows; ``chunked``: for packed steps."""

    def __init__(self, shapes, rows: int, dtype: torch.dtype, device, *, chunked: bool, max_context: int, group: int, in_cols: int = 0):
        """``in_cols``: columns of the projection rows when others share them."""
        self.group = group
        z = lambda *s: torch.zeros(*s, dtype=dtype, device=device)
        self.proj = z(rows, max([s.in_cols for s in shapes] + [in_cols]))
        # queries at the stride of the tensor-core tiles where they have one (padding columns stay zero: one buffer per shape)
        self.q = {(s.heads, s.q_stride, s.dim): z(rows, s.heads * s.q_stride) for s in shapes}
        self.context = max_context
        need = [s.heads * s.splits(max_context) * (s.vdim + 2) for s in shapes]
        self.scratch = torch.empty(min(rows, group) * max(need), dtype=torch.float32, device=device) if any(need) and dtype == torch.bfloat16 else None
        self.ctx = {}
        if chunked and dtype == torch.bfloat16:
            for s in shapes:
                cap = (max_context + 31) // 32 * 32
                if s.window:
                    cap = min(cap, context_rows(rows, s.window)) + ahead_rows(s.most_ahead(max_context))
                key = (s.kv_heads, s.q_stride)
                if s.tiles and (key not in self.ctx or self.ctx[key][0].shape[0] < cap):
                    self.ctx[key] = z(cap, s.kv_heads * s.q_stride), z(s.kv_heads * 128, cap)


class GroupedAttention:
    """One grouped-query attention layer with a gate per head: its weights in the layouts the kernels take, and the launches between the
    packed input projection and the operand of the output projection. The output matrix (``W[p + "o"]``) is the caller's."""

    def __init__(self, shape: GroupedShape, W: Dict[str, torch.Tensor], p: str, device, dtype: torch.dtype):
        """``W[p + name]`` for q, k, v (unless the keys are the values), g, with biases q.b, k.b and with norms q.norm, k.norm."""
        s = shape
        self.shape = s
        get = lambda n: W[p + n].to(device)
        mats = [get(n).to(dtype) for n in ("q", "k") + (() if s.keys_are_values else ("v",)) + (("g",) if s.gated else ())]
        width = mats[0].shape[1]
        self.w_in = torch.zeros(s.in_cols, (width + 7) // 8 * 8, dtype=dtype, device=device)
        self.w_in[:s.offsets[4], :width] = torch.cat(mats, 0)
        self.b_in = None
        if s.bias:
            self.b_in = torch.zeros(s.in_cols, dtype=torch.float32, device=device)
            self.b_in[:s.offsets[1] + s.kv_heads * s.dim] = torch.cat([get("q.b"), get("k.b")]).float()
        vec = lambda n: get(n).float().contiguous() if s.norm else None
        self.q_gain, self.k_gain = vec("q.norm"), vec("k.norm")
        if s.head_norm:
            self.q_gain = self.k_gain = torch.ones(s.dim, dtype=torch.float32, device=device)
        self.slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / s.heads) for h in range(s.heads)], dtype=torch.float32, device=device) if s.biased else None

    def make_pages(self, pages: int, page_tokens: int, device, dtype: torch.dtype) -> tuple:
        """Keys and values of the tokens, then - with blocks - of the blocks."""
        s = self.shape
        z = lambda m, n: torch.zeros(pages, m, s.kv_heads, n, dtype=dtype, device=device)
        m = s.entries(page_tokens)
        return (z(page_tokens, s.dim), z(page_tokens, s.vdim)) + ((z(m, s.dim), z(m, s.vdim)) if m else ())

    def project(self, B: GroupedBuffers, xa: torch.Tensor, status_ptr) -> None:
        N.linear(xa, self.w_in, B.proj[:xa.shape[0], :self.shape.in_cols], bias=self.b_in, status_ptr=status_ptr)

    def attend(self, B: GroupedBuffers, m: int, pages: tuple, rope, pos, slot, plan, table, eps: float, out: torch.Tensor, status_ptr) -> None:
        """``m`` rows of a packed step (``plan``), or decode rows (None), from ``B.proj`` to ``out`` ``[m, >= heads * vdim]``."""
        s = self.shape
        proj, q, bf16 = B.proj[:m], B.q[s.heads, s.q_stride, s.dim][:m], B.proj.dtype == torch.bfloat16
        qo, ko, vo, go, _ = s.offsets
        qk_norm_rope_write(proj, (qo, ko, vo), self.q_gain, self.k_gain, eps, heads=s.heads, kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim, rot=s.rot_dims,
                           interleaved=not s.rot_halves, rope=rope, positions=pos, slots=slot, page_table=table, q_out=q, k_cache=pages[0], v_cache=pages[1],
                           whole=s.norm, status_ptr=status_ptr)
        ahead, pages = Ahead(s.keep, s.pool, pages[2:] or None), pages[:2]
        if s.pool:
            pool_write(*pages, pos, slot, table, ahead, status_ptr)
        gate = proj[:, go:] if s.gated else None
        how = dict(heads=s.heads, window=s.window, scale=s.scale, gate_act="sigmoid" if s.gated else None, gate_head=s.gated, chunked=s.chunked, cap=s.cap, slopes=self.slopes,
                   ahead=ahead, factor=s.factor, status_ptr=status_ptr)
        tiled = plan is not None and bool(plan.runs) and s.tiles and bf16
        if tiled:
            k, vt = B.ctx[s.kv_heads, s.q_stride]
            for r, n, sl, p0 in plan.runs:
                fa_window(q[r:r + n], *pages, table, slot=sl, pos0=p0, ctx_k=k, ctx_vt=vt, out=out[r:r + n], gate=None if gate is None else gate[r:r + n], **how)
        groups = plan.groups if tiled else [(r, min(m, r + B.group)) for r in range(0, m, B.group)]
        rest = plan.step_positions if tiled else pos
        splits = s.splits(B.context) if bf16 else 0
        if splits:
            for lo, hi in groups:
                gqa_window(q[lo:hi], *pages, rest[lo:hi], slot[lo:hi], table, splits=splits, most_ahead=s.most_ahead(B.context), scratch=B.scratch,
                           out=out[lo:hi], gate=None if gate is None else gate[lo:hi], **how)
        elif groups:
            window_attn(q, *pages, rest, slot, table, out=out, gate=gate, **how)
