"""What decoders with an f32 residual stream share: step inputs, the paged-state manager, the output matrix with greedy selection, CUDA
graphs of a launch group, and the packed-step executor with its graphs. A model adds its weights, its per-layer states and its layer
chains.

``StreamDecoder`` runs decode rows (and pieces of prompts up to ``max_tokens`` rows) in one launch chain whose grid depends on the
row count only, so the engine replays it as a CUDA graph; ``StreamRows`` runs a packed step - portions of several prompts beside
decode rows - as matrix-matrix work. Both read the pages and recurrent states of ``decoder.state_manager`` (runtime/paged_state.py)."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..ops import decode as K
from ..ops import stream_norm as N
from ..ops.linear_attn import StepPlan
from ..parallel.fabric import Fabric
from ..runtime.paged_state import PagedState
from .checkpoint import pad8

BF16, F32 = torch.bfloat16, torch.float32
ATTN_ROWS = 64             # rows per launch of the split-KV attention kernels


class StreamDecoder:
    """Decode executor on one GPU: up to ``max_tokens`` (<= 8) rows per step, each with its own position and sequence slot; rows of
    one sequence inside a step are consecutive and in position order. Greedy next tokens land in ``next_ids``.

    A model provides ``_load(weights)`` (tensors on the device, among them ``embed``, ``head``, ``final_norm``), ``_state_bytes()``
    (bytes per token of all paged layers, bytes per sequence of all recurrent layers), ``_make_states()``, ``make_rows(rows,
    chunked)`` (step buffers with ``x``, ``xa`` and ``rows``), ``_layers`` and ``_layers_fused`` (both leave the rows ahead of the
    output matrix in ``xa``), and sets ``fused`` / ``fused_rows``: up to how many rows the fused chain takes."""

    name = "stream"
    chunk = 128            # rows per chunk of a packed step's long runs
    short_rows = 4         # runs of at most this many rows take the decode kernels inside a packed step
    logit_cap = 0.0        # > 0: logits are cap * tanh(logit / cap)
    fused_rows = 2         # beyond this the CUDA-core products are FMA-bound and the GEMMs take over

    def __init__(self, cfg, weights: Dict[str, torch.Tensor], fabric: Fabric, *, max_tokens: int = 8, max_context: int = 1024, num_slots: int = 1,
                 pool_tokens: int = 0, keep_logits: bool = False, dtype: torch.dtype = BF16):
        """``pool_tokens``: tokens the KV page pool holds for all sequences together (0: every slot can reach the full context)."""
        assert 1 <= max_tokens <= 8 and fabric.world == 1, f"the {self.name} decoder runs on one GPU"
        assert dtype in (BF16, F32)
        c, dev = cfg, fabric.device
        self.cfg, self.fabric, self.rank, self.world, self.dtype = cfg, fabric, 0, 1, dtype
        self.T, self.max_context, self.num_slots = max_tokens, max_context, num_slots
        per_slot = (max_context + c.page_tokens - 1) // c.page_tokens
        self.num_pages = (pool_tokens + c.page_tokens - 1) // c.page_tokens if pool_tokens else per_slot * num_slots
        self._load(weights)
        row_bytes, slot_bytes = self._state_bytes()
        self.state_manager = PagedState(model=self.name, context=max_context, residents=num_slots, page_tokens=c.page_tokens, pool_pages=self.num_pages,
                                        row_bytes=row_bytes, slot_bytes=slot_bytes, vocab=c.vocab, device=dev, window=c.window)
        self.page_table = self.state_manager.table
        self._make_states()
        T = max_tokens
        i32 = lambda: torch.zeros(T, dtype=torch.int32, device=dev)
        self.tokens, self.positions, self.slots, self.next_ids = i32(), i32(), i32(), i32()
        self.next_vals = torch.zeros(T, dtype=F32, device=dev)
        self.rows = self.make_rows(T, False)
        self._logits = torch.empty(T, c.vocab, dtype=F32, device=dev)
        self.logits = self._logits if keep_logits else None
        self.partial = torch.empty(((c.vocab + 7) // 8) * 8 * 2, dtype=F32, device=dev)
        self.sample_scratch = torch.empty(T * ((c.vocab + 4095) // 4096) * 128, dtype=F32, device=dev)
        self.inv_temp = torch.full((T,), 1e4, dtype=F32, device=dev)

    # -- weights -----------------------------------------------------------------------------------------------------------
    def _mat(self, W: Dict[str, torch.Tensor], *names: str) -> torch.Tensor:
        """Rows of the named matrices, one after the other, in the activation type; columns padded to 8 elements."""
        t = torch.cat([W[n].to(self.fabric.device) for n in names], 0).to(self.dtype)
        return torch.nn.functional.pad(t, (0, pad8(t.shape[1]) - t.shape[1])).contiguous()

    def _vec(self, W: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
        return W[name].to(self.fabric.device).float().contiguous()

    # -- one step ------------------------------------------------------------------------------------------------------------
    def forward(self, T: Optional[int] = None) -> torch.Tensor:
        n = self.T if T is None else T
        B, tok, pos, slot = self.rows, self.tokens[:n], self.positions[:n], self.slots[:n]
        if self.fused and n <= self.fused_rows:
            self._layers_fused(B, n, tok, pos, slot)
        else:
            self._layers(B, n, tok, pos, slot, None, True)
        if self.dtype == BF16:
            K.lm_head_argmax(B.xa[:n], self.head, self.fabric, vocab_offset=0, partial=self.partial, logits=None if self.logits is None else self.logits[:n],
                             out_ids=self.next_ids[:n], out_vals=self.next_vals[:n], cap=self.logit_cap)
        else:
            N.linear(B.xa[:n], self.head, self._logits[:n], cap=self.logit_cap)
            K.sample_topk(self._logits[:n], self.fabric, top_k=1, inv_temperature=self.inv_temp[:n], scratch=self.sample_scratch, out_ids=self.next_ids[:n])
        return self.next_ids[:n]

    def forward_feedback(self, T: Optional[int] = None) -> torch.Tensor:
        n = self.T if T is None else T
        self.forward(n)
        self.tokens[:n].copy_(self.next_ids[:n])
        self.positions[:n].add_(1)
        return self.next_ids[:n]

    def capture(self, T: Optional[int] = None, feedback: bool = False) -> torch.cuda.CUDAGraph:
        n = self.T if T is None else T
        self.forward(n)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            self.forward_feedback(n) if feedback else self.forward(n)
        return g


class StreamRows:
    """Packed-step executor: up to ``max_rows`` rows of any sequences (portions of prompts, decode rows), rows of one sequence
    consecutive and in position order, as one matrix-matrix pass. Steps without a long run and of at most ``graph_rows_max`` rows
    (a decode row per running sequence) replay a CUDA graph per row count."""

    packed = True              # the engine hands over the rows of a whole step
    batch_threshold = 8

    def __init__(self, dec: StreamDecoder, max_rows: int = 512):
        self.dec, self.M = dec, max_rows
        self.B = dec.make_rows(max_rows, True)
        dev = dec.fabric.device
        self.graph_rows_max = min(64, max_rows)
        self.use_graphs = True
        self._static = torch.zeros(3, self.graph_rows_max, dtype=torch.int32, device=dev)
        self._graphs: Dict[int, torch.cuda.CUDAGraph] = {}

    def plan(self, slots: List[int], positions: List[int]) -> StepPlan:
        return StepPlan(slots, positions, short=self.dec.short_rows, group=ATTN_ROWS, chunk=self.dec.chunk)

    def _run(self, tokens, positions, slots, plan: StepPlan, control, probe) -> None:
        d, m = self.dec, tokens.numel()
        if plan.runs or m > self.graph_rows_max or not self.use_graphs or probe is not None:
            d._layers(self.B, m, tokens, positions, slots, plan.bind(control, positions), False, probe)
            return
        st = self._static[:, :m]
        st[0].copy_(tokens)
        st[1].copy_(positions)
        st[2].copy_(slots)
        g = self._graphs.get(m)
        if g is not None:
            g.replay()
            return
        d._layers(self.B, m, *st, None, False)             # the real run of this step (and the warm-up of the capture)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):                          # records only: no state is touched a second time
            d._layers(self.B, m, *st, None, False)
        self._graphs[m] = g

    def forward_rows(self, tokens: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor, select: torch.Tensor, plan: StepPlan, control: torch.Tensor,
                     probe: Optional[list] = None) -> torch.Tensor:
        """f32 logits ``[len(select), vocab]`` of rows ``select``; ``control``: ``plan.control`` on the device; ``probe`` (a list) receives
        the residual stream after every layer."""
        d, c, m = self.dec, self.dec.cfg, tokens.numel()
        assert 1 <= m <= self.M and plan.rows == m
        self._run(tokens, positions, slots, plan, control, probe)
        xn = torch.zeros(select.numel(), self.B.xa.shape[1], dtype=d.dtype, device=tokens.device)
        N.rms_rows(self.B.x[:m], d.final_norm, c.eps, xn, select.to(torch.int32))
        logits = torch.empty(select.numel(), c.vocab, dtype=F32, device=tokens.device)
        N.linear(xn, d.head, logits, status_ptr=d.fabric.desc.status, cap=d.logit_cap)
        return logits

    def forward(self, tokens: torch.Tensor, pos0: int, slot: int = 0) -> torch.Tensor:
        """A chunk of one sequence; returns the greedy next token (device tensor ``[1]``)."""
        d, m, dev = self.dec, tokens.numel(), tokens.device
        pos = torch.arange(pos0, pos0 + m, dtype=torch.int32, device=dev)
        sl = torch.full((m,), slot, dtype=torch.int32, device=dev)
        plan = self.plan([slot] * m, list(range(pos0, pos0 + m)))
        logits = self.forward_rows(tokens, pos, sl, torch.tensor([m - 1], device=dev), plan, plan.control.to(dev))
        if d.logits is not None:
            d.logits[:1].copy_(logits)
        K.sample_topk(logits, d.fabric, top_k=1, inv_temperature=d.inv_temp[:1], scratch=d.sample_scratch, out_ids=d.next_ids[:1])
        return d.next_ids[:1]
