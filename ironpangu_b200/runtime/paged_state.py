"""Sequence states of an engine whose KV pages come from one pool: pages are taken when tokens arrive, given back when a request
ends - and, for a model all of whose attention is windowed, as soon as every window has passed them - and used again by other
requests. The bookkeeping (free lists, leases with generations, all-or-nothing growth) is the host core's state pool
(``csrc/core/state_pool.h``); this class keeps the page table the kernels read in step with it.

A resident's slot states (recurrent layers) are bound to its sequence slot; kernels start from zero at position 0, so a slot used
again needs no clearing. Table entries of positions a resident does not hold are -1.
Reference: crates/inferfabric-runtime/src/state_pool.rs:13-479 (leases over pages and slots)."""
from __future__ import annotations

import hashlib
import json
from typing import Dict, List, Optional, Tuple

import torch

from .. import compiler


class PagedState:
    KV, SLOT = "kv", "recurrent"

    def __init__(self, *, model: str, context: int, residents: int, page_tokens: int, pool_pages: int, row_bytes: int, slot_bytes: int, vocab: int, device,
                 window: int = 0, max_batched_tokens: int = 1):
        """``row_bytes`` / ``slot_bytes``: bytes per token of all paged layers together / per sequence of all recurrent layers (0: the model
        has none). ``window``: the longest attention window when every attention layer has one, else 0 (pages are kept)."""
        self.context, self.residents, self.page_tokens, self.pool_pages, self.window = context, residents, page_tokens, pool_pages, window
        states = []
        if row_bytes:
            states.append({"name": self.KV, "storage": {"kind": "pages", "page_tokens": page_tokens, "row_bytes": row_bytes}})
        if slot_bytes:
            states.append({"name": self.SLOT, "storage": {"kind": "slot", "slot_bytes": slot_bytes}})
        for i, s in enumerate(states):
            s.update(component=i, dtype="f32" if s["name"] == self.SLOT else "bytes", retention={"kind": "full"})
        manifest = {"format": "inferfabric.serving.v1", "max_context": context, "vocab": vocab, "eos": 0, "resident_sequences": residents,
                    "max_batched_tokens": max_batched_tokens, "states": states,
                    "identity": {"model": model, "program_sha256": hashlib.sha256(json.dumps([model, states]).encode()).hexdigest(), "target": "b200_module_v1",
                                 "tp": 1},
                    "variants": [{"name": "decode", "phase": "decode", "query_tokens": [1], "max_query_tokens": 1, "captured": True, "numerics": "rows"},
                                 {"name": "extend", "phase": "extend", "query_tokens": [], "max_query_tokens": context, "captured": False, "numerics": "rows"}]}
        self.paged = bool(row_bytes)
        self.pool = compiler.pool_create(manifest, {s["name"]: pool_pages if s["name"] == self.KV else residents for s in states}) if states else 0
        self.max_pages = (context + page_tokens - 1) // page_tokens
        self._host = torch.full((residents, self.max_pages), -1, dtype=torch.int32)
        self.table = self._host.to(device)
        self._dirty = False
        self._lease: List[Optional[Tuple[int, int]]] = [None] * residents
        self._held = [0] * residents          # tokens the lease covers
        self._trimmed = [0] * residents       # leading pages given back
        self._requests = 0
        self.pages_taken = self.pages_trimmed = 0

    def _call(self, op: str, **kw):
        try:
            return compiler.pool_call(self.pool, op, **kw)
        except compiler.CompileError as e:
            if e.kind == "capacity":
                raise OverflowError(e.message) from None
            raise

    def _show(self, resident: int, out: Dict) -> None:
        units = out["bindings"].get(self.KV, [])
        self.pages_taken += sum(1 for j in range(len(units)) if units[j] >= 0 and int(self._host[resident, j]) != units[j])
        self._host[resident].fill_(-1)
        if units:
            self._host[resident, :len(units)] = torch.tensor(units, dtype=torch.int32)
        self._dirty = True

    def admit(self, resident: int, reserve: int = 0) -> None:
        """A request starts in sequence slot ``resident``; ``reserve`` tokens get their pages now (0: as they arrive). Raises
        OverflowError when the pool cannot hold them."""
        if self._lease[resident] is not None:
            self.release(resident)
        if not self.pool:
            return
        tokens = max(1, reserve)
        self._requests += 1
        out = self._call("reserve", request=self._requests, tokens=tokens, slot=resident)
        self._lease[resident] = (out["lease"], out["generation"])
        # without a reservation the first pages are taken at once all the same: a lease covers at least one page
        self._held[resident], self._trimmed[resident] = (tokens + self.page_tokens - 1) // self.page_tokens * self.page_tokens, 0
        self._show(resident, out)

    def ensure(self, resident: int, tokens: int) -> None:
        """Positions below ``tokens`` of the resident get pages. Raises OverflowError when the pool is exhausted (nothing changes)."""
        if tokens > self.context:
            raise OverflowError("the sequence runs past the context")
        if not self.paged or tokens <= self._held[resident]:
            return
        if self._lease[resident] is None:
            raise RuntimeError(f"resident {resident} was not admitted")
        lease, gen = self._lease[resident]
        self._show(resident, self._call("extend", lease=lease, generation=gen, tokens=tokens))
        self._held[resident] = (tokens + self.page_tokens - 1) // self.page_tokens * self.page_tokens

    def advance(self, resident: int, position: int) -> None:
        """The next token of the resident is at ``position``: pages that no window will reach again go back to the pool."""
        if not (self.paged and self.window) or self._lease[resident] is None:
            return
        first_live = max(0, position - self.window + 1)
        dead = first_live // self.page_tokens
        if dead > self._trimmed[resident]:
            lease, gen = self._lease[resident]
            self._show(resident, self._call("trim", lease=lease, generation=gen, component=self.KV, first_live=first_live))
            self.pages_trimmed += dead - self._trimmed[resident]
            self._trimmed[resident] = dead

    def release(self, resident: int) -> None:
        if self._lease[resident] is None:
            return
        lease, gen = self._lease[resident]
        self._call("retire", lease=lease, generation=gen)
        self._lease[resident] = None
        self._held[resident] = self._trimmed[resident] = 0
        self._host[resident].fill_(-1)
        self._dirty = True

    def flush(self) -> int:
        """Bring the device table up to date (before a step is launched); returns the bytes copied."""
        if not self._dirty:
            return 0
        self.table.copy_(self._host)          # pageable source: staged before the call returns, later host changes cannot reach it
        self._dirty = False
        return self._host.numel() * 4

    def usage(self) -> Dict:
        u = self._call("usage") if self.pool else {}
        return {"format": "ifab.paged-state.v1", "pages_taken": self.pages_taken, "pages_trimmed": self.pages_trimmed, "components": u}

    def close(self) -> None:
        if self.pool:
            self._call("close")
            self.pool = 0
