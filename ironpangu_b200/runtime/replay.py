"""Trace replay: feeds given token ids through a checkpoint's model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come as JSON lines on standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

one batch each: ``entries`` bring the next tokens of requests and the places among them whose logits are asked for, ``end`` lists
the requests that are finished after the step. A request is admitted at its first entry, into one of ``RESIDENTS`` sequence slots;
its KV pages come from a pool of ``--max-tokens`` tokens. A step in which something is wanted writes ``DIR/<step>.f32`` (f32
``[wanted, vocab]``, in the order of entries and places); after every step a line ``done <step>`` goes to standard output.

The model is opened through ``models/registry.py`` and stepped by the serving engine (``BatchEngine.step_logits``): its batches,
graphs, pages and states."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict

RESIDENTS = 4
ROWS = 1024           # rows of one pass; wider steps take several


class Replay:
    def __init__(self, engine):
        self.engine = engine
        self.slot: Dict[str, int] = {}
        self.position: Dict[str, int] = {}

    def step(self, request: Dict):
        """Run one step; returns the wanted logits (host tensor) or None."""
        slices, tokens, want = [], [], []
        for e in request["entries"]:
            name = e["id"]
            if name not in self.slot:
                free = [r for r in range(self.engine.residents) if r not in self.slot.values()]
                if not free:
                    raise RuntimeError("more live requests than sequence slots")
                self.engine.admit(free[0], {}, 0)
                self.slot[name], self.position[name] = free[0], 0
            n = len(e["tokens"])
            if n == 0:
                continue
            slices.append([self.slot[name], self.position[name], n, False])
            tokens += e["tokens"]
            want.append(list(e.get("want", [])))
            self.position[name] += n
        out = self.engine.step_logits(slices, tokens, want) if slices else None
        for name in request.get("end", []):
            if name in self.slot:
                self.engine.release(self.slot.pop(name))
                del self.position[name]
        return out if out is not None and out.shape[0] else None


def open_engine(checkpoint: str, dtype: str, max_tokens: int):
    import torch

    from ..models import registry
    from ..ops import _lib
    from ..parallel.fabric import Fabric
    from .engine_worker import BatchEngine

    fam = registry.family_of(checkpoint)
    _lib.load(units=getattr(fam.load(), "KERNEL_UNITS", None))
    torch.cuda.set_device(0)
    fab = Fabric(0, 1)
    dec, rows = registry.open_checkpoint(checkpoint, fab, max_rows=min(ROWS, max(64, max_tokens)), max_tokens=8, max_context=max_tokens, num_slots=RESIDENTS,
                                         pool_tokens=max_tokens, keep_logits=True, dtype=torch.float32 if dtype == "float32" else torch.bfloat16)
    return BatchEngine(dec, os.path.basename(os.path.normpath(checkpoint)), max_tokens, dec.cfg.vocab, prefill=rows)


def main() -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits of the steps")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens of the KV page pool")
    args = ap.parse_args()
    from ..models import registry

    if args.dtype == "float32" and not registry.family_of(args.model).exact:
        print("this model family has no 32-bit mode", file=sys.stderr)
        return 3
    os.makedirs(args.out, exist_ok=True)
    replay = Replay(open_engine(args.model, args.dtype, (args.max_tokens + 63) // 64 * 64))
    for line in sys.stdin:
        if not line.strip():
            continue
        request = json.loads(line)
        logits = replay.step(request)
        if logits is not None:
            part = os.path.join(args.out, f".{request['step']}.part")
            logits.numpy().astype("<f4").tofile(part)
            os.replace(part, os.path.join(args.out, f"{request['step']}.f32"))
        print(f"done {request['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
