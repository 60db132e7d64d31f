"""Prefill and decode throughput of the Mikutar design beside its closest other models, and the time of every kernel group of each against its
roofline: the Ponenex decoder (routed experts over an f32 residual, same executors) with the same width, depth, experts per token and parameter
count, and the dense GQA decoder with the same heads and as many parameters as a Mikutar token uses (for attention and dense linears).

    python bench.py --design mikutar                # through the benchmark's command line
    python -m ironpangu_b200.utils.bench_mikutar --sizes small,text

Random weights, synthetic tokens. Model steps are CUDA graphs where the engine replays graphs, device events around them; kernel groups are
timed over all layers of their kind in one graph (distinct weights and pages per layer) with the L2 flushed before every run. Decode rows stand
at the last position of a chunk, where a chunked layer sees most keys."""
from __future__ import annotations

import argparse
import json
from typing import Dict, List

import torch

from .bench_falinex import L_bytes, Timer, _line, _visible, dense_arm, peaks
from .bench_ponenex import _spread_routes, ponenex_arm

BF16 = torch.bfloat16
NAMES = ("layers", "width", "heads", "kv_heads", "ff", "experts", "top", "expert_ff", "shared_ff", "vocab", "window", "chunk")
SIZES = {          # heads of 128 columns
    "small": (8, 1024, 8, 2, 4096, 16, 4, 512, 512, 32000, 512, 512),
    "text": (16, 2048, 16, 4, 6144, 64, 8, 768, 768, 128000, 1024, 1024),
    "wide": (8, 4096, 32, 8, 12288, 64, 8, 1536, 1536, 128000, 2048, 2048),
}
DIM = 128


def mikutar_arm(size, prompt: int, chunk_rows: int, batches: List[int], t: Timer, pk) -> Dict:
    from ironpangu_b200.models import mikutar as M
    from ironpangu_b200.ops import parallel_layer as PL
    from ironpangu_b200.ops import stream_norm as N
    from ironpangu_b200.parallel.fabric import Fabric

    c = dict(zip(NAMES, size))
    dev = torch.device("cuda", 0)
    cfg = M.MikutarConfig.text(dim=DIM, **c)
    fab = Fabric(0, 1)
    nslots, ctx = max(batches), prompt + 512
    w = M.random_weights(cfg, dev)
    dec = M.MikutarDecoder(cfg, w, fab, max_tokens=8, max_context=ctx, num_slots=nslots, keep_logits=True)
    del w
    torch.cuda.empty_cache()
    for i, L in enumerate(dec.layers):
        if L["experts"] is not None:
            _spread_routes(L["experts"].w_router, i)
            L["experts"].w_router.mul_(cfg.width ** -0.5)          # scores that do not saturate
    rows = M.MikutarRows(dec, max_rows=chunk_rows)
    for r in range(nslots):
        dec.state_manager.admit(r, ctx)
    dec.state_manager.flush()
    toks = torch.randint(0, cfg.vocab, (prompt,), dtype=torch.int32, device=dev)
    res = {"params_m": round(cfg.param_count() / 1e6), "active_m": round(cfg.active_params() / 1e6), "prefill": {}, "decode": {}, "kernels": []}

    def prefill():
        for p0 in range(0, prompt, chunk_rows):
            rows.forward(toks[p0:p0 + chunk_rows], p0, 0)

    ms = t.run(prefill, graph=False, flush=False, reps=5)
    res["prefill"] = {"tokens": prompt, "ms": round(ms, 3), "tokens_s": round(prompt / ms * 1e3)}
    for b in batches:
        pos = torch.full((b,), prompt - 1, dtype=torch.int32, device=dev)
        sl = torch.arange(b, dtype=torch.int32, device=dev)
        tk = toks[:b].contiguous()
        if b <= 8:
            dec.tokens[:b].copy_(tk); dec.positions[:b].copy_(pos); dec.slots[:b].copy_(sl)
            ms = t.run(lambda: dec.forward(b), flush=False)
        else:
            plan = rows.plan(list(range(b)), [prompt - 1] * b)
            ctl, sel = plan.control.to(dev), torch.arange(b, device=dev)
            ms = t.run(lambda: rows.forward_rows(tk, pos, sl, sel, plan, ctl), graph=False, flush=False)
        res["decode"][b] = {"ms": round(ms, 4), "tokens_s": round(b / ms * 1e3)}
    st, eps = fab.desc.status, cfg.eps
    dense = [R for R in dec.runs if R["experts"] is None]
    routed = [R for R in dec.runs if R["experts"] is not None]
    win = [R for R in dec.runs if not R["mix"].shape.chunked]
    chu = [R for R in dec.runs if R["mix"].shape.chunked]

    def group(name, Ls, fn, bytes_, flops=0.0):
        ms = t.run(lambda: [fn(L) for L in Ls]) / len(Ls)
        res["kernels"].append(_line(name, ms, bytes_, flops, pk))

    def setup(B, n, pos):
        B.rotary.fill(pos)
        for b in (B.attn.proj, B.xa, B.x, B.y):
            b[:n].normal_()
        for b in B.join.rows.values():
            b[:n].normal_()
        B.experts.start(n)

    H, G = cfg.layers[0].mixer.heads, cfg.layers[0].mixer.kv_heads
    kv_row = 2 * G * DIM * 2.0
    act_row = (H + 2 * G) * DIM * 2 * 2.0
    unit = 2.0 * 3 * cfg.width * c["expert_ff"]
    join_d, join_m = L_bytes(dense[0]["join"].w), L_bytes(routed[0]["join"].w)
    w_in, gu_d, gu_m = L_bytes(dense[0]["mix"].w_in), L_bytes(dense[0]["join"].gate_up), L_bytes(routed[0]["join"].gate_up)
    w_router = L_bytes(routed[0]["experts"].w_router)
    keys = {"windowed": min(c["window"], prompt), "chunked": (prompt - 1) % c["chunk"] + 1}

    def front(R):
        PL.parallel_in(y, None, R["norm1"], eps, x, x2, xa, R["mix"], B.attn.proj[:1], R["join"], B.join, R["experts"], B.experts, fab.ticket_ptr)

    B = dec.rows
    pos, sl = torch.full((1,), prompt - 1, dtype=torch.int32, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    setup(B, 1, pos)
    x, x2, y, xa = B.x[:1], B.x2[:1], B.y[:1], B.xa[:1]
    group("front (residual, norm, projection, unit) of dense layers, 1 row", dense, front, w_in + gu_d)
    group("front (residual, norm, projection, unit, router) of routed layers, 1 row", routed, front, w_in + gu_m + w_router)
    for n in (1, nslots):
        B = dec.rows if n == 1 else rows.B
        pos, sl = torch.full((n,), prompt - 1, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int32, device=dev)
        setup(B, n, pos)
        for what, Ls in (("windowed", win), ("chunked", chu)):
            group(f"{what} attention (norm, rotation, cache write, attention, gate), {n} sequences", Ls, lambda R: dec._attend(B, R, n, pos, sl, None),
                  n * (keys[what] * kv_row + act_row))
    B = dec.rows
    group("output product of dense layers, 1 row", dense, lambda R: R["join"].decode(B.join, 1, y, None), join_d)
    group("output product of routed layers, 1 row", routed, lambda R: R["join"].decode(B.join, 1, y, y), join_m)
    group("routed experts, 1 row", routed, lambda R: R["experts"].decode_chosen(B.experts, 1, xa, y), c["top"] * unit)
    B = rows.B
    for n in (nslots, chunk_rows):
        hit = c["experts"] * (1.0 - (1.0 - c["top"] / c["experts"]) ** n)
        pos = torch.arange(prompt - n, prompt, dtype=torch.int32, device=dev)
        setup(B, n, pos)
        x, xa, y = B.x[:n], B.xa[:n], B.y[:n]
        own = dense[0]["join"].rows(B.join, n, y, st)
        group(f"input projection, {n} rows", dec.runs, lambda R: R["mix"].project(B.attn, xa, st), w_in, n * w_in)
        group(f"gated unit of dense layers, {n} rows", dense, lambda R: R["join"].unit_rows(B.join, xa, st), gu_d, n * gu_d)
        group(f"gated unit of routed layers, {n} rows", routed, lambda R: R["join"].unit_rows(B.join, xa, st), gu_m, n * gu_m)
        group(f"output product of dense layers, {n} rows", dense, lambda R: R["join"].rows(B.join, n, y, st), join_d, n * join_d)
        group(f"output product of routed layers, {n} rows", routed, lambda R: R["join"].rows(B.join, n, y, st), join_m, n * join_m)
        group(f"residual and next norm, {n} rows", dense, lambda R: N.post_norm_add(own, None, eps, x, xa, R["norm1"]), n * cfg.width * 14.0)
        group(f"router, routed experts, residual and next norm, {n} rows", routed, lambda R: R["experts"].rows(B.experts, n, xa, None, R["norm1"], eps, x, st, base=own),
              hit * unit + w_router, n * c["top"] * unit)
    m = chunk_rows
    pos, sl = torch.arange(prompt - m, prompt, dtype=torch.int32, device=dev), torch.zeros(m, dtype=torch.int32, device=dev)
    setup(B, m, pos)
    plan = rows.plan([0] * m, list(range(prompt - m, prompt)))
    dp = plan.bind(plan.control.to(dev), pos)
    pairs = {"windowed": _visible(m, prompt - m, c["window"]), "chunked": float(sum((prompt - m + i) % c["chunk"] + 1 for i in range(m)))}
    for what, Ls in (("windowed", win), ("chunked", chu)):
        group(f"{what} attention, {m} rows", Ls, lambda R: dec._attend(B, R, m, pos, sl, dp), m * (2 * H + 2 * G) * DIM * 2.0, 4.0 * pairs[what] * H * DIM)
    res["fabric_status"] = fab.status()
    dec.state_manager.close()
    fab.close()
    return res


def ponenex_like(size, params: int) -> tuple:
    """Ponenex with the same width, depth, experts per token and window, and as many experts a layer as reach ``params``."""
    from ironpangu_b200.models.ponenex import PonenexConfig

    c = dict(zip(NAMES, size))
    s = lambda e: (c["layers"], c["width"], c["heads"], c["width"] * 3 // 8, e, c["top"], c["expert_ff"], c["vocab"], c["window"])
    count = lambda e: PonenexConfig.text(layers=c["layers"], width=c["width"], heads=c["heads"], q_rank=c["width"] * 3 // 8, experts=e, top=c["top"], ff=c["expert_ff"],
                                         shared_ff=c["expert_ff"], vocab=c["vocab"], window=c["window"]).param_count()
    return s(min(range(c["top"], 257), key=lambda e: abs(count(e) - params)))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="small,text,wide")
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--chunk", type=int, default=2048, help="rows of a prompt step")
    ap.add_argument("--batches", default="1,8,64")
    ap.add_argument("--arms", default="mikutar,ponenex,dense")
    args = ap.parse_args(argv)
    torch.cuda.set_device(0)
    pk, t = peaks(), Timer()
    batches = [int(b) for b in args.batches.split(",")]
    from ironpangu_b200.models.mikutar import MikutarConfig

    for name in args.sizes.split(","):
        s = SIZES[name]
        c = dict(zip(NAMES, s))
        cfg = MikutarConfig.text(dim=DIM, **c)
        out = {"bench": "mikutar", "size": name, "config": c, "prompt": args.prompt, "chunk": args.chunk, "dtype": "bf16", "data": "synthetic, random weights", "peaks": pk}
        for arm in args.arms.split(","):
            if arm == "mikutar":
                out[arm] = mikutar_arm(s, args.prompt, args.chunk, batches, t, pk)
            elif arm == "ponenex":
                ps = ponenex_like(s, cfg.param_count())
                out[arm] = dict(ponenex_arm(ps, args.prompt, args.chunk, batches, t, pk), experts=ps[4])
            else:
                out[arm] = dense_arm((c["width"], c["layers"], c["heads"], c["kv_heads"], DIM, 0, c["vocab"], c["window"]), cfg.active_params(), args.prompt, args.chunk, batches,
                                     t, pk)
            torch.cuda.empty_cache()
        print(json.dumps(out), flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
