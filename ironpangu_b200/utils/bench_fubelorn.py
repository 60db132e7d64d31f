"""Prefill and decode throughput of the Fubelorn design beside the closest existing model - the Falinex decoder (recurrent layers and windowed attention over an
f32 residual, same executors) with the same width, depth, heads and parameter count - and the time of every kernel group of each against its roofline.

    python bench.py --design fubelorn                # through the benchmark's command line
    python -m ironpangu_b200.utils.bench_fubelorn --sizes small,text

Random weights, synthetic tokens. Model steps are CUDA graphs where the engine replays graphs, device events around them; kernel groups are
timed over all layers of their kind in one graph (distinct weights, pages and states per layer) with the L2 flushed before every run."""
from __future__ import annotations

import argparse
import json
from typing import Dict, List

import torch

from .bench_falinex import L_bytes, Timer, _line, _visible, falinex_arm, peaks

BF16 = torch.bfloat16
NAMES = ("layers", "width", "heads", "kv_heads", "ff", "vocab", "window", "keep", "pool", "rec_heads", "streams")
SIZES = {          # heads of 128 columns; recurrences of 128 x 128
    "small": (8, 1024, 8, 4, 4096, 32000, 512, 16, 16, 4, 2),
    "text": (16, 2048, 16, 4, 6144, 128000, 1024, 16, 16, 8, 2),
    "wide": (8, 4096, 32, 8, 16384, 128000, 1024, 16, 16, 16, 4),
}
DIM = 128


def fubelorn_arm(size, prompt: int, chunk_rows: int, batches: List[int], t: Timer, pk) -> Dict:
    from ironpangu_b200.models import fubelorn as M
    from ironpangu_b200.ops import hyper_streams as HS
    from ironpangu_b200.ops import stream_norm as N
    from ironpangu_b200.parallel.fabric import Fabric

    c = dict(zip(NAMES, size))
    dev = torch.device("cuda", 0)
    cfg = M.FubelornConfig.text(dim=DIM, rec_dim=DIM, state=DIM, **c)
    fab = Fabric(0, 1)
    nslots, ctx = max(batches), prompt + 512
    w = M.random_weights(cfg, dev)
    dec = M.FubelornDecoder(cfg, w, fab, max_tokens=8, max_context=ctx, num_slots=nslots, keep_logits=True)
    del w
    torch.cuda.empty_cache()
    rows = M.FubelornRows(dec, max_rows=chunk_rows)
    for r in range(nslots):
        dec.state_manager.admit(r, ctx)
    dec.state_manager.flush()
    toks = torch.randint(0, cfg.vocab, (prompt,), dtype=torch.int32, device=dev)
    res = {"params_m": round(cfg.param_count() / 1e6), "prefill": {}, "decode": {}, "kernels": []}

    def prefill():
        for p0 in range(0, prompt, chunk_rows):
            rows.forward(toks[p0:p0 + chunk_rows], p0, 0)

    ms = t.run(prefill, graph=False, flush=False, reps=5)
    res["prefill"] = {"tokens": prompt, "ms": round(ms, 3), "tokens_s": round(prompt / ms * 1e3)}
    for b in batches:
        pos = torch.full((b,), prompt, dtype=torch.int32, device=dev)
        sl = torch.arange(b, dtype=torch.int32, device=dev)
        tk = toks[:b].contiguous()
        if b <= 8:
            dec.tokens[:b].copy_(tk); dec.positions[:b].copy_(pos); dec.slots[:b].copy_(sl)
            ms = t.run(lambda: dec.forward(b), flush=False)
        else:
            plan = rows.plan(list(range(b)), [prompt] * b)
            ctl, sel = plan.control.to(dev), torch.arange(b, device=dev)
            ms = t.run(lambda: rows.forward_rows(tk, pos, sl, sel, plan, ctl), graph=False, flush=False)
        res["decode"][b] = {"ms": round(ms, 4), "tokens_s": round(b / ms * 1e3)}
    st, W, S, ff = fab.desc.status, cfg.width, max(cfg.streams, 1), c["ff"]
    kinds = {k: [L for L in dec.layers if L["c"].kind == k] for k in M.MIXERS}
    both = kinds["parallel"] + kinds["parallel_2"]

    def group(name, Ls, fn, bytes_, flops=0.0):
        ms = t.run(lambda: [fn(L) for L in Ls]) / len(Ls)
        res["kernels"].append(_line(name, ms, bytes_, flops, pk))

    shape = lambda k: kinds[k][0]["c"].right
    projection = lambda L: 2.0 * L["c"].in_cols * W

    for n in (1, 64):
        B = dec.rows if n <= 8 else rows.B
        pos = torch.full((n,), prompt, dtype=torch.int32, device=dev)
        sl = torch.arange(n, dtype=torch.int32, device=dev)
        B.rotary.fill(pos)
        attend = lambda L: L["left"].attend(B.attn, n, L["pages"], B.rotary.get(*L["c"].left.rotation), pos, sl, None, dec.page_table, cfg.eps, B.mixed[L["c"].mixed][:n], st)
        for k, what in (("parallel", "kept positions"), ("parallel_2", "blocks")):
            l = kinds[k][0]["c"].left
            keys = min(l.window, prompt + 1) + l.most_ahead(prompt + 1)
            group(f"window attention, {what} (norm, rotation, pages, attention, gate), {n} sequences", kinds[k], attend,
                  n * keys * l.row * 2 + n * (l.heads + 2 * l.kv_heads) * l.dim * 4)
        for k, what in (("parallel", "delta rule"), ("mamba2", "state-space"), ("parallel_2", "matrix memory")) if n > 1 else ():
            r = shape(k)
            group(f"recurrence step, {what} (convolution, gates, step, norm), {n} sequences", kinds[k],
                  lambda L: L["right"].mix(B.rec, L["state"], B.attn.proj[:n], pos, sl, None, dec.epoch, cfg.eps, B.mixed[L["c"].mixed][:n, L["c"].mixed[0]:]),
                  n * (8.0 * r.heads * r.E * r.dim + 2 * r.in_cols + 2 * r.inner))
    # the fused launches of one decode row
    B, pos, sl = dec.rows, torch.full((1,), prompt, dtype=torch.int32, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    xs, proj = [t[:1, :, :W] for t in B.streams], B.attn.proj[:1]
    front = lambda L, q, w, out, act=None: HS.gemv_streams(xs[0], xs[1], B.y[:1], L["sub"][0], L["sub"][q], cfg.eps, dec.epoch, pos, sl, w, out, act)
    for k, name in (("parallel", "parallel"), ("mamba2", "state-space")):
        group(f"input projection behind streams, norm and convolution, {name} layer, 1 row", kinds[k], lambda L: front(L, 0, L["in"], proj), projection(kinds[k][0]))
    for k, what in (("parallel", "delta rule"), ("mamba2", "state-space"), ("parallel_2", "matrix memory")):
        r = shape(k)
        group(f"recurrence step, {what} (convolution, gates, step), 1 row", kinds[k], lambda L: L["right"].decode(B.rec, L["state"], proj, pos, sl, dec.epoch),
              8.0 * r.heads * r.E * r.dim + 2 * r.in_cols)
        group(f"output projection behind norm and gate, {what}, 1 row", kinds[k],
              lambda L: L["right"].gemv_mixed(B.rec, proj, cfg.eps, B.mixed[L["c"].mixed][:1], L["c"].mixed[0], L["out"], B.y[:1]), 2.0 * W * sum(kinds[k][0]["c"].mixed))
    group("up projection behind streams, norm and convolution + GELU, 1 row", dec.layers, lambda L: front(L, 1, L["up"], B.act[ff][:1], "gelu_erf"), 2.0 * W * ff)
    group("down projection, 1 row", dec.layers, lambda L: N.gemv_act(B.act[ff][:1], L["down"], B.y[:1]), 2.0 * W * ff)
    for n in (64, chunk_rows):
        B = dec.rows if n <= 8 else rows.B
        pos = torch.arange(prompt - n, prompt, dtype=torch.int32, device=dev) if n == chunk_rows else torch.full((n,), prompt, dtype=torch.int32, device=dev)
        sl = torch.zeros(n, dtype=torch.int32, device=dev) if n == chunk_rows else torch.arange(n, dtype=torch.int32, device=dev)
        xa, a, b = B.xa[:n], B.streams[0][:n, :, :W], B.streams[1][:n, :, :W]
        flops = lambda k: 2.0 * n * k if n > 8 else 0.0
        group(f"streams, norm, convolution, {n} rows", dec.layers, lambda L: HS.streams_rows(a, b, B.y[:n], L["sub"][0], L["sub"][1], L["sub"][1].gain, cfg.eps, dec.epoch, pos, sl, xa),
              n * W * (8.0 * S + 4 + 2) + 4.0 * W * cfg.taps)
        for k, name in (("parallel", "parallel"), ("mamba2", "state-space")):
            group(f"input projection, {name} layer, {n} rows", kinds[k], lambda L: N.linear(xa, L["in"], B.attn.proj[:n, :L["c"].in_cols], status_ptr=st), projection(kinds[k][0]),
                  flops(W * kinds[k][0]["c"].in_cols))
            group(f"output projection, {name} layer, {n} rows", kinds[k], lambda L: dec._product(B, B.mixed[L["c"].mixed][:n], L["out"], n), 2.0 * W * sum(kinds[k][0]["c"].mixed),
                  flops(W * sum(kinds[k][0]["c"].mixed)))
        group(f"up projection + GELU, {n} rows", dec.layers, lambda L: N.linear(xa, L["up"], B.act[ff][:n, :ff], "gelu_erf", status_ptr=st), 2.0 * W * ff, flops(W * ff))
        group(f"down projection, {n} rows", dec.layers, lambda L: dec._product(B, B.act[ff][:n], L["down"], n), 2.0 * W * ff, flops(W * ff))
    m = chunk_rows
    B = rows.B
    pos = torch.arange(prompt - m, prompt, dtype=torch.int32, device=dev)
    sl = torch.zeros(m, dtype=torch.int32, device=dev)
    plan = rows.plan([0] * m, list(range(prompt - m, prompt)))
    dp = plan.bind(plan.control.to(dev), pos)
    B.attn.proj.normal_()
    B.rotary.fill(pos)
    for k, what in (("parallel", "kept positions"), ("parallel_2", "blocks")):
        l = kinds[k][0]["c"].left
        pairs = _visible(m, prompt - m, l.window) + sum(l.most_ahead(prompt - m + i + 1) for i in range(m))
        group(f"window attention, {what}, {m} rows", kinds[k],
              lambda L: L["left"].attend(B.attn, m, L["pages"], B.rotary.get(*L["c"].left.rotation), pos, sl, dp, dec.page_table, cfg.eps, B.mixed[L["c"].mixed][:m], st),
              m * (2 * l.heads + 2 * l.kv_heads) * l.dim * 2, 4.0 * pairs * l.heads * l.dim)
    for k, what in (("parallel", "delta rule"), ("mamba2", "state-space"), ("parallel_2", "matrix memory")):
        r, C = shape(k), dec.chunk
        f = 2.0 * m * r.heads * (C * r.dim + 2 * r.dim * r.E + C * r.E)
        if r.kind == "delta":          # the keys' products among themselves, the triangular solve, the corrections
            f += 2.0 * m * r.heads * (C * r.dim / 2 + C * (r.dim + r.E) / 2 + r.dim * r.E)
        group(f"recurrence chunks, {what} (convolution, gates, norm), {m} rows", kinds[k],
              lambda L: L["right"].mix(B.rec, L["state"], B.attn.proj[:m], pos, sl, dp, dec.epoch, cfg.eps, B.mixed[L["c"].mixed][:m, L["c"].mixed[0]:], st),
              m * (2.0 * r.in_cols + 2 * r.inner), f)
    res["fabric_status"] = fab.status()
    dec.state_manager.close()
    fab.close()
    return res


def like_falinex(size, params_m: int) -> tuple:
    """The Falinex size (its feed-forward width) with that many parameters."""
    from ironpangu_b200.models import falinex as F

    c = dict(zip(NAMES, size))
    make = lambda ff: (c["width"], c["layers"], c["heads"], c["kv_heads"], DIM, ff, c["vocab"], c["window"])
    count = lambda ff: F.FalinexConfig.text2b(layers=c["layers"], width=c["width"], heads=c["heads"], kv_heads=c["kv_heads"], dim=DIM, ff=ff, vocab=c["vocab"],
                                              window=c["window"]).param_count()
    per = (params_m * 1e6 - count(256)) / (2 * c["width"] * c["layers"])
    return make(max(256, 256 + int(per) // 128 * 128))


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="small,text,wide")
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--chunk", type=int, default=2048)
    ap.add_argument("--batches", default="1,8,64")
    ap.add_argument("--only", action="store_true", help="without the other model")
    args = ap.parse_args(argv)
    torch.cuda.set_device(0)
    pk, t = peaks(), Timer()
    batches = [int(b) for b in args.batches.split(",")]
    for name in args.sizes.split(","):
        s = SIZES[name]
        out = {"bench": "fubelorn", "size": name, "config": dict(zip(NAMES, s)), "prompt": args.prompt, "chunk": args.chunk, "dtype": "bf16", "data": "synthetic, random weights",
               "peaks": pk, "fubelorn": fubelorn_arm(s, args.prompt, args.chunk, batches, t, pk)}
        torch.cuda.empty_cache()
        if not args.only:
            f = like_falinex(s, out["fubelorn"]["params_m"])
            out["falinex"] = falinex_arm(f, args.prompt, args.chunk, batches, t, pk)
            out["falinex"]["ffn"] = f[5]
            torch.cuda.empty_cache()
        print(json.dumps(out), flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
