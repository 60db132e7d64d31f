"""Prefill and decode throughput of the Falinex design beside the closest existing model (the dense GQA decoder) at equal size, and
the time of every kernel group against its roofline.

    python bench.py --design falinex                # through the benchmark's command line
    python -m ironpangu_b200.utils.bench_falinex --sizes small,2b

Random weights, synthetic tokens. Model steps are CUDA graphs where the engine replays graphs, device events around them; kernel groups
are timed over all layers of their kind in one graph (distinct weights and states per layer) with the L2 flushed before every run.
The dense model's feed-forward width is chosen so that both models have the same number of parameters per layer."""
from __future__ import annotations

import argparse
import json
import statistics
from pathlib import Path
from typing import Callable, Dict, List

import torch

SIZES = {          # width, layers, heads, kv heads, head size, feed-forward, vocabulary, window
    "small": (1024, 12, 8, 4, 128, 4096, 32000, 512),
    "2b": (2048, 24, 16, 4, 128, 6144, 151936, 1024),
    "8b": (4096, 16, 32, 8, 128, 16384, 128000, 1024),
}


def peaks() -> Dict[str, float]:
    f = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if f.exists():
        j = json.loads(f.read_text())
        return {"hbm_gbs": j["hbm_gbs"], "bf16_tflops": j["bf16_tflops"], "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


class Timer:
    def __init__(self):
        self.flush_buf = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def run(self, fn: Callable[[], None], reps: int = 7, graph: bool = True, flush: bool = True) -> float:
        """Median milliseconds of one execution."""
        fn()
        torch.cuda.synchronize()
        if graph:
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g):
                fn()
            call = g.replay
        else:
            call = fn
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        out = []
        for i in range(reps + 3):
            if flush:
                self.flush_buf.add_(1)
            torch.cuda.synchronize()
            e0.record()
            call()
            e1.record()
            torch.cuda.synchronize()
            if i >= 3:
                out.append(e0.elapsed_time(e1))
        return statistics.median(out)


def _line(name: str, ms: float, bytes_: float, flops: float, pk) -> Dict:
    t_mem, t_mma = bytes_ / pk["hbm_gbs"] / 1e6, flops / pk["bf16_tflops"] / 1e9
    bound = max(t_mem, t_mma)
    return {"kernel": name, "us": round(ms * 1e3, 2), "roofline_us": round(bound * 1e3, 2), "bound": "memory" if t_mem >= t_mma else "tensor",
            "of_measured": round(bound / ms, 3)}


def _visible(n: int, p0: int, window: int) -> float:
    """Query-key pairs of n consecutive queries from position p0."""
    return float(sum(min(p0 + i + 1, window) if window else p0 + i + 1 for i in range(n)))


def falinex_arm(size, prompt: int, chunk: int, batches: List[int], t: Timer, pk) -> Dict:
    from ironpangu_b200.models import falinex as F
    from ironpangu_b200.ops import decode as K
    from ironpangu_b200.ops import stream_norm as N
    from ironpangu_b200.parallel.fabric import Fabric

    width, layers, heads, kv, hd, ff, vocab, window = size
    dev = torch.device("cuda", 0)
    cfg = F.FalinexConfig.text2b(layers=layers, width=width, heads=heads, kv_heads=kv, dim=hd, ff=ff, vocab=vocab, window=window)
    fab = Fabric(0, 1)
    nslots = max(batches)
    dec = F.FalinexDecoder(cfg, F.random_weights(cfg, dev), fab, max_tokens=8, max_context=prompt + 512, num_slots=nslots, keep_logits=True)
    rows = F.FalinexRows(dec, max_rows=chunk)
    for r in range(nslots):
        dec.state_manager.admit(r, prompt + 512)
    dec.state_manager.flush()
    toks = torch.randint(0, vocab, (prompt,), dtype=torch.int32, device=dev)
    res = {"params_m": round(cfg.param_count() / 1e6), "prefill": {}, "decode": {}, "kernels": []}

    def prefill():
        for p0 in range(0, prompt, chunk):
            rows.forward(toks[p0:p0 + chunk], p0, 0)

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
    # ---- kernel groups, all layers of a kind per graph ----
    st = fab.desc.status
    es = 2
    rec = [L for L in dec.layers if L["m"].recurrent]
    att = [L for L in dec.layers if not L["m"].recurrent]
    HV = heads * hd

    def group(name, Ls, fn, bytes_, flops=0.0):
        ms = t.run(lambda: [fn(L) for L in Ls]) / len(Ls)
        res["kernels"].append(_line(name, ms, bytes_, flops, pk))

    for n in (1, 64):
        B = dec.rows if n <= 8 else rows.B
        pos = torch.full((n,), prompt, dtype=torch.int32, device=dev)
        sl = torch.arange(n, dtype=torch.int32, device=dev)
        state = heads * hd * hd * 4
        group(f"recurrence step, {n} sequences", rec, lambda L: dec._mix(B, L, n, pos, sl, None, norm=False), n * (2 * state + 4 * HV * es))
        keys = min(window, prompt + 1)
        group(f"window attention (norm, rotation, cache write, attention, gate), {n} sequences", att, lambda L: dec._mix(B, L, n, pos, sl, None),
              n * keys * 2 * kv * hd * es + n * (heads + 2 * kv) * hd * es * 2)
        if n == 1:
            x, x2, y = B.x[:1], B.x2[:1], B.y[:1]
            group("input projection with output-norm prologue, 1 row", rec, lambda L: N.gemv_post_norm(y, L["norm1"], 1e-5, x, x2, L["in"], B.proj[:1]),
                  L_bytes(rec[0]["in"]))
            group("output projection with group-norm prologue, 1 row", rec,
                  lambda L: N.gemv_group_norm(B.o[:1, :HV], B.proj[:1, L["gate0"]:], L["gate_act"], 1e-5, L["o"], y, L["groups"], L["gain"]), L_bytes(rec[0]["o"]))
            group("up projection with prologue + GELU, 1 row", rec, lambda L: N.gemv_post_norm(y, L["norm1"], 1e-5, x, x2, L["up"], B.act[ff][:1], "gelu_tanh"),
                  L_bytes(rec[0]["up"]))
            group("down projection, 1 row", rec, lambda L: N.gemv_act(B.act[ff][:1], L["down"], y), L_bytes(rec[0]["down"]))
    m = chunk
    B = rows.B
    pos = torch.arange(prompt - m, prompt, dtype=torch.int32, device=dev)
    sl = torch.zeros(m, dtype=torch.int32, device=dev)
    plan = rows.plan([0] * m, list(range(prompt - m, prompt)))
    dp = plan.bind(plan.control.to(dev), pos)
    C = dec.chunk
    flops = 2.0 * m * heads * (C * hd + 2 * hd * hd + C * hd)
    group(f"recurrence chunks, head norm, gate, {m} rows", rec, lambda L: dec._mix(B, L, m, pos, sl, dp), m * 5 * HV * es, flops)
    pairs = _visible(m, prompt - m, window)
    group(f"window attention, {m} rows", att, lambda L: dec._mix(B, L, m, pos, sl, dp), m * (2 * heads + 2 * kv) * hd * es, 4.0 * pairs * heads * hd)
    group(f"output norm + residual, {m} rows", rec, lambda L: N.post_norm_add(B.y[:m], L["norm1"], 1e-5, B.x[:m], B.xa[:m]), m * width * (4 + 4 + 4 + 2))
    group(f"head norm + gate, {m} rows", rec, lambda L: N.group_norm_gate(B.o[:m, :HV], B.proj[:m, L["gate0"]:L["gate0"] + HV], L["gate_act"], 1e-5, B.mixed[HV][:m],
                                                                      L["groups"], L["gain"]), m * HV * (4 + 2 + 2))
    group(f"input projection, {m} rows", rec, lambda L: N.linear(B.xa[:m], L["in"], B.proj[:m, :L["cols"]], status_ptr=st), L_bytes(rec[0]["in"]),
          2.0 * m * width * rec[0]["in"].shape[0])
    group(f"up projection + GELU, {m} rows", rec, lambda L: N.linear(B.xa[:m], L["up"], B.act[ff][:m, :ff], "gelu_tanh", status_ptr=st), 0, 2.0 * m * width * ff)
    group(f"down projection to f32, {m} rows", rec, lambda L: N.linear(B.act[ff][:m], L["down"], B.y[:m, :width], status_ptr=st), 0, 2.0 * m * width * ff)
    res["fabric_status"] = fab.status()
    dec.state_manager.close()
    fab.close()
    return res


def L_bytes(t: torch.Tensor) -> float:
    return float(t.numel() * t.element_size())


def dense_arm(size, params: int, prompt: int, chunk: int, batches: List[int], t: Timer, pk) -> Dict:
    from ironpangu_b200.models import dense_gqa as G
    from ironpangu_b200.models.dense_prefill import DensePrefill
    from ironpangu_b200.ops import decode as K
    from ironpangu_b200.ops import gemm as GM
    from ironpangu_b200.parallel.fabric import Fabric

    width, layers, heads, kv, hd, _, vocab, window = size
    dev = torch.device("cuda", 0)
    cfg = G.DenseConfig(layers=layers, hidden=width, heads=heads, kv_heads=kv, head_dim=hd, ffn=256, vocab=vocab)
    per = (params - cfg.param_count()) / layers / (3 * width)
    cfg.ffn = max(256, 256 + int(per) // 256 * 256)
    fab = Fabric(0, 1)
    nslots = max(batches)
    w = G.random_rank_weights(cfg, 0, 1, dev)
    dec = G.DenseDecoder(cfg, w, fab, max_tokens=8, max_context=prompt + 512, num_slots=nslots, keep_logits=True)
    pre = DensePrefill(dec, max_rows=chunk)
    toks = torch.randint(0, vocab, (prompt,), dtype=torch.int32, device=dev)
    res = {"params_m": round(cfg.param_count() / 1e6), "ffn": cfg.ffn, "prefill": {}, "decode": {}, "kernels": []}

    def prefill():
        for p0 in range(0, prompt, chunk):
            pre.forward(toks[p0:p0 + chunk], p0, 0)

    ms = t.run(prefill, graph=False, flush=False, reps=5)
    res["prefill"] = {"tokens": prompt, "ms": round(ms, 3), "tokens_s": round(prompt / ms * 1e3)}
    for b in batches:
        pos = torch.full((b,), prompt, dtype=torch.int32, device=dev)
        sl = torch.arange(b, dtype=torch.int32, device=dev)
        tk = toks[:b].contiguous()
        if b <= 2:
            dec.tokens[:b].copy_(tk); dec.positions[:b].copy_(pos); dec.slots[:b].copy_(sl)
            ms = t.run(lambda: dec.forward(b), flush=False)
        else:
            sel = torch.arange(b, device=dev)
            ms = t.run(lambda: pre.forward_rows(tk, pos, sl, sel), graph=False, flush=False)
        res["decode"][b] = {"ms": round(ms, 4), "tokens_s": round(b / ms * 1e3)}
    st = fab.desc.status
    scale = hd ** -0.5
    es = 2

    def group(name, fn, bytes_, flops=0.0):
        ms = t.run(lambda: [fn(l) for l in range(layers)]) / layers
        res["kernels"].append(_line(name, ms, bytes_, flops, pk))

    for n, keys in ((1, prompt + 1), (1, window), (64, prompt + 1), (64, window)):      # also as many keys as the window leaves
        q = torch.zeros(n, (heads + 2 * kv) * hd, dtype=torch.bfloat16, device=dev).normal_()
        pos = torch.full((n,), keys - 1, dtype=torch.int32, device=dev)
        sl = torch.arange(n, dtype=torch.int32, device=dev)
        out = torch.empty(n, heads * hd, dtype=torch.bfloat16, device=dev)
        scr = torch.empty(n * heads * dec.max_splits * (hd + 2), dtype=torch.float32, device=dev)

        def attn(l):
            K.gqa_rope_kv_write(q, pos, sl, dec.page_table, dec.k_cache[l], dec.v_cache[l], heads=heads, kv_heads=kv, head_dim=hd, theta=cfg.theta, status_ptr=st)
            K.gqa_decode_attention(q, dec.k_cache[l], dec.v_cache[l], pos, sl, dec.page_table, heads=heads, kv_heads=kv, head_dim=hd, scale=scale,
                                   keys_per_split=dec.kps, max_splits=dec.max_splits, scratch=scr, out=out, status_ptr=st)

        group(f"attention (rotation, cache write, attention), {n} sequences, {keys} keys", attn, n * keys * 2 * kv * hd * es + n * (heads + 2 * kv) * hd * es * 2)
    p = lambda l, s: w[f"layers.{l}.{s}"]
    group("qkv projection with norm prologue, 1 row", lambda l: K.gemv(dec.x[:1], p(l, "qkv"), norm_w=p(l, "attn_norm"), eps=cfg.eps, out=dec.qkv[:1]),
          L_bytes(p(0, "qkv")))
    group("output projection, 1 row", lambda l: K.gemv_allreduce(dec.attn[:1], p(l, "o_proj"), fab, residual=dec.x[:1], out=dec.x[:1]), L_bytes(p(0, "o_proj")))
    group("gate / up with norm prologue + SwiGLU, 1 row",
          lambda l: K.gemv(dec.x[:1], p(l, "gate_up"), norm_w=p(l, "ffn_norm"), eps=cfg.eps, swiglu=True, out=dec.act[:1]), L_bytes(p(0, "gate_up")))
    group("down projection, 1 row", lambda l: K.gemv_allreduce(dec.act[:1], p(l, "down"), fab, residual=dec.x[:1], out=dec.x[:1]), L_bytes(p(0, "down")))
    m = chunk
    pos = torch.arange(prompt - m, prompt, dtype=torch.int32, device=dev)
    sl = torch.zeros(m, dtype=torch.int32, device=dev)
    pre.qkv[:m].normal_()

    def attn_m(l):
        K.gqa_rope_kv_write(pre.qkv[:m], pos, sl, dec.page_table, dec.k_cache[l], dec.v_cache[l], heads=heads, kv_heads=kv, head_dim=hd, theta=cfg.theta,
                            status_ptr=st)
        pre._contig = (prompt - m, 0)
        pre._attention(l, m, pre.qkv[:m], pos, sl, scale, st)
        pre._contig = None

    pairs = _visible(m, prompt - m, 0)
    group(f"attention, {m} rows", attn_m, m * (2 * heads + 2 * kv) * hd * es, 4.0 * pairs * heads * hd)
    group(f"rms norm, {m} rows", lambda l: K.rmsnorm(pre.x[:m], p(l, "attn_norm"), cfg.eps, out=pre.h[:m]), m * width * 4)
    group(f"qkv projection, {m} rows", lambda l: GM.gemm(pre.h[:m], p(l, "qkv"), out=pre.qkv[:m], status_ptr=st), 0, 2.0 * m * width * (heads + 2 * kv) * hd)
    group(f"gate / up + SwiGLU, {m} rows", lambda l: GM.gemm_swiglu(pre.h[:m], p(l, "gate_up"), out=pre.act[:m], status_ptr=st), 0, 4.0 * m * width * cfg.ffn)
    group(f"down projection + residual, {m} rows", lambda l: GM.gemm(pre.act[:m], p(l, "down"), residual=pre.x[:m], out=pre.x[:m], status_ptr=st), 0,
          2.0 * m * width * cfg.ffn)
    res["fabric_status"] = fab.status()
    fab.close()
    return res


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="small,2b,8b")
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--chunk", type=int, default=2048)
    ap.add_argument("--batches", default="1,8,64")
    args = ap.parse_args(argv)
    torch.cuda.set_device(0)
    pk, t = peaks(), Timer()
    batches = [int(b) for b in args.batches.split(",")]
    for name in args.sizes.split(","):
        s = SIZES[name]
        fal = falinex_arm(s, args.prompt, args.chunk, batches, t, pk)
        torch.cuda.empty_cache()
        den = dense_arm(s, int(fal["params_m"] * 1e6), args.prompt, args.chunk, batches, t, pk)
        torch.cuda.empty_cache()
        print(json.dumps({"bench": "falinex", "size": name, "config": dict(zip(("width", "layers", "heads", "kv_heads", "head_dim", "ff", "vocab", "window"), s)),
                          "prompt": args.prompt, "chunk": args.chunk, "dtype": "bf16", "data": "synthetic, random weights", "peaks": pk, "falinex": fal, "dense": den}))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
