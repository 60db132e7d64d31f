"""Prefill and decode throughput of the Ponenex design beside the closest existing model (the MLA + MoE decoder) at the same layer sizes,
window and parameter count, and the time of every kernel group of both against its roofline.

    python bench.py --design ponenex                # through the benchmark's command line
    python -m ironpangu_b200.utils.bench_ponenex --sizes small,text

Random weights, synthetic tokens. Model steps are CUDA graphs where the engine replays graphs, device events around them; kernel groups
are timed over all layers in one graph (distinct weights and pages per layer) with the L2 flushed before every run."""
from __future__ import annotations

import argparse
import json
from typing import Dict, List

import torch

from .bench_falinex import Timer, _line, _visible, peaks

BF16, F32 = torch.bfloat16, torch.float32
SIZES = {          # layers, width, heads, query rank, experts, top, expert ff, vocabulary, window (heads 128 + 64 / 128, latent 512, one shared expert)
    "small": (8, 1024, 8, 384, 16, 4, 512, 32000, 512),
    "text": (16, 2048, 16, 768, 64, 8, 768, 128000, 1024),
    "wide": (5, 4096, 32, 1536, 96, 8, 1536, 153600, 2048),
}
DIM, ROT, VDIM, LATENT = 128, 64, 128, 512


class Costs:
    """Bytes and FLOPs a kernel group cannot do without, the same for both arms."""

    def __init__(self, size):
        self.layers, self.width, self.heads, self.q_rank, self.experts, self.top, self.ff, self.vocab, self.window = size
        H, W = self.heads, self.width
        self.w_in = 2.0 * W * (self.q_rank + LATENT + ROT)
        self.w_attn = 2.0 * (H * (DIM + ROT) * self.q_rank + H * (DIM + VDIM) * LATENT)
        self.w_o = 2.0 * W * H * VDIM
        self.unit = 2.0 * 3 * W * self.ff

    def attention(self, rows: int, keys: int) -> tuple:
        """rows of as many sequences, each over ``keys`` keys: weights once, every sequence's latent rows, queries and results."""
        H = self.heads
        return (self.w_attn + rows * (keys * (LATENT + ROT) * 2 + 2 * (self.q_rank + LATENT + ROT + H * VDIM)),
                2.0 * rows * H * ((DIM + ROT) * self.q_rank + (DIM + VDIM) * LATENT + keys * (2 * LATENT + ROT)))

    def prompt_attention(self, m: int, p0: int) -> tuple:
        H, pairs = self.heads, _visible(m, p0, self.window)
        return (self.w_attn + 2.0 * m * (self.q_rank + LATENT + ROT + H * VDIM),
                2.0 * m * H * ((DIM + ROT) * self.q_rank + (DIM + VDIM) * LATENT) + 2.0 * pairs * H * (DIM + ROT + VDIM))

    def expert_block(self, rows: int) -> tuple:
        routes = rows * self.top
        hit = self.experts * (1.0 - (1.0 - self.top / self.experts) ** rows)            # experts that random routes reach
        return hit * self.unit + self.unit + 2.0 * self.experts * self.width, rows * (self.top + 1) * self.unit


def _result(params) -> Dict:
    return {"params_m": round(params / 1e6), "prefill": {}, "decode": {}, "kernels": []}


def _spread_routes(w_router: torch.Tensor, seed: int) -> None:
    """Routers whose choices spread over the experts whatever the random hidden rows look like."""
    g = torch.Generator(device=w_router.device).manual_seed(seed)
    w_router.normal_(0.0, 1.0, generator=g)


def ponenex_arm(size, prompt: int, chunk: int, batches: List[int], t: Timer, pk) -> Dict:
    from ironpangu_b200.models import ponenex as P
    from ironpangu_b200.ops import stream_norm as N
    from ironpangu_b200.parallel.fabric import Fabric

    C = Costs(size)
    dev = torch.device("cuda", 0)
    cfg = P.PonenexConfig.text(layers=C.layers, width=C.width, heads=C.heads, dim=DIM, rot_dim=ROT, vdim=VDIM, kv_rank=LATENT, q_rank=C.q_rank, experts=C.experts,
                               top=C.top, ff=C.ff, shared_ff=C.ff, vocab=C.vocab, window=C.window)
    fab = Fabric(0, 1)
    nslots, ctx = max(batches), prompt + 512
    w = P.random_weights(cfg, dev)
    dec = P.PonenexDecoder(cfg, w, fab, max_tokens=8, max_context=ctx, num_slots=nslots, keep_logits=True)
    del w
    torch.cuda.empty_cache()
    for i, L in enumerate(dec.layers):
        _spread_routes(L["ff"].w_router, i)
    rows = P.PonenexRows(dec, max_rows=chunk)
    for r in range(nslots):
        dec.state_manager.admit(r, ctx)
    dec.state_manager.flush()
    toks = torch.randint(0, C.vocab, (prompt,), dtype=torch.int32, device=dev)
    res = _result(cfg.param_count())

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
    st, eps, table = fab.desc.status, cfg.eps, dec.page_table
    Ls = dec.layers
    s = Ls[0]["mix"].shape
    HV = s.heads * s.vdim

    def group(name, fn, bytes_, flops=0.0):
        ms = t.run(lambda: [fn(L) for L in Ls]) / len(Ls)
        res["kernels"].append(_line(name, ms, bytes_, flops, pk))

    def setup(B, n, pos):
        B.rotary.fill(pos)
        B.latent.proj[:n].normal_()
        B.xa[:n].normal_()
        B.x[:n].normal_()
        B.y[:n].normal_()
        B.experts.start(n)
        return B.rotary.get(s.rot_dims, s.rot_base)

    keys = min(C.window, prompt + 1)
    B = dec.rows
    pos, sl = torch.full((1,), prompt, dtype=torch.int32, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    rope = setup(B, 1, pos)
    x, x2, y, xa = B.x[:1], B.x2[:1], B.y[:1], B.xa[:1]
    group("input projection, 1 row", lambda L: N.gemv_post_norm(y, L["norm2b"], eps, x, x2, L["mix"].w_in, B.latent.proj[:1, :s.in_cols], next_norm=L["norm1"]), C.w_in)
    group("latent attention, 1 row", lambda L: L["mix"].decode(B.latent, 1, rope, pos, sl, table, eps, st), *C.attention(1, keys))
    group("output projection, 1 row", lambda L: N.gemv_act(B.latent.mixed[HV][:1], L["mix"].w_o, y), C.w_o)
    group("router and experts, 1 row", lambda L: L["ff"].decode(B.experts, 1, y, L["norm1b"], L["norm2"], eps, x, x2, xa, fab.ticket_ptr), *C.expert_block(1))
    B = rows.B
    n = nslots
    pos, sl = torch.full((n,), prompt, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int32, device=dev)
    rope = setup(B, n, pos)
    group(f"latent attention, {n} sequences", lambda L: L["mix"].mix(B.latent, n, rope, pos, sl, None, table, eps, st), *C.attention(n, keys))
    group(f"router and experts, {n} rows", lambda L: L["ff"].rows(B.experts, n, B.xa[:n], L["norm2b"], L["norm1"], eps, B.x[:n], st), *C.expert_block(n))
    m = chunk
    pos, sl = torch.arange(prompt - m, prompt, dtype=torch.int32, device=dev), torch.zeros(m, dtype=torch.int32, device=dev)
    rope = setup(B, m, pos)
    plan = rows.plan([0] * m, list(range(prompt - m, prompt)))
    dp = plan.bind(plan.control.to(dev), pos)
    group(f"input projection, {m} rows", lambda L: N.linear(B.xa[:m], L["mix"].w_in, B.latent.proj[:m, :s.in_cols], status_ptr=st), C.w_in, m * C.w_in)
    group(f"latent attention, {m} rows", lambda L: L["mix"].mix(B.latent, m, rope, pos, sl, dp, table, eps, st), *C.prompt_attention(m, prompt - m))
    group(f"output projection, {m} rows", lambda L: N.linear(B.latent.mixed[HV][:m], L["mix"].w_o, B.y[:m, :C.width], status_ptr=st), C.w_o, m * C.w_o)
    group(f"output norm, residual and next norm, {m} rows", lambda L: N.post_norm_add(B.y[:m], L["norm1b"], eps, B.x[:m], B.xa[:m], L["norm2"]), m * C.width * 14.0)
    group(f"router and experts, {m} rows", lambda L: L["ff"].rows(B.experts, m, B.xa[:m], L["norm2b"], L["norm1"], eps, B.x[:m], st), *C.expert_block(m))
    res["fabric_status"] = fab.status()
    dec.state_manager.close()
    fab.close()
    return res


def mla_arm(size, prompt: int, chunk: int, batches: List[int], t: Timer, pk) -> Dict:
    from ironpangu_b200.models import mla_moe as M
    from ironpangu_b200.models.mla_moe_prefill import MlaMoePrefill
    from ironpangu_b200.ops import decode as K
    from ironpangu_b200.ops import gemm as G
    from ironpangu_b200.parallel.fabric import Fabric

    C = Costs(size)
    dev = torch.device("cuda", 0)
    cfg = M.MlaMoeConfig(layers=C.layers, hidden=C.width, vocab=C.vocab, heads=C.heads, q_lora=C.q_rank, kv_lora=LATENT, nope=DIM, rope=ROT, vdim=VDIM,
                         experts=C.experts, expert_ffn=C.ff, topk=C.top, shared_ffn=C.ff, window=C.window)
    fab = Fabric(0, 1)
    nslots, ctx = max(batches), prompt + 512
    w = M.random_rank_weights(cfg, 0, 1, dev)
    for l in range(C.layers):
        _spread_routes(w[f"layers.{l}.router"], l)
    dec = M.MlaMoeDecoder(cfg, w, fab, max_tokens=8, max_context=ctx, num_slots=nslots, keep_logits=True)
    pre = MlaMoePrefill(dec, max_rows=chunk)
    pre.use_graphs = False                          # chunks of the timed prompt are launched like the other arm's
    toks = torch.randint(0, C.vocab, (prompt,), dtype=torch.int32, device=dev)
    res = _result(cfg.param_count())

    def prefill():
        for p0 in range(0, prompt, chunk):
            pre.forward(toks[p0:p0 + chunk], p0, 0)

    ms = t.run(prefill, graph=False, flush=False, reps=5)
    res["prefill"] = {"tokens": prompt, "ms": round(ms, 3), "tokens_s": round(prompt / ms * 1e3)}
    pre.use_graphs = True
    for b in batches:
        pos = torch.full((b,), prompt, dtype=torch.int32, device=dev)
        sl = torch.arange(b, dtype=torch.int32, device=dev)
        tk = toks[:b].contiguous()
        if b <= 8:
            dec.tokens[:b].copy_(tk); dec.positions[:b].copy_(pos); dec.slots[:b].copy_(sl)
            ms = t.run(lambda: dec.forward(b), flush=False)
        else:
            sel = torch.arange(b, device=dev)
            ms = t.run(lambda: pre.forward_rows(tk, pos, sl, sel), graph=False, flush=False)
        res["decode"][b] = {"ms": round(ms, 4), "tokens_s": round(b / ms * 1e3)}
    st = fab.desc.status
    p = lambda l, n: w[f"layers.{l}.{n}"]

    def group(name, fn, bytes_, flops=0.0):
        ms = t.run(lambda: [fn(l) for l in range(C.layers)]) / C.layers
        res["kernels"].append(_line(name, ms, bytes_, flops, pk))

    keys = min(C.window, prompt + 1)
    c = cfg

    def attend(l, n, pos, sl, qkv):
        if n <= 2 and dec.fused_head:
            K.mla_head_decode(qkv, p(l, "q_a_norm"), p(l, "kv_a_norm"), p(l, "q_b"), p(l, "kv_b"), dec.caches[l], pos, sl, dec.page_table, q_lora=c.q_lora, nope=c.nope,
                              scale=c.scale, eps=c.eps, theta=c.theta, window=c.window, out=dec.attn[:n], status_ptr=st)
            return
        K.mla_kv_write(qkv[:, c.q_lora:], p(l, "kv_a_norm"), pos, sl, dec.page_table, dec.caches[l], latent=c.kv_lora, rope=c.rope, eps=c.eps, theta=c.theta, status_ptr=st)
        q = K.gemv(qkv[:, :c.q_lora], p(l, "q_b"), norm_w=p(l, "q_a_norm"), eps=c.eps, out=dec.q[:n])
        ql = K.mla_q_absorb(q, p(l, "kv_b"), pos, nope=c.nope, rope=c.rope, theta=c.theta, out=dec.q_lat[:n])
        K.mla_decode_attention(ql, dec.caches[l], pos, sl, dec.page_table, p(l, "kv_b"), nope=c.nope, scale=c.scale, window=c.window, keys_per_split=dec.kps,
                               max_splits=dec.max_splits, scratch=dec.scratch, out=dec.attn[:n], status_ptr=st)

    pos, sl = torch.full((1,), prompt, dtype=torch.int32, device=dev), torch.zeros(1, dtype=torch.int32, device=dev)
    dec.x[:1].normal_(); dec.qkv[:1].normal_(); dec.attn[:1].normal_()
    x = dec.x[:1]
    group("input projection, 1 row", lambda l: K.gemv(x, p(l, "qkv_a"), norm_w=p(l, "attn_norm"), eps=c.eps, out=dec.qkv[:1]), C.w_in)
    group("latent attention, 1 row", lambda l: attend(l, 1, pos, sl, dec.qkv[:1]), *C.attention(1, keys))
    group("output projection, 1 row", lambda l: K.gemv_allreduce(dec.attn[:1], p(l, "o_proj"), fab, residual=x, out=x), C.w_o)

    def experts_1(l):
        K.router_topk(x, p(l, "router"), c.topk, norm_w=p(l, "ffn_norm"), eps=c.eps, scoring=c.scoring, scale=c.route_scale, ticket_ptr=fab.ticket_ptr,
                      logits=dec.logits_r[:1], ids=dec.route_ids[:1], wts=dec.route_w[:1], xn=dec.xn[:1])
        K.moe_gate_up(dec.xn[:1], dec.route_ids[:1], p(l, "gate_up"), 0, w_shared_gu=p(l, "shared_gate_up"), act=dec.act[:1])
        K.moe_down_allreduce(dec.act[:1], dec.route_ids[:1], dec.route_w[:1], p(l, "down"), 0, fab, w_shared_down=p(l, "shared_down"), residual=x, out=x)

    group("router and experts, 1 row", experts_1, *C.expert_block(1))
    from ironpangu_b200.ops import prefill as P

    def attention_rows(l, n, contig):
        pos, sl, qkv = pre.positions[:n], pre.slots[:n], pre.qkv[:n]
        K.mla_kv_write(qkv[:, c.q_lora:], p(l, "kv_a_norm"), pos, sl, dec.page_table, dec.caches[l], latent=c.kv_lora, rope=c.rope, eps=c.eps, theta=c.theta, status_ptr=st)
        K.rmsnorm(qkv[:, :c.q_lora], p(l, "q_a_norm"), c.eps, out=pre.qn[:n])
        q = G.gemm(pre.qn[:n], p(l, "q_b"), out=pre.q[:n], status_ptr=st)
        if not contig:
            pre._latent_attention(l, n, q, pre.q_lat[:n], pre.o_lat[:n], pre.attn[:n])
            return
        rows = (prompt + 63) // 64 * 64
        kvb = p(l, "kv_b").view(-1, c.kv_lora)
        P.mla_ctx_gather(dec.caches[l], dec.page_table, 0, prompt, pre.ctx_lat[:rows], pre.ctx_pe[:rows], status_ptr=st)
        G.gemm(pre.ctx_lat[:rows], kvb, out=pre.kv_up[:rows], status_ptr=st)
        G.gemm(kvb, pre.ctx_lat[:rows], out=pre.kvt[:, :rows], status_ptr=st)
        P.mla_q_rope_inplace(q, pos, heads=c.heads, nope=c.nope, rope=c.rope, theta=c.theta)
        P.fa_prefill(q, pre.kv_up, pre.kvt, pre.attn[:n], heads=c.heads, q_head_stride=c.qk_dim, k_head_stride=c.nope + c.vdim, vt_head_stride=c.nope + c.vdim,
                     vt_row0=c.nope, d1=c.nope, d2=c.rope, k2=pre.ctx_pe, ctx=prompt, pos0=prompt - n, scale=c.scale, window=c.window, status_ptr=st)

    def experts_rows(l, n):
        x, h = pre.x[:n], pre.h[:n]
        P.router_block(x, p(l, "router"), c.topk, pre.ids[:n], pre.wts[:n], norm_w=p(l, "ffn_norm"), eps=c.eps, scoring=c.scoring, scale=c.route_scale, xn=h)
        P.moe_dispatch(pre.ids[:n], 0, c.experts, pre.route)
        P.moe_gather(h, pre.route, pre.xp)
        P.grouped_gemm(pre.xp, p(l, "gate_up"), pre.route.tiles, pre.route.num_tiles, pre.act, swiglu=True, status_ptr=st)
        P.grouped_gemm(pre.act, p(l, "down"), pre.route.tiles, pre.route.num_tiles, pre.y, status_ptr=st)
        sgu, sdn = p(l, "shared_gate_up"), p(l, "shared_down")
        if n >= 256 and (sgu.shape[0] // 2) % 32 == 0:
            G.gemm_swiglu(h, sgu, out=pre.sact[:n], status_ptr=st)
        else:
            P.grouped_gemm(h, sgu.unsqueeze(0), pre.shared_tiles, pre.shared_ntiles, pre.sact[:n], swiglu=True, status_ptr=st)
        G.gemm(pre.sact[:n], sdn, out=pre.sd[:n], status_ptr=st)
        P.moe_combine(pre.y, pre.route, pre.wts[:n], shared=pre.sd[:n], residual=x, out=x)

    def setup(n, pos, sl):
        pre.positions[:n].copy_(pos); pre.slots[:n].copy_(sl)
        pre.qkv[:n].normal_(); pre.x[:n].normal_(); pre.h[:n].normal_()
        pre.shared_ntiles.fill_((n + 127) // 128)

    n = nslots
    setup(n, torch.full((n,), prompt, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int32, device=dev))
    group(f"latent attention, {n} sequences", lambda l: attention_rows(l, n, False), *C.attention(n, keys))
    group(f"router and experts, {n} rows", lambda l: experts_rows(l, n), *C.expert_block(n))
    m = chunk
    setup(m, torch.arange(prompt - m, prompt, dtype=torch.int32, device=dev), torch.zeros(m, dtype=torch.int32, device=dev))
    group(f"input projection, {m} rows", lambda l: G.gemm(pre.h[:m], p(l, "qkv_a"), out=pre.qkv[:m], status_ptr=st), C.w_in, m * C.w_in)
    setup(m, pre.positions[:m].clone(), pre.slots[:m].clone())
    group(f"latent attention, {m} rows", lambda l: attention_rows(l, m, True), *C.prompt_attention(m, prompt - m))
    group(f"output projection, {m} rows", lambda l: G.gemm(pre.attn[:m], p(l, "o_proj"), residual=pre.x[:m], out=pre.x[:m], status_ptr=st), C.w_o, m * C.w_o)
    group(f"rms norm, {m} rows", lambda l: K.rmsnorm(pre.x[:m], p(l, "attn_norm"), c.eps, out=pre.h[:m]), m * C.width * 4.0)
    setup(m, pre.positions[:m].clone(), pre.slots[:m].clone())
    group(f"router and experts, {m} rows", lambda l: experts_rows(l, m), *C.expert_block(m))
    res["fabric_status"] = fab.status()
    fab.close()
    return res


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", default="small,text,wide")
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--chunk", type=int, default=2048)
    ap.add_argument("--batches", default="1,8,64")
    args = ap.parse_args(argv)
    torch.cuda.set_device(0)
    pk, t = peaks(), Timer()
    batches = [int(b) for b in args.batches.split(",")]
    names = ("layers", "width", "heads", "q_rank", "experts", "top", "ff", "vocab", "window")
    for name in args.sizes.split(","):
        s = SIZES[name]
        pon = ponenex_arm(s, args.prompt, args.chunk, batches, t, pk)
        torch.cuda.empty_cache()
        mla = mla_arm(s, args.prompt, args.chunk, batches, t, pk)
        torch.cuda.empty_cache()
        print(json.dumps({"bench": "ponenex", "size": name, "config": dict(zip(names, s)), "prompt": args.prompt, "chunk": args.chunk, "dtype": "bf16",
                          "data": "synthetic, random weights", "peaks": pk, "ponenex": pon, "mla_moe": mla}), flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
