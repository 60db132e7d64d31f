"""The Ponenex decoder as a model of the framework: configuration and registry (CPU); whole prompts, portions, token-by-token decoding,
mixed batches, reused pages and slots, long decoding and generation through the engine and the server against the plain restatement
(GPU)."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import ponenex_oracle as O
from ponenex_cases import CASES, config, layer, tokens, weights
from stream_rig import Rig, cut, logit_error, random_batches

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32
# largest allowed error of a row of logits relative to their spread
LIMIT = {F32: 4e-5, BF16: 6e-2}
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def rig(cfg, dtype, seed=0, **kw):
    """In 16 bits the routers have no close calls (a rounding that turns a choice is not a fault)."""
    return Rig(cfg, weights(cfg, seed, separated=dtype == BF16), dtype, **kw)


# ---------------------------------------------------------------------------------------------------------------------------
# CPU
# ---------------------------------------------------------------------------------------------------------------------------
def test_configuration_round_trip_and_checks():
    from ironpangu_b200.models.ponenex import PonenexConfig, weight_shapes

    for c in CASES.values():
        f = PonenexConfig.from_dict(json.loads(json.dumps(c)))
        assert f.to_dict() == c and PonenexConfig.from_dict(f.to_dict()) == f
    assert PonenexConfig.from_dict(CASES["mixed"]).window == 50 and PonenexConfig.from_dict(CASES["tiles"]).window == 0
    for c in (PonenexConfig.tiny(), PonenexConfig.text(layers=2)):
        assert PonenexConfig.from_dict(c.to_dict()) == c
    m = layer()["mixer"]
    bad = [dict(CASES["odd"], architecture="Other"), config([]), config([dict(layer(), type="retention")]), config([layer(rot=3)]), config([layer(rot=18)]),
           config([layer(experts=3, top=4)]), config([layer(kv_rank=2000)]), config([layer(rot_dim=300)]), config([layer(window=-1)]),
           config([dict(layer(), mlp={"kind": "dense", "ff": 3})]), config([dict(layer(), mixer={k: v for k, v in m.items() if k != "scale"})])]
    for c in bad:
        with pytest.raises((ValueError, KeyError)):
            PonenexConfig.from_dict(c)
    s = weight_shapes(PonenexConfig.from_dict(CASES["mixed"]))
    assert s["l0.mlp.e5.down"] == (72, 40) and s["l0.mlp.shared.sg"] == (1, 72) and "l1.norm2" not in s and "l2.mlp.shared.sg" not in s
    assert s["l0.mix.dkv"] == (72 + 24, 72) and s["l0.mix.uq"] == (6 * 64, 48) and s["l1.mix.o"] == (72, 3 * 24)
    c = PonenexConfig.from_dict(CASES["odd"])
    assert c.param_count() == sum(int(np.prod(v)) for v in weight_shapes(c).values())
    assert c.param_count() - c.active_params() == (1 * 3 * 19 + 3 * 3 * 51) * 52 + 130 * 52


def test_checkpoint_and_registry(tmp_path):
    from ironpangu_b200.models import ponenex as P
    from ironpangu_b200.models import registry

    cfg = CASES["mixed"]
    w = weights(cfg)
    P.save_checkpoint(tmp_path, P.PonenexConfig.from_dict(cfg), w)
    assert registry.family_of(tmp_path).decoder == "PonenexDecoder" and {"ponenex-tiny", "falinex-tiny"} <= set(registry.preset_names())
    c, got = P.load_checkpoint(tmp_path)
    assert c == P.PonenexConfig.from_dict(cfg) and set(got) == set(w) and all(torch.equal(got[n], w[n]) for n in w)
    w["l0.mlp.router.b"] = w["l0.mlp.router.b"][:-1]
    P.save_checkpoint(tmp_path, c, w)
    with pytest.raises(ValueError, match="l0.mlp.router.b"):
        P.load_checkpoint(tmp_path)
    del w["l0.mlp.router.b"]
    P.save_checkpoint(tmp_path, c, w)
    with pytest.raises(ValueError, match="l0.mlp.router.b"):
        P.load_checkpoint(tmp_path)


FAULTS = ("window_plus_one", "window_minus_one", "no_gate", "no_rotation", "latent_not_normed", "no_bias", "no_shared", "shared_not_gated")


def test_restatement_notices_planted_faults():
    """The comparison the GPU tests make would fail by a wide margin for every one of these mistakes."""
    for name in ("mixed", "odd", "wide"):
        cfg = CASES[name]
        w, toks = weights(cfg, separated=True), tokens(cfg, 60)
        good = O.forward(cfg, w, toks)
        for fault in FAULTS:
            assert logit_error(O.forward(cfg, w, toks, faults=(fault,)), good) > 2 * LIMIT[BF16], (name, fault)


def test_separated_routers_have_no_close_calls(monkeypatch):
    gaps, route = [], O.route

    def watch(h, r, b, top):
        z = (h @ r.T + b).sort(dim=-1, descending=True).values
        if top < z.shape[1]:
            gaps.append(float((z[:, top - 1] - z[:, top]).min()))
        return route(h, r, b, top)

    monkeypatch.setattr(O, "route", watch)
    for cfg in CASES.values():
        for seed in (0, 1):
            O.forward(cfg, weights(cfg, seed, separated=True), tokens(cfg, 100, seed))
    assert min(gaps) > 0.05


# ---------------------------------------------------------------------------------------------------------------------------
# GPU: the model through the engine
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", list(CASES))
def test_whole_prompts_portions_and_decoding(name, dtype):
    cfg = CASES[name]
    r = rig(cfg, dtype)
    n = 210
    toks = tokens(cfg, n)
    want = O.forward(cfg, r.w, toks)
    rnd = random.Random(name)
    schedules = {"whole": [n], "token by token": [1] * 60, "prompt, then decoding": [n - 70] + [1] * 70, "portions": cut(rnd, n, [2, 3, 5, 9, 17, 33, 64, 65]),
                 "pairs": [2] * 30, "first tokens": [1, 2, 3, 1, 5, 16, 15, 2]}
    for what, cuts in schedules.items():
        got = r.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
        e = logit_error(got, want[:len(got)])
        assert e < LIMIT[dtype], (what, e)
    r.close()


@pytest.mark.gpu
@DTYPES
def test_residual_stream_after_every_layer(dtype):
    cfg = CASES["mixed"]
    r = rig(cfg, dtype)
    toks = tokens(cfg, 80)
    residuals, probe = [], []
    O.forward(cfg, r.w, toks, residuals)
    r.dec.state_manager.admit(0, 80)
    r.dec.state_manager.flush()
    pos = torch.arange(80, dtype=torch.int32, device="cuda")
    plan = r.eng.prefill.plan([0] * 80, list(range(80)))
    r.eng.prefill.forward_rows(torch.tensor(toks, dtype=torch.int32, device="cuda"), pos, torch.zeros_like(pos), torch.tensor([79], device="cuda"), plan,
                               plan.control.cuda(), probe)
    assert len(probe) == len(residuals) == 4
    for got, want in zip(probe, residuals):
        assert float((got.cpu().double() - want).abs().max() / want.abs().max()) < (1e-5 if dtype == F32 else 4e-2)
    r.close()


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", ["mixed", "odd", "tiles"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(name, dtype):
    """More requests than slots over a pool that cannot hold them all at once; portions beside decoded tokens; a request left out of some
    steps; every request equals the restatement (computed alone)."""
    cfg = CASES[name]
    r = rig(cfg, dtype, context=320, pool=448, rows=128)             # rows: wide steps take several passes
    lens = {"a": 150, "b": 23, "c": 97, "d": 5, "e": 64, "f": 33, "g": 121}
    reqs = {k: tokens(cfg, n, i) for i, (k, n) in enumerate(lens.items())}
    want = {k: O.forward(cfg, r.w, t) for k, t in reqs.items()}
    got = r.run(reqs, random_batches(random.Random(7), lens, list(reqs) + ["a#2", "d#2"], 4, 448, [1, 1, 1, 2, 3, 16, 29, 64]))
    for k, g in got.items():
        e = logit_error(g, want[k.split("#")[0]])
        assert e < LIMIT[dtype], (k, e)
    u = r.dec.state_manager.usage()
    assert all(c["occupied_units"] == 0 for c in u["components"].values()) and u["pages_taken"] > u["components"]["kv"]["capacity_units"]
    r.close()


@pytest.mark.gpu
def test_many_sequences_decode_together():
    """Steps of twenty rows replay the packed executor's graphs, of five and eight the launch group's."""
    cfg = CASES["mixed"]
    r = rig(cfg, BF16, residents=20, context=128)
    reqs = {f"r{i}": tokens(cfg, 12 + 2 * i, i) for i in range(20)}
    want = {k: O.forward(cfg, r.w, t) for k, t in reqs.items()}
    steps = [[(k, 4)] for k in reqs]
    for i in range(46):
        steps.append([(k, 1) for k, t in reqs.items() if len(t) - 4 > i])
    got = r.run(reqs, [s for s in steps if s])
    for k, g in got.items():
        rows = [logit_error(g[i:i + 1], want[k][i:i + 1]) for i in range(len(g))]
        assert sorted(rows)[len(rows) * 9 // 10] < LIMIT[BF16] and max(rows) < 2.5 * LIMIT[BF16], k      # a few rows of so many are ill-conditioned
    r.close()


@pytest.mark.gpu
@DTYPES
def test_a_batch_changes_nothing(dtype):
    """Logits of a request alone and beside others, and on other pages and slots, agree far below the model's own rounding."""
    cfg = CASES["tiles"]
    r = rig(cfg, dtype)
    reqs = {k: tokens(cfg, n, i) for i, (k, n) in enumerate({"a": 90, "b": 40, "c": 61}.items())}
    cuts = [[("b", 20), ("a", 50)], [("a", 1), ("b", 1)], [("c", 61), ("a", 1), ("b", 9)]] + [[("a", 1), ("b", 1)]] * 10 + [[("a", 28)]]
    mixed = r.run(reqs, cuts)
    alone = r.run(reqs, [[("a", 50)], [("a", 1)], [("a", 1)]] + [[("a", 1)]] * 10 + [[("a", 28)]])
    assert logit_error(mixed["a"], alone["a"].double()) < (2e-5 if dtype == F32 else 3e-2)
    r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 31, 64])
def test_window_edges_in_prompts_and_decoding(window):
    """Every window against page borders (16) and portion borders; the restatement with the window one token off is far away."""
    cfg = config([layer(4, 64, 32, 64, 128, 64, window=window), layer(3, 20, 8, 24, 40, 16, window=window)], width=64)
    toks = tokens(cfg, 100)
    for dtype in (F32, BF16):
        r = rig(cfg, dtype, rows=128)
        want = O.forward(cfg, r.w, toks)
        off = logit_error(O.forward(cfg, r.w, toks, faults=("window_plus_one",)), want)
        assert off > 3 * LIMIT[dtype]
        for cuts in ([100], [1] * 100, [16] * 6 + [4], [window] * (100 // window) if window > 1 else [3] * 33, [window + 1] * (100 // (window + 1)), [50] + [1] * 50):
            got = r.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
            assert logit_error(got, want[:len(got)]) < min(LIMIT[dtype], off / 3), cuts
        r.close()


@pytest.mark.gpu
@DTYPES
def test_long_decoding_in_a_pool_of_one_window(dtype):
    """Hundreds of decoded tokens while the pages of the window come and go."""
    cfg = config([layer(4, 32, 16, 32, 64, 32, window=40), layer(2, 16, 16, 16, 32, 16, window=23)], width=64)
    r = rig(cfg, dtype, context=700, pool=96, rows=64)
    toks = tokens(cfg, 620)
    want = O.forward(cfg, r.w, toks)
    got = r.run({"a": toks}, [[("a", 40)]] + [[("a", 1)]] * 580)["a"]
    assert logit_error(got, want) < LIMIT[dtype]
    assert r.dec.state_manager.pages_trimmed > 30
    r.close()


@pytest.mark.gpu
@DTYPES
def test_the_first_token_is_seen_by_the_last(dtype):
    """Without a window a far key counts: another first token, other logits at the end, in a prompt and in decoding."""
    cfg = config([layer(2, 64, 64, 64, 256, 64, window=0), layer(4, 24, 8, 16, 40, 24, window=0)], width=64)
    r = rig(cfg, dtype, context=600)
    toks = tokens(cfg, 500)
    for first in (toks[0], (toks[0] + 32) % cfg["vocab"]):
        seq = [first] * 3 + toks[3:]
        want = O.forward(cfg, r.w, seq)
        for cuts in ([500], [440] + [1] * 60, [100, 130, 270]):
            got = r.run({"a": seq}, [[("a", c)] for c in cuts])["a"]
            assert logit_error(got, want) < LIMIT[dtype]
    r.close()


def _greedy(cfg, w, prompt, n):
    toks, margins = list(prompt), []
    for _ in range(n):
        l = O.forward(cfg, w, toks)[-1]
        top = l.topk(2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(l.argmax()))
    return toks[len(prompt):], margins


@pytest.mark.gpu
@DTYPES
def test_greedy_generation_through_the_engine(dtype):
    """Prefill and decode steps of the engine and of the single-sequence engine give the restatement's greedy continuation."""
    from ironpangu_b200.runtime.engine import DecodeEngine

    cfg = CASES["mixed"]
    r = rig(cfg, dtype, residents=2)
    for seed in range(20):                             # a prompt whose continuation has no near tie for some tokens
        prompt = tokens(cfg, 30, seed)
        want, margins = _greedy(cfg, r.w, prompt, 12)
        clear = next((i for i, m in enumerate(margins) if m < (1e-3 if dtype == F32 else 0.15)), 12)
        if clear >= 5:
            break
    r.eng.admit(0, {}, 42)
    r.eng.admit(1, {}, 42)
    got = [r.eng.step([[0, 0, 30, True]], prompt)[0]]
    r.eng.step([[1, 0, 7, True]], prompt[:7])
    for i in range(11):
        got.append(r.eng.step([[0, 30 + i, 1, True], [1, 7 + i, 1, True]], [got[-1], 3])[0])
    assert clear >= 5 and got[:clear] == want[:clear]
    r.eng.release(0)
    r.eng.release(1)
    single = DecodeEngine(r.dec, prefill=r.eng.prefill)
    assert single.generate(prompt, 12)[:clear] == want[:clear]
    single.reset()                                     # the same on the device alone: every sampled token fed back without the host
    first = single.prefill(prompt)
    single.run_device_loop(first, clear - 1)
    assert int(r.dec.next_ids[0]) == want[clear - 1] and single.pos == 30 + clear - 1
    r.close()


@pytest.mark.gpu
def test_generation_through_the_server(tmp_path):
    """A checkpoint directory behind ifab-server: the worker picks the family by config.json; greedy tokens of concurrent requests equal
    the restatement's; seeded sampling repeats."""
    import threading

    from ironpangu_b200.models import ponenex as P
    from test_server import Server

    cfg = dict(CASES["mixed"], vocab=300)
    w = weights(cfg)
    P.save_checkpoint(tmp_path / "ck", P.PonenexConfig.from_dict(cfg), w)
    s = Server("--spawn", f"{sys.executable} -m ironpangu_b200.runtime.engine_worker --model checkpoint --checkpoint {tmp_path / 'ck'} --dtype float32 "
               "--max-num-seqs 2 --max-model-len 128 --kv-pool-tokens 192 --max-num-batched-tokens 48", "--accept-seconds", "300", timeout=400)
    try:
        prompts = [tokens(cfg, n, n) for n in (40, 11, 25)]
        outs = [None] * 3

        def go(i):
            outs[i] = s.post("/inference/v1/generate", {"token_ids": prompts[i], "sampling_params": {"max_tokens": 8}}, timeout=120)

        th = [threading.Thread(target=go, args=(i,)) for i in range(3)]
        [t.start() for t in th]
        [t.join() for t in th]
        for p, (st, o) in zip(prompts, outs):
            want, margins = _greedy(cfg, w, p, 8)
            clear = next((i for i, m in enumerate(margins) if m < 1e-3), 8)
            assert st == 200 and o["token_ids"][:clear] == want[:clear]
        body = {"token_ids": prompts[1], "sampling_params": {"max_tokens": 8, "temperature": 1.2, "top_k": 30, "seed": 5}}
        assert s.post("/inference/v1/generate", body, timeout=120)[1]["token_ids"] == s.post("/inference/v1/generate", body, timeout=120)[1]["token_ids"]
        st, audit = s.request("GET", "/audit")
        eng = json.loads(audit)["engine"]
        assert eng["paged_state"]["components"]["kv"]["occupied_units"] == 0 and eng["fabric_status"] == 0
    finally:
        s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(tmp_path, dtype):
    from ironpangu_b200.models import ponenex as P

    cfg = CASES["odd"]
    w = weights(cfg, separated=True)
    P.save_checkpoint(tmp_path / "ck", P.PonenexConfig.from_dict(cfg), w)
    a, b = tokens(cfg, 40, 1), tokens(cfg, 12, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[3:], "want": [8]}, {"id": "a", "tokens": a[31:], "want": [0, 8]}], "end": ["a", "b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "ck"), "--dtype", dtype, "--out", str(tmp_path / "o"), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = O.forward(cfg, w, a), O.forward(cfg, w, b)
    lim = LIMIT[F32 if dtype == "float32" else BF16]
    load = lambda i: torch.from_numpy(np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])
    assert not (tmp_path / "o" / "1.f32").exists()
    assert logit_error(load(0), wa[[0, 29]]) < lim and logit_error(load(2), torch.stack([wb[11], wa[31], wa[39]])) < lim


@pytest.mark.gpu
def test_worker_preset_and_memory_profile(tmp_path):
    path = tmp_path / "mem.json"
    r = subprocess.run([sys.executable, "-m", "ironpangu_b200.runtime.engine_worker", "--model", "ponenex-tiny", "--max-num-seqs", "2", "--max-model-len", "128",
                        "--kv-pool-tokens", "128", "--prefill-chunk", "64", "--memory-profile", str(path), "--profile-only"], capture_output=True, text=True,
                       timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(path.read_text())["failed_stage"] is None
