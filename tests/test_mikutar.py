"""The Mikutar decoder as a model of the framework: configuration and registry (CPU); whole prompts, portions, token-by-token decoding, mixed
batches, reused pages and slots, long decoding and generation through the engine and the server against the plain restatement (GPU)."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import mikutar_oracle as O
from mikutar_cases import CASES, choice_gap, chunk, config, tokens, weights, window
from stream_rig import Rig, cut, logit_error, random_batches

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32
# largest allowed error of a row of logits relative to their spread
LIMIT = {F32: 4e-5, BF16: 5e-2}
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def rig(cfg, dtype, seed=0, **kw):
    """In 16 bits the routers have no close calls (a rounding that turns a choice is not a fault)."""
    return Rig(cfg, weights(cfg, seed, separated=dtype == BF16), dtype, **kw)


# ---------------------------------------------------------------------------------------------------------------------------
# CPU
# ---------------------------------------------------------------------------------------------------------------------------
def test_configuration_round_trip_and_checks():
    from ironpangu_b200.models.mikutar import MikutarConfig, weight_shapes

    for c in CASES.values():
        f = MikutarConfig.from_dict(json.loads(json.dumps(c)))
        assert f.to_dict() == c and MikutarConfig.from_dict(f.to_dict()) == f
        assert f.order() == O.run_order(c)
    assert MikutarConfig.from_dict(CASES["mixed"]).window == 50
    assert MikutarConfig.from_dict(config([window(), dict(window(), mixer=dict(window()["mixer"], mask=None))])).window == 0
    for c in (MikutarConfig.tiny(), MikutarConfig.text(layers=4, loop=(1, 3, 2))):
        assert MikutarConfig.from_dict(c.to_dict()) == c
    plain = config([window(ff=8), chunk(experts=4, top=2)])
    del plain["loop"], plain["layers"][1]["mlp"]["router"]["groups"]
    f = MikutarConfig.from_dict(plain)
    assert f.order() == [(0, False), (1, False)] and f.layers[1].experts.groups == 1 and f.layers[1].ff == 0
    m = window()["mixer"]
    bad = [dict(CASES["odd"], architecture="Other"), config([]), config([dict(window(), type="retention")]), config([window(rot=3)]), config([window(rot=18)]),
           config([window(heads=5, kv_heads=2)]), config([window(dim=300)]), config([window(size=-1)]), config([chunk(cap=-1.0)]),
           config([dict(window(), mixer=dict(m, vdim=8))]), config([chunk(experts=3, top=4)]), config([chunk(experts=6, top=3, groups=(3, 1))]),
           config([chunk(experts=7, top=2, groups=(2, 1))]), config([chunk(experts=4, top=2, limit=0.0)]), config([chunk(experts=300, top=2)]),
           config([dict(window(), mlp={"kind": "sparse"})]), config([window()], loop=(0, 2, 2)), config([window()], loop=(1, 0, 2)), config([window()], loop=(0, 1, 0)),
           config([window()], cap=-2.0), config([dict(window(), mixer={k: v for k, v in m.items() if k != "scale"})])]
    for c in bad:
        with pytest.raises((ValueError, KeyError)):
            MikutarConfig.from_dict(c)
    s = weight_shapes(MikutarConfig.from_dict(CASES["mixed"]))
    assert s["l0.mix.q.norm"] == (240,) and s["l0.mix.k.b"] == (80,) and "l0.mix.v" not in s and s["l0.mlp.down"] == (72, 200) and "head" not in s
    assert s["l1.mix.v"] == (3 * 56, 72) and "l1.mix.o.b" not in s and s["l1.mlp.shared.up"] == (72, 72) and s["l1.mlp.correction"] == (12,) and "l2.mlp.gate" not in s
    c = MikutarConfig.from_dict(CASES["odd"])
    assert c.param_count() == sum(int(np.prod(v)) for v in weight_shapes(c).values())
    assert c.param_count() - c.active_params() == 7 * 3 * 19 * 53


def test_checkpoint_and_registry(tmp_path):
    from ironpangu_b200.models import mikutar as M
    from ironpangu_b200.models import registry

    cfg = CASES["mixed"]
    w = weights(cfg)
    M.save_checkpoint(tmp_path, M.MikutarConfig.from_dict(cfg), w)
    assert registry.family_of(tmp_path).decoder == "MikutarDecoder" and {"mikutar-tiny", "ponenex-tiny", "falinex-tiny"} <= set(registry.preset_names())
    c, got = M.load_checkpoint(tmp_path)
    assert c == M.MikutarConfig.from_dict(cfg) and set(got) == set(w) and all(torch.equal(got[n], w[n]) for n in w)
    w["l1.mlp.correction"] = w["l1.mlp.correction"][:-1]
    M.save_checkpoint(tmp_path, c, w)
    with pytest.raises(ValueError, match="l1.mlp.correction"):
        M.load_checkpoint(tmp_path)
    del w["l1.mlp.correction"]
    M.save_checkpoint(tmp_path, c, w)
    with pytest.raises(ValueError, match="l1.mlp.correction"):
        M.load_checkpoint(tmp_path)


FAULTS = ("mask_plus_one", "mask_minus_one", "no_gate", "no_projection_bias", "no_output_bias", "norm_per_head", "values_after_norm", "values_are_turned",
          "chunk_is_a_window", "no_score_cap", "no_slopes", "no_limit", "up_without_one", "no_correction", "all_groups", "group_by_best", "closed_groups_score_zero",
          "weights_with_correction", "weights_renormed", "no_shared", "embedding_added_once", "serial", "no_logit_cap")


def test_restatement_notices_planted_faults():
    """The comparison the GPU tests make would fail by a wide margin for every one of these mistakes."""
    cfg = CASES["mixed"]
    for separated in (False, True):
        w, toks = weights(cfg, separated=separated), tokens(cfg, 60)
        good = O.forward(cfg, w, toks)
        # routers whose choices are far apart choose the same under some of the other rules: the 32-bit tests tell these
        for fault in FAULTS if not separated else [f for f in FAULTS if f not in ("all_groups", "group_by_best", "closed_groups_score_zero")]:
            assert logit_error(O.forward(cfg, w, toks, faults=(fault,)), good) > (2 * LIMIT[BF16] if separated else 1000 * LIMIT[F32]), (separated, fault)


def test_separated_routers_have_no_close_calls(monkeypatch):
    from types import SimpleNamespace

    gaps, pick = [], O.choose

    def watch(s, b, top, count, keep, faults=()):
        gaps.append(float(choice_gap(s, s + b, SimpleNamespace(groups=count, keep=keep, top=top)).min()))
        return pick(s, b, top, count, keep, faults)

    monkeypatch.setattr(O, "choose", watch)
    for cfg in CASES.values():
        O.forward(cfg, weights(cfg, separated=True), tokens(cfg, 100))
    assert min(gaps) > 0.012          # a choice score is off by some 0.002 in 16 bits


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
    schedules = {"whole": [n], "token by token": [1] * 70, "prompt, then decoding": [n - 70] + [1] * 70, "portions": cut(rnd, n, [2, 3, 5, 9, 17, 33, 64, 65]),
                 "pairs": [2] * 35, "first tokens": [1, 2, 3, 1, 5, 16, 15, 2], "threes": [3] * 20}
    for what, cuts in schedules.items():
        got = r.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
        e = logit_error(got, want[:len(got)])
        assert e < LIMIT[dtype], (what, e)
    r.close()


@pytest.mark.gpu
@DTYPES
def test_residual_stream_after_every_layer_run(dtype):
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
    assert len(probe) == len(residuals) == 7
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
        assert logit_error(g, want[k]) < LIMIT[BF16], k
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
@pytest.mark.parametrize("size", [1, 2, 15, 16, 17, 31, 64])
@pytest.mark.parametrize("kind", [window, chunk], ids=["window", "chunk"])
def test_edges_in_prompts_and_decoding(kind, size):
    """Every window and chunk against page borders (16) and portion borders; the restatement one token off is far away."""
    sharp = lambda v: {"scale": v} if kind is window else {}
    cfg = config([kind(4, 2, 64, size=size, ff=32, **sharp(0.6)), kind(3, 1, 20, size=size, **sharp(0.9))])
    n = 160
    toks = tokens(cfg, n)
    for dtype in (F32, BF16):
        r = rig(cfg, dtype, rows=128)
        want = O.forward(cfg, r.w, toks)
        off = logit_error(O.forward(cfg, r.w, toks, faults=("mask_plus_one",)), want)
        assert off > 3 * LIMIT[dtype]
        for cuts in ([n], [1] * n, [16] * 10, [size] * (n // size) if size > 1 else [3] * 33, [size + 1] * (n // (size + 1)), [100] + [1] * 60):
            got = r.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
            assert logit_error(got, want[:len(got)]) < min(LIMIT[dtype], off / 3), cuts
        r.close()


@pytest.mark.gpu
@DTYPES
def test_long_decoding_in_a_pool_of_one_window(dtype):
    """Hundreds of decoded tokens while the pages of the window come and go."""
    cfg = config([window(4, 2, 32, size=40, ff=24), chunk(2, 1, 16, size=23)], loop=(0, 1, 2))
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
    """In a wide window or chunk a far key counts: another first token, other logits at the end, in a prompt and in decoding."""
    cfg = config([window(2, 1, 64, size=512, ff=16), chunk(4, 2, 24, size=600, scale=0.02)])
    r = rig(cfg, dtype, context=600)
    toks = tokens(cfg, 500)
    w0 = O.forward(cfg, r.w, toks)
    for first in (toks[0], (toks[0] + 32) % cfg["vocab"]):
        seq = [first] * 40 + toks[40:]
        want = O.forward(cfg, r.w, seq)
        assert logit_error(want[480:], w0[480:]) > 2 * LIMIT[dtype]
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

    cfg = dict(CASES["mixed"], logit_softcap=40.0)
    r = rig(cfg, dtype, residents=2)
    for seed in range(20):                             # a prompt whose continuation has no near tie for some tokens
        prompt = tokens(cfg, 30, seed)
        want, margins = _greedy(cfg, r.w, prompt, 12)
        clear = next((i for i, m in enumerate(margins) if m < (1e-3 if dtype == F32 else 0.3)), 12)
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

    from ironpangu_b200.models import mikutar as M
    from test_server import Server

    cfg = dict(CASES["mixed"], vocab=300)
    w = weights(cfg)
    M.save_checkpoint(tmp_path / "ck", M.MikutarConfig.from_dict(cfg), w)
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
    from ironpangu_b200.models import mikutar as M

    cfg = CASES["odd"]
    w = weights(cfg, separated=True)
    M.save_checkpoint(tmp_path / "ck", M.MikutarConfig.from_dict(cfg), w)
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
    r = subprocess.run([sys.executable, "-m", "ironpangu_b200.runtime.engine_worker", "--model", "mikutar-tiny", "--max-num-seqs", "2", "--max-model-len", "128",
                        "--kv-pool-tokens", "128", "--prefill-chunk", "64", "--memory-profile", str(path), "--profile-only"], capture_output=True, text=True,
                       timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(path.read_text())["failed_stage"] is None
