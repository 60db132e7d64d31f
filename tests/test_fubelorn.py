"""The Fubelorn decoder as a model of the framework: configuration and registry (CPU); whole prompts, portions, token-by-token decoding, mixed
batches, reused pages and slots, long decoding and generation through the engine and the server against the plain restatement (GPU)."""
import copy
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import fubelorn_oracle as O
from fubelorn_cases import CASES, config, delta, kept, memory, pooled, ssd, tokens, weights
from stream_rig import Rig, cut, logit_error, random_batches

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32
# largest allowed error of a row of logits relative to their spread
LIMIT = {F32: 1e-4, BF16: 1.2e-1}
DTYPES = pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])


def rig(cfg, dtype, seed=0, **kw):
    return Rig(cfg, weights(cfg, seed), dtype, **kw)


# ---------------------------------------------------------------------------------------------------------------------------
# CPU
# ---------------------------------------------------------------------------------------------------------------------------
def _but(layer, **change):
    """The layer with changed mixer entries; names with '__' reach into 'left', 'right', 'mask' and 'rot'."""
    out = copy.deepcopy(layer)
    for k, v in change.items():
        *path, last = k.split("__")
        m = out["mixer"]
        for p in path:
            m = m[p]
        m[last] = v
    return out


def test_configuration_round_trip_and_checks():
    from ironpangu_b200.models.fubelorn import FubelornConfig, weight_shapes

    for c in CASES.values():
        f = FubelornConfig.from_dict(json.loads(json.dumps(c)))
        assert FubelornConfig.from_dict(f.to_dict()) == f
        for a, b in zip(f.to_dict()["layers"], c["layers"]):
            assert a == b
        assert f.param_count() == sum(int(np.prod(s)) for s in weight_shapes(f).values())
    for c in (FubelornConfig.tiny(), FubelornConfig.text(layers=4)):
        assert FubelornConfig.from_dict(c.to_dict()) == c
    of = lambda *l, **kw: FubelornConfig.from_dict(config(list(l), **kw))
    # pages may go early only when nothing ahead of a window is seen
    assert of(kept(size=9, keep=0), ssd(), kept(size=14, keep=0)).window == 14 and of(kept(size=9, keep=2)).window == 0 and of(pooled(), kept(keep=0)).window == 0 and of(ssd()).window == 0
    plain = config([kept(keep=0)])
    del plain["streams"], plain["canon"], plain["layers"][0]["mixer"]["left"]["mask"]["keep_first"]
    f = FubelornConfig.from_dict(plain)
    assert f.streams == 0 and f.taps == 0 and f.layers[0].left.keep == 0 and not [n for n in weight_shapes(f) if "hc" in n or "canon" in n or "norm2" in n]
    bad = [dict(CASES["odd"], architecture="Other"), config([]), config([dict(ssd(), type="mamba")]), config([kept(heads=5, kv_heads=2)]), config([kept(dim=300)]), config([kept(keep=-1)]),
           config([kept(size=0, keep=3)]), config([pooled(pool=-4)]), config([pooled(rot=3)]), config([pooled(rot=18)]), config([pooled(scaling=(4.0, 4.0, 1.0, 64))]),
           config([pooled(right=memory(cap=0.0))]), config([kept(right=delta(3, 2))]), config([kept(right=delta(conv=0))]), config([ssd(norm_groups=5)]), config([ssd(heads=3, groups=2)]),
           config([ssd(state=2000)]), config([ssd()], streams=40), config([ssd()], taps=50), config([ssd()], streams=-1), config([dict(ssd(), mlp={"kind": "moe"})]),
           config([_but(kept(), left__scale=None)])]
    for i, c in enumerate(bad):
        with pytest.raises((ValueError, KeyError, TypeError)):
            FubelornConfig.from_dict(c)
            print(i)
    s = weight_shapes(FubelornConfig.from_dict(CASES["mixed"]))
    assert s["l0.mix.right.v.conv"] == (6 * 24, 4) and s["l0.mix.right.norm"] == (24,) and s["l0.hc1.mix"] == (3, 3) and s["l0.canon2"] == (72, 4) and s["l0.norm1"] == ()
    assert s["l1.mix.in"] == (2 * 96 + 2 * 60 + 6, 72) and s["l1.mix.conv.b"] == (96 + 120,) and s["l2.mix.left.g"] == (3, 72) and s["l2.mix.right.norm"] == (120,)
    assert "l2.mlp.up" not in s and "l2.norm2" not in s and s["l2.mix.right.f.b"] == (3,) and "l0.mix.left.g" not in s and s["head"] == (96, 72)


def test_checkpoint_and_registry(tmp_path):
    from ironpangu_b200.models import fubelorn as M
    from ironpangu_b200.models import registry

    cfg = CASES["mixed"]
    w = weights(cfg)
    M.save_checkpoint(tmp_path, M.FubelornConfig.from_dict(cfg), w)
    assert registry.family_of(tmp_path).decoder == "FubelornDecoder" and {"fubelorn-tiny", "fubelorn-text", "mikutar-tiny"} <= set(registry.preset_names())
    c, got = M.load_checkpoint(tmp_path)
    assert c == M.FubelornConfig.from_dict(cfg) and set(got) == set(w) and all(torch.equal(got[n], w[n]) for n in w) and got["final.norm"].shape == ()
    w["l0.mix.right.A_log"] = w["l0.mix.right.A_log"][:-1]
    M.save_checkpoint(tmp_path, c, w)
    with pytest.raises(ValueError, match="l0.mix.right.A_log"):
        M.load_checkpoint(tmp_path)
    del w["l0.mix.right.A_log"]
    M.save_checkpoint(tmp_path, c, w)
    with pytest.raises(ValueError, match="l0.mix.right.A_log"):
        M.load_checkpoint(tmp_path)


def test_random_weights_of_the_presets():
    from ironpangu_b200.models import fubelorn as M

    c = M.FubelornConfig.tiny()
    w = M.random_weights(c, "cpu")
    assert {n: tuple(t.shape) for n, t in w.items()} == M.weight_shapes(c) and all(torch.isfinite(t).all() for t in w.values())
    logits = O.forward(c.to_dict(), w, list(range(40)))
    assert torch.isfinite(logits).all() and float(logits.std()) > 0.05


FAULTS = ("mask_plus_one", "mask_minus_one", "no_kept", "keep_plus_one", "keep_minus_one", "no_qk_norm", "no_scaling", "pool_late", "pool_early", "no_pool", "pool_before_rotation", "no_gate",
          "correct_before_decay", "no_correction", "read_before_write", "taps_reversed", "no_q_factor", "no_conv_bias", "swap_bc", "no_skip", "gate_after_norm", "no_gate_cap", "no_right", "no_canon",
          "canon_reversed", "mix_transposed")


def test_restatement_notices_planted_faults():
    """The comparison the GPU tests make in 32 bits would fail by a wide margin for every one of these mistakes, the one in 16 bits for most."""
    cfg = CASES["mixed"]
    w, toks = weights(cfg), tokens(cfg, 60)
    good = O.forward(cfg, w, toks)
    for fault in FAULTS:
        assert logit_error(O.forward(cfg, w, toks, faults=(fault,)), good) > (500 * LIMIT[F32] if "pool" in fault else 1.5 * LIMIT[BF16]), fault
    assert logit_error(O.forward(cfg, w, toks, faults=("gelu_tanh",)), good) > 10 * LIMIT[F32]


# ---------------------------------------------------------------------------------------------------------------------------
# GPU: the model through the engine
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("name", list(CASES))
def test_whole_prompts_portions_and_decoding(name, dtype):
    if name == "single" and dtype == BF16:
        pytest.skip("a norm over one column is a sign, which a rounding turns")
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
    assert len(probe) == len(residuals) == 6
    for got, want in zip(probe, residuals):
        assert float((got.cpu().double() - want).abs().max() / want.abs().max()) < (2e-5 if dtype == F32 else 5e-2)
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
    assert logit_error(mixed["a"], alone["a"].double()) < (2e-5 if dtype == F32 else 4e-2)
    r.close()


@pytest.mark.gpu
@pytest.mark.parametrize("size", [1, 2, 15, 16, 17, 31, 64])
@pytest.mark.parametrize("kind", ["kept", "pooled"])
def test_edges_in_prompts_and_decoding(kind, size):
    """Every window, with kept positions or blocks, against page borders (16) and portion borders; the restatement one token off is far away."""
    if kind == "kept":
        cfg = config([kept(4, 2, 64, size=size, keep=size % 7 + 1, scale=0.5, ff=32, scales=(1.0, 0.3)), kept(3, 1, 20, size=size, keep=size + 2, scale=0.7, scales=(1.0, 0.3))])
        faults = ("mask_plus_one", "keep_plus_one", "keep_minus_one")
    else:
        cfg = config([pooled(4, 2, 64, size=size, pool=2, scale=1.5, ff=32, scales=(1.0, 0.3)), pooled(3, 1, 20, size=size, pool=2, scale=2.0, scales=(1.0, 0.3))])
        faults = ("mask_plus_one", "pool_late", "pool_early")
    n = 160
    toks = tokens(cfg, n)
    for dtype in (F32, BF16):
        r = rig(cfg, dtype, rows=128)
        want = O.forward(cfg, r.w, toks)
        # one block more or less among dozens of keys shows in 32 bits only
        off = min(logit_error(O.forward(cfg, r.w, toks, faults=(f,)), want) for f in faults if dtype == F32 or "pool" not in f)
        assert off > (3 if dtype == BF16 else 20) * LIMIT[dtype], off
        for cuts in ([n], [1] * n, [16] * 10, [size] * (n // size) if size > 1 else [3] * 33, [size + 1] * (n // (size + 1)), [100] + [1] * 60):
            got = r.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
            e = logit_error(got, want[:len(got)])
            assert e < min(LIMIT[dtype], off / 3), (cuts[:3], e, off)
        r.close()


@pytest.mark.gpu
@DTYPES
def test_long_decoding(dtype):
    """Hundreds of decoded tokens: windows, blocks and states move on; a model of windows alone gives its pages back behind them."""
    cfg = config([kept(4, 2, 32, size=40, keep=7, ff=24), pooled(2, 1, 16, size=23, pool=5), ssd()])
    r = rig(cfg, dtype, context=700, rows=64)
    toks = tokens(cfg, 620)
    want = O.forward(cfg, r.w, toks)
    got = r.run({"a": toks}, [[("a", 40)]] + [[("a", 1)]] * 580)["a"]
    assert logit_error(got, want) < LIMIT[dtype]
    assert r.dec.state_manager.pages_trimmed == 0
    r.close()
    cfg = config([kept(4, 2, 32, size=40, keep=0, ff=24), ssd()])
    r = rig(cfg, dtype, context=700, pool=96, rows=64)
    want = O.forward(cfg, r.w, toks)
    got = r.run({"a": toks}, [[("a", 40)]] + [[("a", 1)]] * 580)["a"]
    assert logit_error(got, want) < LIMIT[dtype] and r.dec.state_manager.pages_trimmed > 30
    r.close()


@pytest.mark.gpu
@DTYPES
def test_models_of_recurrences_alone(dtype):
    """No pages at all; with and without streams and convolution."""
    for kw in ({}, {"streams": 0, "taps": 0}):
        cfg = config([ssd(ff=40), ssd(2, 2, 24, 16, 2, 1)], **kw)
        if not kw.get("streams", 1):
            del cfg["streams"]
        r = rig(cfg, dtype)
        toks = tokens(cfg, 120)
        if kw:          # the restatement knows streams and taps only: one stream of unit weights, taps of zero
            w = dict(r.w)
            for i in (0, 1):
                for q in (1, 2):
                    w.update({f"l{i}.hc{q}.in": torch.ones(1), f"l{i}.hc{q}.out": torch.ones(1), f"l{i}.hc{q}.mix": torch.ones(1, 1), f"l{i}.canon{q}": torch.zeros(64, 1)})
            want = O.forward(dict(cfg, streams=1), w, toks)
        else:
            want = O.forward(cfg, r.w, toks)
        for cuts in ([120], [1] * 40, [50, 2, 3, 60, 1, 1]):
            got = r.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
            assert logit_error(got, want[:len(got)]) < LIMIT[dtype]
        r.close()


@pytest.mark.gpu
@DTYPES
@pytest.mark.parametrize("kind", ["window", "kept", "block"])
def test_the_first_tokens_are_seen_by_the_last(kind, dtype):
    """Far keys count - in a wide window, as kept positions, as a block: other first tokens, other logits at the end, in a prompt and in decoding."""
    off = dict(scales=(1.0, 0.01), right=delta(1, 1, 4, 4))
    layer = {"window": kept(2, 1, 64, size=512, keep=0, scale=0.2, **off), "kept": kept(4, 2, 24, size=30, keep=40, scale=0.4, **off),
             "block": pooled(2, 1, 32, size=30, pool=20, scale=0.2, scales=(1.0, 0.01), right=memory(1, 4, 4))}[kind]
    cfg = config([layer])
    r = rig(cfg, dtype, context=600)
    toks = tokens(cfg, 500)
    seqs = [[first] * 80 + toks[80:] for first in (toks[0], (toks[0] + 32) % cfg["vocab"])]
    wants = [O.forward(cfg, r.w, s) for s in seqs]
    assert logit_error(wants[1][480:], wants[0][480:]) > 2 * LIMIT[dtype]
    for seq, want in zip(seqs, wants):
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
    for seed in range(30):                             # a prompt whose continuation has no near tie for some tokens
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

    from ironpangu_b200.models import fubelorn as M
    from test_server import Server

    cfg = dict(CASES["mixed"], vocab=300)
    w = weights(cfg)
    M.save_checkpoint(tmp_path / "ck", M.FubelornConfig.from_dict(cfg), w)
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
    from ironpangu_b200.models import fubelorn as M

    cfg = CASES["odd"]
    w = weights(cfg)
    M.save_checkpoint(tmp_path / "ck", M.FubelornConfig.from_dict(cfg), w)
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
    r = subprocess.run([sys.executable, "-m", "ironpangu_b200.runtime.engine_worker", "--model", "fubelorn-tiny", "--max-num-seqs", "2", "--max-model-len", "128",
                        "--kv-pool-tokens", "128", "--prefill-chunk", "64", "--memory-profile", str(path), "--profile-only"], capture_output=True, text=True,
                       timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(path.read_text())["failed_stage"] is None
