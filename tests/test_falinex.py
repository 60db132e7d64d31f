"""The Falinex decoder as a model of the framework: configuration and registry, page pool and step plans (CPU); whole prompts,
portions, token-by-token decoding, mixed batches, reused pages and slots, long decoding and generation through the engine and the
server against the plain restatement (GPU)."""
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

import falinex_oracle as O
from falinex_cases import CASES, attention, config, lightning, retention, tokens, weights
from stream_rig import Rig as StreamRig
from stream_rig import cut, logit_error, random_batches

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32
# largest allowed error of a row of logits relative to their spread
LIMIT = {F32: 4e-5, BF16: 6e-2}


# ---------------------------------------------------------------------------------------------------------------------------
# CPU
# ---------------------------------------------------------------------------------------------------------------------------
def test_configuration_round_trip_and_checks():
    from ironpangu_b200.models.falinex import FalinexConfig

    for c in list(CASES.values()):
        f = FalinexConfig.from_dict(json.loads(json.dumps(c)))
        assert f.to_dict() == c and FalinexConfig.from_dict(f.to_dict()) == f
    f = FalinexConfig.from_dict(CASES["mixed"])
    assert [f.owner(i) for i in range(5)] == [0, 1, 2, 1, 0] and f.window == 24
    assert FalinexConfig.from_dict(config([attention(window=5), attention(window=9)])).window == 9
    assert FalinexConfig.from_dict(FalinexConfig.tiny().to_dict()) == FalinexConfig.tiny()
    bad = [dict(CASES["odd"], architecture="Other"), config([retention(decay=[0.5])]), config([attention(heads=3, kv_heads=2)]),
           config([retention(), retention(dim=8, weights_of=0)]), config([retention(weights_of=0)]), config([dict(retention(), type="mamba")]),
           config([retention(rot=17)]), config([dict(retention(), mlp={"kind": "experts", "ff": 3})])]
    for c in bad:
        with pytest.raises((ValueError, KeyError)):
            FalinexConfig.from_dict(c)


def test_checkpoint_and_registry(tmp_path):
    from ironpangu_b200.models import falinex as F
    from ironpangu_b200.models import registry

    cfg = CASES["mixed"]
    w = weights(cfg)
    F.save_checkpoint(tmp_path, F.FalinexConfig.from_dict(cfg), w)
    assert registry.family_of(tmp_path).decoder == "FalinexDecoder"
    c, got = F.load_checkpoint(tmp_path)
    assert c == F.FalinexConfig.from_dict(cfg) and set(got) == set(w) and all(torch.equal(got[n], w[n]) for n in w)
    assert not any(n.startswith(("l3.", "l4.")) for n in got)             # layers that share weights bring none
    del w["l2.mix.norm"]
    F.save_checkpoint(tmp_path, c, w)
    with pytest.raises(ValueError, match="l2.mix.norm"):
        F.load_checkpoint(tmp_path)
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    with pytest.raises(ValueError, match="Unheard"):
        registry.family_of(tmp_path)


def test_restatement_notices_planted_faults():
    """The comparison the GPU tests make would fail by a wide margin for a window that is one token off or a sink left out."""
    for name in ("mixed", "tiles"):
        cfg = CASES[name]
        w, toks = weights(cfg), tokens(cfg, 60)
        good = O.forward(cfg, w, toks)
        for fault in ("no_sink", "window_plus_one", "window_minus_one"):
            if name == "tiles" and fault == "window_minus_one":
                continue                                                   # its window of one token would see nothing
            assert logit_error(O.forward(cfg, w, toks, faults=(fault,)), good) > 3 * LIMIT[BF16], (name, fault)


def test_page_pool_grows_trims_and_reuses():
    from ironpangu_b200.runtime.paged_state import PagedState

    p = PagedState(model="t", context=512, residents=3, page_tokens=16, pool_pages=12, row_bytes=8, slot_bytes=16, vocab=10, device="cpu", window=40)
    p.admit(0)
    p.ensure(0, 100)
    p.flush()
    assert sorted(p.table[0, :7].tolist()) == sorted(set(p.table[0, :7].tolist())) and p.table[0, 7] == -1
    p.advance(0, 100)                                  # positions up to 60 are out of reach: three whole pages
    p.flush()
    assert (p.table[0, :3] == -1).all() and (p.table[0, 3:7] >= 0).all()
    p.advance(0, 102)
    assert p.pages_trimmed == 3
    p.admit(1, reserve=100)
    with pytest.raises(OverflowError):
        p.ensure(0, 512)                               # 25 more pages, one free: refused, nothing changes
    p.ensure(0, 112 + 16)
    p.flush()
    live = [x for x in p.table.flatten().tolist() if x >= 0]
    assert len(live) == len(set(live)) == 12
    with pytest.raises(OverflowError):
        p.admit(2)
    p.release(1)
    p.admit(2)
    p.flush()
    assert p.table[2, 0] >= 0 and (p.table[1] == -1).all()
    p.release(0)
    p.release(2)
    assert all(c["occupied_units"] == 0 for c in p.usage()["components"].values())
    with pytest.raises(OverflowError):
        p.ensure(0, 600)
    p.close()


def test_a_long_request_lives_in_a_window_of_pages():
    from ironpangu_b200.runtime.paged_state import PagedState

    p = PagedState(model="t", context=4096, residents=1, page_tokens=16, pool_pages=6, row_bytes=8, slot_bytes=0, vocab=10, device="cpu", window=33)
    p.admit(0)
    for pos in range(0, 4096, 16):
        p.ensure(0, pos + 16)
        p.advance(0, pos + 16)
        held = (p._host[0] >= 0).sum()
        assert held <= 4
    p.close()


def test_step_plans_cover_every_row_once():
    from ironpangu_b200.ops.linear_attn import StepPlan

    rnd = random.Random(1)
    for _ in range(400):
        slots, pos = [], []
        for s in rnd.sample(range(40), rnd.randint(1, 25)):
            n, p = rnd.choice([1, 1, 2, 3, 4, 5, 9, 70, 130]), rnd.randint(0, 50)
            slots += [s] * n
            pos += list(range(p, p + n))
        chunk = rnd.choice([64, 128])
        plan = StepPlan(slots, pos, short=rnd.choice([0, 4]), group=rnd.choice([8, 64]), chunk=chunk)
        long = {r for a, n, _, _ in plan.runs for r in range(a, a + n)}
        assert sorted(r for a, n, _, _ in plan.chunks for r in range(a, a + n)) == sorted(long)
        assert set(range(len(slots))) - long <= {r for lo, hi in plan.groups for r in range(lo, hi)}
        for a, n, s, f in plan.chunks:
            assert 1 <= n <= chunk and slots[a:a + n] == [s] * n
        i = 0
        while i < len(plan.chunks):
            count = plan.chunks[i][3] >> 1
            assert plan.chunks[i][3] & 1 and all(plan.chunks[i + k][3] == 0 for k in range(1, count))
            assert all(plan.chunks[i + k][1] == chunk for k in range(count - 1))
            i += count
        if plan.masked:
            step = plan.control[4 * len(plan.chunks):].tolist()
            assert step == [-1 if r in long else pos[r] for r in range(len(slots))]


def test_replay_admits_batches_and_releases():
    from ironpangu_b200.runtime.replay import Replay

    class Engine:
        residents = 2

        def __init__(self):
            self.log = []

        def admit(self, r, sampling, reserve):
            self.log.append(("admit", r))

        def release(self, r):
            self.log.append(("release", r))

        def step_logits(self, slices, toks, want):
            self.log.append((slices, toks, want))
            return torch.zeros(sum(len(w) for w in want), 3)

    e = Engine()
    r = Replay(e)
    out = r.step({"step": 0, "entries": [{"id": "a", "tokens": [1, 2], "want": [1]}, {"id": "b", "tokens": [3], "want": []}], "end": ["b"]})
    assert out.shape == (1, 3)
    assert r.step({"step": 1, "entries": [{"id": "c", "tokens": [4], "want": []}, {"id": "a", "tokens": [5], "want": []}], "end": ["a", "c"]}) is None
    assert e.log == [("admit", 0), ("admit", 1), ([[0, 0, 2, False], [1, 0, 1, False]], [1, 2, 3], [[1], []]), ("release", 1), ("admit", 1),
                     ([[1, 0, 1, False], [0, 2, 1, False]], [4, 5], [[], []]), ("release", 0), ("release", 1)]
    r.step({"step": 2, "entries": [{"id": "x", "tokens": [1], "want": []}, {"id": "y", "tokens": [1], "want": []}], "end": []})
    with pytest.raises(RuntimeError):
        r.step({"step": 3, "entries": [{"id": "z", "tokens": [1], "want": []}], "end": []})


# ---------------------------------------------------------------------------------------------------------------------------
# GPU: the model through the engine
# ---------------------------------------------------------------------------------------------------------------------------
def Rig(cfg, dtype, *, seed=0, **kw):
    return StreamRig(cfg, weights(cfg, seed), dtype, **kw)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", list(CASES))
def test_whole_prompts_portions_and_decoding(name, dtype):
    cfg = CASES[name]
    rig = Rig(cfg, dtype)
    n = 210
    toks = tokens(cfg, n)
    want = O.forward(cfg, rig.w, toks)
    rnd = random.Random(name)
    schedules = {"whole": [n], "token by token": [1] * 40, "prompt, then decoding": [n - 70] + [1] * 70, "portions": cut(rnd, n, [2, 3, 5, 9, 17, 33, 64, 65]),
                 "pairs": [2] * 30, "first tokens": [1, 2, 3, 1, 5, 16, 15, 2]}
    for what, cuts in schedules.items():
        got = rig.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
        e = logit_error(got, want[:len(got)])
        assert e < LIMIT[dtype], (what, e)
    rig.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "tiles"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(name, dtype):
    """More requests than slots over a pool that cannot hold them all at once; portions beside decoded tokens; a request left out of some
    steps; every request equals the restatement (computed alone)."""
    cfg = CASES[name]
    rig = Rig(cfg, dtype, context=320, pool=448, rows=128)          # rows: wide steps take several passes
    rnd = random.Random(7)
    lens = {"a": 150, "b": 23, "c": 97, "d": 5, "e": 64, "f": 33, "g": 121}
    reqs = {k: tokens(cfg, n, i) for i, (k, n) in enumerate(lens.items())}
    want = {k: O.forward(cfg, rig.w, t) for k, t in reqs.items()}
    steps = random_batches(rnd, lens, list(reqs) + ["a#2", "d#2"], 4, 448, [1, 1, 1, 2, 3, 16, 29, 64])
    got = rig.run(reqs, steps)
    for k, g in got.items():
        e = logit_error(g, want[k.split("#")[0]])
        assert e < LIMIT[dtype], (k, e)
    u = rig.dec.state_manager.usage()
    assert all(c["occupied_units"] == 0 for c in u["components"].values()) and u["pages_taken"] > u["components"]["kv"]["capacity_units"]
    rig.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
def test_a_batch_changes_nothing(dtype):
    """Logits of a request alone and beside others, and on other pages and slots, agree far below the model's own rounding."""
    cfg = CASES["tiles"]
    rig = Rig(cfg, dtype)
    reqs = {k: tokens(cfg, n, i) for i, (k, n) in enumerate({"a": 90, "b": 40, "c": 61}.items())}
    cuts = [[("b", 20), ("a", 50)], [("a", 1), ("b", 1)], [("c", 61), ("a", 1), ("b", 9)]] + [[("a", 1), ("b", 1)]] * 10 + [[("a", 28)]]
    mixed = rig.run(reqs, cuts)
    alone = rig.run(reqs, [[("a", 50)], [("a", 1)], [("a", 1)]] + [[("a", 1)]] * 10 + [[("a", 28)]])
    assert logit_error(mixed["a"], alone["a"].double()) < (2e-5 if dtype == F32 else 2e-2)
    rig.close()


@pytest.mark.gpu
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 31, 64])
def test_window_edges_in_prompts_and_decoding(window):
    """Every window against page borders (16) and portion borders; the restatement with the window one token off is far away."""
    cfg = config([attention(4, 2, 64, 64, window=window), lightning(2, 32, 32), attention(4, 4, 24, 16, rot=8, window=window)], width=64)
    rig = Rig(cfg, F32, rows=128)
    toks = tokens(cfg, 100)
    want = O.forward(cfg, rig.w, toks)
    off = logit_error(O.forward(cfg, rig.w, toks, faults=("window_plus_one",)), want)
    assert off > 100 * LIMIT[F32]
    for cuts in ([100], [1] * 100, [16] * 6 + [4], [window] * (100 // window) if window > 1 else [3] * 33, [window + 1] * (100 // (window + 1)), [50] + [1] * 50):
        got = rig.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
        assert logit_error(got, want[:len(got)]) < LIMIT[F32], cuts
    rig.close()
    rig = Rig(cfg, BF16, rows=128)
    for cuts in ([100], [1] * 100, [window + 1] * (100 // (window + 1))):
        got = rig.run({"a": toks[:sum(cuts)]}, [[("a", c)] for c in cuts])["a"]
        assert logit_error(got, want[:len(got)]) < min(LIMIT[BF16], off / 3), cuts
    rig.close()


@pytest.mark.gpu
def test_long_decoding_in_a_pool_of_one_window():
    """Hundreds of decoded tokens while the pages of the window come and go; states with slow decay keep what the first tokens left."""
    cfg = config([retention(2, 32, 32, decay=[0.999, 0.9]), attention(4, 2, 64, 64, window=40), lightning(2, 16, 16, decay=[0.9995, 0.7])], width=64)
    rig = Rig(cfg, F32, context=700, pool=96, rows=64)
    toks = tokens(cfg, 620)
    want = O.forward(cfg, rig.w, toks)
    got = rig.run({"a": toks}, [[("a", 40)]] + [[("a", 1)]] * 580)["a"]
    assert logit_error(got, want) < LIMIT[F32]
    assert rig.dec.state_manager.pages_trimmed > 30
    # what the first tokens left is still there: other first tokens, other logits at the end
    other = [(t + 1) % cfg["vocab"] for t in toks[:20]] + toks[20:]
    assert logit_error(O.forward(cfg, rig.w, other)[-1:], want[-1:]) > 100 * LIMIT[F32]
    rig.close()


@pytest.mark.gpu
def test_pool_exhaustion_is_a_capacity_error():
    rig = Rig(CASES["odd"], BF16, context=320, pool=64)
    rig.eng.admit(0, {}, 0)
    with pytest.raises(OverflowError):
        rig.eng.step([[0, 0, 100, True]], tokens(CASES["odd"], 100))
    rig.eng.release(0)
    rig.eng.admit(0, {}, 64)
    assert len(rig.eng.step([[0, 0, 60, True]], tokens(CASES["odd"], 60))) == 1
    with pytest.raises(OverflowError):
        rig.eng.admit(1, {}, 80)                       # a reservation is all or nothing: five pages of a pool of four
    rig.close()


def _greedy(cfg, w, prompt, n):
    toks = list(prompt)
    margins = []
    for _ in range(n):
        l = O.forward(cfg, w, toks)[-1]
        top = l.topk(2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(l.argmax()))
    return toks[len(prompt):], margins


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [F32, BF16], ids=["f32", "bf16"])
def test_greedy_generation_through_the_engine(dtype):
    """Prefill and decode steps of the engine and of the single-sequence engine give the restatement's greedy continuation."""
    from ironpangu_b200.runtime.engine import DecodeEngine

    cfg = CASES["mixed"]
    rig = Rig(cfg, dtype, residents=2)
    for seed in range(20):                             # a prompt whose continuation has no near tie for some tokens
        prompt = tokens(cfg, 30, seed)
        want, margins = _greedy(cfg, rig.w, prompt, 12)
        clear = next((i for i, m in enumerate(margins) if m < (1e-3 if dtype == F32 else 0.2)), 12)
        if clear >= 5:
            break
    rig.eng.admit(0, {}, 42)
    rig.eng.admit(1, {}, 42)
    got = [rig.eng.step([[0, 0, 30, True]], prompt)[0]]
    rig.eng.step([[1, 0, 7, True]], prompt[:7])
    for i in range(11):
        got.append(rig.eng.step([[0, 30 + i, 1, True], [1, 7 + i, 1, True]], [got[-1], 3])[0])
    assert clear >= 5 and got[:clear] == want[:clear]
    rig.eng.release(0)
    rig.eng.release(1)
    single = DecodeEngine(rig.dec, prefill=rig.eng.prefill)
    out = single.generate(prompt, 12)
    assert out[:clear] == want[:clear]
    single.reset()                                     # the same on the device alone: every sampled token fed back without the host
    first = single.prefill(prompt)
    single.run_device_loop(first, clear - 1)
    assert int(rig.dec.next_ids[0]) == want[clear - 1] and single.pos == 30 + clear - 1
    rig.close()


@pytest.mark.gpu
def test_generation_through_the_server(tmp_path):
    """A checkpoint directory behind ifab-server: the worker picks the family by config.json; greedy tokens of concurrent requests equal
    the restatement's; seeded sampling repeats."""
    import threading

    from ironpangu_b200.models import falinex as F
    from test_server import Server

    cfg = dict(CASES["mixed"], vocab=300)
    w = weights(cfg)
    F.save_checkpoint(tmp_path / "ck", F.FalinexConfig.from_dict(cfg), w)
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
    from ironpangu_b200.models import falinex as F

    cfg = CASES["odd"]
    w = weights(cfg)
    F.save_checkpoint(tmp_path / "ck", F.FalinexConfig.from_dict(cfg), w)
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
    r = subprocess.run([sys.executable, "-m", "ironpangu_b200.runtime.engine_worker", "--model", "falinex-tiny", "--max-num-seqs", "2", "--max-model-len", "128",
                        "--kv-pool-tokens", "128", "--prefill-chunk", "64", "--memory-profile", str(path), "--profile-only"], capture_output=True, text=True,
                       timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(path.read_text())["failed_stage"] is None
