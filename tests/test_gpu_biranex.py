"""Biranex through the engine: whole prompts, token by token, portions, mixed batches, pages and slots used again, long
decoding, greedy generation, the command line and the trace replay, against the plain implementation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import biranex as B
from tests import biranex_helpers as H

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", H.CONFIGS)
def test_prompts_portions_and_decoding(name, dtype):
    cfg = H.CONFIGS[name]
    w = H.weights(cfg, 1, match=1.5 if name in ("small", "wide") else 0.0)
    eng = H.engine(H.model(cfg, w, dtype), page_size=64 if name == "wide" else 16)
    tokens = H.far_prompt(150, cfg["vocab"], 2, 70 if name == "wide" else 37)
    want = H.oracle_logits(cfg, w, tokens)
    runs = [H.feed(eng, tokens, cuts) for cuts in ([], range(1, 150), [2, 4, 7, 64, 65, 130, 132], [17, 80, 96, 128, 129], [149])]
    H.check(cfg, w, tokens, runs, want, dtype)
    H.status_clear()


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_after_every_layer(dtype):
    from inference_engine_b200.engine import Step

    cfg = H.CONFIGS["small"]
    w = H.weights(cfg, 3)
    eng = H.engine(H.model(cfg, w, dtype))
    tokens = H.prompt(23, cfg["vocab"])
    want = B.forward(cfg, w, tokens)[1]
    r = eng.open_replay()
    r.pages, r.slot = [eng.pool.free.pop() for _ in range(2)], eng.slots.take()
    with torch.inference_mode():
        eng.fill_mixed(Step([(r, tokens)], 0), 23)
        inp, _ = eng.mixed_views(23)
        trace = []
        eng.model.step(eng.caches, inp, inp.ids, inp.cached_lens, inp.block_table, inp.num_decoding, slots=inp.slots, trace=trace)
    got = torch.stack(trace).cpu().numpy()
    assert np.abs(got - want).max() < (2e-5 if dtype == torch.float32 else 0.15)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_against_each_alone(dtype):
    """Unequal requests in one step, decoding and prompt portions mixed, with graphs: as each request alone."""
    cfg = H.CONFIGS["small"]
    w = H.weights(cfg, 4, match=1.5)
    eng = H.engine(H.model(cfg, w, dtype), graphs=True)
    reqs = [H.far_prompt(n, cfg["vocab"], n) for n in (97, 33, 64, 5)]
    want = [H.oracle_logits(cfg, w, p) for p in reqs]
    live, at, got = [eng.open_replay() for _ in reqs], [0] * 4, [[] for _ in reqs]
    for step in [[60, 3, 0, 0], [2, 1, 64, 0], [1, 1, 0, 5], [1, 20, 0, 0], [33, 8, 0, 0]]:
        entries = [(live[i], reqs[i][at[i] : at[i] + n], list(range(n))) for i, n in enumerate(step) if n]
        logits, o = eng.replay(entries).numpy(), 0
        for i, n in enumerate(step):
            got[i].append(logits[o : o + n])
            o += n
            at[i] += n
    for i in range(4):
        H.check(cfg, w, reqs[i], np.concatenate(got[i]), want[i], dtype)
        eng.close_replay(live[i])
    assert eng.pool.uncommitted() == eng.pool.capacity and eng.pool.committed == 0 and len(eng.slots.free) == eng.slots.capacity
    H.status_clear()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_freed_and_used_again(dtype):
    """A small pool, requests one after the other; what a finished request left behind is poisoned first."""
    cfg = H.CONFIGS["small"]
    w = H.weights(cfg, 5)
    eng = H.engine(H.model(cfg, w, dtype), num_pages=32 + 12, max_len=192, max_batch=2, num_slots=1)
    for seed, n in enumerate((150, 40, 191, 3, 1, 100)):
        tokens = H.prompt(n, cfg["vocab"], seed)
        got = H.feed(eng, tokens, sorted({max(1, c) for c in (n // 3, n // 3 + 2, n - 5, n - 4, n - 3)}))
        H.check(cfg, w, tokens, got, H.oracle_logits(cfg, w, tokens), dtype)
        for cache in eng.caches:
            kv, state = cache if isinstance(cache, tuple) else (None, cache)
            if kv is not None:
                kv.k[..., : kv.k_dim] = float("nan")
                kv.v[..., : kv.v_dim] = float("nan")
            state.state[..., :1] = float("nan")
            state.ring.fill_(float("nan"))


def test_long_decoding_with_graphs():
    cfg = H.CONFIGS["small"]
    w = H.weights(cfg, 6, match=1.5)
    tokens = H.far_prompt(420, cfg["vocab"], 9)
    want = H.oracle_logits(cfg, w, tokens)
    for dtype in DTYPES:
        eng = H.engine(H.model(cfg, w, dtype), graphs=True, max_len=448)
        got = H.feed(eng, tokens, [7] + list(range(8, 420)))
        assert eng.steps_run["decode_graph"] == 413
        H.check(cfg, w, tokens, got, want, dtype)


def greedy(cfg, w, p, n, forced):
    """The plain implementation's logits behind each generated token, for the tokens the engine chose."""
    return H.oracle_logits(cfg, w, p + forced)[len(p) - 1 : len(p) - 1 + n]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler(dtype, graphs):
    cfg = H.CONFIGS["small"]
    w = H.weights(cfg, 7)
    eng = H.engine(H.model(cfg, w, dtype), graphs=graphs, max_batch=3, max_len=128, max_tokens_per_step=40, min_first_chunk=8)
    prompts = [H.prompt(n, cfg["vocab"], n) for n in (60, 3, 1, 35, 17)]
    reqs = eng.generate(prompts, 9)
    assert eng.pool.uncommitted() == eng.pool.capacity and sorted(eng.slots.free) == [0, 1, 2]
    flips = 0
    for p, r in zip(prompts, reqs):
        assert len(r.output) == 9
        for row, tok in zip(greedy(cfg, w, p, 9, r.output[:-1]), r.output):
            if int(row.argmax()) != tok:
                flips += 1
                assert row.max() - row[tok] < (1e-4 if dtype == torch.float32 else 0.2) * row.std()
    assert flips <= (0 if dtype == torch.float32 else 4)
    H.status_clear()


def test_command_line_and_trace_replay(tmp_path):
    from inference_engine_b200.checkpoint import write_safetensors

    cfg = H.CONFIGS["odd"]
    w = H.weights(cfg, 8)
    with open(tmp_path / "config.json", "w") as f:
        json.dump(cfg, f)
    write_safetensors(str(tmp_path / "model.safetensors"), {k: torch.tensor(v).to(torch.bfloat16) for k, v in w.items()})
    p = H.prompt(21, cfg["vocab"], 3)
    out = subprocess.run([sys.executable, "-m", "inference_engine_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt",
                          " ".join(map(str, p)), "--max-new-tokens", "5"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    toks = json.loads(out.stdout.splitlines()[-1])["output"]
    assert [int(r.argmax()) for r in greedy(cfg, w, p, 5, toks[:-1])] == toks
    out = subprocess.run([sys.executable, "-m", "inference_engine_b200", "generate", "--model", str(tmp_path), "--random-weights", "--prompt",
                          "1 2 3"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0 and len(json.loads(out.stdout.splitlines()[-1])["output"]) == 16, out.stderr
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p[9:11], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": p[11:12], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": p, "want": [20]}], "end": ["b"]}]
    res = tmp_path / "out"
    res.mkdir()
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(res),
                          "--max-tokens", "32"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    want = H.oracle_logits(cfg, w, p)
    for n, at in ((0, [0, 8]), (2, [11]), (3, [20])):
        got = np.fromfile(res / f"{n}.f32", "<f4").reshape(len(at), cfg["vocab"])
        assert H.error(got, want[at]).max() < H.FP32_LIMIT


def test_chained_launches_change_nothing():
    """Kernels brought up while their predecessor runs: the same bits, prompts and decoding, with and without."""
    from inference_engine_b200 import kernels as K

    for name in ("wide", "small"):
        cfg = H.CONFIGS[name]
        m = H.model(cfg, H.weights(cfg, 11), torch.bfloat16)
        tokens = H.prompt(420, cfg["vocab"], 5)
        outs = []
        try:
            for chained in (False, True, True):
                K.set_early_start(chained)
                junk = torch.full((1 << 22,), -1, dtype=torch.int32, device="cuda")  # scratch memory starts as nonsense
                del junk
                outs.append(H.feed(H.engine(m), tokens, [380] + list(range(381, 420))))
        finally:
            K.set_early_start(False)
        assert np.array_equal(outs[0], outs[1]) and np.array_equal(outs[0], outs[2])
        H.status_clear()
