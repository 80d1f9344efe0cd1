"""Radivik through the engine: whole prompts, token by token, portions, mixed batches, pages used again, long decoding,
greedy generation, the command line and the trace replay, against the plain implementation."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import radivik as R
from tests import radivik_helpers as H

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]

CONFIGS = {
    "small": H.small(),
    "sharp": H.small(scale=0.9),
    "many_heads": H.config([H.layer(heads=18, kv_heads=1, dim=32, vdim=16, rot_dims=32, experts=9, top=4), H.layer(kv_from=0, heads=2, kv_heads=1,
                            dim=32, vdim=16, rot_dims=32)], vocab=130, width=80),
    "odd": H.config([H.layer(heads=2, kv_heads=1, dim=10, vdim=7, rot_dims=4, ff=9, experts=3, top=1)], vocab=51, width=30, alpha=1.0),
    "wide_heads": H.config([H.layer(heads=2, kv_heads=1, dim=160, vdim=136, rot_dims=64, scaling=H.YARN)], width=128),
    "one_expert": H.config([H.layer(heads=4, kv_heads=4, dim=128, vdim=128, rot_dims=128, experts=1, top=1, ff=136)], width=256),
}


def prompt(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def far_prompt(n, vocab, seed=0):
    """A token rare in the middle comes back at the end and around page and block borders."""
    p = np.random.default_rng(seed).integers(8, vocab, n)
    for at in (0, 1, 15, 16, 63, 64, n // 2, n - 2, n - 1):
        if at < n:
            p[at] = at % 5
    p[-4:] = [0, 1, 3, 4]
    return p.tolist()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_prompts_portions_and_decoding(name, dtype):
    cfg = CONFIGS[name]
    w = H.weights(cfg, 1, match=name != "small")
    eng = H.engine(H.model(cfg, w, dtype), page_size=64 if name == "sharp" else 16)
    tokens = H.settle(cfg, w, far_prompt(150, cfg["vocab"], 2))
    want = H.oracle_logits(cfg, w, tokens)
    for cuts in ([], range(1, 150), [2, 4, 7, 64, 65, 130, 132], [17, 80, 96, 128, 129], [149]):
        assert H.error(H.feed(eng, tokens, cuts), want).max() < H.TOLERANCE[dtype], cuts
    H.status_clear()


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_after_every_layer(dtype):
    cfg = CONFIGS["small"]
    w = H.weights(cfg, 3)
    eng = H.engine(H.model(cfg, w, dtype))
    tokens = H.settle(cfg, w, prompt(23, cfg["vocab"]))
    want = R.forward(cfg, w, tokens)[1]
    r = eng.open_replay()
    r.pages = [eng.pool.free.pop() for _ in range(2)]
    from inference_engine_b200.engine import Step

    with torch.inference_mode():
        eng.fill_mixed(Step([(r, tokens)], 0), 23)
        inp, _ = eng.mixed_views(23)
        trace = []
        eng.model.step(eng.caches, inp, inp.ids, inp.cached_lens, inp.block_table, inp.num_decoding, trace=trace)
    got = torch.stack(trace).cpu().numpy()
    assert np.abs(got - want).max() < (2e-5 if dtype == torch.float32 else 0.15)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_against_each_alone(dtype):
    """Unequal requests in one step, decoding and prompt portions mixed, with graphs: as each request alone."""
    cfg = CONFIGS["sharp"]
    w = H.weights(cfg, 4, match=True)
    m = H.model(cfg, w, dtype)
    eng = H.engine(m, graphs=True)
    reqs = [H.settle(cfg, w, far_prompt(n, cfg["vocab"], n)) for n in (97, 33, 64, 5)]
    want = [H.oracle_logits(cfg, w, p) for p in reqs]
    live, at, got = [eng.open_replay() for _ in reqs], [0] * 4, [[] for _ in reqs]
    plan = [[60, 3, 0, 0], [2, 1, 64, 0], [1, 1, 0, 5], [1, 20, 0, 0], [33, 8, 0, 0]]
    for step in plan:
        entries = [(live[i], reqs[i][at[i] : at[i] + n], list(range(n))) for i, n in enumerate(step) if n]
        logits, o = eng.replay(entries).numpy(), 0
        for i, n in enumerate(step):
            got[i].append(logits[o : o + n])
            o += n
            at[i] += n
    for i in range(4):
        assert H.error(np.concatenate(got[i]), want[i]).max() < H.TOLERANCE[dtype], i
        eng.close_replay(live[i])
    assert eng.pool.uncommitted() == eng.pool.capacity and eng.pool.committed == 0
    H.status_clear()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_freed_and_used_again(dtype):
    """A small pool, requests one after the other; what a finished request left behind is poisoned first."""
    cfg = CONFIGS["small"]
    w = H.weights(cfg, 5)
    eng = H.engine(H.model(cfg, w, dtype), num_pages=32 + 12, max_len=192)
    for seed, n in enumerate((150, 40, 191, 3, 100)):
        tokens = H.settle(cfg, w, prompt(n, cfg["vocab"], seed))
        got = H.feed(eng, tokens, sorted({max(1, c) for c in (n // 3, n // 3 + 2, n - 5, n - 4, n - 3)}))
        assert H.error(got, H.oracle_logits(cfg, w, tokens)).max() < H.TOLERANCE[dtype]
        for c in eng.caches:
            if c is not None:
                c.k[..., : c.k_dim] = float("nan")
                c.v[..., : c.v_dim] = float("nan")


def test_layers_on_another_layers_cache_hold_none():
    cfg = CONFIGS["small"]
    m = H.model(cfg, H.weights(cfg), torch.bfloat16)
    caches = m.make_caches(4, 16, 64)
    assert caches[0] is not None and caches[1] is None and caches[2] is not None
    assert m.layers[1].qkv.shape[0] == 6 * 48


def test_long_decoding_with_graphs():
    cfg = CONFIGS["sharp"]
    w = H.weights(cfg, 6, match=True)
    tokens = H.settle(cfg, w, far_prompt(420, cfg["vocab"], 9))
    want = H.oracle_logits(cfg, w, tokens)
    for dtype in DTYPES:
        eng = H.engine(H.model(cfg, w, dtype), graphs=True, max_len=448)
        got = H.feed(eng, tokens, [7] + list(range(8, 420)))
        assert eng.steps_run["decode_graph"] == 413
        assert H.error(got, want).max() < H.TOLERANCE[dtype]


def greedy(cfg, w, p, n, forced):
    """The plain implementation's logits behind each generated token, for the tokens the engine chose."""
    logits = H.oracle_logits(cfg, w, p + forced)
    return logits[len(p) - 1 : len(p) - 1 + n]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_scheduler(dtype, graphs):
    cfg = CONFIGS["small"]
    w = H.weights(cfg, 7)
    m = H.model(cfg, w, dtype)
    eng = H.engine(m, graphs=graphs, max_batch=3, max_len=128, max_tokens_per_step=40, min_first_chunk=8)
    prompts = [prompt(n, cfg["vocab"], n) for n in (60, 3, 1, 35, 17)]
    reqs = eng.generate(prompts, 9)
    assert eng.pool.uncommitted() == eng.pool.capacity
    flips = 0
    for p, r in zip(prompts, reqs):
        assert len(r.output) == 9
        logits = greedy(cfg, w, p, 9, r.output[:-1])
        for row, tok in zip(logits, r.output):
            if int(row.argmax()) != tok:
                flips += 1
                assert row.max() - row[tok] < (1e-4 if dtype == torch.float32 else 0.2) * row.std()
    assert flips <= (0 if dtype == torch.float32 else 4)
    H.status_clear()


def save(cfg, w, folder):
    from inference_engine_b200.checkpoint import write_safetensors

    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {k: torch.tensor(v).to(torch.bfloat16) for k, v in w.items()})


def test_command_line_and_trace_replay(tmp_path):
    cfg = CONFIGS["small"]
    w = H.weights(cfg, 8)
    save(cfg, w, tmp_path)
    p = prompt(21, cfg["vocab"], 3)
    out = subprocess.run([sys.executable, "-m", "inference_engine_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt",
                          " ".join(map(str, p)), "--max-new-tokens", "5"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert out.returncode == 0, out.stderr
    toks = json.loads(out.stdout.splitlines()[-1])["output"]
    rows = greedy(cfg, w, p, 5, toks[:-1])
    assert [int(r.argmax()) for r in rows] == toks

    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p[9:11], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": p[11:12], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": p, "want": [20]}], "end": ["b"]}]
    res = tmp_path / "out"
    res.mkdir()
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(res),
                          "--max-tokens", "32"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {n}" for n in range(4)]
    assert sorted(os.listdir(res)) == ["0.f32", "2.f32", "3.f32"]
    want = H.oracle_logits(cfg, w, p)
    for n, at in ((0, [0, 8]), (2, [11]), (3, [20])):
        got = np.fromfile(res / f"{n}.f32", "<f4").reshape(len(at), cfg["vocab"])
        assert H.error(got, want[at]).max() < H.TOLERANCE[torch.float32]


def test_chained_launches_change_nothing():
    """Kernels brought up while their predecessor runs: the same bits, prompts and decoding, with and without."""
    from inference_engine_b200 import kernels as K

    for cfg in (CONFIGS["one_expert"], CONFIGS["many_heads"], H.config([H.layer(experts=16, top=3, ff=72)] * 3, width=192)):
        w = H.weights(cfg, 11)
        m = H.model(cfg, w, torch.bfloat16)
        tokens = prompt(420, cfg["vocab"], 5)
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
