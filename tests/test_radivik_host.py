"""Host side of the Radivik decoder: configuration, registry, checkpoint files, the oracle's mechanisms on cases with known
answers, and the C ABI of libb200dec.so.  No GPU."""
import ctypes
import json
import os
import re

import numpy as np
import pytest
import torch

from oracle import radivik as R
from tests import radivik_helpers as H

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_registry_and_configuration():
    from inference_engine_b200.models import load_all, model_class
    from inference_engine_b200.models.radivik import RadivikConfig

    assert {"Radivik", "DecoderScaffold"} <= set(load_all())
    with pytest.raises(ValueError):
        model_class({"architecture": "nothing of the kind"})
    c = RadivikConfig.from_dict(H.small())
    assert [l.mixer.kv_from for l in c.layers] == [None, 0, None] and c.layers[2].mlp is None
    assert c.layers[0].mixer.rotary.scaling == (8.0, 64.0, 8.0, 1.0) and c.layers[2].mixer.rotary.scaling is None


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="something else"),
    lambda c: c["layers"][1]["mixer"].update(kv_from=2),        # not an earlier layer
    lambda c: c["layers"][2]["mixer"].update(kv_from=1),        # a layer without keys of its own
    lambda c: c["layers"][1]["mixer"].update(dim=32),           # other sizes than the cache it uses
    lambda c: c["layers"][0]["mixer"].update(heads=3),          # not a multiple of the key/value heads
    lambda c: c["layers"][0]["mlp"]["router"].update(top=9),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=15),
    lambda c: c["layers"][0]["mlp"].update(kind="dense"),
])
def test_configurations_that_are_refused(change):
    from inference_engine_b200.models.radivik import RadivikConfig

    c = H.small()
    change(c)
    with pytest.raises(ValueError):
        RadivikConfig.from_dict(c)


def test_rotary_frequencies_against_the_plain_ones():
    from inference_engine_b200.ops import Rotary

    for dims, base, sc in ((16, 1e4, H.YARN), (64, 5e5, {"factor": 2.0, "original": 4096, "fast": 32.0, "slow": 1.0}), (2, 100.0, None),
                           (24, 1e4, {"factor": 16.0, "original": 16, "fast": 500.0, "slow": 400.0})):
        r = Rotary(dims, base, None if sc is None else tuple(float(sc[k]) for k in ("factor", "original", "fast", "slow")))
        f, m = R.rotary_frequencies({"dims": dims, "base": base, "scaling": sc})
        assert np.allclose(r.frequencies()[0], f, rtol=1e-13) and r.frequencies()[1] == m
        t = r.table(9, "cpu").numpy()
        assert np.allclose(t[..., 0], np.cos(np.arange(9)[:, None] * f) * m, atol=1e-7)
        assert np.allclose(t[..., 1], np.sin(np.arange(9)[:, None] * f) * m, atol=1e-7)


def test_safetensors_round_trip(tmp_path):
    from inference_engine_b200.checkpoint import Weights, write_safetensors

    g = torch.Generator().manual_seed(0)
    data = {"a": torch.randn(3, 5, generator=g).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, generator=g),
            "d": torch.zeros(0, 4)}
    write_safetensors(str(tmp_path / "model.safetensors"), data)
    w = Weights.open(str(tmp_path))
    assert set(w.tensors) == set(data)
    for k, v in data.items():
        assert torch.equal(w.take(k, *v.shape), v)
    assert w.unused() == []
    with pytest.raises(ValueError):
        w.take("a", 5, 3)
    with pytest.raises(KeyError):
        w.take("nothing", 1)
    with pytest.raises(FileNotFoundError):
        Weights.open(os.path.join(str(tmp_path), ".."))


def test_oracle_known_answers():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(R.rms_norm(x, 0.0), x / np.sqrt(12.5))
    assert np.allclose(R.rms_norm(np.zeros((1, 2)), 1e-6), 0)
    # a quarter turn of a pair: (u, v) -> (-v, u); position 0 does not turn; the channels behind pass
    q = np.array([[[1.0, 2.0, 5.0]], [[1.0, 2.0, 5.0]]])
    rot = {"dims": 2, "base": 10.0}
    y = R.rotate(q, [0, 1], rot)
    assert np.allclose(y[0, 0], [1, 2, 5])
    assert np.allclose(y[1, 0], [np.cos(1) - 2 * np.sin(1), 2 * np.cos(1) + np.sin(1), 5])
    # equal scores: the mean of the visible values; a dominant key: its value; nothing behind the query counts
    k, v = np.zeros((4, 1, 2)), np.arange(4.0).reshape(4, 1, 1)
    assert np.allclose(R.causal_attention(np.ones((4, 2, 2)), k, v, 1.0)[:, 1, 0], [0, 0.5, 1, 1.5])
    k[2] = 50.0
    assert np.allclose(R.causal_attention(np.ones((4, 2, 2)), k, v, 1.0)[:, 0, 0], [0, 0.5, 2, 2])
    # expert: gate limited from above only, up from both sides
    w = {"gate": np.eye(1), "up": np.eye(1), "down": np.eye(1)}
    sig = lambda z: 1 / (1 + np.exp(-z))
    for h in (5.0, 0.5, -5.0):
        g, u = min(h, 2.0), np.clip(h, -2.0, 2.0)
        assert np.allclose(R.expert(np.array([[h]]), w, "", 2.0), g * sig(1.702 * g) * (u + 1))
    ids, s = R.route(np.array([[1.0]]), np.array([[0.0], [2.0], [1.0]]), 2)
    assert ids.tolist() == [[1, 2]] and np.allclose(s, sig(np.array([[2.0, 1.0]])))
    assert np.allclose(R.margin(np.array([[1.0]]), np.array([[0.0], [2.0], [1.0]]), 2), sig(1.0) - 0.5)


def test_oracle_is_causal_and_prefix_stable():
    cfg = H.small()
    w = H.weights(cfg, 2)
    p = np.random.default_rng(0).integers(0, cfg["vocab"], 40).tolist()
    full, part = H.oracle_logits(cfg, w, p), H.oracle_logits(cfg, w, p[:17])
    assert np.allclose(full[:17], part, atol=1e-10)


def test_library_exports_every_declared_symbol():
    from inference_engine_b200 import _lib, build

    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(ROOT, "include", "b200dec.h")).read(), flags=re.S)
    names = sorted(set(re.findall(r"\b(b200dec_[a-z0-9_]+)\s*\(", text)))
    lib = ctypes.CDLL(build.build_library(build.DECODER_LIB))
    assert names == sorted(_lib.DECODER_SIGNATURES)
    for name in names + list(_lib.SHARED_SIGNATURES):
        assert hasattr(lib, name)


def test_invalid_arguments_launch_nothing():
    from inference_engine_b200 import _lib

    lib = _lib.load_decoder()
    fake = 0x10000  # an aligned address nobody dereferences: validation comes first
    cache = _lib.DecCache(fake, fake, 4, 2, 16, 40, 24, 40, 24, 2)
    table, rows = _lib.Table(fake, 4, 4), _lib.DecRows(None, None, fake, fake, 3)
    byref = ctypes.byref
    assert lib.b200dec_attn_rows(None, byref(cache), byref(table), byref(rows), 4, 1.0, fake, None, None) == -1
    assert lib.b200dec_attn_rows(fake, byref(cache), byref(table), byref(rows), 3, 1.0, fake, None, None) == -2
    cache.k_row = 41
    assert lib.b200dec_attn_rows(fake, byref(cache), byref(table), byref(rows), 4, 1.0, fake, None, None) == -2
    cache.k_row = 40
    ws = lib.b200dec_decode_attn_workspace(3, 4, 2, 24, 148)
    assert ws > 0 and ws % 4 == 0
    args = [fake, byref(cache), byref(table), fake, fake, 3, 4, 1.0, fake, 1, fake, ws, 148, None, None]
    assert lib.b200dec_decode_attn(*args[:11], ws - 4, *args[12:]) == -4
    cache.page_size = 24
    assert lib.b200dec_decode_attn(*args) == -2
    assert lib.b200dec_router(fake, fake, 3, 64, 4, 5, fake, fake, fake, fake, None) == -2
    assert lib.b200dec_grouped_linear(fake, fake, 2, fake, 3, 64, 9, 4, 10, 36, None, 1, 1.0, 1.0, fake, 148, 0, None, None) == -1
    assert lib.b200dec_grouped_linear(fake, fake, 2, fake, 3, 64, 9, 4, 10, 36, fake, 1, 1.0, 1.0, fake, 148, 0, None, None) == -2


def test_ops_refuse_cpu_tensors():
    from inference_engine_b200 import ops

    with pytest.raises(RuntimeError):
        ops.embed(torch.zeros(3, 4), torch.zeros(2, dtype=torch.int32))


def test_replay_bookkeeping_without_a_device():
    """Order of entries, pages and wanted rows of the engine's replay, with a stand-in for the device step."""
    from inference_engine_b200 import engine as E

    class Model:
        vocab = 10

        def logits(self, hidden):
            return hidden

    eng = E.Engine.__new__(E.Engine)
    eng.torch, eng.model, eng.page_size, eng.max_len, eng.device, eng.rows = torch, Model(), 4, 32, "cpu", {}
    eng.pool = E.PagePool(9, first=1)
    eng.sched = type("S", (), {"next_id": 0})()
    seen = []

    def run(step):
        seen.append(([len(t) for _, t in step.entries], step.num_decoding))
        flat = [t for _, toks in step.entries for t in toks]
        return type("O", (), {"hidden": torch.tensor(flat, dtype=torch.float32)[:, None]})()

    eng.run = run
    a, b = eng.open_replay(), eng.open_replay()
    assert eng.replay([(a, [1, 2, 3], [2, 0])]).flatten().tolist() == [3, 1]
    # b's first token is a prompt portion, a's single one decodes and moves to the front
    assert eng.replay([(b, [7], [0]), (a, [4], [0])]).flatten().tolist() == [7, 4]
    assert seen == [([3], 0), ([1, 1], 1)]
    assert eng.replay([(a, [5, 6], [])]).shape[0] == 0
    assert len(a.pages) == 2 and a.cached_len == 6
    with pytest.raises(ValueError):
        eng.replay([(b, [11], [])])
    with pytest.raises(ValueError):
        eng.replay([(b, [1] * 40, [])])
    eng.close_replay(a)
    eng.close_replay(b)
    assert eng.pool.uncommitted() == eng.pool.capacity


def test_command_line_lists_models(capsys):
    from inference_engine_b200.__main__ import main, read_prompts

    assert main(["models"]) == 0
    assert "Radivik" in capsys.readouterr().out.split()
    assert read_prompts(["1 2,3"]) == [[1, 2, 3]]


def test_trace_reader_feeds_the_engine(tmp_path):
    from inference_engine_b200 import trace

    class Eng:
        class K:
            @staticmethod
            def check_status(dev):
                return 0

        device, opened, closed = None, 0, 0

        def open_replay(self):
            self.opened += 1
            return self.opened

        def close_replay(self, r):
            self.closed += 1

        def replay(self, entries):
            return torch.tensor([[float(t[w])] * 2 for _, t, want in entries for w in want]).reshape(-1, 2)

    eng, done = Eng(), []
    lines = [json.dumps(x) for x in ({"step": 0, "entries": [{"id": "x", "tokens": [4, 5], "want": [1]}], "end": []},
                                     {"step": 1, "entries": [{"id": "x", "tokens": [6], "want": []}], "end": ["x"]})]
    trace.run(eng, lines, str(tmp_path), done.append)
    assert done == [0, 1] and os.listdir(tmp_path) == ["0.f32"] and (eng.opened, eng.closed) == (1, 1)
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [5.0, 5.0]
