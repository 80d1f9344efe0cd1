"""Host side of the Biranex decoder: configuration, registry, state slots, the oracle's mechanisms on cases with known
answers.  No GPU."""
import copy
import ctypes

import numpy as np
import pytest

from oracle import biranex as B
from tests import biranex_helpers as H


def test_registry_and_configuration():
    from inference_engine_b200.models import load_all
    from inference_engine_b200.models.biranex import BiranexConfig, DeltaConfig

    assert "Biranex" in load_all()
    c = BiranexConfig.from_dict(H.CONFIGS["small"])
    assert [l.ff for l in c.layers] == [40, 0, 0, 24] and isinstance(c.layers[1].mixer, DeltaConfig)
    left, right = c.layers[0].mixer.left, c.layers[0].mixer.right
    assert (left.window, left.rotary.stretch, left.rotary.dims) == (37, 3.0, 16) and (right.groups, right.norm_groups) == (2, 4)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="something else"),
    lambda c: c["layers"][1]["mixer"].update(heads=5),
    lambda c: c["layers"][0]["mixer"]["left"].update(heads=5),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=-4),
    lambda c: c["layers"][0]["mixer"]["right"].update(groups=4),
    lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5),
    lambda c: c["layers"][0]["mlp"].update(kind="moe"),
])
def test_configurations_that_are_refused(change):
    from inference_engine_b200.models.biranex import BiranexConfig

    c = copy.deepcopy(H.CONFIGS["small"])
    change(c)
    with pytest.raises(ValueError):
        BiranexConfig.from_dict(c)


def test_linear_scaling_of_the_frequencies():
    from inference_engine_b200.ops import Rotary

    f, mult = Rotary(12, 500.0, stretch=2.5).frequencies()
    assert np.allclose(f, [500.0 ** (-2 * i / 12) / 2.5 for i in range(6)], rtol=1e-13) and mult == 1.0
    x = np.random.default_rng(0).standard_normal((5, 1, 14))
    y = B.rotate_interleaved(x, range(5), {"dims": 12, "base": 500.0, "scaling": {"factor": 2.5}})
    t = Rotary(12, 500.0, stretch=2.5).table(5, "cpu").numpy()
    assert np.allclose(y[..., 0:12:2][:, 0], x[:, 0, 0:12:2] * t[..., 0] - x[:, 0, 1:12:2] * t[..., 1], atol=1e-6)
    assert np.array_equal(y[..., 12:], x[..., 12:])


def test_oracle_known_answers():
    # a quarter turn mixes neighbours: (u, v) -> (u cos - v sin, v cos + u sin)
    y = B.rotate_interleaved(np.array([[[1.0, 2.0, 5.0]]] * 2), [0, 1], {"dims": 2, "base": 7.0})
    assert np.allclose(y[0, 0], [1, 2, 5]) and np.allclose(y[1, 0], [np.cos(1) - 2 * np.sin(1), 2 * np.cos(1) + np.sin(1), 5])
    # equal scores: the mean of the visible values, the sink taking its share
    k, v = np.zeros((5, 1, 2)), np.arange(5.0).reshape(5, 1, 1)
    q = np.ones((5, 1, 2))
    assert np.allclose(B.window_attention(q, k, v, 1.0, 2)[:, 0, 0], [0, 0.5, 1.5, 2.5, 3.5])
    assert np.allclose(B.window_attention(q, k, v, 1.0, 0, np.array([np.log(2.0)]))[:, 0, 0], [0, 1 / 4, 3 / 5, 6 / 6, 10 / 7])
    # convolution: last column is the current token
    x = np.array([[1.0], [10.0], [100.0]])
    assert np.allclose(B.causal_conv(x, np.array([[2.0, 3.0]]), np.array([0.5]))[:, 0], [3.5, 32.5, 320.5])
    # state space: one channel, no decay (a -> 0) adds up dt b x
    one = np.ones((3, 1, 1))
    s = B.state_space_scan(one, one, one, np.ones((3, 1)), np.array([-60.0]), np.array([0.25]))
    assert np.allclose(s[:, 0, 0], [1.25, 2.25, 3.25])
    s = B.state_space_scan(one, one, one, np.full((3, 1), np.log(2.0)), np.array([0.0]), np.array([0.0]))
    assert np.allclose(s[:, 0, 0] / np.log(2.0), [1, 1.5, 1.75])
    # delta rule: writing the same key again replaces the value (beta 1) or moves half way (beta 1/2); other keys stay
    k = np.array([[[1.0, 0.0]], [[0.0, 1.0]], [[1.0, 0.0]], [[1.0, 0.0]]])
    v = np.array([5.0, 7.0, 9.0, 1.0]).reshape(4, 1, 1)
    o = B.delta_scan(k, k, v, np.array([[1.0], [1.0], [1.0], [0.5]]), np.ones((4, 1, 2)))
    assert np.allclose(o[:, 0, 0], [5, 7, 9, 5])
    # the decay acts on the rows of a key channel, before the correction
    g = np.ones((2, 1, 2))
    g[1, 0, 0] = 0.5
    o = B.delta_scan(k[[0, 0]], k[[0, 0]], v[[0, 0]] * 0 + 4.0, np.array([[1.0], [0.0]]), g)
    assert np.allclose(o[:, 0, 0], [4, 2])
    # the norm's parts are taken by themselves, the gate before it
    y = B.gated_group_norm(np.array([[1.0, 1.0, 30.0, 30.0]]), np.full((1, 4), 50.0), 2, np.ones(4), 0.0)
    assert np.allclose(y, 1.0)
    assert np.allclose(B.softplus(np.array([-800.0, 0.0, 800.0])), [0, np.log(2), 800])


def test_oracle_is_causal_and_prefix_stable():
    for name in ("small", "odd"):
        cfg = H.CONFIGS[name]
        w = H.weights(cfg, 2)
        p = H.prompt(40, cfg["vocab"])
        assert np.allclose(H.oracle_logits(cfg, w, p)[:17], H.oracle_logits(cfg, w, p[:17]), atol=1e-9)


@pytest.mark.parametrize("fault", ["window", "sink", "state", "conv", "rotation", "scale"])
def test_planted_mistakes_show(fault, monkeypatch):
    """The tests' weights are such that a mistake in any mechanism moves the logits by far more than the tolerances."""
    cfg = copy.deepcopy(H.CONFIGS["small"])
    w = H.weights(cfg, 1, match=1.5)
    p = H.far_prompt(100, cfg["vocab"], 2)
    want = H.oracle_logits(cfg, w, p)
    m = cfg["layers"][0]["mixer"]
    if fault == "window":
        m["left"]["mask"]["size"] += 1
    elif fault == "sink":
        w = {**w, "l0.mix.left.sink": w["l0.mix.left.sink"] * 0 - 1e4}
    elif fault == "state":
        real = B.delta_scan
        monkeypatch.setattr(B, "delta_scan", lambda *a: np.concatenate([real(*(x[:64] for x in a)), real(*(x[64:] for x in a))]))
    elif fault == "conv":
        real = B.causal_conv
        monkeypatch.setattr(B, "causal_conv", lambda x, *a: np.concatenate([real(x[:64], *a), real(x[64:], *a)]))
    elif fault == "rotation":
        m["left"]["rot"]["scaling"]["factor"] = 1.0
    else:
        m["right_scale"] = 1.0
    assert H.error(H.oracle_logits(cfg, w, p), want).max() > 0.08


def test_state_slots_follow_the_requests():
    from inference_engine_b200.engine import PagePool, Scheduler, SlotPool

    slots = SlotPool(2)
    s = Scheduler(3, 64, 16, PagePool(40), 64, 4, -1, slots)
    reqs = [s.submit([1] * 5, n) for n in (1, 3, 2)]
    step = s.plan()
    assert [r.slot for r, _ in step.entries] == [0, 1] and reqs[2].slot == -1  # no slot left: the third waits
    assert s.commit(step, [0, 0]) == [reqs[0]] and reqs[0].slot == -1
    step = s.plan()
    assert reqs[2].slot == 0 and reqs[1].slot == 1
    while not s.idle():
        s.commit(step, [0] * len(step.entries))
        step = s.plan()
    assert sorted(slots.free) == [0, 1]
    slots.take(), slots.take()
    with pytest.raises(RuntimeError):
        slots.take()


def test_invalid_arguments_launch_nothing():
    from inference_engine_b200 import _lib

    lib, fake, byref = _lib.load_decoder(), 0x10000, ctypes.byref  # an aligned address nobody dereferences
    rec = _lib.Recurrence(*[fake] * 7, 3, 4, 2, 8, 8, 3, 2, 64, 0, 16, 32, 0, 1, 0, 0.0, 1.0)
    inp, ent = _lib.RecurrenceIn(fake, fake, fake, 64, 4, 4), _lib.Entries(fake, fake, fake, fake, fake, fake, 3, 3)
    scan = lambda: lib.b200dec_recurrence_scan(byref(rec), byref(inp), fake, byref(ent), fake, None, None)  # noqa: E731
    rec.heads = 3  # no multiple of qk_heads
    assert scan() == -2
    rec.heads, rec.off_v = 4, 40  # v would end behind the channels
    assert scan() == -2
    rec.off_v, inp.beta = 32, None
    assert scan() == -1
    inp.beta, ent.slots = fake, None
    assert lib.b200dec_conv_rows(byref(rec), byref(inp), byref(ent), fake, None, None) == -1
    assert lib.b200dec_norm_add(fake, fake, 3, fake, 1.0, 1e-5, None, 2, 8, None) == -2
    assert lib.b200dec_gated_norm(fake, fake, 8, 1, 2, fake, 8, 1e-5, 1.0, fake, 8, 2, 8, 3, None) == -2
    cache, table = _lib.DecCache(fake, fake, 4, 2, 16, 40, 24, 40, 24, 2), _lib.Table(fake, 4, 4)
    rows, opt = _lib.DecRows(None, None, fake, fake, 3), _lib.AttnOptions(-1, None, None, 0, 1.0, 0)
    assert lib.b200dec_attn_rows_opt(fake, byref(cache), byref(table), byref(rows), 4, 1.0, byref(opt), fake, None, None) == -2
    opt.window, opt.out_stride = 4, 100  # rows of 4 * 24 at a stride that is no multiple of 8
    assert lib.b200dec_attn_rows_opt(fake, byref(cache), byref(table), byref(rows), 4, 1.0, byref(opt), fake, None, None) == -2
