"""Every mechanism of the Biranex layers alone, on the GPU, against oracle/biranex.py."""
import numpy as np
import pytest
import torch

from oracle import biranex as B
from tests.biranex_helpers import status_clear

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
DEV = "cuda"


def rnd(g, *shape, dtype=torch.float32, gain=1.0):
    return (torch.from_numpy(g.standard_normal(shape)) * gain).to(DEV, dtype)


def np64(t):
    return t.double().cpu().numpy()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, want, dtype, f32=2e-5, b16=2e-2):
    got, tol = np64(got) if torch.is_tensor(got) else got, f32 if dtype == torch.float32 else b16
    assert np.abs(got - want).max() <= tol * max(1.0, np.abs(want).max()), np.abs(got - want).max()


def step_rows(cached, chunks, nd, page=16, seed=0, slots=None):
    """Rows of a step: entry e brings chunks[e] tokens behind cached[e]; the first nd decode.  Pages in random order."""
    from inference_engine_b200 import ops
    from inference_engine_b200 import scaffold as S

    n, E = sum(chunks), len(chunks)
    plan = S.plan_step(cached[:nd], list(zip(cached[nd:], chunks[nd:])), n, E + 1)
    per = max(1, max(-(-(c + k) // page) for c, k in zip(cached, chunks)))
    order = np.random.default_rng(seed).permutation(E * per)
    table = torch.zeros(E + 1, per, dtype=torch.int32, device=DEV)
    table[:E] = i32(order.reshape(E, per).tolist())
    slots = list(range(E)) if slots is None else slots
    if nd == E:
        return ops.Rows(E, i32(cached), i32([nd]), table[:E], slots=i32(slots)), E * per
    return ops.Rows(n, i32(plan["cached"]), i32(plan["num_decoding"]), table, i32(plan["seq_ids"]), i32(plan["positions"]),
                    i32(plan["cu_seqlens"]), i32(plan["tile_start"]), 128, slots=i32(slots + [-1])), E * per


# ------------------------------------------------------------------ row ops
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width", [(1, 4), (7, 30), (5, 96), (3, 2048), (2, 6400), (2, 9000)])
def test_norm_add(rows, width, dtype):
    from inference_engine_b200 import ops

    g = np.random.default_rng(width)
    x, y, w = rnd(g, rows, width), rnd(g, rows, width, dtype=dtype, gain=3.0), rnd(g, width)
    want = np64(x) + 0.37 * B.rms_norm(np64(y), 1e-5, np64(w))
    xb = ops.norm_add(x, y, w, 0.37, 1e-5, dtype)
    close(x, want, torch.float32, f32=3e-6)
    assert xb.dtype == dtype and torch.equal(xb, x.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,ff", [(3, 9), (2, 40), (65, 1536)])
def test_silu_mul(rows, ff, dtype):
    from inference_engine_b200 import ops

    x = rnd(np.random.default_rng(ff), rows, 2 * ff, dtype=dtype, gain=4.0)
    a = np64(x)
    close(ops.silu_mul(x, ff), B.silu(a[:, :ff]) * a[:, ff:], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,parts,part", [(3, 7, 3), (2, 1, 130), (5, 4, 64), (2, 2, 200), (3, 1, 1536), (2, 2, 4096), (2, 1, 5000)])
def test_gated_norm_before_and_after(rows, parts, part, dtype):
    from inference_engine_b200 import ops

    g = np.random.default_rng(part)
    n = parts * part
    o, wide = rnd(g, rows, n, gain=2.0), rnd(g, rows, n + 8, dtype=dtype, gain=3.0)
    gate, out = wide[:, 8:], torch.empty(rows, n + 24, dtype=dtype, device=DEV)
    w = rnd(g, n)
    ops.gated_norm(o, gate, ops.GatedNorm(w, parts, 1e-5, True, 1.7), out[:, 16 : 16 + n])
    close(out[:, 16 : 16 + n], 1.7 * B.gated_group_norm(np64(o), np64(gate), parts, np64(w), 1e-5), dtype)
    w = rnd(g, part)  # shared by the parts
    ops.gated_norm(o, gate, ops.GatedNorm(w, parts, 1e-5, False), out[:, :n])
    want = B.rms_norm(np64(o).reshape(rows, parts, part), 1e-5, np64(w)).reshape(rows, n) * B.sigmoid(np64(gate))
    close(out[:, :n], want, dtype)


# ------------------------------------------------------------------ norm of whole projections, rotation, cache write
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim,dims", [(4, 2, 64, 48, 64), (6, 3, 24, 40, 8), (3, 1, 9, 7, 4), (2, 2, 160, 136, 0)])
def test_norm_rotation_and_write(heads, kv, dim, vdim, dims, dtype):
    from inference_engine_b200 import ops

    g = np.random.default_rng(dim)
    rows, pages = step_rows([33, 5, 0], [1, 20, 9], 1)
    n = rows.num_rows
    cache = ops.make_paged_kv(pages, kv, 16, dim, vdim, dtype, DEV)
    wide = rnd(g, n, heads * dim + kv * (dim + vdim) + 8, dtype=dtype, gain=2.0)
    qkv = wide[:, : wide.shape[1] - 8]
    qn, kn = rnd(g, heads * dim), rnd(g, kv * dim)
    rot = {"dims": dims, "base": 300.0, "scaling": {"factor": 1.5}}
    table = ops.Rotary(dims, 300.0, stretch=1.5).table(64, DEV) if dims else None
    q = ops.norm_rope_write(qkv, rows, cache, qn, kn, 1e-5, table, heads)
    a, pos = np64(qkv), np64(rows.positions)
    want_q = B.rotate_interleaved(B.rms_norm(a[:, : heads * dim], 1e-5, np64(qn)).reshape(n, heads, dim), pos, rot)
    want_k = B.rotate_interleaved(B.rms_norm(a[:, heads * dim : (heads + kv) * dim], 1e-5, np64(kn)).reshape(n, kv, dim), pos, rot)
    close(q[..., :dim], want_q, dtype)
    assert (q[..., dim:] == 0).all()
    for r in range(n):
        p = int(pos[r])
        page = int(rows.block_table[int(rows.seq_ids[r]), p // 16])
        close(cache.k[page, :, p % 16, :dim], want_k[r], dtype)
        assert torch.equal(cache.v[page, :, p % 16, :vdim].reshape(-1), qkv[r, (heads + kv) * dim :])
    status_clear()


# ------------------------------------------------------------------ attention: window, sink, gate
def attention_case(g, dtype, cached, chunks, nd, heads, kv, dim, vdim, page):
    """Random keys and values of whole sequences in a cache, and the queries of a step's rows."""
    from inference_engine_b200 import ops

    rows, pages = step_rows(cached, chunks, nd, page)
    cache = ops.make_paged_kv(pages, kv, page, dim, vdim, dtype, DEV)
    cache.k.fill_(float("nan"))  # nothing behind a sequence may count
    cache.v.fill_(float("nan"))
    keys, values = [], []
    for e, (c, n) in enumerate(zip(cached, chunks)):
        k, v = rnd(g, c + n, kv, dim, dtype=dtype), rnd(g, c + n, kv, vdim, dtype=dtype)
        for p in range(c + n):
            at = int(rows.block_table[e, p // page])
            cache.k[at, :, p % page] = 0
            cache.v[at, :, p % page] = 0
            cache.k[at, :, p % page, :dim] = k[p]
            cache.v[at, :, p % page, :vdim] = v[p]
        keys.append(k)
        values.append(v)
    q = torch.zeros(rows.num_rows, heads, cache.k.shape[3], dtype=dtype, device=DEV)
    q[..., :dim] = rnd(g, rows.num_rows, heads, dim, dtype=dtype)
    return rows, cache, q, keys, values


def attention_want(rows, cached, chunks, q, keys, values, dim, scale, window, sink, gate, out_scale):
    out, at = [], 0
    for e, (c, n) in enumerate(zip(cached, chunks)):
        full = np.zeros((c + n, q.shape[1], dim))
        full[c:] = np64(q[at : at + n, :, :dim])
        o = B.window_attention(full, np64(keys[e]), np64(values[e]), scale, window, None if sink is None else np64(sink))[c:]
        out.append(o)
        at += n
    o = np.concatenate(out) * out_scale
    return o if gate is None else o * B.sigmoid(np64(gate))[..., None]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 64, 64), (18, 1, 128, 40), (6, 3, 24, 128), (3, 1, 10, 7), (2, 1, 160, 136)])
@pytest.mark.parametrize("window", [0, 1, 5, 64, 77, 130])
def test_window_sink_and_gate(heads, kv, dim, vdim, window, dtype):
    from inference_engine_b200 import ops

    g = np.random.default_rng(window + dim)
    for cached, chunks, nd, page in (([200, 64, 63, 3, 0], [1, 1, 1, 1, 1], 5, 64), ([130, 0, 100, 7], [1, 150, 70, 2], 1, 16)):
        rows, cache, q, keys, values = attention_case(g, dtype, cached, chunks, nd, heads, kv, dim, vdim, page)
        n = rows.num_rows
        sink, gate = rnd(g, heads, gain=2.0), rnd(g, n, heads + 3, dtype=dtype, gain=2.0)[:, 2 : 2 + heads]
        wide = torch.full((n, (heads * vdim + 7) // 8 * 8 + 16), 7.0, dtype=dtype, device=DEV)
        out = wide[:, : heads * vdim].unflatten(1, (heads, vdim))
        ops.paged_attention(q, cache, rows, dim ** -0.5, ops.AttnOptions(window, sink, gate, 1.3), out)
        want = attention_want(rows, cached, chunks, q, keys, values, dim, dim ** -0.5, window, sink, gate, 1.3)
        close(out, want, dtype)
        assert (wide[:, heads * vdim :] == 7.0).all()
        o = ops.paged_attention(q, cache, rows, dim ** -0.5, ops.AttnOptions(window))
        close(o, attention_want(rows, cached, chunks, q, keys, values, dim, dim ** -0.5, window, None, None, 1.0), dtype)
    status_clear()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [63, 64, 65, 100, 136])
def test_a_key_at_the_windows_edge(window, dtype):
    """One key outweighs all others by e^20; the queries a window later see it or do not, in prompts and decoding, and a sink
    as strong takes half."""
    from inference_engine_b200 import ops

    g = np.random.default_rng(1)
    T, dim = 260, 64
    for at in (0, 15, 16, 63, 64, 100):
        for cached, n in ((0, T), (at + window - 1, 2), (at + window - 2, 1), (at + window - 1, 1), (at + window, 1)):
            nd = 1 if n == 1 and cached else 0
            rows, cache, q, keys, values = attention_case(g, dtype, [cached], [n], nd, 2, 1, dim, 64, 16)
            q[..., :dim] = 1.0
            if at < cached + n:
                keys[0][at] = 20.0 / dim
                cache.k[int(rows.block_table[0, at // 16]), :, at % 16, :dim] = 20.0 / dim
            for k in range(cached + n):
                if k != at:
                    keys[0][k] = 0.0
                    cache.k[int(rows.block_table[0, k // 16]), :, k % 16, :dim] = 0.0
            sink = torch.tensor([20.0, -50.0], device=DEV)
            out = ops.paged_attention(q, cache, rows, 1.0, ops.AttnOptions(window, sink))
            close(out, attention_want(rows, [cached], [n], q, keys, values, dim, 1.0, window, sink, None, 1.0), dtype)
    status_clear()


# ------------------------------------------------------------------ recurrent layers
def make_rec(g, kind, heads, groups, dim, vdim, taps, strong=False):
    from inference_engine_b200 import ops

    qk, v = groups * dim, heads * vdim
    conv = rnd(g, taps, 2 * qk + v)
    a_log = rnd(g, heads, gain=1.5) + (3.0 if strong else -1.5)
    if kind == "delta":
        rec = ops.Recurrence(heads, groups, dim, vdim, conv, None, -a_log.exp(), rnd(g, heads * dim), None, 0, qk, 2 * qk, True, True, 1e-6,
                             dim ** -0.5)
    else:
        rec = ops.Recurrence(heads, groups, dim, vdim, conv, rnd(g, 2 * qk + v, gain=0.5), -a_log.exp(), rnd(g, heads), rnd(g, heads), v + qk, v, 0)
    return rec, np64(a_log)


def rec_inputs(g, rec, n, dtype):
    wide = rnd(g, n, rec.channels + 16, dtype=dtype)
    step = rnd(g, n, rec.dt_bias.numel() + 5, dtype=dtype)[:, : rec.dt_bias.numel()]
    beta = rnd(g, n, rec.heads, dtype=dtype) if rec.correct else None
    return wide[:, 8 : 8 + rec.channels], step, beta


def rec_want(rec, a_log, x, step, beta):
    """o [T, heads, vdim] of one whole sequence."""
    T, H, G, D, P = len(x), rec.heads, rec.qk_heads, rec.dim, rec.vdim
    c = B.silu(B.causal_conv(np64(x), np64(rec.conv_w).T, None if rec.conv_b is None else np64(rec.conv_b)))
    q, k = c[:, rec.off_q : rec.off_q + G * D].reshape(T, G, D), c[:, rec.off_k : rec.off_k + G * D].reshape(T, G, D)
    v = c[:, rec.off_v : rec.off_v + H * P].reshape(T, H, P)
    dt = B.softplus(np64(step) + np64(rec.dt_bias))
    if not rec.correct:
        return B.state_space_scan(v, k, q, dt, a_log, np64(rec.skip))
    decay = np.exp(-np.exp(a_log)[:, None] * dt.reshape(T, H, D))
    return B.delta_scan(B.unit(q) * D ** -0.5, B.unit(k), v, B.sigmoid(np64(beta)), decay)


KINDS = ["delta", "state_space"]
SIZES = [(4, 4, 32, 32, 4), (4, 2, 40, 24, 3), (2, 2, 8, 72, 4), (6, 3, 20, 28, 3), (2, 1, 128, 128, 4), (3, 1, 9, 7, 5), (1, 1, 64, 48, 1), (2, 2, 144, 264, 2), (2, 1, 260, 40, 3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,groups,dim,vdim,taps", SIZES)
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("form", [None, "scan"])
def test_recurrence_portions_and_decoding(heads, groups, dim, vdim, taps, kind, dtype, strong, form):
    """Three sequences in random slots, cut in different ways, prompts beside decoding entries; the slots start as nonsense.
    form "scan": the kernels for any size."""
    from inference_engine_b200 import ops

    g = np.random.default_rng(dim + heads)
    rec, a_log = make_rec(g, kind, heads, groups, dim, vdim, taps, strong)
    st = ops.make_recurrent_state(rec, 5, dtype, DEV)
    st.state.fill_(float("nan"))
    st.ring.fill_(float("nan"))
    T = [70, 41, 24]
    seqs = [rec_inputs(g, rec, t, dtype) for t in T]
    want = [rec_want(rec, a_log, *s) for s in seqs]
    slots, at = [4, 0, 2], [0, 0, 0]
    for chunks in ([1, 17, 2], [2, 1, 0], [33, 2, 0], [1, 1, 2], [1, 1, 1], [32, 19, 19]):
        live = [e for e in range(3) if chunks[e]]
        live.sort(key=lambda e: not (chunks[e] == 1 and at[e] > 0))  # decoding entries first
        nd = sum(chunks[e] == 1 and at[e] > 0 for e in live)
        rows, _ = step_rows([at[e] for e in live], [chunks[e] for e in live], nd, slots=[slots[e] for e in live])
        join = lambda i: torch.cat([seqs[e][i][at[e] : at[e] + chunks[e]] for e in live])  # noqa: E731
        x, step, beta = torch.cat([torch.zeros(rows.num_rows, 8, dtype=dtype, device=DEV), join(0)], 1)[:, 8:], join(1), None
        if rec.correct:
            beta = join(2)
        out = torch.empty(rows.num_rows, heads * vdim, device=DEV)
        ops.recurrence_decode(rec, st, x, step, beta, rows, out, variant=int(form == "scan"))
        if rows.seq_ids is not None:
            ops.recurrence_prefill(rec, st, x, step, beta, rows, out, form)
        o = 0
        for e in live:
            close(out[o : o + chunks[e]].view(-1, heads, vdim), want[e][at[e] : at[e] + chunks[e]], dtype, f32=5e-5, b16=3e-2)
            o += chunks[e]
            at[e] += chunks[e]
    assert at == T
    assert torch.isnan(st.state[1]).all() and torch.isnan(st.ring[3].float()).all()  # the other slots are as they were
    status_clear()


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,groups,dim,vdim", [(2, 1, 64, 64), (16, 4, 128, 72), (40, 8, 16, 16), (100, 4, 32, 8)])
def test_long_portions_beside_others(kind, heads, groups, dim, vdim):
    """Portions long enough to be cut into pieces that run side by side: one alone, two in a step, three beside a decoding one."""
    from inference_engine_b200 import ops

    g = np.random.default_rng(heads)
    dtype = torch.bfloat16
    rec, a_log = make_rec(g, kind, heads, groups, dim, vdim, 4)
    st = ops.make_recurrent_state(rec, 4, dtype, DEV)
    seqs = [rec_inputs(g, rec, 400, dtype) for _ in range(4)]
    want = [rec_want(rec, a_log, *s) for s in seqs]
    at = [0] * 4
    for chunks in ([257, 0, 0, 0], [0, 129, 150, 0], [1, 64, 130, 200]):
        live = [e for e in range(4) if chunks[e]]
        rows, _ = step_rows([at[e] for e in live], [chunks[e] for e in live], int(chunks[0] == 1), slots=live)
        x, step, beta = (None if i == 2 and not rec.correct else torch.cat([seqs[e][i][at[e] : at[e] + chunks[e]] for e in live]) for i in range(3))
        out = torch.empty(rows.num_rows, heads * vdim, device=DEV)
        ops.recurrence_decode(rec, st, x, step, beta, rows, out)
        ops.recurrence_prefill(rec, st, x, step, beta, rows, out)
        o = 0
        for e in live:
            close(out[o : o + chunks[e]].view(-1, heads, vdim), want[e][at[e] : at[e] + chunks[e]], dtype, b16=3e-2)
            o += chunks[e]
            at[e] += chunks[e]
    status_clear()


@pytest.mark.parametrize("dtype", DTYPES)
def test_decode_with_the_gated_norm_inside(dtype):
    from inference_engine_b200 import ops

    g = np.random.default_rng(8)
    for heads, groups, dim, vdim, taps in SIZES:
        rec, _ = make_rec(g, "delta", heads, groups, dim, vdim, taps)
        a, b = (ops.make_recurrent_state(rec, 3, dtype, DEV) for _ in range(2))
        rows, _ = step_rows([9, 4, 0], [1, 1, 1], 3, slots=[2, 0, 1])
        rows.num_decoding.fill_(2)  # the last row is idle
        x, step, beta = rec_inputs(g, rec, 3, dtype)
        for s in (a, b):
            s.state[..., :vdim] = rnd(np.random.default_rng(1), *s.state[..., :vdim].shape)
            s.ring.copy_(rnd(np.random.default_rng(2), *s.ring.shape, dtype=dtype))
        gate, norm = rnd(g, 3, heads * vdim, dtype=dtype), ops.GatedNorm(rnd(g, vdim), heads, 1e-5, False)
        out, raw = (torch.full((3, heads * vdim), float("nan"), dtype=t, device=DEV) for t in (dtype, torch.float32))
        ops.recurrent_mixer(rec, a, x, step, beta, gate, norm, rows, out)
        ops.recurrence_decode(rec, b, x, step, beta, rows, raw, variant=1)  # the form for any size
        want = B.rms_norm(np64(raw).reshape(3, heads, vdim), 1e-5, np64(norm.weight)).reshape(3, -1) * B.sigmoid(np64(gate))
        close(out, want, dtype)
        assert (out[2] == 0).all() and torch.allclose(a.state, b.state, rtol=1e-5, atol=1e-5) and torch.equal(a.ring, b.ring)
    status_clear()


@pytest.mark.parametrize("kind", KINDS)
def test_far_token_in_the_state(kind):
    """With almost no decay a single strong write is read back hundreds of tokens later, over portions and decoding."""
    from inference_engine_b200 import ops

    g = np.random.default_rng(3)
    rec, _ = make_rec(g, kind, 2, 1, 64, 64, 2)
    rec.neg_a.fill_(-1e-6)
    a_log = np.log(1e-6) * np.ones(2)
    for dtype in DTYPES:
        st = ops.make_recurrent_state(rec, 1, dtype, DEV)
        x, step, beta = rec_inputs(g, rec, 700, dtype)
        x[1:-1] *= 0.05
        want, at = rec_want(rec, a_log, x, step, beta), 0
        for n in [300, 1, 2, 390] + [1] * 7:
            rows, _ = step_rows([at], [n], int(n == 1 and at > 0), slots=[0])
            out, cut = torch.empty(n, 128, device=DEV), slice(at, at + n)
            args = (rec, st, torch.cat([x.new_zeros(n, 8), x[cut]], 1)[:, 8:], step[cut], None if beta is None else beta[cut], rows, out)
            (ops.recurrence_prefill if rows.seq_ids is not None else ops.recurrence_decode)(*args)
            close(out.view(n, 2, 64), want[cut], dtype, f32=5e-5, b16=3e-2)
            at += n


def test_bad_slots_are_reported_and_nothing_is_written():
    from inference_engine_b200 import kernels as K
    from inference_engine_b200 import ops

    g = np.random.default_rng(4)
    rec, _ = make_rec(g, "delta", 2, 1, 16, 16, 3)
    st = ops.make_recurrent_state(rec, 2, torch.bfloat16, DEV)
    x, step, beta = rec_inputs(g, rec, 20, torch.bfloat16)
    rows, _ = step_rows([3, 5], [1, 19], 1, slots=[7, -5])
    out = torch.full((20, 32), 3.0, device=DEV)
    ops.recurrence_decode(rec, st, x, step, beta, rows, out)
    ops.recurrence_prefill(rec, st, x, step, beta, rows, out)
    assert K.check_status() != 0
    K.status_word(torch.device("cuda", 0)).zero_()
    assert (out == 3.0).all() and (st.state == 0).all() and (st.ring == 0).all()
