"""Each mechanism of the decoder ops alone, against the plain implementation."""
import numpy as np
import pytest
import torch

from oracle import radivik as R
from tests import radivik_helpers as H

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
DEV = "cuda"


def t(x, dtype=torch.float32):
    return torch.as_tensor(np.asarray(x, np.float32)).to(dtype).to(DEV)


def i32(x):
    return torch.as_tensor(np.asarray(x, np.int32)).to(DEV)


def close(got, want, dtype, tol=None):
    got, want = got.detach().float().cpu().numpy(), np.asarray(want)
    tol = tol or (3e-6 if dtype == torch.float32 else 1e-2)
    err = np.abs(got - want).max() / max(1.0, np.abs(want).max())
    assert err < tol, err


def make_rows(entries, page=16, pages_extra=3, seed=0):
    """entries: [(cached, new)]; decoding ones (new == 1 and cached > 0) first.  A scattered block table."""
    from inference_engine_b200 import ops
    from inference_engine_b200.scaffold import plan_step

    nd = 0
    while nd < len(entries) and entries[nd][1] == 1 and entries[nd][0] > 0:
        nd += 1
    n = sum(x for _, x in entries)
    plan = plan_step([c for c, _ in entries[:nd]], entries[nd:], n, len(entries) + 1)
    need = [(c + x + page - 1) // page for c, x in entries]
    perm = np.random.default_rng(seed).permutation(sum(need) + pages_extra)
    table = np.full((len(entries) + 1, max(need)), -1, np.int32)
    at = 0
    for b, k in enumerate(need):
        table[b, :k] = perm[at : at + k]
        at += k
    rows = ops.Rows(n, i32(plan["cached"]), i32([nd]), i32(table), i32(plan["seq_ids"]), i32(plan["positions"]), i32(plan["cu_seqlens"]),
                    i32(plan["tile_start"]), 128)
    return rows, table, len(perm), plan


def fill(cache, table, b, k, v):
    """Place keys [n, heads, dim] and values of an entry in the cache by its pages."""
    P = cache.page_size
    for j in range(k.shape[0]):
        cache.k[int(table[b, j // P]), :, j % P, : k.shape[2]] = k[j]
        cache.v[int(table[b, j // P]), :, j % P, : v.shape[2]] = v[j]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,top", [(64, 1), (2052, 3), (33, 2)])
def test_scaled_add_norm(dtype, width, top):
    from inference_engine_b200 import ops

    g = np.random.default_rng(1)
    x, w = g.standard_normal((7, width)), H.bf16(1 + 0.3 * g.standard_normal(width))
    d = H.bf16(g.standard_normal((7 * top, width)))
    index = g.permutation(7 * top).reshape(7, top)
    want = R.rms_norm(2.25 * np.float32(x) + d[index].sum(1), 1e-3, w)
    zero = torch.ones(5, dtype=torch.int32, device=DEV)
    y, yb = ops.scaled_add_norm(t(x), t(d, dtype), t(w), 2.25, 1e-3, dtype, index=i32(index), zero=zero)
    close(y, want, torch.float32)
    close(yb, want, dtype)
    assert zero.sum().item() == 0
    x0 = t(x)
    _, only = ops.scaled_add_norm(x0, None, t(w), 1.0, 1e-3, dtype, keep=False)
    close(only, R.rms_norm(np.float32(x), 1e-3, w), dtype)
    close(x0, x, torch.float32)  # untouched


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scaling", [None, H.YARN])
@pytest.mark.parametrize("dim,vdim,rot", [(48, 40, 16), (20, 36, 20), (7, 130, 2)])
def test_rotation_unit_norm_and_write(dtype, scaling, dim, vdim, rot):
    from inference_engine_b200 import ops

    g = np.random.default_rng(2)
    heads, kv, eps = 4, 2, 1e-4
    rows, table, pages, plan = make_rows([(33, 1), (15, 1), (0, 5), (14, 40)])
    cache = ops.make_paged_kv(pages, kv, 16, dim, vdim, dtype, DEV)
    rd = {"dims": rot, "base": 500.0, **({"scaling": scaling} if scaling else {})}
    rotary = ops.Rotary(rot, 500.0, None if not scaling else tuple(float(scaling[k]) for k in ("factor", "original", "fast", "slow")))
    f, mult = R.rotary_frequencies(rd)
    assert np.allclose(rotary.frequencies()[0], f, rtol=1e-12) and rotary.frequencies()[1] == mult
    qkv = H.bf16(g.standard_normal((rows.num_rows, (heads + kv) * dim + kv * vdim)))
    q = ops.rope_write(t(qkv, dtype), rows, cache, rotary.table(64, DEV), heads, True, True, eps)
    pos, seq = np.array(plan["positions"]), np.array(plan["seq_ids"])
    n = rows.num_rows
    close(q[..., :dim], R.rms_norm(R.rotate(qkv[:, : heads * dim].reshape(n, heads, dim), pos, rd), eps), dtype)
    assert q[..., dim:].abs().sum().item() == 0
    k = R.rms_norm(R.rotate(qkv[:, heads * dim : (heads + kv) * dim].reshape(n, kv, dim), pos, rd), eps)
    v = qkv[:, (heads + kv) * dim :].reshape(n, kv, vdim)
    page, slot = table[seq, pos // 16], pos % 16
    close(cache.k[page, :, slot][..., :dim], k, dtype)
    close(cache.v[page, :, slot][..., :vdim], v, dtype)
    touched = np.zeros((pages, 16), bool)
    touched[page, slot] = True
    assert cache.k.permute(0, 2, 1, 3)[torch.as_tensor(~touched)].abs().sum().item() == 0  # nothing else was written
    # queries only: the cache stays as it is
    before = cache.k.clone()
    q2 = ops.rope_write(t(qkv[:, : heads * dim], dtype), rows, cache, rotary.table(64, DEV), heads, False, True, eps)
    assert torch.equal(q, q2) and torch.equal(before, cache.k)
    H.status_clear()


CASES = [  # heads, kv heads, key size, value size
    (4, 2, 48, 40), (3, 1, 128, 64), (8, 8, 64, 128), (12, 1, 104, 88), (40, 2, 16, 24), (2, 1, 36, 12), (2, 2, 10, 7),
]


@pytest.mark.parametrize("heads,kv,dim,vdim", CASES)
@pytest.mark.parametrize("page", [16, 64])
def test_attention_single_key_stands_out(heads, kv, dim, vdim, page):
    """Every query matches one key far above all others (its own position, the first key, both sides of page and block
    borders, the key just outside the causal edge as a decoy), in prompt portions and decoding rows of one step."""
    from inference_engine_b200 import ops

    g = np.random.default_rng(3)
    entries = [(16, 1), (63, 1), (64, 1), (700, 1), (0, 130), (61, 67), (257, 2)]
    rows, table, pages, plan = make_rows(entries, page)
    cache = ops.make_paged_kv(pages, kv, page, dim, vdim, torch.bfloat16, DEV)
    cache.k.fill_(float("nan"))  # whatever no token was written to must not matter
    cache.v.fill_(float("nan"))
    cache.k[..., dim:] = 0
    cache.v[..., vdim:] = 0
    q = np.zeros((rows.num_rows, heads, dim))
    want = np.zeros((rows.num_rows, heads, vdim))
    at = 0
    scale = 24.0 / np.sqrt(dim)
    for b, (c, x) in enumerate(entries):
        n = c + x
        k = H.bf16(R.rms_norm(g.standard_normal((n, kv, dim)), 1e-6))
        v = H.bf16(g.standard_normal((n, kv, vdim)))
        fill(cache, table, b, t(k, torch.bfloat16), t(v, torch.bfloat16))
        for i in range(x):
            p = c + i
            targets = [p, 0, max(0, p - 1), min(p, 15), min(p, 16), min(p, 63), min(p, 64), p // 64 * 64, min(n - 1, p + 1)]
            for h in range(heads):
                q[at + i, h] = k[targets[(i + h) % len(targets)], h // (heads // kv)]
        q[at : at + x] = H.bf16(q[at : at + x])
        want[at : at + x] = R.causal_attention(q[at : at + x], k, v, scale, c)
        at += x
    qd = torch.zeros(rows.num_rows, heads, cache.k.shape[3], device=DEV, dtype=torch.bfloat16)
    qd[..., :dim] = t(q, torch.bfloat16)
    close(ops.attention_rows(qd, cache, rows, scale), want, torch.bfloat16)
    assert ops.tensor_core_attention(cache)
    for _ in range(2):  # the second call finds the workspace as the first left it
        close(ops.paged_attention(qd, cache, rows, scale), want, torch.bfloat16, 2e-2)
    H.status_clear()


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_beyond_the_tensor_core_sizes(dtype):
    from inference_engine_b200 import ops

    g = np.random.default_rng(4)
    rows, table, pages, _ = make_rows([(37, 1), (5, 30)])
    cache = ops.make_paged_kv(pages, 1, 16, 200, 260, dtype, DEV)
    assert not ops.tensor_core_attention(cache)
    q = H.bf16(g.standard_normal((31, 2, 200)))
    want, at = np.zeros((31, 2, 260)), 0
    for b, (c, x) in enumerate([(37, 1), (5, 30)]):
        k, v = H.bf16(g.standard_normal((c + x, 1, 200))), H.bf16(g.standard_normal((c + x, 1, 260)))
        fill(cache, table, b, t(k, dtype), t(v, dtype))
        want[at : at + x] = R.causal_attention(q[at : at + x], k, v, 0.1, c)
        at += x
    close(ops.paged_attention(t(q, dtype), cache, rows, 0.1), want, dtype)


def test_decode_attention_splits_and_idle_rows():
    """Long and short entries over the whole persistent grid, entries past num_decoding, and one entry alone."""
    from inference_engine_b200 import ops

    g = np.random.default_rng(5)
    heads, kv, dim, vdim, page = 6, 3, 40, 72, 64
    for lens in ([5000, 1, 64, 65, 900, 128, 127, 2300], [3000], [70] * 40):
        B = len(lens) + 2  # two idle rows
        need = [(n + page - 1) // page for n in lens]
        table = np.full((B, max(need)), -1, np.int32)
        perm, at = g.permutation(sum(need)), 0
        for b, m in enumerate(need):
            table[b, :m] = perm[at : at + m]
            at += m
        cache = ops.make_paged_kv(sum(need), kv, page, dim, vdim, torch.bfloat16, DEV)
        cache.k[..., :dim] = torch.randn(cache.k.shape[:3] + (dim,), device=DEV)
        cache.v[..., :vdim] = torch.randn(cache.v.shape[:3] + (vdim,), device=DEV)
        rows = ops.Rows(B, i32([n - 1 for n in lens] + [7, 7]), i32([len(lens)]), i32(table))
        q = torch.randn(B, heads, dim, device=DEV).to(torch.bfloat16)
        got = ops.paged_attention(q, cache, rows, 0.3)
        again = ops.paged_attention(q, cache, rows, 0.3)
        assert torch.equal(got, again)
        assert got[len(lens) :].abs().sum().item() == 0
        kk, vv, qq = cache.k.float().cpu().numpy(), cache.v.float().cpu().numpy(), q.float().cpu().numpy()
        for b, n in enumerate(lens):
            flat = lambda x, d: np.concatenate([x[p] for p in table[b, : need[b]]], axis=1)[:, :n, :d].transpose(1, 0, 2)
            want = R.causal_attention(qq[b : b + 1], flat(kk, dim), flat(vv, vdim), 0.3, n - 1)
            close(got[b : b + 1], want, torch.bfloat16)
        close(ops.attention_rows(q, cache, rows, 0.3)[: len(lens)], got[: len(lens)].float().cpu().numpy(), torch.bfloat16)
        H.status_clear()


MOE = [  # rows, width, ff, experts, top, limit
    (1, 64, 40, 4, 1, 2.0), (37, 64, 24, 5, 3, 0.5), (5, 72, 64, 8, 8, 1.0), (700, 136, 200, 3, 2, 7.0), (300, 64, 64, 40, 6, 1.5),
    (33, 30, 18, 3, 2, 1.0), (260, 520, 96, 2, 1, 2.0),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,ff,experts,top,limit", MOE)
def test_mixture(dtype, rows, width, ff, experts, top, limit):
    from inference_engine_b200 import ops

    g = np.random.default_rng(6)
    mat = lambda o, i, s: H.bf16(g.standard_normal((o, i)) * s * i ** -0.5)
    w = {"router": mat(experts, width, 2.0)}
    for e in range(experts):
        w.update({f"e{e}.gate": mat(ff, width, 3.0), f"e{e}.up": mat(ff, width, 3.0), f"e{e}.down": mat(width, ff, 1.0)})
    x = H.bf16(g.standard_normal((rows, width)))
    tt = lambda k: t(w[k], torch.bfloat16)
    ex = ops.make_experts(tt("router"), [tt(f"e{e}.gate") for e in range(experts)], [tt(f"e{e}.up") for e in range(experts)],
                          [tt(f"e{e}.down") for e in range(experts)], top, limit, 1.702, dtype, torch.device(DEV))
    want = R.mixture(np.float64(x), w, "", {"router": {"experts": experts, "top": top}, "expert": {"limit": limit}})
    ids, _ = R.route(np.float64(x), w["router"], top)
    for variant in (None, 1):
        ex.counts.zero_()
        y, places = ops.mixture(t(x), t(x, dtype), ex, variant)
        assert sorted(places.flatten().tolist()) == list(range(rows * top))
        assert ex.counts.tolist() == np.bincount(ids.flatten(), minlength=experts).tolist()
        got = y.float()[places.long()].sum(1)
        close(got, want, dtype, 1e-5 if dtype == torch.float32 else 2e-2)
    H.status_clear()


def test_router_takes_rows_that_are_not_numbers():
    """Idle rows of a padded step may hold anything; they must not disturb the others or leave the expert range."""
    from inference_engine_b200 import ops

    m = H.model(H.small(), H.weights(H.small()), torch.bfloat16)
    ex = m.layers[0].experts
    x = torch.randn(9, 64, device=DEV)
    x[3] = float("nan")
    ex.counts.zero_()
    y, places = ops.mixture(x, x.to(torch.bfloat16), ex)
    assert sorted(places.flatten().tolist()) == list(range(18))
    ex.counts.zero_()
    keep = [i for i in range(9) if i != 3]
    y2, places2 = ops.mixture(x[keep].contiguous(), x[keep].to(torch.bfloat16), ex)
    assert torch.equal(y[places[keep].long()].sum(1), y2[places2.long()].sum(1))
