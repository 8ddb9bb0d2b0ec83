"""Grouped-query attention with any head size, its cache, post-norms and the router alone, against float64 numpy."""
import numpy as np
import pytest

import dipisun_oracle as do
from homura_b200 import synth

pytestmark = pytest.mark.gpu

PAGE = 64
LN2 = float(np.log(2.0))


def bf16_round(x):
    return synth.bf16_to_f32(synth.f32_to_bf16_rne(np.ascontiguousarray(x, np.float32)))


def make_cache(hm, heads, kv_heads, dim, vdim, dt, lens, seed, spare=3, k_edit=None):
    """A cache filled with random keys and values on shuffled pages; returns it and the stored (keys, values) per sequence."""
    g = np.random.default_rng(seed)
    per = (max(lens) + PAGE - 1) // PAGE
    table = g.permutation(len(lens) * per + spare)[: len(lens) * per].reshape(len(lens), per)
    cache = hm.GqaCache(heads, kv_heads, dim, vdim, dt, table)
    stored = []
    for s, n in enumerate(lens):
        raw = g.standard_normal((n, heads * dim + kv_heads * (dim + vdim))).astype(np.float32)
        if k_edit:
            k_edit(s, raw)
        cache.write(raw, np.full(n, s), np.arange(n))
        k = raw[:, heads * dim : heads * dim + kv_heads * dim].reshape(n, kv_heads, dim)
        v = raw[:, heads * dim + kv_heads * dim :].reshape(n, kv_heads, vdim)
        stored.append(tuple((bf16_round(a) if dt == hm.DType.BF16 else a).astype(np.float64) for a in (k, v)))
    return cache, stored


def reference(q, stored, row_seq, row_pos, bias=None):
    """q as base-2 exponents per unit of key."""
    M, H, _ = q.shape
    k0, v0 = stored[0]
    out = np.empty((M, H, v0.shape[2]))
    for m in range(M):
        k, v = (a[: row_pos[m] + 1] for a in stored[row_seq[m]])
        dist = row_pos[m] - np.arange(row_pos[m] + 1)
        for h in range(H):
            g = h // (H // k.shape[1])
            s = k[:, g] @ q[m, h].astype(np.float64)
            if bias is not None:
                s = s + bias[h][np.minimum(dist, bias.shape[1] - 1)].astype(np.float64)
            p = np.exp2(s - s.max())
            out[m, h] = p @ v[:, g] / p.sum()
    return out


def check(got, want, tol):
    err = np.abs(got - want).max()
    assert err <= tol * max(1.0, np.abs(want).max()), err


# (heads, key heads, dim, vdim): one of everything; odd; unequal key and value sizes on both sides of 16, 64, 128, 256; groups of one,
# more than eight and more than sixteen heads
SHAPES = [(1, 1, 1, 1), (3, 1, 5, 7), (4, 2, 24, 40), (16, 4, 64, 64), (6, 6, 72, 16), (24, 2, 128, 80), (18, 1, 48, 128), (10, 2, 100, 33), (4, 1, 200, 160), (2, 1, 260, 64), (3, 3, 64, 272)]


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
def test_prompt_and_decode_rows(hm, heads, kv_heads, dim, vdim, dtype):
    dt = hm.DType[dtype]
    cache, stored = make_cache(hm, heads, kv_heads, dim, vdim, dt, [1, 63, 64, 65, 130, 300], dim)
    g = np.random.default_rng(dim + 1)
    # a mixed batch: single tokens, portions across a page, the first tokens of a sequence, two tokens
    rows = [(0, 0), (1, 62)] + [(4, p) for p in range(115, 130)] + [(2, 63), (3, 64)] + [(5, p) for p in range(0, 21)] + [(5, 298), (5, 299)]
    rs, rp = np.array([r[0] for r in rows]), np.array([r[1] for r in rows])
    q = (g.standard_normal((len(rows), heads, dim)) * 2.0 * dim**-0.5).astype(np.float32)
    bias = g.standard_normal((heads, 41)).astype(np.float32) * 2
    # exact products in both: what differs is the order of the sums (and one rounding of a stored value to bf16, done alike)
    for b in (None, bias):
        want = reference(q, stored, rs, rp, b)
        for nsplit in (0, 1, 3):
            check(cache.attend(q, rs, rp, b, nsplit), want, 2e-5)


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("length", [2, 16, 17, 64, 65, 129, 700])
def test_one_key_stands_out(hm, length, dtype):
    """A query that matches one key among many returns that key's value: first, last, and on both sides of units of 16 and of pages."""
    dt = hm.DType[dtype]
    heads, dim = 3, 56
    cache, stored = make_cache(hm, heads, 1, dim, 24, dt, [length], 7 * length)
    k, v = stored[0]
    targets = sorted({t for t in (0, 1, 15, 16, 63, 64, 127, 128, 511, 512, length - 17, length - 2, length - 1) if 0 <= t < length})
    for i in range(0, len(targets), heads):
        t = [targets[min(i + h, len(targets) - 1)] for h in range(heads)]
        q = np.stack([3 * k[j, 0] for j in t])[None].astype(np.float32)
        got = cache.attend(q, [0], [length - 1])
        check(got, reference(q, stored, [0], [length - 1]), 2e-5)
        for h, j in enumerate(t):
            assert np.abs(got[0, h] - v[j, 0]).max() < 1e-3
        # a row in front of a target does not see it
        for h, j in enumerate(t):
            if j > 0:
                seen = cache.attend(q, [0], [j - 1])
                check(seen, reference(q, stored, [0], [j - 1]), 2e-5)


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
def test_bias_picks_a_distance(hm, dtype):
    """Without a query the bias alone decides: a large entry returns the value that many tokens back, the last entry all beyond."""
    dt = hm.DType[dtype]
    heads, n, reach = 6, 200, 70
    cache, stored = make_cache(hm, heads, 2, 32, 48, dt, [n, n], 5)
    v = stored[1][1]
    for dist in ((0, 1, 15, 16, 63, 69), (17, 31, 32, 64, 65, 70)):
        bias = np.zeros((heads, reach + 1), np.float32)
        for h, d in enumerate(dist):
            bias[h, d] = 60.0
        pos = list(range(100, 148))
        got = cache.attend(np.zeros((len(pos), heads, 32), np.float32), [1] * len(pos), pos, bias)
        for m, p in enumerate(pos):
            for h, d in enumerate(dist):
                want = v[p - d, h // 3] if d < reach else v[: p - reach + 1, h // 3].mean(0)
                assert np.abs(got[m, h] - want).max() < 1e-4


def test_bf16_pages_hold_rounded_rows(hm):
    """Both page types store what they are given, at the slot of its position, and nothing else changes."""
    g = np.random.default_rng(3)
    for dt in (hm.DType.F32, hm.DType.BF16):
        cache, stored = make_cache(hm, 2, 2, 20, 36, dt, [70, 5], 11)
        one = g.standard_normal((1, 2 * 20 + 2 * 56)).astype(np.float32)
        cache.write(one, [1], [4])
        stored[1][0][4] = one[0, 40:80].reshape(2, 20)
        stored[1][1][4] = one[0, 80:].reshape(2, 36)
        if dt == hm.DType.BF16:
            stored[1] = tuple(bf16_round(a).astype(np.float64) for a in stored[1])
        q = g.standard_normal((2, 2, 20)).astype(np.float32)
        check(cache.attend(q, [0, 1], [69, 4]), reference(q, stored, [0, 1], [69, 4]), 2e-5)


@pytest.mark.parametrize("norm", [0, 1, 2])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(1, 1, 1, 1), (5, 1, 11, 9), (12, 4, 96, 40), (8, 8, 130, 24)])
def test_norms_temperature_and_blended_values(hm, norm, heads, kv_heads, dim, vdim):
    g = np.random.default_rng(heads + norm)
    M, eps, coef, every = 9, 1e-2, 0.6, 5
    nq, nk, nv = heads * dim, kv_heads * dim, kv_heads * vdim
    raw = (g.standard_normal((M, nq + nk + nv)) * 3).astype(np.float32)
    qn, kn = (1 + 0.3 * g.standard_normal(n).astype(np.float32) for n in ((dim, dim) if norm == 1 else (nq, nk)))
    pos = np.array([0, 3, 4, 5, 9, 10, 44, 100, 127])
    cache = hm.GqaCache(heads, kv_heads, dim, vdim, hm.DType.F32, np.arange(2 * M).reshape(M, 2)[:, ::-1])
    first = np.zeros((M, nv), np.float32)
    got = cache.write(raw, np.arange(M), pos, qn, kn, norm, eps, 0.25, (coef, every), v_first=first)
    r = raw.astype(np.float64)
    q, k, v = r[:, :nq], r[:, nq : nq + nk], r[:, nq + nk :]
    if norm == 1:
        q, k = do.norm_each_head(q, qn, heads, eps), do.norm_each_head(k, kn, kv_heads, eps)
    elif norm == 2:
        q, k = do.norm_all_heads(q, qn, eps), do.norm_all_heads(k, kn, eps)
    want_q = q * do.temperature(pos, coef, every)[:, None] * 0.25
    check(got.reshape(M, -1), want_q, 1e-5)
    assert np.array_equal(first, raw[:, nq + nk :])
    # keys and values through the attention: a row alone with its own key returns its own value, two rows weigh their keys
    one = cache.attend(got, np.arange(M), pos * 0)
    assert one.shape == (M, heads, vdim)
    cache.write(raw, np.arange(M), np.zeros(M, np.int64), qn, kn, norm, eps, 0.25, (coef, every), v_first=first, v_lambda=0.375)
    blend = do.blend_values(v, first.astype(np.float64), 0.375)
    stored = [(k[m].reshape(1, kv_heads, dim), blend[m].reshape(1, kv_heads, vdim)) for m in range(M)]
    check(cache.attend(got, np.arange(M), np.zeros(M, np.int64)), reference(got, stored, np.arange(M), np.zeros(M, np.int64)), 1e-5)
    other = (g.standard_normal((M, nv)) * 2).astype(np.float32)
    cache.write(raw, np.arange(M), np.ones(M, np.int64), qn, kn, norm, eps, 0.25, (coef, every), v_first=other, v_lambda=0.375)
    blend2 = do.blend_values(v, other.astype(np.float64), 0.375)
    stored = [(np.stack([k[m], k[m]]).reshape(2, kv_heads, dim), np.stack([blend[m], blend2[m]]).reshape(2, kv_heads, vdim)) for m in range(M)]
    check(cache.attend(got, np.arange(M), np.ones(M, np.int64)), reference(got, stored, np.arange(M), np.ones(M, np.int64)), 1e-5)


@pytest.mark.parametrize("M,W", [(1, 1), (1, 96), (3, 130), (2, 1536), (64, 200), (17, 2056)])
@pytest.mark.parametrize("identity", [False, True])
def test_post_norm(hm, M, W, identity):
    g = np.random.default_rng(W)
    y, x = (g.standard_normal((M, W)).astype(np.float32) * s for s in (5, 2))
    w, idw = 1 + 0.2 * g.standard_normal(W).astype(np.float32), g.random(M).astype(np.float32)
    got = hm.post_norm_route(y, x, w, 0.35, 1e-3, idw if identity else None)
    yy = y.astype(np.float64) + (idw[:, None] * x.astype(np.float64) if identity else 0)
    check(got, x + 0.35 * do.rms(yy, 1e-3) * w, 2e-6)


# (rows, width, experts, identity experts, top): more outputs than a warp, a cluster's rows, every output chosen, a width that is not
# a multiple of eight
@pytest.mark.parametrize("M,W,E,I,top", [(1, 96, 5, 2, 3), (4, 130, 1, 0, 1), (1, 1536, 100, 7, 8), (64, 64, 33, 31, 10), (30, 256, 4, 3, 7), (2, 17, 2, 6, 5)])
def test_router(hm, M, W, E, I, top):
    g = np.random.default_rng(E * W)
    y, x = g.standard_normal((M, W)).astype(np.float32), g.standard_normal((M, W)).astype(np.float32)
    w = np.ones(W, np.float32)
    router = synth.f32_to_bf16_rne((g.standard_normal((E + I, W)) * 2 * W**-0.5).astype(np.float32))
    corr = (0.3 * g.standard_normal(E + I)).astype(np.float32)
    new, ids, wts, idw = hm.post_norm_route(y, x, w, 0.5, 1e-5, router=router, correction=corr, experts=E, top=top)
    want_x = x + 0.5 * do.rms(y.astype(np.float64), 1e-5)
    check(new, want_x, 2e-6)
    chosen, weights = do.route(want_x @ synth.bf16_to_f32(router).astype(np.float64).T, corr.astype(np.float64), top)
    assert np.array_equal(np.where(chosen < E, chosen, -1), ids)
    check(wts, weights, 1e-5)
    check(idw, np.where(chosen >= E, weights, 0).sum(1), 1e-5)


def test_bad_arguments_are_refused(hm):
    cache, _ = make_cache(hm, 4, 2, 16, 16, hm.DType.F32, [10], 1)
    q = np.zeros((1, 4, 16), np.float32)
    for rs, rp in (([1], [0]), ([0], [64]), ([-1], [0]), ([0], [-1])):
        with pytest.raises(hm.HomuraError):
            cache.attend(q, rs, rp)
    with pytest.raises(hm.HomuraError):
        cache.attend(q, [0], [5], nsplit=9)
    with pytest.raises(hm.HomuraError):
        hm.GqaCache(4, 3, 16, 16, hm.DType.F32, np.zeros((1, 1))).attend(q, [0], [0])
