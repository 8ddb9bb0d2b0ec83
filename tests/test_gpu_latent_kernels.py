"""Latent cache and attention kernels alone, against float64 numpy."""
import numpy as np
import pytest

from homura_b200 import synth

pytestmark = pytest.mark.gpu

PAGE = 64


def bf16_round(x):
    return synth.bf16_to_f32(synth.f32_to_bf16_rne(np.ascontiguousarray(x, np.float32)))


def make_cache(hm, rank, dt, lens, seed, spare=3):
    """A cache filled with unit latents of the given lengths on shuffled pages; returns it and the stored latents."""
    g = np.random.default_rng(seed)
    per = (max(lens) + PAGE - 1) // PAGE
    table = g.permutation(len(lens) * per + spare)[: len(lens) * per].reshape(len(lens), per)
    cache = hm.LatentCache(rank, dt, table)
    stored = []
    w = np.ones(rank, np.float32)
    for s, n in enumerate(lens):
        c = g.standard_normal((n, rank)).astype(np.float32)
        cache.write(c, w, 1e-6, np.full(n, s), np.arange(n))
        c = c.astype(np.float64)
        c /= np.sqrt((c**2).mean(1, keepdims=True) + 1e-6)
        stored.append(bf16_round(c).astype(np.float64) if dt == hm.DType.BF16 else c)
    return cache, stored


def reference(q, stored, scale, row_seq, row_pos):
    out = np.empty(q.shape, np.float64)
    for m in range(q.shape[0]):
        c = stored[row_seq[m]][: row_pos[m] + 1]
        s = scale * (q[m].astype(np.float64) @ c.T)
        p = np.exp(s - s.max(1, keepdims=True))
        out[m] = (p / p.sum(1, keepdims=True)) @ c
    return out


def check(got, want, tol):
    err = np.abs(got - want).max()
    assert err <= tol * max(1.0, np.abs(want).max()), err


# (rank, heads): one element; odd; below, at and above a 64-element block; several slices; more heads than a tile's pairs; wide
SHAPES = [(1, 1), (5, 3), (48, 2), (64, 16), (72, 5), (128, 8), (192, 24), (320, 40), (512, 20), (640, 4)]


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("rank,heads", SHAPES)
def test_prompt_and_decode_rows(hm, rank, heads, dtype):
    dt = hm.DType[dtype]
    lens = [1, 63, 64, 65, 130, 300]
    cache, stored = make_cache(hm, rank, dt, lens, rank)
    g = np.random.default_rng(rank + 1)
    # a mixed batch: single tokens, a portion that crosses a page and a 128-token tile, the first tokens of a sequence
    rows = [(0, 0), (1, 62)] + [(4, p) for p in range(120, 130)] + [(2, 63), (3, 64)] + [(5, p) for p in range(0, 9)] + [(5, 299)]
    rs, rp = np.array([r[0] for r in rows]), np.array([r[1] for r in rows])
    q = g.standard_normal((len(rows), heads, rank)).astype(np.float32)
    scale = 2.0 * rank**-0.5
    want = reference(q, stored, scale, rs, rp)
    # float32 weights against float32 sums; on bf16 pages a latent may round to the neighbouring bf16 value
    for nsplit in (0, 1, 3):
        check(cache.attend(q, scale, rs, rp, nsplit), want, 2e-5 if dtype == "F32" else 5e-3)


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("length", [2, 64, 65, 128, 129, 257, 1000])
def test_one_key_stands_out(hm, length, dtype):
    """A query that matches one key among many returns that key's latent: first, last, and on both sides of every page."""
    dt = hm.DType[dtype]
    rank, heads = 80, 3
    cache, stored = make_cache(hm, rank, dt, [length], 7 * length)
    targets = sorted({t for t in (0, 1, 63, 64, 127, 128, 191, 192, 255, 256, 640, length - 2, length - 1) if 0 <= t < length})
    for row_pos, expect_hit in ((length - 1, True), (max(0, length // 2), None)):
        for i in range(0, len(targets), heads):
            t = [targets[min(i + h, len(targets) - 1)] for h in range(heads)]
            q = np.stack([stored[0][k] for k in t])[None].astype(np.float32)
            want = reference(q, stored, 1.0, [0], [row_pos])
            got = cache.attend(q, 1.0, [0], [row_pos])
            check(got, want, 2e-5 if dtype == "F32" else 5e-3)
            if expect_hit:
                for h, k in enumerate(t):
                    assert np.abs(got[0, h] - stored[0][k]).max() < 1e-2


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
def test_the_next_key_is_never_seen(hm, dtype):
    """Rows of a portion see their own position and not the one behind, wherever the portion lies relative to pages and tiles."""
    dt = hm.DType[dtype]
    rank, heads = 64, 2
    cache, stored = make_cache(hm, rank, dt, [400], 11)
    for start in (0, 1, 40, 60, 63, 64, 100, 126, 127, 128, 250, 340):
        n = 33
        rp = np.arange(start, start + n)
        # head 0 asks for the row's own key, head 1 for the one behind it
        q = np.stack([np.stack([stored[0][p], stored[0][p + 1]]) for p in rp]).astype(np.float32)
        got = cache.attend(q, 1.0, np.zeros(n, int), rp)
        check(got, reference(q, stored, 1.0, np.zeros(n, int), rp), 2e-5 if dtype == "F32" else 5e-3)
        assert np.abs(got[:, 0] - stored[0][rp]).max() < 1e-2
        assert np.abs(got[:, 1] - stored[0][rp + 1]).max(1).min() > 0.5


def test_scores_that_grow_with_the_position(hm):
    """The reference maximum has to move again and again, by little and by much, without losing what was summed before."""
    rank, n = 64, 900
    table = np.arange(15)[None, ::-1].copy()
    for growth in (0.01, 0.08, 0.5):
        cache = hm.LatentCache(rank, hm.DType.BF16, table)
        c = np.zeros((n, rank), np.float32)
        # unit vectors whose first element carries the score and the others identify the token
        c[:, 0] = np.linspace(-1, 1, n)
        c[np.arange(n), 1 + np.arange(n) % 63] = 1.5
        w = np.ones(rank, np.float32)
        cache.write(c, w, 1e-6, np.zeros(n, int), np.arange(n))
        cn = c.astype(np.float64) / np.sqrt((c.astype(np.float64) ** 2).mean(1, keepdims=True) + 1e-6)
        stored = [bf16_round(cn).astype(np.float64)]
        q = np.zeros((1, 4, rank), np.float32)
        q[0, :, 0] = [growth * n / 8, growth * n / 2, -growth * n / 2, 0.0]
        check(cache.attend(q, 1.0, [0], [n - 1], 1), reference(q, stored, 1.0, [0], [n - 1]), 5e-3)


def test_weights_and_rank_of_the_write(hm):
    rank, n = 72, 70
    g = np.random.default_rng(3)
    c, w = g.standard_normal((n, rank)).astype(np.float32) * 3, g.standard_normal(rank).astype(np.float32)
    cache = hm.LatentCache(rank, hm.DType.F32, np.array([[4, 1]]))
    cache.write(c, w, 0.5, np.zeros(n, int), np.arange(n))
    stored = [c / np.sqrt((c.astype(np.float64) ** 2).mean(1, keepdims=True) + 0.5) * w]
    q = g.standard_normal((2, 3, rank)).astype(np.float32)
    check(cache.attend(q, 0.2, [0, 0], [0, n - 1]), reference(q, stored, 0.2, [0, 0], [0, n - 1]), 2e-5)
    raw = cache.pages.download(np.float32, 5 * PAGE * rank).reshape(5, PAGE, rank)
    assert np.allclose(raw[4], stored[0][:64], atol=1e-5) and np.allclose(raw[1, :6], stored[0][64:], atol=1e-5)
    assert not raw[[0, 2, 3]].any() and not raw[1, 6:].any()


def test_bad_rows_are_errors(hm):
    cache, _ = make_cache(hm, 16, hm.DType.F32, [64], 1)
    q = np.zeros((1, 1, 16), np.float32)
    for seq, pos in ((1, 0), (-1, 0), (0, 64), (0, -1)):
        with pytest.raises(hm.HomuraError):
            cache.attend(q, 1.0, [seq], [pos])


@pytest.mark.parametrize("heads", [1, 3, 12])
def test_portions_behind_a_long_context(hm, heads):
    """Rows that share a CTA, in passes whose contexts are long enough for the wider tiles, with a key that stands out far away."""
    rank, length = 64, 4300
    cache, stored = make_cache(hm, rank, hm.DType.BF16, [length, 30], 17)
    rows = [(0, p) for p in range(4200, 4233)] + [(1, p) for p in range(5, 25)] + [(0, 1)]
    rs, rp = np.array([r[0] for r in rows]), np.array([r[1] for r in rows])
    g = np.random.default_rng(heads)
    q = g.standard_normal((len(rows), heads, rank)).astype(np.float32) * 0.3
    q[3, 0], q[20, heads - 1] = stored[0][2], stored[0][4095]
    want = reference(q, stored, 1.0, rs, rp)
    for nsplit in (0, 1, 5):
        check(cache.attend(q, 1.0, rs, rp, nsplit), want, 5e-3)
