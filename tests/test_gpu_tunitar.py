"""Tunitar models on the engine, against the plain float64 oracle."""
import functools

import numpy as np
import pytest
from conftest import record_error
from tunitar_cases import NAMES, model

from homura_b200 import synth
from homura_b200.serving import Scheduler, Session
from tunitar_oracle import Oracle

pytestmark = pytest.mark.gpu

# relative to the largest reference value: f32 throughout; bf16 pages against an oracle that rounds its latents alike (a latent on
# the edge of a rounding step may go the other way)
TOL = {"F32": 3e-5, "BF16": 6e-3}


def bf16_round(x):
    return synth.bf16_to_f32(synth.f32_to_bf16_rne(np.ascontiguousarray(x, np.float32))).astype(np.float64)


@functools.lru_cache(maxsize=None)
def weights(name):
    return synth.tunitar_weights(model(name), 21)


@functools.lru_cache(maxsize=None)
def oracle_of(name, dtype):
    return Oracle(model(name), {k: synth.bf16_to_f32(v) for k, v in weights(name).items()}, cache_round=bf16_round if dtype == "BF16" else None)


@functools.lru_cache(maxsize=None)
def expected(name, dtype, seed, n):
    """(ids, logits, residual stream after every layer) of a seeded prompt."""
    ids = tuple(int(t) for t in synth.prompt_ids(seed, n, model(name)["vocab"]))
    o = oracle_of(name, dtype)
    logits = o.forward(ids, keep_layers=True)
    return ids, logits, np.stack(o.layers)


@pytest.fixture(scope="module")
def engines(hm, tmp_path_factory):
    """name, dtype -> loaded model (from files)."""
    cache = {}

    def get(name, dtype):
        if (name, dtype) not in cache:
            d = synth.write_tunitar_model(str(tmp_path_factory.mktemp(name)), model(name), 21, weights(name))
            cache[name, dtype] = hm.HfModel.load_with_dtype(d, hm.DType[dtype])
        return cache[name, dtype]

    yield get
    for m in cache.values():
        m.close()


def close(got, want, dtype, what):
    err, ref = float(np.abs(got - want).max()), float(np.abs(want).max())
    record_error(f"tunitar {what} ({dtype})", err, ref)
    assert err <= TOL[dtype] * max(ref, 1e-3), (what, err, ref)


def run_portions(m, ids, portions, seq=0, hidden=False):
    """Logits of every position, the prompt cut into the given portions (the last one repeats)."""
    out, layers, pos, i = [], [], 0, 0
    while pos < len(ids):
        n = min(portions[min(i, len(portions) - 1)], len(ids) - pos)
        lg, _, h = m.step([(seq, ids[pos : pos + n], range(n))], want_hidden=hidden)
        out.append(lg)
        layers.append(h)
        pos, i = pos + n, i + 1
    return (np.concatenate(out), np.concatenate(layers, axis=1)) if hidden else np.concatenate(out)


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("name", NAMES)
def test_layers_and_logits_of_a_prompt(hm, engines, name, dtype):
    ids, want, layers = expected(name, dtype, 1, 150)
    m = engines(name, dtype)
    assert m.architecture() == "Tunitar"
    m.init_kv_cache(256, batch=2, kv_dtype=hm.DType[dtype])
    got, hidden = run_portions(m, ids, [150], seq=1, hidden=True)
    for i in range(len(layers)):
        close(hidden[i], layers[i], dtype, "residual stream")
    close(got, want, dtype, "logits of a prompt")


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("portions", [[1], [2], [3, 64, 5, 2, 61], [7], [9], [63, 1, 65]])
def test_cuts_do_not_matter(hm, engines, name, dtype, portions):
    """Token by token (up to the first page's edge and beyond), portions of two tokens, portions across pages and passes."""
    ids, want, _ = expected(name, dtype, 1, 150)
    m = engines(name, dtype)
    m.init_kv_cache(256, batch=1, kv_dtype=hm.DType[dtype])
    close(run_portions(m, ids, portions), want, dtype, "logits of portions")


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_decoding_far_into_a_sequence(hm, engines, name, dtype):
    """Prompt through hm_prefill, then the captured decode step token by token: across several pages and a 128-token tile."""
    ids, want, _ = expected(name, dtype, 2, 420)
    m = engines(name, dtype)
    m.init_kv_cache(448, batch=1, kv_dtype=hm.DType[dtype])
    n0 = 187
    tok, lg = m.prefill(ids[:n0], want_logits=True)
    close(lg, want[n0 - 1], dtype, "logits of a prefill")
    got = np.stack([m.decode_step([t])[0][0] for t in ids[n0:]])
    close(got, want[n0:], dtype, "logits of decoded tokens")
    assert m.kv_cache_len() == 420


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_mixed_batches_and_reused_pages(hm, engines, name, dtype):
    """Unequal requests in shared batches, pausing and ending, over a pool too small for all of them at once."""
    m = engines(name, dtype)
    session = Session(m, 3, 6 * 64, kv_dtype=hm.DType[dtype])
    lengths = {"a": 130, "b": 3, "c": 64, "d": 129, "e": 1, "f": 65, "g": 190}
    full = {k: expected(name, dtype, 30 + i, n) for i, (k, n) in enumerate(lengths.items())}
    g = np.random.default_rng(4)
    at, waiting, live = dict.fromkeys(lengths, 0), list(lengths), []
    pages = lambda k: -(-lengths[k] // 64)
    while waiting or live:
        while waiting and len(live) < 3 and sum(map(pages, live)) + pages(waiting[0]) <= 6:
            live.append(waiting.pop(0))
        chosen = [k for k in live if g.random() < 0.8] or live[:1]
        entries, want = [], []
        for k in chosen:
            n = min(int(g.choice([1, 1, 2, 5, 29, 64])), lengths[k] - at[k])
            places = [p for p in range(n) if g.random() < 0.6]
            entries.append((k, full[k][0][at[k] : at[k] + n], places))
            want += [full[k][1][at[k] + p] for p in places]
            at[k] += n
        logits, _ = session.step(entries)
        if want:
            close(logits, np.stack(want), dtype, "logits of mixed batches")
        for k in chosen:
            if at[k] == lengths[k]:
                session.end(k)
                live.remove(k)
    assert m.free_tokens() == 6 * 64


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
def test_a_slot_starts_from_nothing(hm, engines, dtype):
    """The first token of a request that takes over a slot sees neither the old cache nor the old predecessor row."""
    m = engines("mixed", dtype)
    m.init_kv_cache(128, batch=1, kv_dtype=hm.DType[dtype], pool_tokens=128)
    a, b = expected("mixed", dtype, 50, 100), expected("mixed", dtype, 51, 20)
    for ids, want, _ in (a, b, a):
        m.reset_kv_cache(0)
        close(run_portions(m, ids[:1], [1]), want[:1], dtype, "first token")
        close(run_portions(m, ids[1:], [17]), want[1:], dtype, "reused slot")


def test_latents_in_the_cache(hm, engines):
    ids, _, _ = expected("mixed", "F32", 60, 90)
    o = oracle_of("mixed", "F32")
    o.forward(ids)
    m = engines("mixed", "F32")
    m.init_kv_cache(128, batch=2, kv_dtype=hm.DType.F32)
    run_portions(m, ids, [90], seq=1)
    for layer, owner in ((0, 0), (1, 1), (2, 0), (3, 1)):
        c = o.latents[owner]
        close(m.latent_view(layer, c.shape[1], seq=1), c, "F32", "cached latents")
    with pytest.raises(hm.HomuraError):
        m.kv_view(0)
