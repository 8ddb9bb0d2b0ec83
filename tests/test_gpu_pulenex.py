"""Pulenex models on the engine, against the plain float64 oracle."""
import functools
import json

import numpy as np
import pytest
from conftest import record_error
from pulenex_cases import NAMES, RANKS, model

from pulenex_oracle import Oracle, layer_norm, rotate_neighbours, rotation_frequencies, short_convolution
from homura_b200 import synth
from homura_b200.serving import Scheduler, Session

pytestmark = pytest.mark.gpu

# relative to the largest reference value: f32 throughout; bf16 pages against an oracle that rounds its keys and values alike (one on
# the edge of a rounding step may go the other way)
TOL = {"F32": 3e-5, "BF16": 4e-3}


def bf16_round(x):
    return synth.bf16_to_f32(synth.f32_to_bf16_rne(np.ascontiguousarray(x, np.float32))).astype(np.float64)


@functools.lru_cache(maxsize=None)
def weights(name):
    return synth.pulenex_weights(model(name), 21, RANKS[name])


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
            d = synth.write_pulenex_model(str(tmp_path_factory.mktemp(name)), model(name), 21, weights(name), RANKS[name])
            cache[name, dtype] = hm.HfModel.load_with_dtype(d, hm.DType[dtype])
        return cache[name, dtype]

    yield get
    for m in cache.values():
        m.close()


def close(got, want, dtype, what):
    rows = np.abs(got - want).reshape(-1, want.shape[-1]).max(1)
    err, ref = float(rows.max()), float(np.abs(want).max())
    record_error(f"pulenex {what} ({dtype})", err, ref)
    assert err <= TOL[dtype] * max(ref, 1e-3), (what, int(rows.argmax()), len(rows), err, ref)


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
    assert m.architecture() == "Pulenex"
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
@pytest.mark.parametrize("name", ["mixed", "odd", "far", "windows", "shared", "large"])
def test_decoding_far_into_a_sequence(hm, engines, name, dtype):
    """Prompt through hm_prefill, then the captured decode step token by token: across pages and windows."""
    n = 700 if name == "far" else 330
    ids, want, _ = expected(name, dtype, 2, n)
    m = engines(name, dtype)
    m.init_kv_cache(n + 20, batch=1, kv_dtype=hm.DType[dtype])
    n0 = 187
    tok, lg = m.prefill(ids[:n0], want_logits=True)
    close(lg, want[n0 - 1], dtype, "logits of a prefill")
    got = np.stack([m.decode_step([t])[0][0] for t in ids[n0:]])
    close(got, want[n0:], dtype, "logits of decoded tokens")
    assert m.kv_cache_len() == n


def conspicuous(cfg, w, token):
    """Every query of a one-layer model looks for one token: its key stands out by far, whatever the distance."""
    w = dict(w)
    f = {k: synth.bf16_to_f32(v).copy() for k, v in w.items()}
    m, p = cfg["layers"][0]["mixer"], "l0.mix."
    e = f["embed"]
    e[:, :2] = 0
    e[:, 1] = 3.0       # an element that all tokens share: the queries' direction
    e[token] = 0
    e[token, :2] = 8.0  # and one that only this token has
    if "left" in m:
        m, p = m["left"], p + "left."
        f["l0.mix.right.out"] *= 0  # (a state forgets slowly)
        for t in "qk":
            f[p + t + ".conv"] *= 0
            f[p + t + ".conv"][:, -1] = 1
        f[p + "talk"] = np.abs(f[p + "talk"])
        q, k, last = f[p + "q"] * 0, f[p + "k"] * 0.05, m["dim"] - 1  # the last element of a head is not rotated
        assert m["rot"]["dims"] < m["dim"]
        q[last :: m["dim"], 1] = 8.0
        k[last :: m["dim"], 0] = 8.0
        f[p + "k"] = k
    else:
        q, d = f[p + "q"] * 0, m["dim"]
        q[0 :: d + m["rot_dim"], 1] = 8.0  # an unrotated element
        f[p + "dkv"] *= 0.05
        f[p + "dkv"][0, 0] = 8.0           # the first of a latent
        f[p + "uk"] *= 0.05
        f[p + "uk"][0::d, 0] = 4.0
    f[p + "q"] = q
    return {k: synth.f32_to_bf16_rne(v.astype(np.float32)) for k, v in f.items()}


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("name,layer", [("far", 0), ("far", 1), ("parallel", 0), ("latent", 0), ("windows", 0), ("windows", 2), ("windows", 3), ("windows", 4), ("windows", 8), ("shared", 3)])
def test_a_conspicuous_key_is_seen_exactly_inside_its_window_or_chunk(hm, tmp_path, name, layer, dtype):
    """One token that every query looks for, at page borders and at the edges of chunks: its value comes back up to the last place that
    sees it and not one further, in prompts and in decoding."""
    cfg = model(name)
    spec = cfg["layers"][layer]
    spec["mixer"].pop("kv_from", None)
    cfg["layers"] = [{**spec, "mlp": None}]
    w = conspicuous(cfg, synth.pulenex_weights(cfg, 21, RANKS[name]), 7)
    chunked = "left" in spec["mixer"]
    size = (spec["mixer"]["left"] if chunked else spec["mixer"])["mask"]["size"]
    o = Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in w.items()}, cache_round=bf16_round if dtype == "BF16" else None)
    n = 2 * size + 200
    ids = [int(t) if t != 7 else 8 for t in synth.prompt_ids(3, n, cfg["vocab"])]
    m = hm.HfModel.load_with_dtype(synth.write_pulenex_model(str(tmp_path), cfg, 21, w, RANKS[name]), hm.DType[dtype])
    without = o.forward(ids)
    for at in sorted({0, 63, 64, 100, size - 1, size}):
        with_it = ids[:at] + [7] + ids[at + 1 :]
        want = o.forward(with_it)
        changed = np.abs(want - without).max(1) / np.abs(want).max()
        end = (at // size + 1) * size if chunked else at + size  # the first place that does not see it
        if end - 1 > at:
            assert changed[end - 1] > 1e-2
        assert changed[max(end, at + 1) :].max() < 1e-6  # (queries look at no other token's embedding)
        m.init_kv_cache(n + 20, batch=1, kv_dtype=hm.DType[dtype])
        cut = max(end - 6, 3)
        got = run_portions(m, with_it[:cut], [cut - 2, 2])
        close(got, want[:cut], dtype, "logits of a prompt with one conspicuous key")
        got = np.stack([m.decode_step([t])[0][0] for t in with_it[cut : cut + 12]])
        close(got, want[cut : cut + 12], dtype, "logits of tokens decoded around an edge")
        got = run_portions(m, with_it[cut + 12 :], [2, 30])
        close(got, want[cut + 12 :], dtype, "logits behind an edge")
    m.close()


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
def test_a_strong_sink_and_a_weak_one(hm, tmp_path, dtype):
    """Sinks that swallow nearly everything, or nothing."""
    cfg = model("mixed")
    ids = synth.prompt_ids(5, 90, cfg["vocab"])
    for value in (30.0, -40.0):
        w = {k: synth.f32_to_bf16_rne(np.where(np.arange(len(v)) % 2 == 0, value, synth.bf16_to_f32(v)).astype(np.float32)) if k.endswith("sink") else v for k, v in weights("mixed").items()}
        o = Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in w.items()}, cache_round=bf16_round if dtype == "BF16" else None)
        m = hm.HfModel.load_with_dtype(synth.write_pulenex_model(str(tmp_path / str(value)), cfg, 21, w, RANKS["mixed"]), hm.DType[dtype])
        want = o.forward(ids)
        for portions in ([90], [50, 1, 2]):
            m.init_kv_cache(128, batch=1, kv_dtype=hm.DType[dtype])
            close(run_portions(m, ids, portions), want, dtype, "logits with sinks")
        m.close()


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("fast", [True, False])
def test_decays_of_every_speed(hm, tmp_path, fast, dtype):
    """Delta-rule channels that forget at once (their logarithm far below what a product of decays could keep) or hardly ever, with steps
    near one and near zero; retention from nothing to everything."""
    cfg = model("parallel")
    cfg["layers"].append({**synth.pulenex_retention(4, 16, 24, decay=[0.0, 0.125, 1.0, 0.9990234375]), "mlp": None})
    w = {k: synth.bf16_to_f32(v).copy() for k, v in synth.pulenex_weights(cfg, 21, RANKS["parallel"]).items()}
    w["l0.mix.right.A_log"][:] = [3.0, 2.0, 0.0, -8.0] if fast else [-12.0, -6.0, -4.0, -9.0]
    w["l0.mix.right.dt_bias"] += np.where(np.arange(len(w["l0.mix.right.dt_bias"])) % 3 == 0, 30.0, 3.0) if fast else -4.0
    w["l0.mix.right.b"] *= 8.0
    w = {k: synth.f32_to_bf16_rne(v.astype(np.float32)) for k, v in w.items()}
    o = Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in w.items()}, cache_round=bf16_round if dtype == "BF16" else None)
    ids = synth.prompt_ids(6, 400, cfg["vocab"])
    want = o.forward(ids)
    m = hm.HfModel.load_with_dtype(synth.write_pulenex_model(str(tmp_path), cfg, 21, w, RANKS["parallel"]), hm.DType[dtype])
    for portions in ([400], [200, 2, 1, 31]):
        m.init_kv_cache(512, batch=1, kv_dtype=hm.DType[dtype])
        close(run_portions(m, ids, portions), want, dtype, "logits with extreme decays")
    m.close()


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
def test_a_state_carries_a_token_a_long_way(hm, tmp_path, dtype):
    """Retention that forgets nothing, queries that look for one token's key: its value is still there hundreds of tokens later, whatever
    the cuts."""
    cfg = synth.pulenex_config(64, 80, [(synth.pulenex_retention(4, 24, 24, synth.pulenex_rot(16), [1.0] * 4), None)])
    f = {k: synth.bf16_to_f32(v).copy() for k, v in synth.pulenex_weights(cfg, 21).items()}
    f["embed"][:, :2] = [0, 3.0]
    f["embed"][7] = 0
    f["embed"][7, :2] = 8.0
    for t, c in (("q", 1), ("k", 0)):
        f["l0.mix." + t] *= 0.02
        f["l0.mix." + t][23::24, c] = 8.0  # an element that is not rotated
    w = {k: synth.f32_to_bf16_rne(v) for k, v in f.items()}
    o = Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in w.items()})
    ids = [int(t) if t != 7 else 8 for t in synth.prompt_ids(3, 600, 80)]
    without = o.forward(ids)
    m = hm.HfModel.load_with_dtype(synth.write_pulenex_model(str(tmp_path), cfg, 21, w), hm.DType[dtype])
    for at in (0, 64, 70):
        with_it = ids[:at] + [7] + ids[at + 1 :]
        want = o.forward(with_it)
        assert np.abs(want - without)[-1].max() > 0.01 * np.abs(want).max()
        m.init_kv_cache(640, batch=1, kv_dtype=hm.DType[dtype])
        close(run_portions(m, with_it[:590], [at + 1, 2, 100]), want[:590], dtype, "logits far behind a conspicuous token")
        got = np.stack([m.decode_step([t])[0][0] for t in with_it[590:]])
        close(got, want[590:], dtype, "logits decoded far behind a conspicuous token")
    m.close()


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
    all_got, all_want = [], []
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
            all_got.append(logits)
            all_want += want
        for k in chosen:
            if at[k] == lengths[k]:
                session.end(k)
                live.remove(k)
    close(np.concatenate(all_got), np.stack(all_want), dtype, "logits of mixed batches")
    assert m.free_tokens() == 6 * 64


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
@pytest.mark.parametrize("name", ["large", "parallel", "retention", "odd", "mixed"])
def test_many_sequences_in_a_pass(hm, engines, name, dtype):
    """Forty sequences: a prompt each, then passes that mix single tokens with portions, then the captured step."""
    m = engines(name, dtype)
    m.init_kv_cache(64, batch=40, kv_dtype=hm.DType[dtype])
    full = [expected(name, dtype, 100 + b % 4, 24) for b in range(40)]
    m.step([(b, full[b][0][: 3 + b % 5], []) for b in range(40)], want_logits=False)
    at = [3 + b % 5 for b in range(40)]
    for wide in (0, 1):
        n = [1 + (b % 3 if wide else 0) for b in range(40)]
        got, _, _ = m.step([(b, full[b][0][at[b] : at[b] + n[b]], [n[b] - 1]) for b in range(40)])
        at = [a + k for a, k in zip(at, n)]
        close(got, np.stack([full[b][1][at[b] - 1] for b in range(40)]), dtype, "logits of many sequences")
    lg, _ = m.decode_step([full[b][0][at[b]] for b in range(40)])
    close(lg, np.stack([full[b][1][at[b]] for b in range(40)]), dtype, "logits of a captured step of many sequences")


@pytest.mark.parametrize("dtype", ["F32", "BF16"])
def test_a_slot_starts_from_nothing(hm, engines, dtype):
    """A request that takes over a slot sees neither the old keys nor the old states."""
    m = engines("mixed", dtype)
    m.init_kv_cache(128, batch=1, kv_dtype=hm.DType[dtype], pool_tokens=128)
    a, b = expected("mixed", dtype, 50, 100), expected("mixed", dtype, 51, 20)
    for ids, want, _ in (a, b, a):
        m.reset_kv_cache(0)
        close(run_portions(m, ids[:1], [1]), want[:1], dtype, "first token")
        close(run_portions(m, ids[1:], [17]), want[1:], dtype, "reused slot")


def test_what_is_in_a_batch_does_not_matter(hm, engines):
    """The same request alone and beside others, on the same kernels: equal to the last bit where the shapes are equal."""
    m = engines("mixed", "BF16")
    ids, _, _ = expected("mixed", "BF16", 1, 150)
    m.init_kv_cache(256, batch=3, kv_dtype=hm.DType.BF16)
    m.step([(0, ids[:60], [])], want_logits=False)
    alone, _, _ = m.step([(0, ids[60:70], range(10))])
    m.reset_kv_cache()
    m.step([(0, ids[:60], []), (1, ids[5:9], [])], want_logits=False)
    beside, _, _ = m.step([(1, ids[:3], []), (0, ids[60:70], range(10)), (2, ids[:2], [])])
    assert np.abs(alone - beside).max() < 1e-4 * np.abs(alone).max()


def test_caches_can_be_read(hm, engines):
    ids, _, _ = expected("mixed", "F32", 60, 90)
    m = engines("mixed", "F32")
    m.init_kv_cache(128, batch=2, kv_dtype=hm.DType.F32)
    run_portions(m, ids, [90], seq=1)
    o = oracle_of("mixed", "F32")
    h = layer_norm(o.w["embed"][list(ids)], o.w["l0.norm1"], o.eps)
    mx = model("mixed")["layers"][0]["mixer"]["left"]
    k, v = m.kv_view(0, seq=1, shape=(mx["kv_heads"], mx["dim"], mx["vdim"]))
    plain = short_convolution(h @ o.w["l0.mix.left.k"].T, o.w["l0.mix.left.k.conv"]).reshape(90, mx["kv_heads"], -1)
    turned = rotate_neighbours(plain, rotation_frequencies(mx["rot"]["dims"], mx["rot"]["base"]))
    for got, want in ((k, turned), (v, plain)):
        close(got[0], want.transpose(1, 0, 2), "F32", "cached keys and values")
    lat = model("mixed")["layers"][2]["mixer"]
    c, again = (m.latent_view(i, lat["kv_rank"] + lat["rot_dim"], seq=1) for i in (2, 4))
    assert c.shape[-1] == lat["kv_rank"] + lat["rot_dim"] and np.isfinite(c).all() and (c == again).all()
    for layer in (1, 2):
        with pytest.raises(hm.HomuraError):
            m.kv_view(layer, seq=1, shape=(1, 8, 8))


# ---- generation through the engine's own loops and the scheduler ---------------------------------


@functools.lru_cache(maxsize=None)
def greedy(name, seed, n_prompt, n_new):
    ids = tuple(int(t) for t in synth.prompt_ids(seed, n_prompt, model(name)["vocab"]))
    return ids, tuple(oracle_of(name, "F32").greedy(ids, n_new))


def test_greedy_generation(hm, engines):
    ids, want = greedy("mixed", 70, 37, 60)
    m = engines("mixed", "F32")
    m.init_kv_cache(128, batch=1, kv_dtype=hm.DType.F32)
    assert tuple(m.generate_ids(ids, 60, hm.SamplingConfig.greedy())) == want


def test_batched_decode_graph(hm, engines):
    """Three, twelve (tensor-core projections) and seventy sequences decode together what each decodes alone."""
    for batch in (3, 12, 70):
        m = engines("mixed", "F32" if batch == 3 else "BF16")
        m.init_kv_cache(64, batch=batch, kv_dtype=hm.DType.F32)
        refs = [greedy("mixed", 80 + b % 6, 5 + b % 6, 12) for b in range(batch)]
        first = [m.prefill(ids, seq=b) for b, (ids, _) in enumerate(refs)]
        rest = m.decode_greedy_n(first, 11)
        for b, (_, want) in enumerate(refs):
            assert (first[b], *rest[b].tolist()) == want


def test_scheduler_generates_what_each_prompt_generates_alone(hm, engines):
    refs = [greedy("mixed", 90 + i, n, 20) for i, n in enumerate((70, 1, 33, 150, 2, 64))]
    m = engines("mixed", "F32")
    sched = Scheduler(Session(m, 3, 5 * 64, kv_dtype=hm.DType.F32), portion=24, batch_tokens=40)
    assert [tuple(o) for o in sched.run([ids for ids, _ in refs], 20)] == [want for _, want in refs]
    assert m.free_tokens() == 5 * 64
    with pytest.raises(hm.KvCacheFull):
        sched.run([[1] * 400], 4)


def test_sampled_generation_matches_the_host_sampler(hm, engines):
    cfg = hm.SamplingConfig(temperature=0.8, top_k=12, top_p=0.9, repetition_penalty=1.2, seed=5)
    ids, _ = greedy("mixed", 70, 37, 60)
    m = engines("mixed", "F32")
    m.init_kv_cache(128, batch=1, kv_dtype=hm.DType.F32)
    got = m.generate_ids(ids, 25, cfg)
    m.reset_kv_cache()
    cur, rng, out = m.prefill(ids), 5 | 1, []
    out.append(cur)
    for _ in range(24):
        lg, _ = m.decode_step([cur])
        cur, rng = hm.sample_token(lg[0], cfg, out, rng)
        out.append(cur)
    assert got == out


def test_a_conversation_goes_on_after_the_end_token(hm, tmp_path):
    """Generation runs ahead of the host in blocks; what the end token cut off must leave no trace in the next turn."""
    cfg = model("mixed")
    ids, out = greedy("mixed", 70, 37, 60)
    k = next(i for i in range(5, 31) if out[i] not in out[:i])
    cfg["eos_token_id"] = int(out[k])
    m = hm.HfModel.load_with_dtype(synth.write_pulenex_model(str(tmp_path), cfg, 21, weights("mixed"), RANKS["mixed"]), hm.DType.F32)
    m.init_kv_cache(128, batch=1, kv_dtype=hm.DType.F32)
    got = m.generate_ids(ids, 60, hm.SamplingConfig.greedy())
    assert tuple(got) == out[:k] and m.kv_cache_len() == len(ids) + k
    more = [3, 1, 4, 1, 5]
    _, lg = m.prefill(more, want_logits=True)
    close(lg, oracle_of("mixed", "F32").forward([*ids, *out[:k], *more])[-1], "F32", "second turn")
    m.close()


def test_tensors_one_by_one_and_missing_ones(hm):
    cfg = model("odd")
    tensors = [(n, hm.DType.BF16, s, weights("odd")[n]) for n, s, _ in synth.pulenex_tensor_specs(cfg, RANKS["odd"])]
    tensors.sort(key=lambda t: t[0][::-1])  # any order will do
    ids, want, _ = expected("odd", "F32", 1, 150)
    m = hm.HfModel.from_config_json(json.dumps(cfg), tensors, hm.DType.F32)
    m.init_kv_cache(64, batch=1, kv_dtype=hm.DType.F32)
    close(run_portions(m, ids[:30], [30]), want[:30], "F32", "logits of a prompt")
    m.close()
    for drop in ("embed", "head", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.left.q.conv", "l0.mix.left.talk", "l0.mix.left.temp", "l0.mix.left.sink", "l0.mix.left.out", "l0.mix.right.a1", "l0.mix.right.g1",
                 "l0.mix.right.g2", "l0.mix.right.v.conv", "l0.mix.right.A_log", "l0.mix.right.dt_bias", "l0.mix.right.norm", "l0.mix.right.o", "l0.mlp.gate.b", "l0.mlp.down.b", "l1.mix.dkv.norm", "l1.mix.uk", "l1.mix.g", "l2.mix.v", "l2.mlp.up"):
        with pytest.raises(hm.HomuraError) as e:
            hm.HfModel.from_config_json(json.dumps(cfg), [t for t in tensors if t[0] != drop])
        assert "missing weight" in e.value.message
    sizes = [t for t in tensors if t[0] in ("l0.mix.right.a1", "l0.mix.right.g1")]
    for name, shape in (("l0.mix.left.q.conv", (55, 3)), ("l0.mix.left.talk", (5, 4)), ("l0.mix.left.v", (11, 130)), ("l0.mix.right.a2", (42, 3)), ("l0.mix.right.k", (42, 130)), ("l0.mlp.up", (34, 130)), ("l0.mlp.up.b", (34,)),
                        ("l1.mix.q", (44, 130)), ("l1.mix.dkv", (29, 130)), ("l1.mix.g", (33, 130)), ("l2.mix.q", (36, 130)), ("l3.norm2", (130,)), ("head", (76, 130))):
        with pytest.raises(hm.HomuraError):
            hm.HfModel.from_config_json(json.dumps(cfg), sizes + [(name, hm.DType.BF16, shape, np.zeros(shape, np.uint16))])


def test_a_sharded_checkpoint(hm, tmp_path):
    """Shapes that tell sizes may lie in another shard than the tensors they size."""
    d = synth.write_pulenex_model(str(tmp_path / "one"), model("mixed"), 21, weights("mixed"), RANKS["mixed"])
    ids, want, _ = expected("mixed", "F32", 1, 150)
    for n in (2, 5):
        m = hm.HfModel.load_with_dtype(synth.shard_hf_model(d, str(tmp_path / str(n)), n), hm.DType.F32)
        m.init_kv_cache(256, batch=1, kv_dtype=hm.DType.F32)
        close(run_portions(m, ids, [150]), want, "F32", "logits of a sharded checkpoint")
        m.close()


def test_step_refuses_bad_entries_and_keeps_its_state(hm, engines):
    ids, want, _ = expected("mixed", "F32", 1, 150)
    m = engines("mixed", "F32")
    m.init_kv_cache(128, batch=2, kv_dtype=hm.DType.F32, pool_tokens=128)
    close(run_portions(m, ids[:40], [40]), want[:40], "F32", "logits of a prompt")
    for bad in ([(0, [1], [0]), (0, [2], [])], [(2, [1], [])], [(0, [], [])], [(0, [100], [])], [(0, [1, 2], [1, 0])]):
        with pytest.raises(hm.HomuraError):
            m.step(bad)
    with pytest.raises(hm.KvCacheFull):
        m.step([(0, [1] * 60, []), (1, [1] * 10, [])])
    assert (m.kv_cache_len(0), m.kv_cache_len(1), m.free_tokens()) == (40, 0, 64)
    close(run_portions(m, ids[40:90], [50]), want[40:90], "F32", "logits after a refusal")


def test_the_trace_runner_replays_steps(hm, tmp_path):
    import os
    import subprocess
    import sys

    ids, want, _ = expected("odd", "F32", 1, 150)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    d = synth.write_pulenex_model(str(tmp_path / "model"), model("odd"), 21, weights("odd"), RANKS["odd"])
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": ids[:50], "want": [2, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": ids[:9], "want": []}, {"id": "p", "tokens": ids[50:51], "want": []}], "end": ["p"]},
             {"step": 2, "entries": [{"id": "q", "tokens": ids[9:11], "want": [1]}, {"id": "r", "tokens": ids[:64], "want": [63]}], "end": ["q", "r"]}]
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(map(json.dumps, steps)), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    read = lambda n: np.fromfile(out / f"{n}.f32", "<f4").reshape(-1, 77)
    close(read(0), want[[2, 49]], "F32", "replayed logits")
    assert not (out / "1.f32").exists()
    close(read(2), want[[10, 63]], "F32", "replayed logits")


def test_generation_on_the_command_line(hm, tmp_path, capsys):
    from homura_b200.__main__ import main

    d = synth.write_pulenex_model(str(tmp_path), model("mixed"), 21, weights("mixed"), RANKS["mixed"])
    refs = [greedy("mixed", 70, 37, 60), greedy("mixed", 90, 70, 20)]
    args = ["generate", d, "--max-new", "20", "--dtype", "f32"]
    for ids, _ in refs:
        args += ["--ids", ",".join(map(str, ids))]
    assert main(args) == 0
    assert capsys.readouterr().out.split() == [",".join(map(str, want[:20])) for _, want in refs]
