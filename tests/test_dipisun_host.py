"""CPU tests of the Dipisun design: config reader, checkpoint description, oracle."""
import copy
import json

import numpy as np
import pytest
from dipisun_cases import BUCKETS, NAMES, model

import dipisun_oracle as do
from homura_b200 import synth


def oracle_of(cfg, seed=5, buckets=12, **kw):
    return do.Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in synth.dipisun_weights(cfg, seed, buckets).items()}, **kw)


@pytest.mark.parametrize("name", NAMES)
def test_checkpoint_info_reads_the_layer_list(hm, tmp_path, name):
    cfg = model(name)
    info = hm.checkpoint_info(synth.write_dipisun_model(str(tmp_path), cfg, 1, buckets=BUCKETS[name]))
    c = info["config"]
    assert c["architecture"] == "Dipisun"
    assert (c["hidden_size"], c["vocab_size"], c["num_hidden_layers"]) == (cfg["width"], cfg["vocab"], len(cfg["layers"]))
    first = next((i for i, e in enumerate(cfg["layers"]) if e["mixer"].get("v_mix")), None)
    for got, want in zip(c["layers"], cfg["layers"]):
        m = want["mixer"]
        assert [got[k] for k in ("heads", "kv_heads", "dim", "vdim")] == [m[k] for k in ("heads", "kv_heads", "dim", "vdim")]
        assert got["scale"] == pytest.approx(m["scale"], rel=1e-6) and got["bias_reach"] == m.get("bias_max", 0)
        t = m.get("q_temp") or {"coef": 0, "every": 0}
        assert (got["temp_coef"], got["temp_every"]) == (pytest.approx(t["coef"]), t["every"])
        assert got["v_first"] == (first if m.get("v_mix") else None)
        assert got["qk_norm"] == ("all" if want["type"] == "attention" else "head")
        f = want["mlp"]
        assert [got[k] for k in ("ff", "experts", "identity", "top")] == ([f["expert"]["ff"], f["router"]["experts"], f["router"]["identity"], f["router"]["top"]] if f else [0, 0, 0, 0])
    assert len(info["tensors"]) == len(synth.dipisun_tensor_specs(cfg))


@pytest.mark.parametrize("edit", [
    lambda c: c.pop("width"),
    lambda c: c.pop("residual_mult"),
    lambda c: c["norm"].pop("eps"),
    lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="attention_3"),
    lambda c: c["layers"][0]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mixer"].pop("bias_max"),
    lambda c: c["layers"][0]["mixer"]["q_temp"].pop("every"),
    lambda c: c["layers"][0]["mixer"].update(kv_heads=4),          # does not divide the heads
    lambda c: c["layers"][2]["mixer"].update(vdim=47),             # blends values of another size
    lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=8),       # more than there are
    lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"),
])
def test_config_errors_are_reported(hm, tmp_path, edit):
    cfg = copy.deepcopy(model("mixed"))
    edit(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(hm.HomuraError) as e:
        hm.checkpoint_info(str(tmp_path))
    assert "config.json" in e.value.message and e.value.status == hm.HM_ERR_IO


# ---- the oracle's pieces against values worked out by hand -------------------------------------


def test_position_vectors():
    v = do.position_vectors([0, 3], 4)
    assert np.allclose(v, [[0, 1, 0, 1], [np.sin(3), np.cos(3), np.sin(0.03), np.cos(0.03)]])
    assert np.allclose(do.position_vectors([1], 3), [[np.sin(1), np.cos(1), np.sin(10000 ** (-2 / 3))]])


def test_temperature_steps_after_every_so_many_tokens():
    t = do.temperature([0, 6, 7, 14, 15, 22], 0.5, 8)
    assert np.allclose(t, 1 + 0.5 * np.log([1, 1, 2, 2, 3, 3]))


def test_distance_buckets():
    # eight rows: distances 0..3 by themselves, then steps of a factor 2 up to 64
    want = {0: 0, 3: 3, 4: 4, 7: 4, 8: 5, 15: 5, 16: 6, 31: 6, 32: 7, 63: 7, 64: 7, 1000: 7}
    assert {n: do.distance_bucket(n, 8, 64) for n in want} == want
    assert [do.distance_bucket(n, 2, 3) for n in range(4)] == [0, 1, 1, 1]
    assert [do.distance_bucket(n, 7, 33) for n in (2, 3, 5, 6, 32, 33)] == [2, 3, 3, 4, 6, 6]


def test_norms_of_queries():
    q = np.array([[3.0, 4.0, 0.0, 2.0]])
    w = np.array([1.0, 2.0])
    assert np.allclose(do.norm_each_head(q, w, 2, 0.0), [[3 / 12.5**0.5, 8 / 12.5**0.5, 0.0, 4 / 2**0.5]])
    assert np.allclose(do.norm_all_heads(q, np.array([1.0, 2.0, 3.0, 4.0]), 0.0), np.array([[3.0, 8.0, 0.0, 8.0]]) / 7.25**0.5)


def test_grouped_attention_by_hand():
    # two query heads of one key head: one picks the largest key, the other is driven by its bias to the token before
    k = np.array([[1.0], [5.0], [3.0]])
    bias = np.zeros((3, 3, 2))
    bias[1:, :, 1] = -1e3
    bias[1, 0, 1] = bias[2, 1, 1] = 0
    out = do.grouped_attention(np.array([[100.0, 0.0]] * 3), k, k * 10, 2, 1, 1.0, bias)
    assert np.allclose(out, [[10, 10], [50, 10], [50, 50]])


def test_router_weights_are_the_scores_of_a_corrected_choice():
    z = np.log(np.array([[0.5, 0.3, 0.15, 0.05]]))
    chosen, weights = do.route(z, np.array([0.0, 0.0, 0.0, 0.4]), 2)
    assert chosen.tolist() == [[0, 3]] and np.allclose(weights, [[0.5, 0.05]])


def test_expert_clamps():
    one = np.ones((1, 1))
    f = lambda g, u: do.clamped_expert(np.array([[1.0]]), one * g, one * u, one, 2.0)[0, 0]
    sig = lambda z: 1 / (1 + np.exp(-z))
    assert f(5, 7) == pytest.approx(2 * sig(3.404) * 3)          # both held at the limit
    assert f(-5, -7) == pytest.approx(-5 * sig(-8.51) * -1)      # the gate has no lower limit
    assert f(1, 0.5) == pytest.approx(sig(1.702) * 1.5)


def test_mixture_with_identity_experts():
    h = np.array([[2.0, -1.0]])
    z = np.log(np.array([0.6, 0.3, 0.1]))
    router = z[:, None] * np.array([[0.5, 0.0]])  # logits of this token: z
    out = do.mixture(h, router, np.zeros(3), 2, [lambda t: t * 10, lambda t: t, lambda t: t])
    assert np.allclose(out, h * (6.0 + 0.3))


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_oracle_is_causal(name):
    cfg = model(name)
    o = oracle_of(cfg, buckets=BUCKETS[name])
    ids = synth.prompt_ids(3, 40, cfg["vocab"])
    whole = o.forward(ids)
    assert np.allclose(o.forward(ids[:17]), whole[:17], rtol=0, atol=1e-10)


def _weights(o, end, value):
    o.w.update({k: np.full_like(v, value) for k, v in o.w.items() if k.endswith(end)})


# Each mistake must show in the logits of the test models far above the tolerances of the GPU tests.
MISTAKES = {
    "no distance bias": lambda o: _weights(o, ".rel", 0.0),
    "no query temperature": lambda o: [e["mixer"].pop("q_temp", None) for e in o.cfg["layers"]],
    "temperature one token late": lambda o: [e["mixer"]["q_temp"].update(every=17) for e in o.cfg["layers"] if "q_temp" in e["mixer"]],
    "no query norm weight": lambda o: _weights(o, "q.norm", 1.0),
    "no key norm weight": lambda o: _weights(o, "k.norm", 1.0),
    "values not blended": lambda o: _weights(o, ".vmix", 0.0),
    "no correction": lambda o: _weights(o, ".correction", 0.0),
    "no residual multiplier": lambda o: setattr(o, "mult", 1.0),
    "scale of one": lambda o: [e["mixer"].update(scale=1.0) for e in o.cfg["layers"]],
    "another limit": lambda o: [e["mlp"]["expert"].update(limit=7.0) for e in o.cfg["layers"] if e["mlp"]],
    "another reach": lambda o: [e["mixer"].update(bias_max=25) for e in o.cfg["layers"] if "bias_max" in e["mixer"]],
    "no output norm weight": lambda o: _weights(o, "norm2", 1.0),
    "another eps": lambda o: setattr(o, "eps", o.eps + 0.1),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_shows_in_the_logits(mistake):
    cfg = model("mixed")
    ids = synth.prompt_ids(9, 64, cfg["vocab"])
    want = oracle_of(cfg).forward(ids)
    wrong = oracle_of(copy.deepcopy(cfg))
    MISTAKES[mistake](wrong)
    assert np.abs(wrong.forward(ids) - want).max() > 0.02 * np.abs(want).max()


def test_info_on_the_command_line(hm, tmp_path, capsys):
    from homura_b200.__main__ import main

    assert main(["info", synth.write_dipisun_model(str(tmp_path), model("mixed"), 1, buckets=12)]) == 0
    out = capsys.readouterr().out
    assert "architecture: Dipisun" in out and "layer 3:" in out and "l0.mix.rel  BF16  [12, 6]" in out and "l1.mix.vmix  BF16  []" in out
