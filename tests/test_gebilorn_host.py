"""CPU tests of the Gebilorn design: config reader, checkpoint description, oracle."""
import copy
import json

import numpy as np
import pytest
from gebilorn_cases import NAMES, RANKS, model

import gebilorn_oracle as go
from homura_b200 import synth


def oracle_of(cfg, seed=5, rank=12, **kw):
    return go.Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in synth.gebilorn_weights(cfg, seed, rank).items()}, **kw)


@pytest.mark.parametrize("name", NAMES)
def test_checkpoint_info_reads_the_layer_list(hm, tmp_path, name):
    cfg = model(name)
    info = hm.checkpoint_info(synth.write_gebilorn_model(str(tmp_path), cfg, 1, decay_rank=RANKS[name]))
    c = info["config"]
    assert c["architecture"] == "Gebilorn" and c["tie_word_embeddings"]
    assert (c["hidden_size"], c["vocab_size"], c["num_hidden_layers"]) == (cfg["width"], cfg["vocab"], len(cfg["layers"]))
    for got, want in zip(c["layers"], cfg["layers"]):
        m, f = want["mixer"], want["mlp"]
        if want["type"] == "latent_attention":
            assert got["type"] == "latent_attention"
            assert [got[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")] == [m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")]
        else:
            a = m["left"] if want["type"] == "parallel" else m
            assert got["type"] == ("parallel" if want["type"] == "parallel" else "windowed_attention")
            assert [got[k] for k in ("heads", "kv_heads", "dim", "vdim")] == [a[k] for k in ("heads", "kv_heads", "dim", "vdim")]
            assert (got["window"], got["keep_first"], got["conv"]) == (a["mask"]["size"], a["mask"].get("keep_first", 0), a.get("conv", 0))
            m = a
        assert got["scale"] == pytest.approx(m["scale"], rel=1e-6)
        if "rot" in m:
            s = m["rot"].get("scaling") or {}
            assert (got["rot"]["dims"], got["rot"]["base"]) == (m["rot"]["dims"], m["rot"]["base"]) and {k: got["rot"][k] for k in s} == s
        if want["type"] == "parallel":
            r = want["mixer"]["right"]
            assert got["linear"] == {k: pytest.approx(r[k]) for k in ("heads", "dim", "vdim", "tau")}
            assert (got["left_scale"], got["right_scale"]) == (pytest.approx(want["mixer"]["left_scale"]), pytest.approx(want["mixer"]["right_scale"]))
        moe = f is not None and f["kind"] == "moe"
        assert got["ff"] == (0 if f is None else f["expert"]["ff"] if moe else f["ff"])
        assert [got[k] for k in ("experts", "top", "shared_ff")] == ([f["router"]["experts"], f["router"]["top"], f["shared"]["ff"]] if moe else [0, 0, 0])
    assert len(info["tensors"]) == len(synth.gebilorn_tensor_specs(cfg))


@pytest.mark.parametrize("edit", [
    lambda c: c.pop("width"),
    lambda c: c["norm"].pop("eps"),
    lambda c: c["embedding"].pop("scale"),
    lambda c: c["embedding"]["bigram"].pop("mul_cur"),
    lambda c: c.update(logit_softcap=-1.0),
    lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="attention_2"),
    lambda c: c["layers"][0]["mixer"].pop("left_scale"),
    lambda c: c["layers"][0]["mixer"]["left"].pop("mask"),
    lambda c: c["layers"][0]["mixer"]["right"].update(tau=0),
    lambda c: c["layers"][0]["mlp"].pop("ff"),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][1]["mixer"].pop("q_rank"),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10),      # not the rotated part's size
    lambda c: c["layers"][1]["mlp"]["router"].update(top=8),       # more than there are
    lambda c: c["layers"][1]["mlp"]["router"].pop("scale"),
    lambda c: c["layers"][2]["mixer"].update(kv_heads=3),          # does not divide the heads
    lambda c: c["layers"][2]["mixer"]["rot"].update(dims=30),      # more than a head has
    lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("low"),
])
def test_config_errors_are_reported(hm, tmp_path, edit):
    cfg = copy.deepcopy(model("mixed"))
    edit(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(hm.HomuraError) as e:
        hm.checkpoint_info(str(tmp_path))
    assert "config.json" in e.value.message and e.value.status == hm.HM_ERR_IO


# ---- the oracle's pieces against values worked out by hand -------------------------------------


def test_offset_norm():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(go.offset_norm(x, np.array([0.0, -0.5]), 0.0), [[3 / 12.5**0.5, 2 / 12.5**0.5]])
    assert np.allclose(go.rms(np.zeros((1, 2)), 1e-2), 0)


def test_activations():
    assert go.silu(np.array([2.0]))[0] == pytest.approx(2 / (1 + np.exp(-2)))
    assert go.gelu_tanh(np.array([1.0]))[0] == pytest.approx(0.5 * (1 + np.tanh(np.sqrt(2 / np.pi) * 1.044715)))
    assert np.isfinite(go.sigmoid(np.array([-800.0, 800.0]))).all()


def test_bigram_rows():
    assert go.bigram_rows([4, 9, 2], 10, 3, 7) == [10, (12 + 63) % 10, (27 + 14) % 10]


def test_rotation():
    f = go.rotation_frequencies(4, 100.0)
    assert np.allclose(f, [1.0, 0.1])
    x = np.array([1.0, 2.0, 3.0, 4.0, 5.0]).reshape(1, 1, 5).repeat(3, axis=0)
    y = go.rotate(x, f)
    c, s = np.cos([2.0, 0.2]), np.sin([2.0, 0.2])
    assert np.allclose(y[0, 0], x[0, 0])
    assert np.allclose(y[2, 0], [c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1], 5])


def test_scaled_frequencies():
    # wavelengths 2 pi, 2 pi 10, 2 pi 100, 2 pi 1000 against bounds 32 (kept below) and 512 (slowed above)
    f = go.rotation_frequencies(8, 10000.0, {"factor": 4.0, "low": 1.0, "high": 16.0, "original": 512})
    s = (512 / (20 * np.pi) - 1) / 15
    assert np.allclose(f, [1.0, ((1 - s) / 4 + s) * 0.1, 0.01 / 4, 0.001 / 4])


def test_windows():
    m = go.window_mask(6, 2, 1)
    assert [r.nonzero()[0].tolist() for r in m] == [[0], [0, 1], [0, 1, 2], [0, 2, 3], [0, 3, 4], [0, 4, 5]]
    assert go.window_mask(3).sum() == 6


def test_sink_takes_its_share():
    p = go.softmax_with_sink(np.log(np.array([1.0, 2.0])), np.log(5.0))
    assert np.allclose(p, [1 / 8, 2 / 8])
    assert np.allclose(go.softmax_with_sink(np.array([0.0, -np.inf]), 900.0), 0)


def test_masked_attention_by_hand():
    q = np.array([[[100.0], [0.0]]] * 3)
    k = np.array([[[5.0]], [[1.0]], [[3.0]]])
    out = go.masked_attention(q, k, k * 10, 1.0, go.window_mask(3, 2))
    assert np.allclose(out[..., 0], [[50, 50], [50, 30], [30, 20]])


def test_short_convolution():
    u = np.array([[1.0, 1.0], [2.0, 0.0], [4.0, 0.0]])
    w = np.array([[0.5, 10.0, 1.0], [1.0, 2.0, 3.0]])
    assert np.allclose(go.short_convolution(u, w), [[1, 3], [12, 2], [24.5, 1]])
    assert np.allclose(go.short_convolution(u, w[:, :1]), u * [0.5, 1.0])


def test_gated_linear_attention():
    one = np.ones((3, 1, 1))
    k, v, a = one * 2, np.array([1.0, 10.0, 100.0]).reshape(3, 1, 1), np.array([0.3, 0.5, 0.25]).reshape(3, 1, 1)
    assert np.allclose(go.gated_linear_attention(one, k, v, a).ravel(), [2, 21, 21 / 4 + 200])
    assert np.allclose(go.decay(np.array([0.0, 50.0]), 2.0), [0.5**0.5, 1.0])
    # the decay belongs to the rows of the keys
    k2, v2 = np.array([[[1.0, 1.0]], [[0.0, 0.0]]]), np.array([[[1.0, 2.0]], [[0.0, 0.0]]])
    a2 = np.array([[[1.0, 1.0]], [[0.5, 0.1]]])
    assert np.allclose(go.gated_linear_attention(np.array([[[1.0, 0.0]], [[1.0, 0.0]]]), k2, v2, a2)[1, 0], [0.5, 1.0])


def test_router_weights_are_scores_of_all_experts():
    chosen, weights = go.route(np.log(np.array([[0.2, 0.5, 0.3]])), 2, 10.0)
    assert chosen.tolist() == [[1, 2]] and np.allclose(weights, [[5, 3]])


# ---- what the oracle ignores would show ----------------------------------------------------------


@pytest.mark.parametrize("edit", [
    lambda c, w: c["layers"][2]["mixer"]["mask"].update(size=49),
    lambda c, w: c["layers"][2]["mixer"]["mask"].update(size=51),
    lambda c, w: c["layers"][2]["mixer"]["mask"].update(keep_first=8),
    lambda c, w: c["layers"][2]["mixer"]["mask"].update(keep_first=10),
    lambda c, w: c["layers"][2]["mixer"]["rot"].pop("scaling"),
    lambda c, w: c["layers"][0]["mixer"]["left"]["mask"].update(size=29),
    lambda c, w: c["layers"][0]["mixer"].update(left_scale=1.2),
    lambda c, w: c["layers"][0]["mixer"].update(right_scale=0.5),
    lambda c, w: c["layers"][0]["mixer"]["right"].update(tau=7.0),
    lambda c, w: c["layers"][1]["mlp"]["router"].update(scale=1.0),
    lambda c, w: c["embedding"].update(scale=1.0),
    lambda c, w: c.update(logit_softcap=30.0),
    lambda c, w: w.update({"l2.mix.sink": w["l2.mix.sink"] - 50}),
    lambda c, w: w.update({"l0.mix.left.sink": w["l0.mix.left.sink"] - 50}),
    lambda c, w: w.update({"l3.mix.left.v.conv": w["l3.mix.left.v.conv"] * [0, 1, 1, 1]}),
    lambda c, w: w.update({"bigram": w["bigram"] * (np.arange(len(w["bigram"])) < len(w["bigram"]) - 1)[:, None]}),
    lambda c, w: w.update({"l1.mlp.shared.sg": w["l1.mlp.shared.sg"] * 0}),
])
def test_every_constant_shows_in_the_logits(edit):
    """A wrong constant changes the logits by far more than the tolerances of the GPU tests."""
    cfg = model("mixed")
    o = oracle_of(cfg, 21)
    ids = synth.prompt_ids(1, 150, cfg["vocab"])
    want = o.forward(ids)
    other = copy.deepcopy(cfg)
    w = dict(o.w)
    edit(other, w)
    assert np.abs(go.Oracle(other, w).forward(ids) - want).max() > 0.01 * np.abs(want).max()


def test_oracle_rows_do_not_depend_on_later_tokens():
    o = oracle_of(model("mixed"))
    ids = synth.prompt_ids(3, 40, 100)
    assert np.allclose(o.forward(ids)[:17], o.forward(ids[:17]), atol=1e-9)
