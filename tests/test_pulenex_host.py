"""CPU tests of the Pulenex design: config reader, checkpoint description, oracle."""
import copy
import json

import numpy as np
import pytest
from pulenex_cases import NAMES, RANKS, model

import pulenex_oracle as po
from homura_b200 import synth


def oracle_of(cfg, seed=5, ranks=(12, 20), **kw):
    return po.Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in synth.pulenex_weights(cfg, seed, ranks).items()}, **kw)


@pytest.mark.parametrize("name", NAMES)
def test_checkpoint_info_reads_the_layer_list(hm, tmp_path, name):
    cfg = model(name)
    info = hm.checkpoint_info(synth.write_pulenex_model(str(tmp_path), cfg, 1, ranks=RANKS[name]))
    c = info["config"]
    assert c["architecture"] == "Pulenex" and not c["tie_word_embeddings"]
    assert (c["hidden_size"], c["vocab_size"], c["num_hidden_layers"]) == (cfg["width"], cfg["vocab"], len(cfg["layers"]))
    for got, want in zip(c["layers"], cfg["layers"]):
        m, f = want["mixer"], want["mlp"]
        assert got["type"] == want["type"]
        if want["type"] == "retention":
            assert [got[k] for k in ("heads", "dim", "vdim")] == [m[k] for k in ("heads", "dim", "vdim")]
            assert got["decay"] == pytest.approx(m["decay"])
        elif want["type"] == "latent_attention":
            keys = ("heads", "dim", "rot_dim", "vdim", "kv_rank")
            assert [got[k] for k in keys] == [m[k] for k in keys]
            assert (got["window"], got["kv_from"]) == (m["mask"]["size"], m.get("kv_from"))
            assert got["scale"] == pytest.approx(m["scale"], rel=1e-6)
        else:
            assert got["linear"] == m["right"]
            m = m["left"]
            assert [got[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv")] == [m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv")]
            assert got["chunk"] == m["mask"]["size"] and got["scale"] == pytest.approx(m["scale"], rel=1e-6)
        assert got["rot"] == m["rot"]
        assert (got["ff"], got["limit"]) == ((0, 0) if f is None else (f["ff"], pytest.approx(f["limit"])))
    assert len(info["tensors"]) == len(synth.pulenex_tensor_specs(cfg))


@pytest.mark.parametrize("edit", [
    lambda c: c.pop("width"),
    lambda c: c["norm"].pop("eps"),
    lambda c: c.pop("logit_scale"),
    lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="attention"),
    lambda c: c["layers"][0]["mixer"].pop("right"),
    lambda c: c["layers"][0]["mixer"]["left"].pop("mask"),
    lambda c: c["layers"][0]["mixer"]["left"].pop("conv"),
    lambda c: c["layers"][0]["mixer"]["left"].update(vdim=23),       # the values are the keys
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4),    # does not divide the heads
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=26),
    lambda c: c["layers"][0]["mixer"]["right"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"]["right"].pop("vdim"),
    lambda c: c["layers"][0]["mlp"].pop("limit"),
    lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    lambda c: c["layers"][1]["mixer"].pop("rot"),
    lambda c: c["layers"][1]["mixer"]["decay"].pop(),
    lambda c: c["layers"][2]["mixer"].update(kv_rank=0),
    lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10),        # not the rotated part's size
    lambda c: c["layers"][4]["mixer"].update(kv_from=4),             # itself
    lambda c: c["layers"][4]["mixer"].update(kv_from=1),             # no latents there
    lambda c: c["layers"][4]["mixer"].update(kv_rank=64),            # not that layer's
    lambda c: c["layers"][4]["mixer"].pop("mask"),
])
def test_config_errors_are_reported(hm, tmp_path, edit):
    cfg = copy.deepcopy(model("mixed"))
    edit(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(hm.HomuraError) as e:
        hm.checkpoint_info(str(tmp_path))
    assert "config.json" in e.value.message and e.value.status == hm.HM_ERR_IO


# ---- the oracle's pieces against values worked out by hand -------------------------------------


def test_norms():
    x = np.array([[1.0, 5.0]])
    assert np.allclose(po.layer_norm(x, np.array([1.0, 0.5]), 0.0), [[-1.0, 0.5]])
    assert np.allclose(po.layer_norm(x, np.ones(2), 5.0), [[-2 / 3, 2 / 3]])
    assert np.allclose(po.rms(np.array([[3.0, 4.0]]), 0.0), [[3 / 12.5**0.5, 4 / 12.5**0.5]])
    assert np.allclose(po.unit(np.array([[3.0, 4.0]])), [[0.6, 0.8]]) and np.allclose(po.unit(np.zeros((1, 2))), 0)


def test_activations():
    assert po.silu(np.array([2.0]))[0] == pytest.approx(2 / (1 + np.exp(-2)))
    assert np.isfinite(po.sigmoid(np.array([-800.0, 800.0]))).all()
    assert po.softplus(np.array([0.0, 50.0])) == pytest.approx([np.log(2), 50.0])
    sig = lambda z: 1 / (1 + np.exp(-z))
    got = po.clamped_glu(np.array([9.0, -9.0, 0.5]), np.array([9.0, -9.0, 0.25]), 2.0)
    assert got == pytest.approx([2 * sig(3.404) * 3, -9 * sig(-9 * 1.702) * -1, 0.5 * sig(0.851) * 1.25])


def test_rotations():
    f = po.rotation_frequencies(4, 100.0)
    assert np.allclose(f, [1.0, 0.1])
    x = np.array([1.0, 2.0, 3.0, 4.0, 5.0]).reshape(1, 1, 5).repeat(3, axis=0)
    c, s = np.cos([2.0, 0.2]), np.sin([2.0, 0.2])
    y = po.rotate_halves(x, f)
    assert np.allclose(y[0], x[0]) and np.allclose(y[2, 0], [c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1], 5])
    y = po.rotate_neighbours(x, f)
    assert np.allclose(y[0], x[0]) and np.allclose(y[2, 0], [c[0] - 2 * s[0], 2 * c[0] + s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1], 5])


def test_masks():
    assert [r.nonzero()[0].tolist() for r in po.window_mask(4, 2)] == [[0], [0, 1], [1, 2], [2, 3]]
    assert [r.nonzero()[0].tolist() for r in po.chunk_mask(5, 2)] == [[0], [0, 1], [2], [2, 3], [4]]


def test_sink_takes_its_share():
    assert np.allclose(po.softmax(np.log(np.array([1.0, 2.0])), np.log(5.0)), [1 / 8, 2 / 8])
    assert np.allclose(po.softmax(np.array([0.0, -np.inf]), 900.0), 0)


def test_talking_scores():
    q, k = np.array([[[1.0], [2.0]]] * 2), np.array([[[3.0]], [[5.0]]])
    s = po.talking_scores(q, k, 0.5, np.array([1.0, 10.0]), np.array([[1.0, 0.0], [2.0, 1.0]]))
    assert np.allclose(s[:, 0], [[1.5, 2.5], [33.0, 55.0]])


def test_short_convolution():
    u = np.array([[1.0, 1.0], [2.0, 0.0], [4.0, 0.0]])
    w = np.array([[0.5, 10.0, 1.0], [1.0, 2.0, 3.0]])
    assert np.allclose(po.short_convolution(u, w), [[1, 3], [12, 2], [24.5, 1]])
    assert np.allclose(po.short_convolution(u, w[:, :1]), u * [0.5, 1.0])


def test_recurrences():
    one = np.ones((3, 1, 1))
    v = np.array([1.0, 10.0, 100.0]).reshape(3, 1, 1)
    assert np.allclose(po.retention(one, one * 2, v, np.array([0.5])).ravel(), [2, 21, 210.5])
    # with a key of length one and a full step the state forgets what it held for that key
    assert np.allclose(po.gated_delta_rule(one, one, v, one * 0.5, np.ones((3, 1))).ravel(), [1, 10, 100])
    assert np.allclose(po.gated_delta_rule(one, one, v, one * 0.5, np.full((3, 1), 0.5)).ravel(), [0.5, 0.25 + 0.5 * 9.75, 2.5625 + 0.5 * (100 - 2.5625)])
    # the decay belongs to the rows of the keys
    k2, v2 = np.array([[[1.0, 0.0]], [[0.0, 0.0]]]), np.array([[[1.0, 2.0]], [[0.0, 0.0]]])
    g2 = np.array([[[1.0, 1.0]], [[0.5, 0.1]]])
    assert np.allclose(po.gated_delta_rule(np.array([[[1.0, 0.0]]] * 2), k2, v2, g2, np.ones((2, 1)))[1, 0], [0.5, 1.0])
    assert np.allclose(po.channel_decay(np.zeros((1, 1, 1)), np.array([np.log(2.0)])), 0.25)


# ---- what the oracle ignores would show ----------------------------------------------------------


@pytest.mark.parametrize("edit", [
    lambda c, w: c["layers"][0]["mixer"]["left"]["mask"].update(size=29),
    lambda c, w: c["layers"][0]["mixer"]["left"]["mask"].update(size=31),
    lambda c, w: c["layers"][0]["mixer"]["left"].update(scale=0.25),
    lambda c, w: c["layers"][0]["mixer"]["left"]["rot"].update(dims=14),
    lambda c, w: c["layers"][0]["mixer"]["left"]["rot"].update(base=900.0),
    lambda c, w: c["layers"][0]["mlp"].update(limit=1.4),
    lambda c, w: c["layers"][1]["mixer"]["decay"].__setitem__(4, 0.9),
    lambda c, w: c["layers"][1]["mixer"]["rot"].update(base=600.0),
    lambda c, w: c["layers"][2]["mixer"]["mask"].update(size=32),
    lambda c, w: c["layers"][2]["mixer"].update(scale=0.2),
    lambda c, w: c["layers"][4]["mixer"]["mask"].update(size=51),
    lambda c, w: c["layers"][4]["mixer"]["rot"].update(base=200.0),
    lambda c, w: c.update(logit_scale=0.8),
    lambda c, w: c["norm"].update(eps=0.1),
    lambda c, w: w.update({"l0.mix.left.sink": w["l0.mix.left.sink"] - 50}),
    lambda c, w: w.update({"l0.mix.left.temp": w["l0.mix.left.temp"] * 0 + 1}),
    lambda c, w: w.update({"l0.mix.left.talk": np.eye(6)}),
    lambda c, w: w.update({"l0.mix.left.talk": w["l0.mix.left.talk"].T}),
    lambda c, w: w.update({"l0.mix.left.k.conv": w["l0.mix.left.k.conv"] * [0, 1, 1]}),
    lambda c, w: w.update({"l0.mix.right.v.conv": w["l0.mix.right.v.conv"] * [0, 1, 1, 1]}),
    lambda c, w: w.update({"l0.mix.right.A_log": w["l0.mix.right.A_log"] + 0.5}),
    lambda c, w: w.update({"l0.mix.right.dt_bias": w["l0.mix.right.dt_bias"] * 0}),
    lambda c, w: w.update({"l0.mix.right.b": w["l0.mix.right.b"] * 0}),
    lambda c, w: w.update({"l0.mix.right.g2": w["l0.mix.right.g2"] * 0}),
    lambda c, w: w.update({"l0.mlp.up.b": w["l0.mlp.up.b"] * 0}),
    lambda c, w: w.update({"l2.mix.g": w["l2.mix.g"] * 0}),
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
    assert np.abs(po.Oracle(other, w).forward(ids) - want).max() > 0.01 * np.abs(want).max()


def test_oracle_rows_do_not_depend_on_later_tokens():
    o = oracle_of(model("mixed"))
    ids = synth.prompt_ids(3, 40, 100)
    assert np.allclose(o.forward(ids)[:17], o.forward(ids[:17]), atol=1e-9)
