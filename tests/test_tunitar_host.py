"""CPU tests of the Tunitar design: config reader, checkpoint description, oracle."""
import copy
import json

import numpy as np
import pytest
from tunitar_cases import NAMES, model

from homura_b200 import synth
from tunitar_oracle import Oracle, group_norm, latent_attention, token_shift


def oracle_of(cfg, seed=5, **kw):
    return Oracle(cfg, {k: synth.bf16_to_f32(v) for k, v in synth.tunitar_weights(cfg, seed).items()}, **kw)


@pytest.mark.parametrize("name", NAMES)
def test_checkpoint_info_reads_the_layer_list(hm, tmp_path, name):
    cfg = model(name)
    info = hm.checkpoint_info(synth.write_tunitar_model(str(tmp_path), cfg, 1))
    c = info["config"]
    assert c["architecture"] == "Tunitar" and c["norm_groups"] == cfg["norm"]["groups"]
    assert (c["hidden_size"], c["vocab_size"], c["num_hidden_layers"]) == (cfg["width"], cfg["vocab"], len(cfg["layers"]))
    for got, want in zip(c["layers"], cfg["layers"]):
        m = want["mixer"]
        assert [got[k] for k in ("heads", "dim", "vdim", "kv_rank")] == [m[k] for k in ("heads", "dim", "vdim", "kv_rank")]
        assert got["kv_from"] == m.get("kv_from") and got["scale"] == pytest.approx(m["scale"], rel=1e-6)
        assert got["ff"] == (want["mlp"]["ff"] if want["mlp"] else 0)
    assert len(info["tensors"]) == len(synth.tunitar_tensor_specs(cfg))


def _broken(edit):
    cfg = copy.deepcopy(model("mixed"))
    edit(cfg)
    return cfg


@pytest.mark.parametrize("edit", [
    lambda c: c.update(architecture="Tunitarium"),
    lambda c: c.pop("width"),
    lambda c: c["norm"].update(groups=7),
    lambda c: c["norm"].pop("eps"),
    lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="convolution"),
    lambda c: c["layers"][0]["mixer"].pop("scale"),
    lambda c: c["layers"][0]["mixer"].update(kv_from=0),       # itself
    lambda c: c["layers"][1]["mixer"].update(kv_from=2),       # a later layer
    lambda c: c["layers"][3]["mixer"].update(kv_from=2),       # a layer without latents of its own
    lambda c: c["layers"][3]["mixer"].update(kv_from=0),       # another kv_rank
    lambda c: c["layers"][1]["mlp"].update(kind="sparse"),
])
def test_config_errors_are_reported(hm, tmp_path, edit):
    (tmp_path / "config.json").write_text(json.dumps(_broken(edit)))
    with pytest.raises(hm.HomuraError) as e:
        hm.checkpoint_info(str(tmp_path))
    assert "config.json" in e.value.message and e.value.status == hm.HM_ERR_IO


# ---- the oracle's pieces against values worked out by hand -------------------------------------


def test_group_norm_divides_each_run_by_its_own_size():
    x = np.array([[3.0, 4.0, 0.0, 2.0]])
    w = np.array([1.0, 2.0, 3.0, 4.0])
    a, b = np.sqrt(12.5), np.sqrt(2.0)
    assert np.allclose(group_norm(x, w, 2, 0.0), [[3 / a, 8 / a, 0.0, 8 / b]])
    assert np.allclose(group_norm(np.zeros((1, 4)), w, 2, 1e-6), 0.0)


def test_token_shift_reads_the_row_before_its_own_shift():
    h = np.array([[1.0, 10.0], [2.0, 20.0], [4.0, 40.0]])
    assert np.allclose(token_shift(h, np.array([1.0, 0.25])), [[0.0, 7.5], [1.0, 17.5], [2.0, 35.0]])


def test_latent_attention_by_hand():
    # one head whose query picks the token with the largest latent; identity projections, a gate of one half
    c = np.array([[1.0], [5.0], [3.0]])
    h = np.ones((3, 1))
    one, zero = np.ones((1, 1)), np.zeros((1, 1))
    out = latent_attention(h, c, one * 100, one, one, zero, one, 1, 1, 1, 1.0)
    assert np.allclose(out[:, 0], [0.5, 2.5, 2.5])  # token 2 still sees token 1


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_oracle_is_causal(name):
    cfg = model(name)
    o = oracle_of(cfg)
    ids = synth.prompt_ids(3, 40, cfg["vocab"])
    whole = o.forward(ids)
    assert np.allclose(o.forward(ids[:17]), whole[:17], rtol=0, atol=1e-10)


# Each mistake must show in the logits of the test models far above the tolerances of the GPU tests (1e-4, and 1e-2 on bf16 pages).
MISTAKES = {
    "no gate": lambda o: o.w.update({k: np.full_like(v, 0.0) for k, v in o.w.items() if k.endswith("mix.g")}),
    "no shift": lambda o: o.w.update({k: np.zeros_like(v) for k, v in o.w.items() if k.endswith("shift")}),
    "norm over the whole row": lambda o: setattr(o, "groups", 1),
    "no layer scale": lambda o: o.w.update({k: np.ones_like(v) for k, v in o.w.items() if k.endswith(".ls1")}),
    "no MLP layer scale": lambda o: o.w.update({k: np.ones_like(v) for k, v in o.w.items() if k.endswith(".ls2")}),
    "no latent norm weight": lambda o: o.w.update({k: np.ones_like(v) for k, v in o.w.items() if k.endswith("dkv.norm")}),
    "scale of one": lambda o: [m["mixer"].update(scale=1.0) for m in o.cfg["layers"]],
    "another eps": lambda o: setattr(o, "eps", o.eps + 0.1),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_a_mistake_shows_in_the_logits(mistake):
    cfg = model("mixed")
    ids = synth.prompt_ids(9, 24, cfg["vocab"])
    want = oracle_of(cfg).forward(ids)
    wrong = oracle_of(copy.deepcopy(cfg))
    MISTAKES[mistake](wrong)
    assert np.abs(wrong.forward(ids) - want).max() > 0.05 * np.abs(want).max()


def test_shared_latents_are_the_named_layers():
    cfg = model("mixed")
    ids = synth.prompt_ids(9, 24, cfg["vocab"])
    o = oracle_of(cfg)
    want = o.forward(ids)
    assert sorted(o.latents) == [0, 1]
    swapped = copy.deepcopy(cfg)  # layer 3 could also be given latents of the same rank from elsewhere
    swapped["layers"][3]["mixer"]["kv_rank"] = 72
    swapped["layers"][3]["mixer"]["kv_from"] = 0
    w = {k: synth.bf16_to_f32(v) for k, v in synth.tunitar_weights(cfg, 5).items()}
    for k in ("uk", "uv"):
        w[f"l3.mix.{k}"] = np.pad(w[f"l3.mix.{k}"], ((0, 0), (0, 24)))
    assert np.abs(Oracle(swapped, w).forward(ids) - want).max() > 0.05 * np.abs(want).max()


def test_info_on_the_command_line(hm, tmp_path, capsys):
    from homura_b200.__main__ import main

    assert main(["info", synth.write_tunitar_model(str(tmp_path), model("mixed"), 1)]) == 0
    out = capsys.readouterr().out
    assert "architecture: Tunitar" in out and "layer 2:" in out and "l1.mix.dkv.norm  BF16  [48]" in out
