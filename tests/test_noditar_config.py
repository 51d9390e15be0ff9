"""The Noditar configuration reader and the description it builds (no device needed)."""
import copy

import numpy as np
import pytest

from noditar_helpers import CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_E, biased, config, dense, draw_weights, latent, mamba2, tokens
from plain import noditar_plain as P
from purhie_b200.config import ConfigError, ModelConfig, registered_architectures, registered_parts
from purhie_b200.weights import expected_tensors


def test_the_architecture_and_its_parts_are_registered():
    assert "Noditar" in registered_architectures()
    assert {"latent_attention", "attention", "mamba2"} <= set(registered_parts("mixer"))
    assert "hyper_connection" in registered_parts("arrangement")


def test_the_description_follows_the_layer_list():
    cfg = ModelConfig.from_dict(CONFIG_A)
    assert cfg.architecture == "Noditar"
    spec = cfg.model_spec()
    assert spec["residual_lanes"] == 2
    layers = spec["layers"]
    kinds = [(l["arrangement"], l["parts"]["mixer"]["kind"], l["parts"].get("feed_forward", {}).get("kind")) for l in layers]
    assert kinds == [("hyper_connection", "latent_attention", "swiglu"), ("hyper_connection", "mamba2", "swiglu"), ("hyper_connection", "attention", None),
                     ("hyper_connection", "attention", "swiglu"), ("hyper_connection", "latent_attention", None)]
    assert layers[0]["params"]["lanes"] == 2 and layers[0]["params"]["mixer_names"] == {"in": "l0.hc1.in", "out": "l0.hc1.out", "mix": "l0.hc1.mix"}
    assert layers[0]["params"]["feed_forward_names"]["mix"] == "l0.hc2.mix" and "feed_forward_names" not in layers[2]["params"]
    assert "feed_forward_norm" not in layers[2]["parts"]
    a = layers[0]["parts"]["mixer"]["params"]
    assert (a["num_heads"], a["head_dim"], a["rot_dim"], a["value_dim"], a["kv_rank"], a["scale"], a["gate"]) == (3, 16, 0, 24, 40, 0.3, "values")
    assert a["q_rank"] is None and a["position"] is None and a["norm_eps"] == 1e-6
    m = layers[1]["parts"]["mixer"]["params"]
    assert (m["num_heads"], m["value_dim"], m["state"], m["groups"], m["conv"], m["norm_groups"]) == (6, 8, 12, 3, 3, 4)
    b = layers[2]["parts"]["mixer"]["params"]
    assert (b["num_heads"], b["num_kv_heads"], b["head_dim"], b["value_dim"], b["scale"]) == (4, 2, 12, 20, 0.4)
    assert b["qk_norm_weight"] is False and b["qk_norm_eps"] == 1e-6 and b["sink_value"] == 0.0 and b["names"]["gate_proj"] == "l2.mix.g"
    assert b["distance_slopes"] == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    assert np.allclose(layers[3]["parts"]["mixer"]["params"]["distance_slopes"], P.head_slopes(5))
    assert layers[0]["parts"]["feed_forward"]["params"]["activation"] == {"kind": "clamped_swish", "alpha": 1.702, "limit": 1.1, "shift": 1.0}
    assert [(c["layer"], c["pass"], c["cache_from"]) for c in spec["schedule"]] == [(i, 0, None) for i in range(5)]
    assert spec["head"]["params"]["names"] == {"weight": "head"} and spec["keep_embedding_output"] is False


def test_the_tensor_list_has_every_name_with_its_shape():
    t = expected_tensors(CONFIG_A)
    shape = lambda n: tuple(t[n].shape)
    assert shape("embed") == (80, 48) and shape("head") == (80, 48) and shape("final.norm") == (48,)
    assert shape("l0.mix.q") == (48, 48) and shape("l0.mix.dkv") == (40, 48) and shape("l0.mix.dkv.norm") == (40,)
    assert shape("l0.mix.uk") == (48, 40) and shape("l0.mix.uv") == (72, 40) and shape("l0.mix.g") == (72, 48) and shape("l0.mix.o") == (48, 72)
    assert shape("l1.mix.in") == (48 + 48 + 2 * 36 + 6, 48) and shape("l1.mix.conv") == (48 + 72, 3) and shape("l1.mix.conv.b") == (120,)
    assert shape("l1.mix.dt_bias") == shape("l1.mix.A_log") == shape("l1.mix.D") == (6,) and shape("l1.mix.norm") == (48,) and shape("l1.mix.o") == (48, 48)
    assert shape("l2.mix.q") == (48, 48) and shape("l2.mix.k") == (24, 48) and shape("l2.mix.v") == (40, 48) and shape("l2.mix.g") == (80, 48)
    assert shape("l3.hc2.in") == shape("l3.hc2.out") == (2,) and shape("l3.hc2.mix") == (2, 2)
    assert "l2.norm2" not in t and "l2.hc2.in" not in t and "l2.mlp.up" not in t and "l2.mix.sink" not in t and "l2.mix.q.norm" not in t
    assert shape("l0.mlp.gate") == shape("l0.mlp.up") == (64, 48) and shape("l0.mlp.down") == (48, 64)


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="mamba1"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(limit=-1.0), "limit"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("streams"), "streams"),
    (lambda c: c.update(streams=33), "streams"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_a_configuration_that_does_not_fit_is_refused_by_name(change, word):
    c = copy.deepcopy(CONFIG_A)
    change(c)
    with pytest.raises(ConfigError) as e:
        ModelConfig.from_dict(c)
    assert word in str(e.value)


def test_a_random_model_folder_of_this_design_is_written_and_passes_the_folder_check(tmp_path):
    from purhie_b200.config import load_config
    from purhie_b200.weights import check_model_folder, list_tensors, write_random_model
    write_random_model(str(tmp_path), CONFIG_B, seed=3, std=0.05, scale_low=0.8, scale_high=1.2, dtype="bfloat16")
    check_model_folder(str(tmp_path))
    names = {t["name"]: t for t in list_tensors(str(tmp_path))}
    assert set(names) == set(expected_tensors(CONFIG_B))
    assert names["l0.hc1.mix"]["shape"] == [5, 5] and names["l3.mix.conv"]["shape"] == [96 + 2 * 132, 1]
    assert load_config(str(tmp_path)).to_dict()["layers"] == CONFIG_B["layers"]


def test_what_each_mixer_asks_the_cache_manager_for():
    from purhie_b200.parts import PartProbe
    cfg = config(32, 20, 2, [(latent(4, 8, 12, 24), None), (biased(4, 2, 8, 12), dense(16, 1.0)), (mamba2(4, 8, 6, 2, 3, 1), None)])
    spec = ModelConfig.from_dict(cfg).model_spec()
    need = [PartProbe("mixer", l["parts"]["mixer"]["kind"], l["parts"]["mixer"]["params"]).cache_need() for l in spec["layers"]]
    # one row of the latent per token, nothing else; keys and values of the kv heads; S and the convolution's last inputs
    assert (need[0]["kind"], need[0]["kv_heads"], need[0]["head_dim"], need[0]["window"]) == ("pages", 1, 24, None) and not need[0]["state_shape"]
    assert (need[1]["kind"], need[1]["kv_heads"], need[1]["head_dim"], need[1]["value_dim"]) == ("pages", 2, 8, 12)
    assert need[2]["kind"] == "state" and need[2]["state_shape"] == [4 * 8 * 6 + 2 * (32 + 24)]


# ---- the plain implementation itself: statements that do not need the engine ---------------------------------------------
@pytest.mark.parametrize("cfg", [CONFIG_A, CONFIG_B, CONFIG_E])
def test_the_plain_implementation_gives_a_position_the_same_logits_whatever_follows(cfg):
    w = {k: np.asarray(v, dtype=np.float64) for k, v in draw_weights(cfg, 5).items()}
    toks = tokens(30, cfg["vocab"], 1)
    whole = P.forward(cfg, w, toks)
    for n in (1, 2, 17):
        assert np.allclose(P.forward(cfg, w, toks[:n]), whole[:n], rtol=1e-9, atol=1e-9)


def test_streams_with_an_identity_mix_are_the_ordinary_residual():
    rng = np.random.default_rng(0)
    X = np.stack([rng.normal(size=(4, 6))] * 3)
    y = rng.normal(size=(4, 6))
    out = P.streams_update(X, np.eye(3), np.ones(3), y)
    assert np.allclose(out, X + y)
    M = np.zeros((3, 3)); M[0, 2] = 1.0                     # [from, to]: the third stream becomes the first one
    X[0] += 1.0
    moved = P.streams_update(X, M, np.zeros(3), y)
    assert np.allclose(moved[2], X[0]) and np.allclose(moved[:2], 0.0)
    assert np.allclose(P.streams_read(X, np.array([0.5, 0.0, 2.0])), 0.5 * X[0] + 2.0 * X[2])
