"""The Defapel configuration reader, the description it builds, and the plain implementation itself (no device needed)."""
import copy

import numpy as np
import pytest

from defapel_helpers import (CONFIG_A, CONFIG_B, CONFIG_C, CONFIG_D, SCALING, channel, config, delta, draw_weights, moe, parallel, rot, scaling, tokens,
                             window)
from plain import defapel_plain as P
from purhie_b200.config import ConfigError, ModelConfig, registered_architectures, registered_parts
from purhie_b200.weights import expected_tensors


def test_the_architecture_and_its_parts_are_registered():
    assert "Defapel" in registered_architectures()
    assert {"attention", "delta_rule", "side_by_side"} <= set(registered_parts("mixer"))


def test_the_description_follows_the_layer_list():
    cfg = ModelConfig.from_dict(CONFIG_A)
    assert cfg.architecture == "Defapel"
    spec = cfg.model_spec()
    layers = spec["layers"]
    kinds = [(l["arrangement"], l["parts"]["mixer"]["kind"], l["parts"].get("feed_forward", {}).get("kind")) for l in layers]
    assert kinds == [("pre_norm", "side_by_side", "routed_glu"), ("pre_norm", "delta_rule", "routed_glu"), ("pre_norm", "side_by_side", None),
                     ("pre_norm", "delta_rule", "routed_glu")]
    n = layers[0]["parts"]["mixer_norm"]["params"]
    assert (n["size"], n["eps"], n["weight_offset"], n["names"]["weight"]) == (48, 1e-6, 1.0, "l0.norm1")
    both = layers[0]["parts"]["mixer"]["params"]
    assert (both["combine"], both["left_factor"], both["right_factor"]) == ("weighted_sum", 0.8, 1.3)
    a = both["left"]["params"]
    assert (a["num_heads"], a["num_kv_heads"], a["head_dim"], a["value_dim"], a["window"], a["softcap"]) == (4, 2, 12, 20, 11, 4.0)
    assert a["qk_norm_over"] == "row" and a["bias"] is True and a["names"]["gate_proj"] == "l0.mix.left.g" and a["names"]["q_bias"] == "l0.mix.left.q.b"
    assert a["position"]["params"] == {"theta": 1e4, "n_rot": 8, "max_position": 65536, "pairing": "interleaved",
                                       "scaling": dict(SCALING, kind="wavelength")}
    assert "scaling" not in layers[2]["parts"]["mixer"]["params"]["left"]["params"]["position"]["params"]
    r = both["right"]["params"]
    assert (r["num_heads"], r["num_kv_heads"], r["head_dim"], r["value_dim"], r["conv"], r["decay"], r["gate"]) == (6, 2, 8, 12, 3, "head", "silu")
    assert r["names"]["decay_proj"] == "l0.mix.right.a" and r["names"]["gate_proj"] == "l0.mix.right.g"
    d = layers[1]["parts"]["mixer"]["params"]
    assert (d["num_heads"], d["num_kv_heads"], d["head_dim"], d["value_dim"], d["conv"], d["decay"], d["gate"]) == (3, 1, 10, 14, 4, "channel", "sigmoid")
    assert (d["decay_rank"], d["gate_rank"]) == (5, 3) and d["names"]["decay_down"] == "l1.mix.a1" and d["names"]["gate_up"] == "l1.mix.g2"
    f = layers[0]["parts"]["feed_forward"]["params"]
    assert (f["experts"], f["top"], f["intermediate_size"], f["weight_on"], f["scoring"]["kind"]) == (5, 2, 24, "input", "sigmoid")
    assert spec["head"]["params"]["tied_to"] == "embed" and spec["head"]["params"]["scale"] == 0.7


def test_the_tensor_list_has_every_name_with_its_shape():
    t = expected_tensors(CONFIG_A)
    shape = lambda n: tuple(t[n].shape)
    assert shape("embed") == (80, 48) and "head" not in t and shape("final.norm") == (48,)
    assert shape("l0.mix.left.q") == (48, 48) and shape("l0.mix.left.k") == (24, 48) and shape("l0.mix.left.v") == (40, 48)
    assert shape("l0.mix.left.q.b") == (48,) and shape("l0.mix.left.v.b") == (40,)
    assert shape("l0.mix.left.q.norm") == (48,) and shape("l0.mix.left.k.norm") == (24,) and shape("l0.mix.left.g") == (80, 48)
    assert shape("l0.mix.left.o") == (48, 80)
    assert shape("l0.mix.right.q") == shape("l0.mix.right.k") == (16, 48) and shape("l0.mix.right.v") == (72, 48)
    assert shape("l0.mix.right.q.conv") == (16, 3) and shape("l0.mix.right.v.conv") == (72, 3) and shape("l0.mix.right.b") == (6, 48)
    assert shape("l0.mix.right.a") == (6, 48) and shape("l0.mix.right.dt_bias") == shape("l0.mix.right.A_log") == (6,)
    assert shape("l0.mix.right.norm") == (12,) and shape("l0.mix.right.g") == (72, 48) and shape("l0.mix.right.o") == (48, 72)
    assert shape("l1.mix.a1") == (5, 48) and shape("l1.mix.a2") == (30, 5) and shape("l1.mix.dt_bias") == (30,)
    assert shape("l1.mix.g1") == (3, 48) and shape("l1.mix.g2") == (42, 3) and shape("l1.mix.A_log") == (3,)
    assert "l1.mix.a" not in t and "l1.mix.g" not in t and "l2.norm2" not in t and "l2.mlp.router" not in t
    assert shape("l0.mlp.router") == (5, 48) and shape("l0.mlp.e4.gate") == (24, 48) and shape("l0.mlp.e4.down") == (48, 24)


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="delta"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=2), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"].update(gate_rank=0), "gate_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(softcap=0.0), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=14), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=3), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(base=0.0), "base"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(scaling=scaling(8.0, 5.0, 4.0, 64)), "low"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(scaling={"factor": 2.0}), "original"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(heads=5), "kv_heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
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
    assert load_config(str(tmp_path)).to_dict()["layers"] == CONFIG_B["layers"]


def test_ranks_that_the_configuration_leaves_out_are_whatever_is_stored():
    c = copy.deepcopy(CONFIG_A)
    for l in c["layers"]:
        l["mixer"].pop("decay_rank", None)
        l["mixer"].pop("gate_rank", None)
    t = expected_tensors(c)
    assert tuple(t["l1.mix.a1"].shape) == (-1, 48) and tuple(t["l1.mix.g2"].shape) == (42, -1)


def test_what_each_mixer_asks_the_cache_manager_for():
    from purhie_b200.parts import PartProbe
    spec = ModelConfig.from_dict(CONFIG_A).model_spec()
    need = [PartProbe("mixer", l["parts"]["mixer"]["kind"], l["parts"]["mixer"]["params"]).cache_need() for l in spec["layers"]]
    # keys and values of the window, and beside them S with the convolution's last inputs
    assert (need[0]["kind"], need[0]["kv_heads"], need[0]["head_dim"], need[0]["value_dim"], need[0]["window"]) == ("pages", 2, 12, 20, 11)
    assert need[0]["state_shape"] == [6 * 12 * 8 + 2 * (32 + 72)]
    assert need[1]["kind"] == "state" and need[1]["state_shape"] == [3 * 14 * 10 + 3 * (20 + 42) + 2]     # rounded up to 4
    assert need[3]["state_shape"] == [4 * 8 * 16]                                                        # one tap keeps no inputs


# ---- the plain implementation itself: statements that do not need the engine ---------------------------------------------
@pytest.mark.parametrize("cfg", [CONFIG_A, CONFIG_B, CONFIG_D])
def test_the_plain_implementation_gives_a_position_the_same_logits_whatever_follows(cfg):
    w = {k: np.asarray(v, dtype=np.float64) for k, v in draw_weights(cfg, 5).items()}
    toks = tokens(30, cfg["vocab"], 1)
    whole = P.forward(cfg, w, toks)
    for n in (1, 2, 17):
        assert np.allclose(P.forward(cfg, w, toks[:n]), whole[:n], rtol=1e-9, atol=1e-9)


def test_the_delta_rule_writes_a_value_where_its_key_points_and_overwrites_it():
    D, V = 4, 3
    k = np.eye(D)[[0, 1, 0]][:, None, :]
    v = np.arange(9.0).reshape(3, 1, V) + 1.0
    one, no_decay = np.ones((3, 1)), np.ones((3, 1, D))
    o, S = P.delta_scan(k, k, v, one, no_decay)
    assert np.allclose(o, v)                                        # the read-out sees the current token's write
    assert np.allclose(S[0, 0], v[2, 0]) and np.allclose(S[0, 1], v[1, 0])       # the third token replaced the first one's value
    half, _ = P.delta_scan(k, k, v, 0.5 * one, no_decay)
    assert np.allclose(half[2], 0.5 * v[0] * 0.5 + 0.5 * v[2])
    g = no_decay.copy()
    g[2, 0, 0] = 0.25                                                # the decay comes before the correction
    half, _ = P.delta_scan(k, k, v, 0.5 * one, g)
    assert np.allclose(half[2], 0.25 * 0.5 * v[0] * 0.5 + 0.5 * v[2])


def test_frequencies_are_kept_blended_or_divided_by_their_wavelength():
    r = rot(16, 1e4, scaling(8.0, 1.0, 4.0, 64))
    f, plain = P.frequencies(r), P.frequencies(rot(16, 1e4))
    wave = 2.0 * np.pi / plain
    assert np.allclose(f[wave < 16.0], plain[wave < 16.0]) and np.allclose(f[wave > 64.0], plain[wave > 64.0] / 8.0)
    between = (wave >= 16.0) & (wave <= 64.0)
    assert between.any() and (wave < 16.0).any() and (wave > 64.0).any()
    assert ((f[between] > plain[between] / 8.0) & (f[between] < plain[between])).all()


def test_a_window_sees_itself_and_the_tokens_before():
    seen = P.window_seen(10, 3)
    assert seen[5].nonzero()[0].tolist() == [3, 4, 5] and seen[1].nonzero()[0].tolist() == [0, 1]


def test_the_weight_of_an_expert_counts_inside_its_activation():
    cfg = config(8, 10, [(channel(1, 1, 4, 4, 1, 2, 2), moe(6, 3, 2))])
    w = {k: np.asarray(v, dtype=np.float64) for k, v in draw_weights(cfg, 2, std=1.0).items()}
    h = np.random.default_rng(0).normal(size=(5, 8))
    y = P.experts(h, w, "l0.mlp.", cfg["layers"][0]["mlp"])
    s = P.sigmoid(h @ w["l0.mlp.router"].T)
    on_output = sum(np.where(np.argsort(-s, axis=-1).argsort(axis=-1)[:, e:e + 1] < 2, s[:, e:e + 1], 0.0) * P.expert(h, w, f"l0.mlp.e{e}.")
                    for e in range(3))
    assert np.abs(y - on_output).max() > 0.1 * np.abs(y).max()
