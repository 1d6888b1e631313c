"""Zabozen on the host: from config.json to the plan, the tensor table and a random-weights folder.  No GPU needed."""
import copy

import numpy as np
import pytest

import plain_zabozen as P
import zabozen_configs as C


def test_the_architecture_is_registered():
    import velomind_b200 as vm
    assert "Zabozen" in vm.registered_architectures()
    d = vm.describe_config(C.config("a"))
    assert d["architecture"] == "Zabozen" and d["hidden_size"] == 88 and d["vocab_size"] == 150 and d["max_positions"] == 0
    assert d["runs"] == 5 and len(d["blocks"]) == 5


def test_tensor_table_follows_the_layer_list():
    import velomind_b200 as vm
    t = {k: v["shape"] for k, v in vm.weight_table(C.config("a")).items()}
    assert t["embed"] == [150, 88] and t["head"] == [150, 88] and t["final.norm"] == [88]
    # a norm in front of and behind every sublayer; a layer without a feed-forward has one pair
    assert t["l0.norm1"] == t["l0.norm1b"] == t["l0.norm2"] == t["l0.norm2b"] == [88]
    assert "l1.norm2" not in t and "l1.norm2b" not in t and t["l1.norm1b"] == [88] and "l1.mlp.gate" not in t
    # the delta rule: shared queries and keys, convolutions on all three, two gates of the recurrence, no biases
    assert t["l0.mix.q"] == [24, 88] and t["l0.mix.k"] == [24, 88] and t["l0.mix.v"] == [120, 88] and t["l0.mix.g"] == [120, 88]
    assert t["l0.mix.q.conv"] == [24, 4] and t["l0.mix.v.conv"] == [120, 4] and t["l0.mix.b"] == [6, 88] and t["l0.mix.a"] == [6, 88]
    assert t["l0.mix.A_log"] == [6] and t["l0.mix.dt_bias"] == [6] and t["l0.mix.norm"] == [20] and t["l0.mix.o"] == [88, 120]
    assert "l0.mix.q.b" not in t
    # attention with biases everywhere; a layer on another one's keys has queries and an output alone
    assert t["l1.mix.q"] == [60, 88] and t["l1.mix.k.b"] == [20] and t["l1.mix.v"] == [12, 88] and t["l1.mix.o.b"] == [88]
    assert t["l3.mix.q.b"] == [60] and t["l3.mix.o"] == [88, 36] and not any(k.startswith(("l3.mix.k", "l3.mix.v", "l4.mix.k", "l4.mix.v")) for k in t)
    # latent attention: queries straight from the input, one gate row per head
    assert t["l2.mix.q"] == [48, 88] and t["l2.mix.dkv"] == [42, 88] and t["l2.mix.dkv.norm"] == [36] and t["l2.mix.uk"] == [30, 36]
    assert t["l2.mix.uv"] == [42, 36] and t["l2.mix.g"] == [3, 88] and t["l2.mix.o"] == [88, 42]
    assert t["l2.mlp.gate"] == [40, 88] and t["l2.mlp.down"] == [88, 40]


@pytest.mark.parametrize("damage,word", [
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(conv=17), "taps"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(dim=513), "dim"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(mask={"size": 0}), "size"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=2), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=8), "rotary_dim"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_a_wrong_configuration_is_refused_by_name(damage, word):
    import velomind_b200 as vm
    cfg = copy.deepcopy(C.config("a"))
    damage(cfg)
    with pytest.raises(vm.ConfigError) as e:
        vm.weight_table(cfg)
    assert word in str(e.value)


def test_random_weights_folder_matches_the_model(tmp_path):
    import velomind_b200 as vm
    for which in C.ALL:
        folder = vm.write_random_model(str(tmp_path / which), C.config(which), seed=1)
        vm.check_model_folder(folder)
        assert set(vm.safetensors_info(folder + "/model.safetensors")) == set(vm.weight_table(C.config(which)))


# ----------------------------------------------------------------------------- the plain implementation itself, on cases that have an answer
def test_plain_delta_rule_overwrites_what_it_holds_under_a_key():
    """With orthonormal keys and full writes the memory is a dictionary: reading a key gives its LAST value, whatever came between."""
    d, dv = 4, 3
    rng = np.random.default_rng(0)
    order = [0, 1, 2, 0, 3, 1, 0]
    k = np.eye(d)[order]
    v = rng.normal(size=(len(order), dv))
    o = P.delta_rule(k, k, v, np.ones(len(order)), np.ones(len(order)))
    np.testing.assert_allclose(o, v, atol=1e-12)
    q = np.eye(d)[[1] * len(order)]
    o = P.delta_rule(q, k, v, np.ones(len(order)), np.full(len(order), 0.5))
    np.testing.assert_allclose(o[4], v[1] * 0.5 ** 3, atol=1e-12)         # written at place 1, forgotten three times, untouched by other keys
    np.testing.assert_allclose(o[6], v[5] * 0.5, atol=1e-12)


def test_plain_rotation_depends_on_the_distance_alone():
    rng = np.random.default_rng(1)
    x, y = rng.normal(size=(1, 1, 6)), rng.normal(size=(1, 1, 6))
    q, k = P.turn_halves(np.repeat(x, 30, axis=0), 50.0, 6)[:, 0], P.turn_halves(np.repeat(y, 30, axis=0), 50.0, 6)[:, 0]
    np.testing.assert_allclose(q[25] @ k[20], q[9] @ k[4], atol=1e-12)
    assert abs(q[25] @ k[20] - q[25] @ k[19]) > 1e-3


def test_plain_slopes_and_windows():
    np.testing.assert_allclose(P.slopes(8), [0.5 ** (h + 1) for h in range(8)])
    m = P.sees(5, 2)
    assert m.sum() == 9 and m[4, 3] and not m[4, 2] and not m[2, 3]
