"""Depunex on the host: from config.json to the plan, the tensor table and a random-weights folder.  No GPU needed."""
import copy

import numpy as np
import pytest

import depunex_configs as C
import plain_depunex as P


def test_the_architecture_is_registered():
    import velomind_b200 as vm
    assert "Depunex" in vm.registered_architectures()
    d = vm.describe_config(C.config("a"))
    assert d["architecture"] == "Depunex" and d["hidden_size"] == 90 and d["vocab_size"] == 150 and d["max_positions"] == 0
    assert d["runs"] == 4 and len(d["blocks"]) == 4


def test_tensor_table_follows_the_layer_list():
    import velomind_b200 as vm
    t = {k: v["shape"] for k, v in vm.weight_table(C.config("a")).items()}
    assert t["embed"] == [150, 90] and t["bigram"] == [62, 90] and t["side.embed"] == [150, 40] and t["final.norm"] == [90] and "head" not in t
    # one norm a layer, a scale for each sublayer, the token's own input
    assert t["l0.norm1"] == t["l0.ls1"] == t["l0.ls2"] == [90] and "l0.norm2" not in t and "l1.ls2" not in t and "l1.mlp.gate" not in t
    assert t["l0.side.gate"] == [10, 90] and t["l0.side.proj"] == [90, 10] and t["l1.side.norm"] == [90]
    # attention without biases beside the selective scan
    assert t["l0.mix.left.q"] == [42, 90] and t["l0.mix.left.k"] == [14, 90] and t["l0.mix.left.v"] == [10, 90] and t["l0.mix.left.o"] == [90, 30]
    assert "l0.mix.left.q.b" not in t and t["l0.mix.right.in"] == [84, 90] and t["l0.mix.right.conv"] == [42, 3] and t["l0.mix.right.conv.b"] == [42]
    assert t["l0.mix.right.x"] == [17, 42] and t["l0.mix.right.dt"] == [42, 5] and t["l0.mix.right.dt.b"] == [42] and t["l0.mix.right.A_log"] == [42, 6]
    assert t["l0.mix.right.D"] == [42] and t["l0.mix.right.o"] == [90, 42]
    # Mamba-2: z | x | B | C | dt
    assert t["l1.mix.in"] == [42 + 42 + 33 + 33 + 6, 90] and t["l1.mix.conv"] == [108, 3] and t["l1.mix.norm"] == [42] and t["l1.mix.A_log"] == [6]
    # routed experts without a correction or a shared expert
    assert t["l2.mlp.router"] == [9, 90] and t["l2.mlp.e8.gate"] == [26, 90] and t["l2.mlp.e0.down"] == [90, 26]
    assert not any(k.startswith(("l2.mlp.e9", "l2.mlp.shared", "l2.mlp.correction")) for k in t)
    # everything optional left out
    assert set(k for k in vm.weight_table(C.config("c")) if not k.startswith("l")) == {"embed", "final.norm"}
    assert not any(".side." in k for k in vm.weight_table(C.config("c")))


@pytest.mark.parametrize("damage,word", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=2), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(mask={"size": 0}), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(mask=7), "mask"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=16), "rotary_dim"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(original=0), "original"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("dt_rank"), "dt_rank"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(state=1000), "state"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(conv=65), "conv"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="other"), "kind"),
    (lambda c: c["layers"][1]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][2]["mlp"]["router"]["groups"].update(count=2), "groups"),
    (lambda c: c["layers"][2]["mlp"]["router"].pop("experts"), "experts"),
    (lambda c: c["embedding"]["bigram"].pop("buckets"), "buckets"),
    (lambda c: c["token_side"].update(dim=0), "dim"),
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
def test_plain_frequencies_on_the_three_sides_of_the_two_borders():
    rot = {"base": 10000.0, "dims": 16, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 1000}}
    plain = P.frequencies({"base": 10000.0, "dims": 16})
    f = P.frequencies(rot)
    wave = 2 * np.pi / plain
    fast, slow = wave < 250, wave > 1000
    assert fast.any() and slow.any() and (~fast & ~slow).any()
    np.testing.assert_allclose(f[fast], plain[fast])
    np.testing.assert_allclose(f[slow], plain[slow] / 8)
    mid = ~fast & ~slow
    assert ((f[mid] < plain[mid]) & (f[mid] > plain[mid] / 8)).all()
    # continuous at both borders
    for w, share in ((250.0, 1.0), (1000.0, 1.0 / 8)):
        x = 2 * np.pi / w                                                # (of four dimensions, pair 1 turns at base^(-1/2))
        lo, hi = (float(P.frequencies({"base": (x * (1 + e)) ** -2.0, "dims": 4, "scaling": rot["scaling"]})[1]) for e in (-1e-9, 1e-9))
        assert abs(lo - hi) < 1e-8 * x and abs(lo - share * x) < 1e-6 * x


def test_plain_chunks_count_from_the_sequences_start():
    m = P.sees(7, 3)
    assert [int(r.sum()) for r in m] == [1, 2, 3, 1, 2, 3, 1]
    assert m[2, 0] and not m[3, 2] and m[5, 3] and not m[6, 5]
    assert P.sees(7, None)[6].all()


def test_plain_routing_keeps_to_the_best_groups():
    z = np.array([3.0, -9.0, -9.0, 2.0, 1.9, -9.0, 0.5, 0.6, 0.4])       # group scores: one high alone, two high, three middling
    order, w = P.choose_experts(z, 2, {"count": 3, "keep": 1})
    assert sorted(order.tolist()) == [3, 4]                              # the best single expert's group has no second one
    np.testing.assert_allclose(w.sum(), 1.0)
    order, _ = P.choose_experts(z, 3, {"count": 3, "keep": 2})
    assert sorted(order.tolist()) == [3, 4, 7]
    assert P.choose_experts(z, 1)[0].tolist() == [0]


def test_plain_scans_agree_where_both_apply():
    """One head of one column whose state decays alike for all its values is the channel scan of one channel."""
    rng = np.random.default_rng(3)
    n, N = 9, 5
    x, dt, B, Cc = rng.normal(size=(n, 1)), rng.uniform(0.1, 1.0, (n, 1)), rng.normal(size=(n, N)), rng.normal(size=(n, N))
    a = P.channel_scan(x, dt, np.full((1, N), -np.exp(0.3)), B, Cc, [0.7])
    b = P.head_scan(x[:, :, None], dt, [0.3], B[:, None], Cc[:, None], [0.7])
    np.testing.assert_allclose(a[:, 0], b[:, 0, 0], atol=1e-12)
