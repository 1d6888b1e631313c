"""The Zabozen design in the library against the plain implementation (tests/plain_zabozen.py): each mechanism alone (through the
probe architecture of the tests' plug-in, which lets one part's output reach the logits), the wiring, whole models cut into steps in
several ways, weights shaped so that a fault would show where random ones would hide it, and generation through the entry points."""
import copy
import os
import subprocess
import sys

import numpy as np
import pytest

import plain_zabozen as P
import schedules as S
import zabozen_configs as C
from test_kogilix_gpu import mixer_block, probe_config, random_tensors, rounded_to_bf16, run_cuts, standard_cuts, steps_in_pieces, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
MIX = "layers.0.mixer."
EPS = 1e-5


# ----------------------------------------------------------------------------- a part's arguments, from the configuration's own object
def attention_args(hidden, m):
    return {"hidden": hidden, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"], "eps": EPS,
            "window": m["mask"]["size"] if m.get("mask") else 0, "bias": 1, "out_bias": 1, "unit_heads": 1, "slopes": 1}


def latent_args(hidden, m):
    return {"hidden": hidden, "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "q_rank": 0, "kv_rank": m["kv_rank"], "rot_dim": m["rot_dim"],
            "scale": m["scale"], "eps": EPS, "gate": 1, "gate_per_head": 1,
            "position": {"kind": "rotary_half_split", "args": {"head_dim": m["rot_dim"], "theta": m["rot"]["base"], "rotary_dim": m["rot"]["dims"],
                                                               "exact_frequencies": 1}}}


def delta_args(hidden, m):
    return {"hidden": hidden, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "taps": m["conv"], "eps": EPS}


PARTS = {"attention": ("general_attention", attention_args), "latent_attention": ("latent_attention", latent_args), "delta": ("delta_rule", delta_args)}

# name -> (type, hidden, the configuration's own object)
MECHANISMS = {
    # grouped keys (3 on 1), sizes that are no multiple of 8, a window that ends inside a page
    "attention": ("attention", 80, C.attention(3, 1, 20, 12, 0.5, 50)),
    # sizes the tensor-core kernel of prompts takes (bfloat16), a window of exactly one page; slopes of a head count that is no power of two
    "attention_tiles": ("attention", 128, C.attention(6, 2, 64, 32, 0.1, 64)),
    "attention_over_pages": ("attention", 64, C.attention(2, 2, 32, 64, 0.3, 130)),
    "attention_one_token": ("attention", 48, C.attention(2, 1, 8, 8, 0.4, 1)),
    "attention_no_window": ("attention", 64, C.attention(4, 4, 16, 24, 0.3)),
    # odd sizes; sizes of the tensor-core kernel (64 + 16, 128 + 64); a latent wider than the decode kernel takes
    "latent": ("latent_attention", 72, C.latent(3, 10, 6, 14, 36, 0.4, base=50.0)),
    "latent_tiles": ("latent_attention", 128, C.latent(5, 24, 16, 40, 64, 0.3)),
    "latent_tiles_wide": ("latent_attention", 64, C.latent(2, 64, 64, 64, 128, 0.15, base=1e6)),
    "latent_320": ("latent_attention", 64, C.latent(2, 12, 8, 20, 320, 0.3)),
    "latent_one_head": ("latent_attention", 48, C.latent(1, 4, 2, 6, 8, 0.8)),
    # sizes no vector kernel takes; one tap; five taps; chunked prompts and the one-launch decode step at several sizes, among them keys wider than
    # a chunk, values that leave a ragged slice of columns, equal and grouped heads
    "delta_odd": ("delta", 56, C.delta(3, 1, 10, 14, 3)),
    "delta_one_tap": ("delta", 64, C.delta(2, 1, 16, 24, 1)),
    "delta_many_taps": ("delta", 64, C.delta(4, 2, 12, 20, 5)),
    "delta_equal_heads": ("delta", 64, C.delta(3, 3, 32, 32, 4)),
    "delta_128": ("delta", 64, C.delta(2, 1, 128, 128, 4)),
    "delta_wide_keys": ("delta", 64, C.delta(2, 2, 200, 40, 2)),
    "delta_wide_values": ("delta", 64, C.delta(2, 1, 36, 168, 3)),
    "delta_widest_keys": ("delta", 48, C.delta(1, 1, 400, 8, 2)),
    "delta_odd_keys": ("delta", 48, C.delta(2, 1, 18, 16, 4)),
}


def shape_weights(w, rng, prefix=MIX):
    """Random weights that let every branch show: strong taps and biases, decays that spread between almost nothing and almost all."""
    for name in list(w):
        if name.endswith(".conv"):
            w[name] = rng.normal(0.0, 0.7, w[name].shape).astype(np.float32)
        elif name.endswith(".b") and w[name].ndim == 1:
            w[name] = rng.normal(0.0, 0.5, w[name].shape).astype(np.float32)
        elif name.endswith("A_log"):
            w[name] = rng.uniform(-3.0, 1.0, w[name].shape).astype(np.float32)
        elif name.endswith("dt_bias"):
            w[name] = rng.uniform(-3.0, 1.0, w[name].shape).astype(np.float32)
    return w


def probe_model(tmp_path, vm, kind, hidden, m, dtype, seed, std=0.3, change=None):
    part, args = PARTS[kind]
    cfg = probe_config(hidden, mixer_block(part, args(hidden, m)))
    rng = np.random.default_rng(seed)
    w = shape_weights(random_tensors(vm.weight_table(cfg), rng, std), rng)
    if change:
        change(w)
    if dtype == "bfloat16":
        w = rounded_to_bf16(w)              # stored as bfloat16; the plain implementation runs on the same rounded numbers
    return w, write_model(str(tmp_path / f"{kind}_{dtype}"), cfg, w, as_bf16=dtype == "bfloat16")


def plain_mixer(kind, m, w, tokens):
    x = w["embed.weight"].astype(np.float64)[tokens]
    return x, P.MIXERS[kind](x, P.sub(w, MIX), m, EPS)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_each_mechanism_alone(name, dtype, toy_plugin, tmp_path):
    import velomind_b200 as vm
    kind, hidden, m = MECHANISMS[name]
    w, folder = probe_model(tmp_path, vm, kind, hidden, m, dtype, sum(name.encode()))
    engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 6, max_slots=3)      # few pages and slots: both are used again
    requests = S.make_requests(hidden, (70, 5, 130, 64, 1, 65), seed=3)
    plain = {}
    for rid, toks in requests.items():
        x, y = plain_mixer(kind, m, w, toks)
        plain[rid] = x + y
    cuts = standard_cuts(requests)
    cuts["pieces"] = steps_in_pieces(requests, (2, 3, 64, 1, 65))
    cuts["small pieces"] = steps_in_pieces({"r0": requests["r0"]}, (2, 2, 5, 1))
    run_cuts(engine, requests, plain, cuts, 3e-5 if dtype == "float32" else 2.5e-2)


# ----------------------------------------------------------------------------- the wiring
def both_norms_config(hidden, kinds, share, head=None, final=None):
    """Layers of the wiring, one after another: kinds is a list of "full" (attention whose output bias the wiring takes along, feed-forward),
    "mixer" (attention alone: its bias stays with it) and "prenorm" (a layer of another wiring)."""
    ident = {"kind": "identity", "args": {"size": hidden}}
    norm = {"kind": "rmsnorm", "args": {"size": hidden, "eps": EPS}}
    none = {"kind": "none", "args": {}}
    mixer = {"kind": "general_attention", "args": attention_args(hidden, C.attention(2, 1, 16, 8, 0.4, 40))}
    ff = {"kind": "gated", "args": {"hidden": hidden, "intermediate": 40, "activation": "silu", "gate": "gate", "up": "up", "down": "down"}}
    blocks = []
    for kind in kinds:
        alone = kind == "mixer"
        b = {"arrangement": "prenorm" if kind == "prenorm" else "both_norms", "mixer": mixer, "feed_forward": none if alone else ff, "mixer_norm": norm,
             "feed_forward_norm": none if alone else norm}
        if kind != "prenorm":
            b["arrangement_args"] = {"hidden": hidden, "eps": EPS, "share": share, "mixer_out": "after1", "feed_forward_out": "after2",
                                     "feed_forward": 0 if alone else 1}
        blocks.append(copy.deepcopy(b))
    return {"architectures": ["ProbeForCausalLM"], "hidden": hidden, "vocab": hidden, "limit": 4096, "final_norm": final or ident, "head": head or ident,
            "embedding": {"kind": "token_table", "args": {"vocab": hidden, "hidden": hidden}}, "blocks": blocks}


def plain_wiring(w, kinds, share, tokens):
    m = C.attention(2, 1, 16, 8, 0.4, 40)
    x = w["embed.weight"].astype(np.float64)[tokens]
    for l, kind in enumerate(kinds):
        u = P.sub(w, f"layers.{l}.")
        mix, ff = (lambda a: P.mixer_attention(a, P.sub(u, "mixer."), m, EPS)), (lambda a: P.gated_unit(a, P.sub(u, "feed_forward.")))
        if kind == "prenorm":
            x = x + mix(P.rms_norm(x, u["mixer_norm.weight"], EPS))
            x = x + ff(P.rms_norm(x, u["feed_forward_norm.weight"], EPS))
            continue
        x = P.sublayer(x, u["mixer_norm.weight"], u["after1"], EPS, share, mix)
        if kind == "full":
            x = P.sublayer(x, u["feed_forward_norm.weight"], u["after2"], EPS, share, ff)
    return x


@pytest.mark.parametrize("hidden", [50, 64, 1040])
@pytest.mark.parametrize("kinds", [("full", "full"), ("mixer", "full", "mixer"), ("full", "prenorm", "full", "prenorm")])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_norm_on_both_sides_of_every_sublayer(hidden, kinds, dtype, toy_plugin, tmp_path):
    """A layer's last result joins the stream in the next layer's first kernel (of this wiring, or of another), the last layer's in the
    model's own; the identity as final norm shows the stream itself."""
    import velomind_b200 as vm
    share = 0.45
    cfg = both_norms_config(hidden, kinds, share)
    rng = np.random.default_rng(len(kinds) + hidden)
    w = shape_weights(random_tensors(vm.weight_table(cfg), rng, 0.25), rng)
    if dtype == "bfloat16":
        w = rounded_to_bf16(w)
    folder = write_model(str(tmp_path / "wiring"), cfg, w, as_bf16=dtype == "bfloat16")
    engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 6, max_slots=3)
    requests = S.make_requests(hidden, (70, 5, 90, 1), seed=13)
    plain = {rid: plain_wiring(w, kinds, share, toks) for rid, toks in requests.items()}
    cuts = standard_cuts(requests)
    cuts["pieces"] = steps_in_pieces(requests, (2, 1, 1, 30, 1))
    run_cuts(engine, requests, plain, cuts, 3e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("vocab", [77, 96])
def test_the_last_sum_joins_the_final_norm_and_logits_are_capped(vocab, toy_plugin, tmp_path):
    """An RMS norm behind the last layer (its kernel then carries the last layer's sum at the wanted rows alone) and a head whose logits would go
    far beyond the cap; rows that start on no 16-byte boundary when the vocabulary is odd."""
    import velomind_b200 as vm
    hidden, cap, kinds = 64, 2.5, ("full", "full")
    cfg = both_norms_config(hidden, kinds, 0.7, head={"kind": "linear", "args": {"vocab": vocab, "hidden": hidden, "soft_cap": cap}},
                            final={"kind": "rmsnorm", "args": {"size": hidden, "eps": EPS}})
    cfg["vocab"] = vocab
    cfg["embedding"]["args"]["vocab"] = vocab
    rng = np.random.default_rng(vocab)
    w = shape_weights(random_tensors(vm.weight_table(cfg), rng, 0.4), rng)
    folder = write_model(str(tmp_path / "capped"), cfg, w)
    engine = vm.Engine(vm.load_model(folder, "float32", "cuda:0"), 64 * 6, max_slots=3, max_step_tokens=33)      # (long prompts come in several pieces)
    requests = S.make_requests(vocab, (70, 5, 90, 1), seed=14)
    plain = {}
    for rid, toks in requests.items():
        z = P.lin(P.rms_norm(plain_wiring(w, kinds, 0.7, toks), w["norm.weight"], EPS), w["head.weight"])
        assert np.abs(z).max() > 2 * cap or len(toks) < 10
        plain[rid] = P.soft_cap(z, cap)
    run_cuts(engine, requests, plain, standard_cuts(requests), 3e-5)


# ----------------------------------------------------------------------------- shaped: sharp scores, so that one key off shows
@pytest.mark.parametrize("window", [33, 64, 75])
def test_keys_at_the_windows_edges_decide(window, toy_plugin, tmp_path):
    """With sharp scores a window one token longer or shorter, or slopes left out, give another answer at many places (checked on the plain
    implementation first); the library must give the right one, in prompts, pieces and decode steps."""
    import velomind_b200 as vm
    m = C.attention(4, 2, 16, 16, 2.5, window)
    requests = S.make_requests(64, (330, 150), seed=window)
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 3e-2)):
        w, folder = probe_model(tmp_path, vm, "attention", 64, m, dtype, 100 + window)
        plain = {}
        places = {"longer": 0, "shorter": 0, "level": 0}
        for rid, toks in requests.items():
            x, y = plain_mixer("attention", m, w, toks)
            plain[rid] = x + y
            level, P.slopes = P.slopes, lambda H: [0.0] * H
            flat = plain_mixer("attention", m, w, toks)[1]
            P.slopes = level
            for key, other in (("longer", plain_mixer("attention", dict(m, mask={"size": window + 1}), w, toks)[1]),
                               ("shorter", plain_mixer("attention", dict(m, mask={"size": window - 1}), w, toks)[1]), ("level", flat)):
                places[key] += int((np.abs(other - y).max(axis=1)[window:] > 0.05 * np.abs(y).max()).sum())
        assert min(places.values()) >= 3, places
        engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 8, max_slots=2)
        cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=120),
                "batches": S.steps_unequal_batches(requests, tails=(90, 40)), "pieces": steps_in_pieces(requests, (70, 2, 64, 1, 33))}
        run_cuts(engine, requests, plain, cuts, tol)


@pytest.mark.parametrize("window", [64, 130, 200])
def test_one_planted_key_decides_to_the_last_place_of_the_window(window, toy_plugin, tmp_path):
    """Every query points the same way (a large bias), and one rare token's key does too: while it is visible it takes nearly all the weight,
    and the answer jumps at the very place where it leaves the window (checked on the plain implementation)."""
    import velomind_b200 as vm
    m = C.attention(2, 1, 16, 16, 2.0, window)

    def plant(w):
        way = np.random.default_rng(5).normal(0.0, 1.0, 16).astype(np.float32)
        w[MIX + "q.b"][:] = 20.0 * np.concatenate([way, way])
        w["embed.weight"][:, 0] = 0.0                    # one direction of the stream belongs to the rare token alone
        w["embed.weight"][0] = 0.0
        w["embed.weight"][0, 0] = 4.0
        w[MIX + "k"][:, 0] = 6.0 * way

    requests = S.make_requests(64, (460, 300), seed=window)
    for toks in requests.values():
        for i in range(len(toks)):
            toks[i] = 0 if i % (window + 20) == 30 else max(toks[i], 1)
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 3e-2)):
        w, folder = probe_model(tmp_path, vm, "attention", 64, m, dtype, 3, change=plant)
        plain = {}
        for rid, toks in requests.items():
            x, y = plain_mixer("attention", m, w, toks)
            plain[rid] = x + y
            leaves = [i + window for i in range(30, len(toks) - window, window + 20)]          # the first place that no longer sees it
            longer = plain_mixer("attention", dict(m, mask={"size": window + 1}), w, toks)[1]
            shorter = plain_mixer("attention", dict(m, mask={"size": window - 1}), w, toks)[1]
            for i in leaves:
                assert np.abs(longer[i] - y[i]).max() > 0.3 * np.abs(y).max() and np.abs(shorter[i - 1] - y[i - 1]).max() > 0.3 * np.abs(y).max(), i
        engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 10, max_slots=2)
        cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=250),
                "batches": S.steps_unequal_batches(requests, tails=(240, 200)), "pieces": steps_in_pieces(requests, (70, 2, 64, 1, 33))}
        run_cuts(engine, requests, plain, cuts, tol)


def test_far_keys_decide_where_every_token_is_visible(toy_plugin, tmp_path):
    """Latent attention with sharp scores: keys hundreds of tokens back carry much of the weight (checked on the plain implementation: a
    rotation off by one place, or hiding everything beyond 128 tokens, gives another answer), across page borders, in prompts, pieces and 200
    decode steps."""
    import velomind_b200 as vm
    m = C.latent(2, 16, 8, 24, 32, 1.5, base=100.0)
    requests = S.make_requests(64, (450, 130), seed=21)
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 4e-2)):
        w, folder = probe_model(tmp_path, vm, "latent_attention", 64, m, dtype, 11)
        plain = {}
        for rid, toks in requests.items():
            x, y = plain_mixer("latent_attention", m, w, toks)
            plain[rid] = x + y
            if len(toks) > 400:
                whole, P.sees = P.sees, lambda n, window=None: whole(n, 128)
                near = plain_mixer("latent_attention", m, w, toks)[1]
                P.sees = whole
                assert (np.abs(near - y).max(axis=1)[200:] > 0.05 * np.abs(y).max()).sum() >= 20
        engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 10, max_slots=2)
        cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=200),
                "batches": S.steps_unequal_batches(requests, tails=(150, 60)), "pieces": steps_in_pieces(requests, (70, 2, 64, 1, 129))}
        run_cuts(engine, requests, plain, cuts, tol)


@pytest.mark.parametrize("m", [C.delta(2, 1, 16, 16, 3), C.delta(2, 2, 64, 64, 4)], ids=["16", "64"])
def test_the_memory_is_carried_far(m, toy_plugin, tmp_path):
    """Decays close to 1 and small writes: what the first tokens wrote still decides the answer hundreds of tokens later (checked on the
    plain implementation: other first tokens, another last row), through a prompt in pieces and 300 decode steps."""
    import velomind_b200 as vm

    def long_memory(w):
        w[MIX + "A_log"][:] = -4.0
        w[MIX + "dt_bias"][:] = -2.0
        w[MIX + "b"][:] = w[MIX + "b"] * 0.3          # (writes of about a half)

    w, folder = probe_model(tmp_path, vm, "delta", 64, m, "float32", 41, change=long_memory)
    requests = S.make_requests(64, (420, 35), seed=6)
    for i, toks in enumerate(requests["r0"]):
        if i >= 20:
            requests["r0"][i] = toks % 3               # three tokens keep coming; what only the first twenty wrote stays where it is
    plain = {}
    for rid, toks in requests.items():
        x, y = plain_mixer("delta", m, w, toks)
        plain[rid] = x + y
        if len(toks) > 400:
            other = [(t + 7) % 64 for t in toks[:20]] + toks[20:]
            y2 = plain_mixer("delta", m, w, other)[1]
            assert np.abs(y2[-1] - y[-1]).max() > 0.1 * np.abs(y).max()
    engine = vm.Engine(vm.load_model(folder, "float32", "cuda:0"), 64 * 8, max_slots=2)
    cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=300), "pieces": steps_in_pieces(requests, (100, 2, 64, 1, 7))}
    run_cuts(engine, requests, plain, cuts, 1e-4)


def test_keys_that_come_again_are_corrected_inside_a_chunk(toy_plugin, tmp_path):
    """The same few tokens over and over with full writes and no forgetting: the corrections inside a chunk of 64 tokens then cancel almost
    everything (the triangular system is far from the identity), and very strong decays beside weak ones in one chunk leave sums of logarithms of
    several hundred, whose differences still have to be exact."""
    import velomind_b200 as vm
    m = C.delta(3, 1, 16, 16, 2)
    for name, change in (("repeats", lambda w: (w[MIX + "A_log"].fill(-8.0), w[MIX + "b"].__imul__(6.0))),
                         ("decays", lambda w: (w[MIX + "A_log"].fill(2.5), w[MIX + "a"].__imul__(8.0)))):
        w, folder = probe_model(tmp_path / name, vm, "delta", 64, m, "float32", 43, change=change)
        requests = {"r0": [3, 9, 3, 4] * 45, "r1": S.make_requests(64, (150,), seed=8)["r0"]}
        plain = {}
        for rid, toks in requests.items():
            x, y = plain_mixer("delta", m, w, toks)
            plain[rid] = x + y
        engine = vm.Engine(vm.load_model(folder, "float32", "cuda:0"), 64 * 8, max_slots=2)
        cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=60), "batches": S.steps_unequal_batches(requests, tails=(70, 33)),
                "pieces": steps_in_pieces(requests, (65, 2, 63, 1))}
        run_cuts(engine, requests, plain, cuts, 1e-4)


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def zab_folders(tmp_path_factory):
    import velomind_b200 as vm
    root = tmp_path_factory.mktemp("zabozen")
    return {k: vm.write_random_model(str(root / k), C.config(k), seed=s, std=0.12, norm_jitter=0.2, dtype="float32")
            for k, s in (("a", 5), ("b", 6), ("c", 7), ("d", 8), ("e", 9))}


def plain_logits(folder, requests):
    cfg, w = P.read_model(folder)
    return cfg, {rid: P.forward(cfg, w, toks) for rid, toks in requests.items()}


@pytest.mark.parametrize("which", ["a", "b", "c", "d", "e"])
def test_whole_model_float32(which, zab_folders):
    import velomind_b200 as vm
    engine = vm.Engine(vm.load_model(zab_folders[which], "float32", "cuda:0"), 64 * 7, max_slots=3)     # few pages and slots: both are used again
    requests = S.make_requests(C.config(which)["vocab"], (50, 6, 140, 64, 2, 129), seed=8)
    cfg, plain = plain_logits(zab_folders[which], requests)
    cuts = standard_cuts(requests)
    cuts["pieces"] = steps_in_pieces(requests, (3, 2, 64, 70, 1))
    run_cuts(engine, requests, plain, cuts, 1e-4)
    engine.cache.check()


@pytest.mark.parametrize("which", ["a", "b", "c", "d", "e"])
def test_whole_model_bfloat16(which, zab_folders, tmp_path):
    """The serving precision: weights rounded to bfloat16, then compared with the plain implementation on the SAME rounded weights."""
    import velomind_b200 as vm
    cfg, w = P.read_model(zab_folders[which])
    bits = rounded_to_bf16(w)
    folder = write_model(str(tmp_path / "b16"), cfg, bits, as_bf16=True)
    engine = vm.Engine(vm.load_model(folder, "bfloat16", "cuda:0"), 64 * 16, max_slots=4)
    requests = S.make_requests(cfg["vocab"], (200, 31, 330), seed=9)
    plain = {rid: P.forward(cfg, bits, toks) for rid, toks in requests.items()}
    scale = max(float(np.abs(v).max()) for v in plain.values())
    for steps in (S.steps_whole(requests), S.steps_tail_one_by_one(requests, tail=40), S.steps_unequal_batches(requests, tails=(30, 11, 45))):
        got = S.run_steps_in_process(engine, steps)
        exp = S.expected_rows(steps, requests, plain)
        err = np.concatenate([np.abs(got[k] - exp[k]).max(axis=1) for k in exp]) / scale
        # (a head of the delta rule that reads almost nothing is still divided by its root mean square: at a few places rounding is magnified)
        assert np.median(err) < 0.02 and np.quantile(err, 0.98) < 0.06, (float(np.median(err)), float(np.quantile(err, 0.98)), float(err.max()))


@pytest.mark.parametrize("keeper,reader", [(20, 90), (90, 20), (20, None), (None, 20)])
def test_a_layer_on_another_ones_keys_sees_with_its_own_window(keeper, reader, tmp_path):
    """Two layers on the same keys with sharp scores and unlike windows: the keys stay as long as the wider of the two needs them, and
    either window one token off would show (checked on the plain implementation)."""
    import velomind_b200 as vm
    cfg = C.config("e")
    first, second = C.attention(2, 1, 16, 16, 2.0, keeper), C.attention(2, 1, 16, 16, 2.5, reader, kv_from=0)
    cfg.update(width=64, vocab=64, layers=[C.layer("attention", first, 48), C.layer("attention", second, None)])
    folder = vm.write_random_model(str(tmp_path / "shared"), cfg, seed=3, std=0.3, norm_jitter=0.2, dtype="float32")
    requests = S.make_requests(64, (230, 60), seed=31)
    _, plain = plain_logits(folder, requests)
    w = P.read_model(folder)[1]
    for l, size in ((0, keeper), (1, reader)):
        other = copy.deepcopy(cfg)
        other["layers"][l]["mixer"]["mask"] = {"size": size + 1 if size else 150}
        moved = np.abs(P.forward(other, w, requests["r0"]) - plain["r0"]).max(axis=1)
        assert (moved > 0.02 * np.abs(plain["r0"]).max()).sum() >= 3
    engine = vm.Engine(vm.load_model(folder, "float32", "cuda:0"), 64 * 6, max_slots=2)
    cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=190), "batch": S.steps_unequal_batches(requests, batch=2, tails=(150, 30)),
            "pieces": steps_in_pieces(requests, (65, 2, 40, 1))}
    run_cuts(engine, requests, plain, cuts, 1e-4)


def test_long_decoding_passes_windows_over_decoded_tokens(zab_folders):
    """300 decode steps behind a short prompt: every window of model a (33, 70 and 9 tokens, all on one layer's keys) moves over decoded
    tokens only, pages that fell out of the widest go back, and steps are replayed from graphs."""
    import velomind_b200 as vm
    engine = vm.Engine(vm.load_model(zab_folders["a"], "float32", "cuda:0"), 64 * 8, max_slots=2)
    assert engine.use_graphs
    requests = S.make_requests(150, (310, 40), seed=10)
    cfg, plain = plain_logits(zab_folders["a"], requests)
    run_cuts(engine, requests, plain, {"tail": S.steps_tail_one_by_one(requests, tail=300), "batch": S.steps_unequal_batches(requests, batch=2, tails=(290, 30))}, 1e-4)
    assert engine.graphs_captured > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_row_does_not_depend_on_its_batch(dtype, zab_folders):
    """The same requests alone, in a batch, and on other slots and pages: decode steps of one batch size share their kernels, so the rows of a
    batch of equal requests are equal bit for bit."""
    import velomind_b200 as vm
    engine = vm.Engine(vm.load_model(zab_folders["b"], dtype, "cuda:0"), 64 * 24, max_slots=6)
    toks = S.make_requests(352, (150,), seed=17)["r0"]
    spare = engine.open()
    engine.step([vm.Entry(spare, toks[:70], [])])                   # (other pages and another slot for the ones that follow)
    slots = [engine.open() for _ in range(3)]
    for lo, hi in ((0, 100), (100, 101), (101, 102), (102, 104), (104, 150)):
        got = engine.step([vm.Entry(s, toks[lo:hi], list(range(hi - lo))) for s in slots]).float().cpu().numpy().reshape(3, hi - lo, -1)
        assert np.array_equal(got[0], got[1]) and np.array_equal(got[0], got[2]), (lo, hi)
    for s in slots + [spare]:
        engine.close(s)
    engine.cache.check()


# ----------------------------------------------------------------------------- through the entry points
def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(P.forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


def test_greedy_generation_through_the_entry_point(zab_folders):
    import velomind_b200 as vm
    cfg, w = P.read_model(zab_folders["a"])
    te = vm.load(zab_folders["a"], dtype="float32", max_tokens=2048)
    prompts = [[1, 2, 3, 4, 5], [100, 7], [9] * 70]
    out = te.generate(prompts, temperature=0.0, max_tokens=6, stop_tokens=())
    assert [len(r.tokens) for r in out] == [6, 6, 6]
    for prompt, r in zip(prompts, out):
        seq = list(prompt)
        for tok in r.tokens:
            row = P.forward(cfg, w, seq)[-1]
            assert row[tok] >= row.max() - 1e-4, (seq, tok, int(row.argmax()))
            seq.append(tok)
    # several decode steps queued on the device give the same tokens: memories and kept rows move on there
    again = te.generate(prompts, temperature=0.0, max_tokens=6, stop_tokens=(), steps_per_sync=4)
    assert [r.tokens for r in again] == [r.tokens for r in out]


def test_the_console_program_generates(zab_folders):
    cfg, w = P.read_model(zab_folders["e"])
    want = greedy(cfg, w, [5, 6, 7, 8], 5)
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "smollm2_chat"), "--model", zab_folders["e"], "--dtype", "float32", "--temp", "0",
                           "--max-tokens", "5", "--prompt-ids", "5,6,7,8"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    line = [ln for ln in proc.stdout.splitlines() if ln.startswith("Output: ")][0]
    assert line == "Output: " + "".join(f"[{t}]" for t in want)


def test_trace_replay_program(zab_folders, tmp_path):
    requests = S.make_requests(150, (40, 3, 90), seed=12)
    cfg, plain = plain_logits(zab_folders["a"], requests)
    steps = S.steps_unequal_batches(requests, tails=(20, 2, 33))
    out = str(tmp_path / "out")
    for dtype, tol in (("float32", 1e-4), ("bfloat16", None)):
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", zab_folders["a"], "--dtype", dtype, "--out", out,
                               "--max-tokens", str(64 * 6)], input=S.to_jsonl(steps), text=True, capture_output=True, timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [ln for ln in proc.stdout.splitlines() if ln.startswith("done ")] == [f"done {s['step']}" for s in steps]
        want = S.expected_rows(steps, requests, plain)
        scale = max(1.0, max(float(np.abs(v).max()) for v in want.values()))
        for step, rows in want.items():
            got = np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])
            assert got.shape == rows.shape
            if tol is not None:
                assert float(np.abs(got - rows).max()) <= tol * scale, step
            else:
                assert np.isfinite(got).all()
