"""The Depunex design in the library against the plain implementation (tests/plain_depunex.py): each mechanism alone (through the
probe architecture of the tests' plug-in, which lets one part's output reach the logits), the wiring with its input of the token's own, whole
models cut into steps in several ways, weights shaped so that a fault would show where random ones would hide it, and generation through
the entry points."""
import copy
import os
import subprocess
import sys

import numpy as np
import pytest

import depunex_configs as C
import plain_depunex as P
import schedules as S
from test_kogilix_gpu import ff_block, mixer_block, probe_config, random_tensors, rounded_to_bf16, run_cuts, standard_cuts, steps_in_pieces, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
MIX, FF = "layers.0.mixer.", "layers.0.feed_forward."
EPS = 1e-5


# ----------------------------------------------------------------------------- a part's arguments, from the configuration's own object
def attention_args(hidden, m):
    a = {"hidden": hidden, "heads": m["heads"], "kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"], "scale": m["scale"], "eps": EPS,
         "chunk": m["mask"]["size"] if m.get("mask") else 0}
    if m.get("rot"):
        rot = {"head_dim": m["dim"], "theta": m["rot"]["base"], "rotary_dim": m["rot"]["dims"], "exact_frequencies": 1}
        if m["rot"].get("scaling"):
            rot["scaling"] = m["rot"]["scaling"]
        a["position"] = {"kind": "rotary_half_split", "args": rot}
    return a


def scan_args(hidden, m):
    return dict(m, hidden=hidden)


def mamba2_args(hidden, m):
    return dict(m, hidden=hidden, eps=EPS)


def parallel_args(hidden, m):
    return {"hidden": hidden, "left": {"kind": "general_attention", "args": attention_args(hidden, m["left"])},
            "right": {"kind": "selective_scan", "args": scan_args(hidden, m["right"])}, "join": "weighted", "left_scale": m["left_scale"],
            "right_scale": m["right_scale"]}


def dense_args(hidden, m):
    return {"hidden": hidden, "intermediate": m["ff"], "limit": m["limit"], "alpha": 1.702, "gate": "gate", "up": "up", "down": "down"}


def moe_args(hidden, m):
    r = m["router"]
    a = {"hidden": hidden, "experts": r["experts"], "top": r["top"], "ff": m["expert"]["ff"], "routing": "sigmoid", "normalize": 1, "glu": 3, "activation": "silu"}
    if r.get("groups"):
        a.update(groups=r["groups"]["count"], groups_keep=r["groups"]["keep"], groups_top=2)
    return a


PARTS = {"attention": ("general_attention", attention_args, P.attention_mixer), "scan": ("selective_scan", scan_args, P.mamba_mixer),
         "mamba2": ("mamba2", mamba2_args, lambda h, w, m: P.mamba2_mixer(h, w, m, EPS)), "parallel": ("side_by_side", parallel_args, P.parallel_mixer),
         "dense": ("gated", dense_args, lambda h, w, m: P.clamped_unit(h, w, m["limit"])), "moe": ("routed_experts", moe_args, P.routed)}

SLOWED = (5.0, 1.0, 3.0, 80)

# name -> (kind, hidden, the configuration's own object)
MECHANISMS = {
    # grouped keys (3 on 1), sizes that are no multiple of 8, a chunk that ends inside a page; frequencies on all sides of both borders
    "attention": ("attention", 80, C.attention(3, 1, 20, 12, 0.5, 50, 60.0, 16, SLOWED)),
    # sizes the tensor-core kernel of prompts takes (bfloat16), a chunk of exactly one page, chunks that straddle pages and tiles
    "attention_tiles": ("attention", 128, C.attention(6, 2, 64, 32, 0.1, 64, 1000.0, 32)),
    "attention_tiles_over_pages": ("attention", 64, C.attention(2, 2, 32, 64, 0.3, 100, 500.0, None, SLOWED)),
    "attention_tiles_wide": ("attention", 64, C.attention(2, 1, 128, 128, 0.1, 33, 7000.0, 96)),
    "attention_one_token": ("attention", 48, C.attention(2, 1, 8, 8, 0.4, 1)),
    "attention_small_chunk": ("attention", 48, C.attention(2, 2, 16, 16, 0.5, 7)),
    "attention_no_mask": ("attention", 64, C.attention(4, 4, 16, 24, 0.3, None, 100.0, 8)),
    "attention_no_rotation": ("attention", 64, C.attention(4, 2, 32, 32, 0.2, 130, dims=0)),
    # sizes no 16-byte copy takes; one tap; five taps; states of one, of six (padded to eight), of 24, of 100 and of 128 values per channel
    "scan_odd": ("scan", 56, C.scan(37, 5, 7, 3)),
    "scan_one_tap": ("scan", 64, C.scan(48, 4, 16, 1)),
    "scan_many_taps": ("scan", 64, C.scan(40, 8, 12, 5)),
    "scan_state_one": ("scan", 48, C.scan(20, 1, 1, 2)),
    "scan_16": ("scan", 64, C.scan(128, 32, 16, 4)),
    "scan_24": ("scan", 64, C.scan(72, 10, 24, 3)),
    "scan_40": ("scan", 48, C.scan(24, 16, 40, 4)),
    "scan_100": ("scan", 48, C.scan(32, 20, 100, 2)),
    "scan_128": ("scan", 64, C.scan(16, 8, 128, 4)),
    # so many channels that a few sequences fill the GPU: one pass over the tokens instead of pieces
    "scan_many_channels": ("scan", 32, C.scan(2400, 8, 8, 4)),
    "mamba2_groups": ("mamba2", 64, C.mamba2(6, 10, 14, 3, 3, 4)),
    "mamba2_two_taps": ("mamba2", 64, C.mamba2(2, 40, 32, 1, 2, 1)),
    "parallel": ("parallel", 64, C.parallel(C.attention(2, 1, 16, 24, 0.4, 40, 100.0), C.scan(48, 6, 12, 4), 0.7, 1.3)),
    "parallel_negative": ("parallel", 50, C.parallel(C.attention(1, 1, 10, 6, 0.6, 65), C.scan(30, 3, 5, 2), -0.4, 0.9)),
    "dense": ("dense", 64, C.dense(96, 0.7)),
    "dense_odd": ("dense", 50, C.dense(42, 1.9)),
    "dense_one": ("dense", 96, C.dense(64, 1.0)),
    "moe_groups": ("moe", 64, C.moe(12, 3, 32, (4, 2))),
    "moe_odd": ("moe", 50, C.moe(9, 2, 18, (3, 1))),
    "moe_no_groups": ("moe", 64, C.moe(7, 4, 40)),
    "moe_top_one": ("moe", 48, C.moe(6, 1, 16, (2, 1))),
    # more tokens than the tensor-core tiles of the experts need, at sizes they take
    "moe_tiles": ("moe", 128, C.moe(8, 4, 64, (4, 3))),
}


def shape_weights(w, rng):
    """Random weights that let every branch show: strong taps and biases, decays that spread between almost nothing and almost all."""
    for name in list(w):
        if name.endswith(".conv"):
            w[name] = rng.normal(0.0, 0.7, w[name].shape).astype(np.float32)
        elif name.endswith(("conv.b", ".D")):
            w[name] = rng.normal(0.0, 0.5, w[name].shape).astype(np.float32)
        elif name.endswith("A_log"):
            w[name] = rng.uniform(-3.0, 1.0, w[name].shape).astype(np.float32)
        elif name.endswith(("dt_bias", "dt.b")):
            w[name] = rng.uniform(-3.0, 1.0, w[name].shape).astype(np.float32)
    return w


def probe_model(tmp_path, vm, kind, hidden, m, dtype, seed, std=0.3, change=None):
    part, args, _ = PARTS[kind]
    block = ff_block if kind in ("dense", "moe") else mixer_block
    cfg = probe_config(hidden, block(part, args(hidden, m)))
    rng = np.random.default_rng(seed)
    w = shape_weights(random_tensors(vm.weight_table(cfg), rng, std), rng)
    if change:
        change(w)
    if dtype == "bfloat16":
        w = rounded_to_bf16(w)              # stored as bfloat16; the plain implementation runs on the same rounded numbers
    return w, write_model(str(tmp_path / f"{kind}_{dtype}"), cfg, w, as_bf16=dtype == "bfloat16")


def plain_part(kind, m, w, tokens):
    x = w["embed.weight"].astype(np.float64)[tokens]
    return x, PARTS[kind][2](x, P.under(w, FF if kind in ("dense", "moe") else MIX), m)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_each_mechanism_alone(name, dtype, toy_plugin, tmp_path):
    import velomind_b200 as vm
    kind, hidden, m = MECHANISMS[name]
    w, folder = probe_model(tmp_path, vm, kind, hidden, m, dtype, sum(name.encode()), std=0.15 if kind == "scan" else 0.3)
    engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 6, max_slots=3)      # few pages and slots: both are used again
    lengths = (70, 5, 130, 64, 1, 65) if name != "moe_tiles" else (300, 5, 70)
    requests = S.make_requests(hidden, lengths, seed=3)
    plain = {}
    for rid, toks in requests.items():
        x, y = plain_part(kind, m, w, toks)
        plain[rid] = x + y
    if kind == "moe":        # the test sees a wrong expert only if the routing spreads
        z = P.lin(w["embed.weight"].astype(np.float64), w[FF + "router"])
        assert len({int(e) for row in z for e in P.choose_experts(row, m["router"]["top"], m["router"].get("groups"))[0]}) == m["router"]["experts"]
    cuts = standard_cuts(requests)
    cuts["pieces"] = steps_in_pieces(requests, (2, 3, 64, 1, 65))
    cuts["small pieces"] = steps_in_pieces({"r0": requests["r0"]}, (2, 2, 5, 1))
    run_cuts(engine, requests, plain, cuts, 5e-5 if dtype == "float32" else 3e-2)


def test_clamping_decides_on_both_sides(toy_plugin, tmp_path):
    """Gates beyond the limit above (cut), far below (not cut), and ups beyond it on both sides, in the plain implementation first."""
    import velomind_b200 as vm
    m = C.dense(96, 0.7)
    for dtype, tol in (("float32", 3e-5), ("bfloat16", 2.5e-2)):
        w, folder = probe_model(tmp_path, vm, "dense", 64, m, dtype, 5, std=0.5)
        x = w["embed.weight"].astype(np.float64)
        g, u = P.lin(x, w[FF + "gate"]), P.lin(x, w[FF + "up"])
        assert (g > 0.7).mean() > 0.1 and (g < -3).mean() > 0.05 and (u > 0.7).mean() > 0.1 and (u < -0.7).mean() > 0.1
        requests = S.make_requests(64, (90, 7), seed=4)
        plain = {rid: sum(plain_part("dense", m, w, toks)) for rid, toks in requests.items()}
        engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 6, max_slots=3)
        run_cuts(engine, requests, plain, standard_cuts(requests), tol)


# ----------------------------------------------------------------------------- the wiring and the token's own input
def wiring_config(hidden, kinds, token_dim, vocab, final=None, embedding_scale=1.0):
    """Layers one after another: "full" (mixer and feed-forward), "mixer" (a mixer alone), "two" (two mixers side by side: the wiring
    carries their weighted sum out), "prenorm" (a layer of another wiring)."""
    ident = {"kind": "identity", "args": {"size": hidden}}
    norm = {"kind": "rmsnorm", "args": {"size": hidden, "eps": EPS, "about_one": 1}}
    none = {"kind": "none", "args": {}}
    att = {"kind": "general_attention", "args": attention_args(hidden, ATT)}
    par = {"kind": "side_by_side", "args": parallel_args(hidden, PAR)}
    ff = {"kind": "gated", "args": dense_args(hidden, C.dense(40, 0.9))}
    blocks = []
    for l, kind in enumerate(kinds):
        alone = kind == "mixer"
        b = {"arrangement": "prenorm" if kind == "prenorm" else "shared_norm", "mixer": par if kind == "two" else att, "feed_forward": none if alone else ff,
             "mixer_norm": norm, "feed_forward_norm": norm if kind == "prenorm" else none}
        if kind != "prenorm":
            b["arrangement_args"] = {"hidden": hidden, "eps": EPS, "mixer_scale": "s1", "feed_forward_scale": "s2", "feed_forward": 0 if alone else 1}
            if token_dim:
                b["arrangement_args"].update(token="own", token_dim=token_dim, token_offset=l * token_dim)
        blocks.append(copy.deepcopy(b))
    emb = {"kind": "token_pairs_table", "args": {"vocab": vocab, "hidden": hidden, "tensor": "weight", "pairs_tensor": "pairs", "buckets": PAIRS["buckets"],
                                                "mul_prev": PAIRS["mul_prev"], "mul_cur": PAIRS["mul_cur"], "scale": embedding_scale}}
    if token_dim:
        emb = {"kind": "with_token_rows", "args": {"embedding": emb, "vocab": vocab, "cols": token_dim * len(kinds), "rows_tensor": "rows"}}
    return {"architectures": ["ProbeForCausalLM"], "hidden": hidden, "vocab": hidden, "limit": 4096, "final_norm": final or ident, "head": ident,
            "embedding": emb, "blocks": blocks}


ATT = C.attention(2, 1, 16, 8, 0.4, 40, 100.0)
PAR = C.parallel(ATT, C.scan(24, 4, 6, 3), 0.6, -0.8)
PAIRS = {"buckets": 29, "mul_prev": 5, "mul_cur": 3}


def plain_wiring(w, kinds, token_dim, tokens, embedding_scale=1.0):
    x = P.embed(tokens, w["embed.weight"], embedding_scale, w["embed.pairs"], PAIRS)
    for l, kind in enumerate(kinds):
        u = P.under(w, f"layers.{l}.")
        mix = (lambda a: P.parallel_mixer(a, P.under(u, "mixer."), PAR)) if kind == "two" else (lambda a: P.attention_mixer(a, P.under(u, "mixer."), ATT))
        ff = lambda a: P.clamped_unit(a, P.under(u, "feed_forward."), 0.9)  # noqa: E731
        h = P.norm_about_one(x, u["mixer_norm.weight"], EPS)
        if kind == "prenorm":
            x = x + mix(h)
            x = x + ff(P.norm_about_one(x, u["feed_forward_norm.weight"], EPS))
            continue
        x = x + mix(h) * u["s1"] + (0.0 if kind == "mixer" else ff(h) * u["s2"])
        if token_dim:
            part = w["embed.rows"].astype(np.float64)[np.asarray(tokens), l * token_dim:(l + 1) * token_dim]
            x = P.token_input(x, part, u["own.gate"], u["own.proj"], u["own.norm"], EPS)
    return x


@pytest.mark.parametrize("hidden,token_dim", [(50, 6), (64, 32), (1040, 9), (64, 0), (50, 0)])
@pytest.mark.parametrize("kinds", [("full", "two", "full"), ("mixer", "full", "mixer"), ("two", "prenorm", "full", "prenorm")])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_norm_for_both_sublayers_and_the_tokens_own_input(hidden, token_dim, kinds, dtype, toy_plugin, tmp_path):
    """A layer's token input joins the stream in the next layer's first kernel (of this wiring, or of another), the last layer's in the model's
    own; the identity as final norm shows the stream itself."""
    import velomind_b200 as vm
    vocab = 60
    cfg = wiring_config(hidden, kinds, token_dim, vocab, embedding_scale=1.6)
    rng = np.random.default_rng(len(kinds) + hidden)
    w = shape_weights(random_tensors(vm.weight_table(cfg), rng, 0.14 if hidden < 500 else 0.03), rng)
    for name in w:
        if name.endswith(("norm.weight", ".s1", ".s2")):
            w[name] = rng.normal(0.0, 0.4, w[name].shape).astype(np.float32) + (0.0 if "norm" in name else 0.8)
    if dtype == "bfloat16":
        w = rounded_to_bf16(w)
    folder = write_model(str(tmp_path / "wiring"), cfg, w, as_bf16=dtype == "bfloat16")
    engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 6, max_slots=3)
    requests = S.make_requests(min(vocab, hidden), (70, 5, 90, 1), seed=13)
    plain = {rid: plain_wiring(w, kinds, token_dim, toks, 1.6) for rid, toks in requests.items()}
    cuts = standard_cuts(requests)
    cuts["pieces"] = steps_in_pieces(requests, (2, 1, 1, 30, 1))
    run_cuts(engine, requests, plain, cuts, 4e-5 if dtype == "float32" else 6e-2)


def test_every_branch_of_the_wiring_changes_the_answer(toy_plugin):
    """In the plain implementation: the pair table, the embedding's scale, the layer scales, the weight stored about zero and the layer's own part
    of the token's rows all show, so the comparison above would catch any of them left out."""
    import velomind_b200 as vm
    cfg = wiring_config(50, ("full", "two"), 6, 60)
    rng = np.random.default_rng(1)
    w = shape_weights(random_tensors(vm.weight_table(cfg), rng, 0.14), rng)
    toks = S.make_requests(50, (30,), seed=2)["r0"]
    base = plain_wiring(w, ("full", "two"), 6, toks)
    for change in (lambda v: v["embed.pairs"].fill(0), lambda v: v["layers.0.s1"].fill(1), lambda v: v["layers.1.s2"].fill(1),
                   lambda v: v["layers.0.mixer_norm.weight"].__isub__(1), lambda v: v["embed.rows"].__setitem__(slice(None), np.roll(v["embed.rows"], 6, 1))):
        v = {k: a.copy() for k, a in w.items()}
        change(v)
        assert np.abs(plain_wiring(v, ("full", "two"), 6, toks) - base).max() > 0.02 * np.abs(base).max()
    assert np.abs(plain_wiring(w, ("full", "two"), 6, toks, 1.2) - base).max() > 0.02 * np.abs(base).max()


# ----------------------------------------------------------------------------- shaped: one key off would show
@pytest.mark.parametrize("chunk", [33, 64, 100])
def test_keys_at_the_chunks_edges_decide(chunk, toy_plugin, tmp_path):
    """With sharp scores chunks one token longer or shorter, a sliding window of the same size, or chunks counted from another place give another
    answer at many places (checked on the plain implementation first); the library must give the right one, in prompts, pieces and decode steps."""
    import velomind_b200 as vm
    m = C.attention(4, 2, 16, 16, 2.5, chunk, 100.0, 8)
    requests = S.make_requests(64, (330, 150), seed=chunk)
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 4e-2)):
        w, folder = probe_model(tmp_path, vm, "attention", 64, m, dtype, 100 + chunk)
        plain = {}
        chunked = P.sees
        others = {"longer": lambda n, c: chunked(n, c + 1), "shorter": lambda n, c: chunked(n, c - 1), "shifted": lambda n, c: chunked(n + 7, c)[7:, 7:],
                  "sliding": lambda n, c: np.tril(np.ones((n, n), bool)) & ~np.tril(np.ones((n, n), bool), -c)}
        places = {key: 0 for key in others}
        for rid, toks in requests.items():
            x, y = plain_part("attention", m, w, toks)
            plain[rid] = x + y
            for key, mask in others.items():
                P.sees = mask
                try:
                    other = plain_part("attention", m, w, toks)[1]
                finally:
                    P.sees = chunked
                places[key] += int((np.abs(other - y).max(axis=1)[chunk:] > 0.05 * np.abs(y).max()).sum())
        assert min(places.values()) >= 3, places
        engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 8, max_slots=2)
        cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=120),
                "batches": S.steps_unequal_batches(requests, tails=(90, 40)), "pieces": steps_in_pieces(requests, (70, 2, 64, 1, 33))}
        run_cuts(engine, requests, plain, cuts, tol)


@pytest.mark.parametrize("chunk", [64, 90, 130])
def test_one_planted_key_decides_to_the_last_place_of_its_chunk(chunk, toy_plugin, tmp_path):
    """Every query points the same way and one rare token's key does too: while it is visible it takes nearly all the weight, and the answer
    jumps at the very place where the next chunk begins (checked on the plain implementation)."""
    import velomind_b200 as vm
    m = C.attention(2, 1, 16, 16, 0.2, chunk, dims=0)

    def plant(w):
        way = np.random.default_rng(5).normal(0.0, 1.0, 16).astype(np.float32)
        w["embed.weight"][:, 1] = 1.0                    # one direction of the stream is every token's, and the queries follow it
        w["embed.weight"][:, 0] = 0.0                    # another belongs to the rare token alone
        w["embed.weight"][0] = 0.0
        w["embed.weight"][0, :2] = 4.0, 1.0
        w[MIX + "q"][:, 1] = np.concatenate([way, way])
        w[MIX + "k"][:, 0] = 6.0 * way
        w[MIX + "k"][:, 1] = 0.0

    requests = S.make_requests(64, (460, 300), seed=chunk)
    for toks in requests.values():
        for i in range(len(toks)):
            toks[i] = 0 if i % chunk == chunk // 3 else max(toks[i], 1)
    for dtype, tol in (("float32", 5e-5), ("bfloat16", 4e-2)):
        w, folder = probe_model(tmp_path, vm, "attention", 64, m, dtype, 3, change=plant)
        plain = {}
        for rid, toks in requests.items():
            x, y = plain_part("attention", m, w, toks)
            plain[rid] = x + y
            longer = plain_part("attention", dict(m, mask={"size": 10000}), w, toks)[1]
            for i in range(chunk, len(toks), chunk):     # the first place of a chunk no longer sees it, the last place of the one before does
                assert np.abs(longer[i] - y[i]).max() > 0.2 * np.abs(y).max() and np.abs(longer[i - 1] - y[i - 1]).max() < 0.3 * np.abs(y).max(), i
        engine = vm.Engine(vm.load_model(folder, dtype, "cuda:0"), 64 * 10, max_slots=2)
        cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=250),
                "batches": S.steps_unequal_batches(requests, tails=(240, 200)), "pieces": steps_in_pieces(requests, (70, 2, 64, 1, 33))}
        run_cuts(engine, requests, plain, cuts, tol)


def test_pages_of_finished_chunks_go_back(tmp_path):
    """Three sequences of 320 tokens decode together in a cache of six pages (384 tokens): within chunks of 40 tokens each holds two at most."""
    import velomind_b200 as vm
    cfg = C.config("a")
    cfg["layers"] = [cfg["layers"][0]]
    cfg["layers"][0]["mixer"]["left"]["mask"] = {"size": 40}
    folder = vm.write_random_model(str(tmp_path / "small"), cfg, seed=3, std=0.2, dtype="float32")
    engine = vm.Engine(vm.load_model(folder, "float32", "cuda:0"), 64 * 6, max_slots=3)
    requests = S.make_requests(150, (320, 310, 300), seed=31)
    _, plain = plain_logits(folder, requests)
    run_cuts(engine, requests, plain, {"batch": S.steps_unequal_batches(requests, batch=3, tails=(280, 290, 270))}, 1e-4)


@pytest.mark.parametrize("kind,m", [("scan", C.scan(32, 4, 16, 3)), ("scan", C.scan(40, 3, 6, 4)), ("mamba2", C.mamba2(4, 16, 16, 2, 4, 1))],
                         ids=["scan_16", "scan_6", "mamba2"])
def test_the_state_is_carried_far(kind, m, toy_plugin, tmp_path):
    """Decays close to 1: what the first tokens wrote still decides the answer hundreds of tokens later (checked on the plain implementation:
    other first tokens, another last row), through a prompt in pieces and 300 decode steps."""
    import velomind_b200 as vm

    def long_memory(w):
        w[MIX + "A_log"][:] = -4.5
        w[MIX + ("dt.b" if kind == "scan" else "dt_bias")][:] = -2.0
        for name in (MIX + "dt",):
            if name in w:
                w[name][:] *= 0.2
        w[MIX + "D"][:] = 0.0

    w, folder = probe_model(tmp_path, vm, kind, 64, m, "float32", 41, change=long_memory)
    requests = S.make_requests(64, (420, 35), seed=6)
    for i, tok in enumerate(requests["r0"]):
        if i >= 20:
            requests["r0"][i] = tok % 3                # three tokens keep coming; what only the first twenty wrote fades slowly
    plain = {}
    for rid, toks in requests.items():
        x, y = plain_part(kind, m, w, toks)
        plain[rid] = x + y
        if len(toks) > 400:
            other = [(t + 7) % 64 for t in toks[:20]] + toks[20:]
            y2 = plain_part(kind, m, w, other)[1]
            assert np.abs(y2[-1] - y[-1]).max() > 1e-3 * np.abs(y).max()
    engine = vm.Engine(vm.load_model(folder, "float32", "cuda:0"), 64 * 8, max_slots=2)
    cuts = {"whole": S.steps_whole(requests), "tail": S.steps_tail_one_by_one(requests, tail=300), "pieces": steps_in_pieces(requests, (100, 2, 64, 1, 7))}
    run_cuts(engine, requests, plain, cuts, 5e-5)


def test_strong_decays_and_step_sizes_stay_exact(toy_plugin, tmp_path):
    """Step sizes between a few thousandths and more than ten and rates up to e^3: products that underflow to zero beside decays that hardly move."""
    import velomind_b200 as vm
    m = C.scan(48, 6, 16, 4)

    def strong(w):
        rng = np.random.default_rng(9)
        w[MIX + "A_log"][:] = rng.uniform(-6.0, 3.0, w[MIX + "A_log"].shape)
        w[MIX + "dt.b"][:] = rng.uniform(-6.0, 12.0, w[MIX + "dt.b"].shape)

    w, folder = probe_model(tmp_path, vm, "scan", 64, m, "float32", 44, std=0.2, change=strong)
    requests = S.make_requests(64, (200, 64, 17), seed=7)
    plain = {rid: sum(plain_part("scan", m, w, toks)) for rid, toks in requests.items()}
    engine = vm.Engine(vm.load_model(folder, "float32", "cuda:0"), 64 * 8, max_slots=3)
    cuts = standard_cuts(requests)
    cuts["pieces"] = steps_in_pieces(requests, (65, 2, 63, 1))
    run_cuts(engine, requests, plain, cuts, 5e-5)


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def dep_folders(tmp_path_factory):
    import velomind_b200 as vm
    root = tmp_path_factory.mktemp("depunex")
    out = {}
    for k, seed in (("a", 5), ("b", 6), ("c", 7), ("d", 8), ("e", 9)):
        rng = np.random.default_rng(seed)
        w = shape_weights(random_tensors(vm.weight_table(C.config(k)), rng, 0.12), rng)
        out[k] = write_model(str(root / k), C.config(k), w)
    return out


def plain_logits(folder, requests):
    cfg, w = P.read_model(folder)
    return cfg, {rid: P.forward(cfg, w, toks) for rid, toks in requests.items()}


@pytest.mark.parametrize("which", ["a", "b", "c", "d", "e"])
def test_whole_model_float32(which, dep_folders):
    import velomind_b200 as vm
    engine = vm.Engine(vm.load_model(dep_folders[which], "float32", "cuda:0"), 64 * 7, max_slots=3)     # few pages and slots: both are used again
    requests = S.make_requests(C.config(which)["vocab"], (50, 6, 140, 64, 2, 129), seed=8)
    cfg, plain = plain_logits(dep_folders[which], requests)
    cuts = standard_cuts(requests)
    cuts["pieces"] = steps_in_pieces(requests, (3, 2, 64, 70, 1))
    run_cuts(engine, requests, plain, cuts, 1e-4)
    engine.cache.check()


@pytest.mark.parametrize("routed", [True, False])
@pytest.mark.parametrize("which", ["a", "b", "c", "d", "e"])
def test_whole_model_bfloat16(which, routed, dep_folders, tmp_path):
    """The serving precision: weights rounded to bfloat16, then compared with the plain implementation on the SAME rounded weights.  A router's
    close call may go the other way in bfloat16 (and the states carry what that changed), so the bound that holds for nearly every place is set
    for the same layers without routed experts."""
    import velomind_b200 as vm
    cfg, w = P.read_model(dep_folders[which])
    if not routed:
        for L in cfg["layers"]:
            if L["mlp"] and L["mlp"]["kind"] == "moe":
                L["mlp"] = C.dense(64, 1.2)
        rng = np.random.default_rng(3)
        w = shape_weights(random_tensors(vm.weight_table(cfg), rng, 0.12), rng)
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
        share, bound = (0.85, 0.08) if routed else (0.98, 0.06)
        assert np.median(err) < 0.02 and np.quantile(err, share) < bound, (float(np.median(err)), float(np.quantile(err, share)), float(err.max()))


def test_long_decoding_passes_chunks_over_decoded_tokens(dep_folders):
    """300 decode steps behind a short prompt: both chunk sizes of model a begin again and again among decoded tokens, pages of finished chunks
    go back, and steps are replayed from graphs."""
    import velomind_b200 as vm
    engine = vm.Engine(vm.load_model(dep_folders["a"], "float32", "cuda:0"), 64 * 8, max_slots=2)
    assert engine.use_graphs
    requests = S.make_requests(150, (310, 40), seed=10)
    cfg, plain = plain_logits(dep_folders["a"], requests)
    run_cuts(engine, requests, plain, {"tail": S.steps_tail_one_by_one(requests, tail=300), "batch": S.steps_unequal_batches(requests, batch=2, tails=(290, 30))}, 1e-4)
    assert engine.graphs_captured > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_row_does_not_depend_on_its_batch(dtype, dep_folders):
    """The same requests alone, in a batch, and on other slots and pages: decode steps of one batch size share their kernels, so the rows of a
    batch of equal requests are equal bit for bit."""
    import velomind_b200 as vm
    engine = vm.Engine(vm.load_model(dep_folders["b"], dtype, "cuda:0"), 64 * 24, max_slots=6)
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


def test_greedy_generation_through_the_entry_point(dep_folders):
    import velomind_b200 as vm
    cfg, w = P.read_model(dep_folders["a"])
    te = vm.load(dep_folders["a"], dtype="float32", max_tokens=2048)
    prompts = [[1, 2, 3, 4, 5], [100, 7], [9] * 70]
    out = te.generate(prompts, temperature=0.0, max_tokens=6, stop_tokens=())
    assert [len(r.tokens) for r in out] == [6, 6, 6]
    for prompt, r in zip(prompts, out):
        seq = list(prompt)
        for tok in r.tokens:
            row = P.forward(cfg, w, seq)[-1]
            assert row[tok] >= row.max() - 1e-4, (seq, tok, int(row.argmax()))
            seq.append(tok)
    # several decode steps queued on the device give the same tokens: states, kept rows and previous tokens move on there
    again = te.generate(prompts, temperature=0.0, max_tokens=6, stop_tokens=(), steps_per_sync=4)
    assert [r.tokens for r in again] == [r.tokens for r in out]


def test_the_console_program_generates(dep_folders):
    cfg, w = P.read_model(dep_folders["e"])
    want = greedy(cfg, w, [5, 6, 7, 8], 5)
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "smollm2_chat"), "--model", dep_folders["e"], "--dtype", "float32", "--temp", "0",
                           "--max-tokens", "5", "--prompt-ids", "5,6,7,8"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    line = [ln for ln in proc.stdout.splitlines() if ln.startswith("Output: ")][0]
    assert line == "Output: " + "".join(f"[{t}]" for t in want)


def test_trace_replay_program(dep_folders, tmp_path):
    requests = S.make_requests(150, (40, 3, 90), seed=12)
    cfg, plain = plain_logits(dep_folders["a"], requests)
    steps = S.steps_unequal_batches(requests, tails=(20, 2, 33))
    out = str(tmp_path / "out")
    for dtype, tol in (("float32", 1e-4), ("bfloat16", None)):
        proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", dep_folders["a"], "--dtype", dtype, "--out", out,
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
