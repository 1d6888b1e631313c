// Depunex as a plan of parts: a decoder whose config.json lists its layers one by one.  A layer has ONE norm (RMSNorm, weights stored about
// zero) and both its mixer and its feed-forward read its output, each scaled per column before the sum (arrangement `shared_norm`); then an
// input of the token's own follows, gated by the stream.  The embedding is scaled and a second table read by a hash of (previous token,
// token) is added; the head is the embedding table itself, with softly capped logits.  Mixers:
//   "mamba2":    the state-space mixer with a matrix state per head (part `mamba2`)
//   "parallel":  left: grouped-query softmax attention without biases, rotary positions (pairs i, i + dims / 2) with slowed long wave
//                lengths, a chunked mask (a token sees its own chunk of places); right: the selective state-space mixer with a state per
//                channel (part `selective_scan`); joined as left_scale * left + right_scale * right
// Feed-forward: the clamped gated unit, or routed experts (sigmoid scores, the `top` largest among the experts of the best groups, a group's
// score being the sum of its two largest; weights are the scores over their sum; SiLU-gated experts), or none.
//
// config.json: "architecture": "Depunex", "vocab", "width", "norm": {"eps"}, "embedding": {"scale", "bigram": {"buckets", "mul_prev",
//   "mul_cur"}}, "token_side": {"dim"}, "logit_softcap", "layers": [{"type", "mixer": {...}, "mlp": {...} | null}].
//   mamba2 mixer:      heads, vdim, state, groups, conv, norm_groups
//   parallel mixer:    left: {heads, kv_heads, dim, vdim, scale, mask: {size}, rot: {base, dims, scaling: {factor, low, high, original}}},
//                      right: {inner, dt_rank, state, conv}, left_scale, right_scale
//   mlp kind "dense":  ff, limit
//   mlp kind "moe":    expert: {ff}, router: {experts, top, groups: {count, keep}}
// Tensors: embed, bigram, side.embed, final.norm, and per layer l<i>.norm1, l<i>.ls1, l<i>.ls2, l<i>.side.*, l<i>.mix.*, l<i>.mlp.*.
#include <cmath>

#include "velomind_b200/velomind.h"

namespace vmb {

namespace {

const json::Value& need(const json::Value& o, const char* key, const std::string& where) {
    const json::Value* v = o.is_object() ? o.find(key) : nullptr;
    if (!v) throw ConfigError(where + ": missing required key '" + key + "'");
    return *v;
}

const json::Value& need_object(const json::Value& o, const char* key, const std::string& where) {
    const json::Value& v = need(o, key, where);
    if (!v.is_object()) throw ConfigError(where + ": key '" + key + "' must be an object");
    return v;
}

const json::Value* optional_object(const json::Value& o, const char* key, const std::string& where) {
    const json::Value* v = o.find(key);
    if (!v || v->is_null()) return nullptr;
    if (!v->is_object()) throw ConfigError(where + ": key '" + key + "' must be an object or null");
    return v;
}

json::Value part(const std::string& kind, const json::Value& args) {
    json::Value p;
    p.set("kind", kind);
    p.set("args", args);
    return p;
}

// {"kind": rotary_half_split, "args": {...}} from a mixer's "rot": {base, dims, scaling}
json::Value rotation(const json::Value& rot, long long dim, const std::string& where) {
    KeyReader r(rot, where);
    const long long dims = r.integer_or("dims", dim, 0);
    if (dims == 0) return part("none", json::Value());
    json::Value a;
    a.set("head_dim", dim);
    a.set("theta", r.number("base"));
    a.set("rotary_dim", dims);
    a.set("exact_frequencies", 1);
    if (const json::Value* s = optional_object(rot, "scaling", where)) {
        KeyReader k(*s, where + ".scaling");
        json::Value sc;
        for (const char* key : {"factor", "low", "high", "original"}) sc.set(key, k.number(key));
        a.set("scaling", sc);
    }
    return part("rotary_half_split", a);
}

json::Value attention(const json::Value& mx, int width, double eps, const std::string& where) {
    KeyReader m(mx, where);
    json::Value a;
    a.set("hidden", width);
    const long long heads = m.integer("heads"), dim = m.integer("dim");
    a.set("heads", heads);
    a.set("kv_heads", m.integer_or("kv_heads", heads));
    a.set("dim", dim);
    a.set("vdim", m.integer_or("vdim", dim));
    a.set("scale", m.number("scale", false));
    a.set("eps", eps);
    if (const json::Value* rot = optional_object(mx, "rot", where)) a.set("position", rotation(*rot, dim, where + ".rot"));
    if (const json::Value* mask = optional_object(mx, "mask", where)) a.set("chunk", KeyReader(*mask, where + ".mask").integer("size"));
    return part("general_attention", a);
}

json::Value selective_scan(const json::Value& mx, int width, const std::string& where) {
    KeyReader m(mx, where);
    json::Value a;
    a.set("hidden", width);
    for (const char* key : {"inner", "dt_rank", "state", "conv"}) a.set(key, m.integer(key));
    return part("selective_scan", a);
}

PartSpec mixer_parallel(const json::Value& mx, int width, double eps, const std::string& where) {
    KeyReader m(mx, where);
    json::Value a;
    a.set("hidden", width);
    a.set("left", attention(need_object(mx, "left", where), width, eps, where + ".left"));
    a.set("right", selective_scan(need_object(mx, "right", where), width, where + ".right"));
    a.set("join", "weighted");
    a.set("left_scale", m.number("left_scale", false));
    a.set("right_scale", m.number("right_scale", false));
    return PartSpec{"side_by_side", a};
}

PartSpec mixer_mamba2(const json::Value& mx, int width, double eps, const std::string& where) {
    KeyReader m(mx, where);
    json::Value a;
    a.set("hidden", width);
    for (const char* key : {"heads", "vdim", "state", "conv"}) a.set(key, m.integer(key));
    a.set("groups", m.integer_or("groups", 1));
    a.set("norm_groups", m.integer_or("norm_groups", 1));
    a.set("eps", eps);
    return PartSpec{"mamba2", a};
}

PartSpec routed(const json::Value& mlp, int width, const std::string& where) {
    const json::Value& rj = need_object(mlp, "router", where);
    KeyReader router(rj, where + ".router");
    json::Value f;
    f.set("hidden", width);
    f.set("experts", router.integer("experts"));
    f.set("top", router.integer("top"));
    f.set("ff", KeyReader(need_object(mlp, "expert", where), where + ".expert").integer("ff"));
    f.set("routing", "sigmoid");
    f.set("normalize", 1);
    f.set("glu", 3);                         // SiLU-gated experts, the routing weight on their output
    f.set("activation", "silu");
    if (const json::Value* groups = optional_object(rj, "groups", where + ".router")) {
        KeyReader g(*groups, where + ".router.groups");
        const long long count = g.integer("count");
        f.set("groups", count);
        f.set("groups_keep", g.integer_or("keep", count));
        f.set("groups_top", 2);              // a group's score: the sum of its two largest scores
    }
    return PartSpec{"routed_experts", f};
}

ModelPlan depunex_plan(const json::Value& config, const std::string& where) {
    KeyReader top(config, where);
    const int vocab = static_cast<int>(top.integer("vocab")), width = static_cast<int>(top.integer("width"));
    const double eps = KeyReader(need_object(config, "norm", where), where + ": norm").number("eps");
    const json::Value& layers = need(config, "layers", where);
    if (!layers.is_array() || layers.as_array().empty()) throw ConfigError(where + ": key 'layers' must be a list of layers");
    const int n = static_cast<int>(layers.as_array().size());
    const json::Value* side = optional_object(config, "token_side", where);
    const long long side_dim = side ? KeyReader(*side, where + ": token_side").integer("dim") : 0;

    auto norm = [&]() {
        json::Value a;
        a.set("size", width);
        a.set("eps", eps);
        a.set("tensor", "");                    // the prefix is the tensor's whole name
        a.set("about_one", 1);
        return PartSpec{"rmsnorm", a};
    };

    ModelPlan plan;
    plan.hidden_size = width;
    plan.vocab_size = vocab;
    int n_mamba2 = 0, n_parallel = 0, n_dense = 0, n_moe = 0;
    for (int l = 0; l < n; ++l) {
        const json::Value& L = layers.as_array()[l];
        const std::string lw = format("%s: layers[%d]", where.c_str(), l);
        if (!L.is_object()) throw ConfigError(lw + " must be an object");
        const json::Value& type = need(L, "type", lw);
        const json::Value& mx = need_object(L, "mixer", lw);
        BlockSpec b;
        b.prefix = format("l%d.", l);
        b.names = {{"mixer", "mix."}, {"feed_forward", "mlp."}, {"mixer_norm", "norm1"}};
        const std::string t = type.is_string() ? type.as_string() : "?";
        if (t == "mamba2") { b.mixer = mixer_mamba2(mx, width, eps, lw + ".mixer"); ++n_mamba2; }
        else if (t == "parallel") { b.mixer = mixer_parallel(mx, width, eps, lw + ".mixer"); ++n_parallel; }
        else throw ConfigError(format("%s: type '%s' is not a mixer of this architecture (mamba2, parallel)", lw.c_str(), t.c_str()));
        b.mixer_norm = norm();
        b.feed_forward_norm = PartSpec{"none", json::Value()};
        b.arrangement = "shared_norm";
        json::Value w;
        w.set("hidden", width);
        w.set("eps", eps);
        w.set("mixer_scale", "ls1");
        w.set("feed_forward_scale", "ls2");
        if (side) {
            w.set("token", "side");
            w.set("token_dim", side_dim);
            w.set("token_offset", l * side_dim);
        }
        const json::Value* mlp = optional_object(L, "mlp", lw);
        if (!mlp) {
            w.set("feed_forward", 0);
            b.feed_forward = PartSpec{"none", json::Value()};
        } else {
            const std::string fw = lw + ".mlp";
            const json::Value& kind = need(*mlp, "kind", fw);
            const std::string k = kind.is_string() ? kind.as_string() : "?";
            if (k == "dense") {
                KeyReader d(*mlp, fw);
                json::Value f;
                f.set("hidden", width);
                f.set("intermediate", d.integer("ff"));
                f.set("limit", d.number("limit"));
                f.set("alpha", 1.702);           // the design's constant
                f.set("gate", "gate");
                f.set("up", "up");
                f.set("down", "down");
                b.feed_forward = PartSpec{"gated", f};
                ++n_dense;
            } else if (k == "moe") {
                b.feed_forward = routed(*mlp, width, fw);
                ++n_moe;
            } else {
                throw ConfigError(fw + ": kind must be 'dense' or 'moe'");
            }
        }
        b.arrangement_args = w;
        plan.blocks.push_back(std::move(b));
        plan.schedule.push_back(ScheduleEntry{l, -1});
    }

    json::Value emb;
    emb.set("vocab", vocab);
    emb.set("hidden", width);
    emb.set("tensor", "embed");
    std::string kind = "token_table";
    if (const json::Value* e = optional_object(config, "embedding", where)) {
        emb.set("scale", KeyReader(*e, where + ": embedding").number_or("scale", 1.0, false));
        if (const json::Value* big = optional_object(*e, "bigram", where + ": embedding")) {
            KeyReader k(*big, where + ": embedding.bigram");
            kind = "token_pairs_table";
            emb.set("pairs_tensor", "bigram");
            emb.set("buckets", k.integer("buckets"));
            emb.set("mul_prev", k.integer("mul_prev", 0));
            emb.set("mul_cur", k.integer("mul_cur", 0));
        }
    }
    plan.embedding = PartSpec{kind, emb};
    plan.embedding_prefix = "";
    if (side) {
        json::Value r;
        r.set("embedding", part(kind, emb));
        r.set("vocab", vocab);
        r.set("cols", side_dim * n);
        r.set("rows_tensor", "side.embed");
        plan.embedding = PartSpec{"with_token_rows", r};
    }
    json::Value h;
    h.set("vocab", vocab);
    h.set("hidden", width);
    h.set("tensor", "");
    if (top.has("logit_softcap")) h.set("soft_cap", top.number("logit_softcap"));
    plan.final_norm = norm();
    plan.final_norm_prefix = "final.norm";
    plan.head = PartSpec{"linear", h};
    plan.head_prefix = "embed";                  // the embedding table itself (one tensor on the device, unscaled)
    plan.max_positions = 0;                      // rotary angles are computed from the position itself: no limit of its own
    json::Value d;
    d.set("Vocab", format("%d tokens", vocab));
    d.set("Hidden", width);
    d.set("Layers", format("%d (%d Mamba-2, %d parallel)", n, n_mamba2, n_parallel));
    d.set("FeedForward", format("%d dense, %d routed", n_dense, n_moe));
    plan.describe = d;
    return plan;
}

struct RegisterDepunex {
    RegisterDepunex() { register_architecture("Depunex", depunex_plan); }
} register_depunex;

}  // namespace

}  // namespace vmb
