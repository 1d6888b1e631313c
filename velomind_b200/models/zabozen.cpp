// Zabozen as a plan of parts: a decoder whose config.json lists its layers one by one, with a norm in front of and behind every sublayer
// (x += residual_mult * norm_b(sublayer(norm(x))), arrangement `both_norms`), an untied head and softly capped logits.  Mixers:
//   "attention":         grouped-query softmax attention without rotation: biases on q, k, v and the output, every q and k head divided by its
//                        root mean square, a bias linear in the distance (one fixed slope per head), a sliding window; a layer with `kv_from`
//                        reads another layer's keys and values with its own queries and window
//   "latent_attention":  queries straight from the layer's input, keys and values from a cached low-rank latent, a rotated key part shared by all
//                        heads (pairs i, i + dims / 2), every earlier token visible, a sigmoid gate per head
//   "delta":             the gated delta rule over a matrix memory per head, behind short convolutions with SiLU, with a SiLU gate and a norm
//                        per head on its output
// Feed-forward: a SiLU-gated unit, or none.
//
// config.json: "architecture": "Zabozen", "vocab", "width", "norm": {"eps"}, "residual_mult", "logit_softcap" (optional),
//   "layers": [{"type", "mixer": {...}, "mlp": {"kind": "dense", "ff"} | null}].
//   mixer of "attention":         heads, kv_heads, dim, vdim, scale, mask: {size}, kv_from (optional)
//   mixer of "latent_attention":  heads, dim, rot_dim, vdim, kv_rank, scale, rot: {base, dims}
//   mixer of "delta":             heads, kv_heads, dim, vdim, conv
// Tensors: embed, head, final.norm, and per layer l<i>.norm1, l<i>.norm1b, l<i>.norm2, l<i>.norm2b, l<i>.mix.*, l<i>.mlp.*.
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

long long window_of(const json::Value& mixer, const std::string& where) {
    const json::Value* mask = mixer.find("mask");
    if (!mask || mask->is_null()) return 0;
    if (!mask->is_object()) throw ConfigError(where + ": key 'mask' must be an object or null");
    return KeyReader(*mask, where + ".mask").integer_or("size", 0);
}

PartSpec attention(const json::Value& mx, int width, double eps, bool own_kv, const std::string& where) {
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
    a.set("window", window_of(mx, where));
    a.set("bias", 1);
    a.set("out_bias", 1);
    a.set("unit_heads", 1);
    a.set("slopes", 1);
    a.set("own_kv", own_kv ? 1 : 0);
    return PartSpec{"general_attention", a};
}

PartSpec latent_attention(const json::Value& mx, int width, double eps, bool own_kv, const std::string& where) {
    KeyReader m(mx, where);
    json::Value a;
    a.set("hidden", width);
    const long long dim = m.integer("dim"), rot_dim = m.integer_or("rot_dim", 0, 0);
    a.set("heads", m.integer("heads"));
    a.set("dim", dim);
    a.set("vdim", m.integer_or("vdim", dim));
    a.set("q_rank", 0);
    a.set("kv_rank", m.integer("kv_rank"));
    a.set("scale", m.number("scale"));
    a.set("eps", eps);
    a.set("window", window_of(mx, where));
    a.set("gate", 1);
    a.set("gate_per_head", 1);
    a.set("own_latent", own_kv ? 1 : 0);
    a.set("rot_dim", rot_dim);
    if (rot_dim > 0) {
        KeyReader rot(need_object(mx, "rot", where), where + ".rot");
        json::Value pa;
        pa.set("head_dim", rot_dim);
        pa.set("theta", rot.number("base"));
        pa.set("rotary_dim", rot.integer_or("dims", rot_dim));
        pa.set("exact_frequencies", 1);          // base^(-2i / dims) in double precision, rounded once
        json::Value pos;
        pos.set("kind", "rotary_half_split");
        pos.set("args", pa);
        a.set("position", pos);
    }
    return PartSpec{"latent_attention", a};
}

PartSpec delta(const json::Value& mx, int width, double eps, const std::string& where) {
    KeyReader m(mx, where);
    json::Value a;
    a.set("hidden", width);
    const long long heads = m.integer("heads"), dim = m.integer("dim");
    a.set("heads", heads);
    a.set("kv_heads", m.integer_or("kv_heads", heads));
    a.set("dim", dim);
    a.set("vdim", m.integer_or("vdim", dim));
    a.set("taps", m.integer("conv"));
    a.set("q_scale", 1.0 / std::sqrt(static_cast<double>(dim)));
    a.set("eps", eps);
    return PartSpec{"delta_rule", a};
}

ModelPlan zabozen_plan(const json::Value& config, const std::string& where) {
    KeyReader top(config, where);
    const int vocab = static_cast<int>(top.integer("vocab")), width = static_cast<int>(top.integer("width"));
    const double eps = KeyReader(need_object(config, "norm", where), where + ": norm").number("eps");
    const double share = top.number_or("residual_mult", 1.0, false), cap = top.number_or("logit_softcap", 0.0);
    const json::Value& layers = need(config, "layers", where);
    if (!layers.is_array() || layers.as_array().empty()) throw ConfigError(where + ": key 'layers' must be a list of layers");

    auto norm = [&]() {
        json::Value a;
        a.set("size", width);
        a.set("eps", eps);
        a.set("tensor", "");                    // the prefix is the tensor's whole name
        return PartSpec{"rmsnorm", a};
    };

    ModelPlan plan;
    plan.hidden_size = width;
    plan.vocab_size = vocab;
    const int n = static_cast<int>(layers.as_array().size());
    int n_att = 0, n_lat = 0, n_delta = 0, n_borrowed = 0, n_dense = 0;
    for (int l = 0; l < n; ++l) {
        const json::Value& L = layers.as_array()[l];
        const std::string lw = format("%s: layers[%d]", where.c_str(), l);
        if (!L.is_object()) throw ConfigError(lw + " must be an object");
        const json::Value& type = need(L, "type", lw);
        const json::Value& mx = need_object(L, "mixer", lw);
        const std::string t = type.is_string() ? type.as_string() : "?";
        int from = -1;                           // the layer whose keys and values (or latents) this one reads
        if (const json::Value* f = mx.find("kv_from"); f && !f->is_null()) {
            if (!f->is_integer() || f->as_int() < 0 || f->as_int() >= l) throw ConfigError(lw + ".mixer: kv_from must name an earlier layer");
            from = static_cast<int>(f->as_int());
            const json::Value& other = need(layers.as_array()[from], "type", format("%s: layers[%d]", where.c_str(), from));
            const json::Value& om = need_object(layers.as_array()[from], "mixer", format("%s: layers[%d]", where.c_str(), from));
            const json::Value* again = om.find("kv_from");
            if (t == "delta" || !(other == type) || (again && !again->is_null()))
                throw ConfigError(format("%s.mixer: kv_from names layer %d, which has no keys and values of its own for this mixer", lw.c_str(), from));
            ++n_borrowed;
        }
        BlockSpec b;
        b.prefix = format("l%d.", l);
        b.names = {{"mixer", "mix."}, {"feed_forward", "mlp."}, {"mixer_norm", "norm1"}, {"feed_forward_norm", "norm2"}};
        if (t == "attention") { b.mixer = attention(mx, width, eps, from < 0, lw + ".mixer"); ++n_att; }
        else if (t == "latent_attention") { b.mixer = latent_attention(mx, width, eps, from < 0, lw + ".mixer"); ++n_lat; }
        else if (t == "delta") { b.mixer = delta(mx, width, eps, lw + ".mixer"); ++n_delta; }
        else throw ConfigError(format("%s: type '%s' is not a mixer of this architecture (attention, latent_attention, delta)", lw.c_str(), t.c_str()));
        b.mixer_norm = norm();
        json::Value wiring;
        wiring.set("hidden", width);
        wiring.set("eps", eps);
        wiring.set("share", share);
        wiring.set("mixer_out", "norm1b");
        wiring.set("feed_forward_out", "norm2b");
        b.arrangement = "both_norms";
        const json::Value* mlp = L.find("mlp");
        if (!mlp || mlp->is_null()) {
            wiring.set("feed_forward", 0);
            b.feed_forward = PartSpec{"none", json::Value()};
            b.feed_forward_norm = PartSpec{"none", json::Value()};
        } else {
            const std::string fw = lw + ".mlp";
            const json::Value& kind = need(*mlp, "kind", fw);
            if (!kind.is_string() || kind.as_string() != "dense") throw ConfigError(fw + ": kind must be 'dense'");
            json::Value f;
            f.set("hidden", width);
            f.set("intermediate", KeyReader(*mlp, fw).integer("ff"));
            f.set("activation", "silu");
            f.set("gate", "gate");
            f.set("up", "up");
            f.set("down", "down");
            b.feed_forward = PartSpec{"gated", f};
            b.feed_forward_norm = norm();
            ++n_dense;
        }
        b.arrangement_args = wiring;
        plan.blocks.push_back(std::move(b));
        plan.schedule.push_back(ScheduleEntry{l, from});
    }
    json::Value e;
    e.set("vocab", vocab);
    e.set("hidden", width);
    e.set("tensor", "");
    plan.embedding = PartSpec{"token_table", e};
    plan.embedding_prefix = "embed";
    plan.final_norm = norm();
    plan.final_norm_prefix = "final.norm";
    json::Value head = e;
    head.set("soft_cap", cap);
    plan.head = PartSpec{"linear", head};
    plan.head_prefix = "head";
    plan.max_positions = 0;                      // rotary angles are computed from the position itself: no table, no limit of its own
    json::Value d;
    d.set("Vocab", format("%d tokens", vocab));
    d.set("Hidden", width);
    d.set("Layers", format("%d attention, %d latent attention, %d delta (%d on another layer's keys)", n_att, n_lat, n_delta, n_borrowed));
    d.set("FeedForward", format("%d dense", n_dense));
    plan.describe = d;
    return plan;
}

struct RegisterZabozen {
    RegisterZabozen() { register_architecture("Zabozen", zabozen_plan); }
} register_zabozen;

}  // namespace

}  // namespace vmb
