// Position encodings.  A position part owns constants only; the mixer's kernels apply them.
#include "args.h"
#include "velomind_b200/kernels.h"

namespace vmb {

// Rotary positions.  Frequencies as the reference builds them, in float32: inv_freq[j] = 1 / pow(theta, 2j / rotary_dim)
// (examples/common/llama/llama_rope_mask.cpp:17-19); the angle pos * inv_freq[j] and its sine and cosine are computed in
// float32 on the device.  With `exact_frequencies` the frequencies are computed in double precision and rounded to float32 once.
// `scaling` slows the pairs of long wave lengths, l = 2 pi / f: f stays where l < original / high, becomes f / factor where
// l > original / low, and in between (1 - s) f / factor + s f with s = (original / l - low) / (high - low), in double precision.
// Which two values of a head make pair j is the `pairing`: the reference's half-split
// (j, j + rotary_dim/2) (src/cpu/ops/rotary_embedding.cpp:30-44), or interleaved (2j, 2j + 1).
class Rotary : public Position {
public:
    struct Scaling { double factor = 1.0, low = 1.0, high = 1.0, original = 0.0; };      // original 0: none
    Rotary(int head_dim, double theta, int rotary_dim, int pairing, bool exact, const Scaling& scaling)
        : head_dim_(head_dim), rotary_dim_(rotary_dim), pairing_(pairing), theta_(theta), exact_(exact), scaling_(scaling) {
        if (rotary_dim_ % 2 || rotary_dim_ <= 0 || rotary_dim_ > head_dim_)
            throw ConfigError(format("rotary_dim %d must be even and within the head size %d", rotary_dim_, head_dim_));
    }
    bool graph_safe() const override { return true; }
    std::vector<float> inv_freq_host() const {
        std::vector<float> f(static_cast<size_t>(rotary_dim_ / 2));
        for (int j = 0; j < rotary_dim_ / 2; ++j) {
            if (exact_) {                    // theta^(-2j / rotary_dim) in double precision, rounded once
                f[j] = static_cast<float>(scaled(std::pow(theta_, -2.0 * j / rotary_dim_)));
                continue;
            }
            const float exponent = (2.0f * static_cast<float>(j)) / static_cast<float>(rotary_dim_);
            f[j] = 1.0f / powf(static_cast<float>(theta_), exponent);
            if (scaling_.original > 0.0) f[j] = static_cast<float>(scaled(f[j]));
        }
        return f;
    }
    double scaled(double f) const {
        const Scaling& s = scaling_;
        if (!(s.original > 0.0)) return f;
        const double wave = 6.283185307179586476925286766559 / f;
        if (wave < s.original / s.high) return f;
        if (wave > s.original / s.low) return f / s.factor;
        const double share = (s.original / wave - s.low) / (s.high - s.low);
        return (1.0 - share) * f / s.factor + share * f;
    }
    RotaryTable tables(BindContext& bc) override {
        if (!table_.ptr) table_ = bc.upload_floats(inv_freq_host());
        return RotaryTable{static_cast<const float*>(table_.ptr), rotary_dim_, pairing_};
    }

private:
    int head_dim_, rotary_dim_, pairing_;
    double theta_;
    bool exact_;
    Scaling scaling_;
    DeviceTensor table_;
};

// No position encoding: queries and keys pass unrotated.
class NoPosition : public Position {
public:
    bool graph_safe() const override { return true; }
    RotaryTable tables(BindContext&) override { return RotaryTable{}; }
};

namespace {
std::shared_ptr<Part> make_rotary(const json::Value& a, int pairing, const char* kind) {
    const int head_dim = static_cast<int>(arg_int(a, "head_dim", kind));
    Rotary::Scaling sc;
    if (const json::Value* s = a.find("scaling")) {
        sc.factor = arg_number(*s, "factor", kind);
        sc.low = arg_number(*s, "low", kind);
        sc.high = arg_number(*s, "high", kind);
        sc.original = arg_number(*s, "original", kind);
        if (!(sc.factor > 0.0 && sc.low > 0.0 && sc.high > 0.0 && sc.original > 0.0))
            throw ConfigError(format("part '%s': factor, low, high and original of the scaling must be positive", kind));
    }
    return std::make_shared<Rotary>(head_dim, arg_number(a, "theta", kind), static_cast<int>(arg_int_or(a, "rotary_dim", head_dim, kind)), pairing,
                                    arg_int_or(a, "exact_frequencies", 0, kind) != 0, sc);
}
RegisterPart reg_half("position", "rotary_half_split", [](const json::Value& a) { return make_rotary(a, VM_PAIR_HALF_SPLIT, "rotary_half_split"); });
RegisterPart reg_inter("position", "rotary_interleaved", [](const json::Value& a) { return make_rotary(a, VM_PAIR_INTERLEAVED, "rotary_interleaved"); });
RegisterPart reg_none("position", "none", [](const json::Value&) { return std::make_shared<NoPosition>(); });
}  // namespace

}  // namespace vmb
