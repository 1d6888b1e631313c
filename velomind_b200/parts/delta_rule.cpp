// The gated delta rule over a matrix memory per head, as a mixer.
//
//   q, k = W_q x, W_k x  [kv_heads, dim];  v = W_v x  [heads, vdim];  head h reads q and k of number h / (heads / kv_heads)
//   every channel of q, k, v: a short causal convolution over time (`taps` K, tensors q.conv, k.conv, v.conv [channels, K]; the last K - 1
//   projected rows of a sequence are part of its state), then SiLU;  q, k <- x / sqrt(sum x^2 + 1e-6) per head;  q *= q_scale
//   beta = sigmoid(W_b x)_h;   g = exp(-exp(A_log_h) softplus((W_a x)_h + dt_bias_h))
//   per head  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q             S [dim, vdim], zero at the sequence's start
//   every head's o is divided by its root mean square, times `norm` [vdim], times silu(W_g x) value by value;  then W_o
//
// q | k | v | g | b | a come out of one stacked product as float32 (its rows filled up to a multiple of eight); everything between that
// product and the gated heads is float32, and the memory lives in the cache's float32 state area of the sequence.
#include <cmath>

#include "args.h"
#include "linear.h"

namespace vmb {

class DeltaRule : public Mixer {
public:
    explicit DeltaRule(const json::Value& a) {
        const char* k = "delta_rule";
        hidden_ = static_cast<int>(arg_int(a, "hidden", k));
        H_ = static_cast<int>(arg_int(a, "heads", k));
        G_ = static_cast<int>(arg_int_or(a, "kv_heads", H_, k));
        Dk_ = static_cast<int>(arg_int(a, "dim", k));
        Dv_ = static_cast<int>(arg_int_or(a, "vdim", Dk_, k));
        K_ = static_cast<int>(arg_int(a, "taps", k));
        q_scale_ = static_cast<float>(arg_number_or(a, "q_scale", 1.0 / std::sqrt(static_cast<double>(Dk_)), k));
        eps_ = static_cast<float>(arg_number_or(a, "eps", 1e-6, k));
        if (H_ <= 0 || G_ <= 0 || H_ % G_) throw ConfigError(format("part '%s': heads (%d) must be a multiple of kv_heads (%d)", k, H_, G_));
        if (Dk_ <= 0 || Dv_ <= 0) throw ConfigError(format("part '%s': dim and vdim must be positive", k));
        if (Dk_ > 512) throw ConfigError(format("part '%s': dim (%d) above 512 has no kernel", k, Dk_));
        if (K_ < 1 || K_ > 16) throw ConfigError(format("part '%s': taps (%d) must be within 1..16", k, K_));
    }

    WeightTable weight_specs() const override {
        const long long nqk = static_cast<long long>(G_) * Dk_, nv = static_cast<long long>(H_) * Dv_;
        WeightTable t;
        t["q"].shape = t["k"].shape = {nqk, hidden_};
        t["v"].shape = t["g"].shape = {nv, hidden_};
        t["q.conv"].shape = t["k.conv"].shape = {nqk, K_};
        t["v.conv"].shape = {nv, K_};
        t["b"].shape = t["a"].shape = {H_, hidden_};
        t["A_log"].shape = t["dt_bias"].shape = {H_};
        t["norm"].shape = {Dv_};
        t["norm"].init_ones = true;
        t["o"].shape = {hidden_, nv};
        return t;
    }

    void bind(const Weights& w, BindContext& bc) override {
        proj_.bind({&w.at("q"), &w.at("k"), &w.at("v"), &w.at("g"), &w.at("b"), &w.at("a")}, bc, 8);
        out_.bind({&w.at("o")}, bc);
        taps_ = bc.upload_stacked({&w.at("q.conv"), &w.at("k.conv"), &w.at("v.conv")}, DType::F32);
        A_log_ = bc.upload(w.at("A_log"), DType::F32);
        dt_bias_ = bc.upload(w.at("dt_bias"), DType::F32);
        norm_ = bc.upload(w.at("norm"), DType::F32);
    }

    bool graph_safe() const override { return true; }

    CacheNeed cache_need() const override {
        CacheNeed n;
        n.state_floats = vm_delta_state_floats(H_, G_, Dk_, Dv_, K_);
        return n;
    }

    void forward(StepContext& ctx, const void* x, void* out) override {
        const int ld = static_cast<int>(proj_.out_features);
        float* proj = static_cast<float*>(ctx.take_tokens(ld, DType::F32));
        project_f32(ctx, proj_, x, proj);
        ops::DeltaArgs d;
        d.g_off = 2 * G_ * Dk_ + H_ * Dv_;
        d.b_off = d.g_off + H_ * Dv_;
        d.a_off = d.b_off + H_;
        d.taps = static_cast<const float*>(taps_.ptr);
        d.K = K_;
        d.A_log = static_cast<const float*>(A_log_.ptr);
        d.dt_bias = static_cast<const float*>(dt_bias_.ptr);
        d.norm_w = static_cast<const float*>(norm_.ptr);
        d.eps = eps_;
        d.q_scale = q_scale_;
        d.H = H_;
        d.G = G_;
        d.Dk = Dk_;
        d.Dv = Dv_;
        void* heads = ctx.take_tokens(static_cast<long long>(H_) * Dv_, ctx.act_dtype);
        ops::delta_rule(proj, ld, d, ctx, heads);
        ctx.give(proj);
        project(ctx, out_, heads, out);
        ctx.give(heads);
    }

private:
    int hidden_ = 0, H_ = 0, G_ = 0, Dk_ = 0, Dv_ = 0, K_ = 1;
    float q_scale_ = 1.f, eps_ = 1e-6f;
    Linear proj_, out_;
    DeviceTensor taps_, A_log_, dt_bias_, norm_;
};

namespace {
RegisterPart reg("mixer", "delta_rule", [](const json::Value& a) { return std::make_shared<DeltaRule>(a); });
}  // namespace

}  // namespace vmb
