// The selective state-space mixer of the first Mamba, as a mixer with a fixed-size state per sequence.
//
//   W_in h = [x | z]                       (C columns each)
//   x passes a short causal convolution per channel (taps `conv`, with bias) and SiLU
//   W_x x = [r | B | C]                    (dt_rank, state, state columns);   dt = softplus(W_dt r + dt.b), one per channel
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,  A = -exp(A_log);    y_c = sum_n S[c, n] C_n + D_c x_c
//   out = W_o (y * silu(z))
//
// What it keeps of a sequence, float32, in the cache's state area of the sequence's slot: S of all channels and the convolution's last
// conv - 1 inputs.  Both start at zero when the slot is opened and are carried from step to step.  The kernels are in
// csrc/selective_scan.cu; the projections are the library's or the weight-streaming products, except that a decode step makes the step
// sizes inside the recurrence's own kernel.
#include <cmath>

#include "args.h"
#include "linear.h"

namespace vmb {

class SelectiveScan : public Mixer {
public:
    explicit SelectiveScan(const json::Value& a) {
        const char* k = "selective_scan";
        hidden_ = static_cast<int>(arg_int(a, "hidden", k));
        C_ = static_cast<int>(arg_int(a, "inner", k));
        R_ = static_cast<int>(arg_int(a, "dt_rank", k));
        N_ = static_cast<int>(arg_int(a, "state", k));
        K_ = static_cast<int>(arg_int_or(a, "conv", 4, k));
        if (hidden_ <= 0 || C_ <= 0 || R_ <= 0) throw ConfigError(format("part '%s': hidden, inner and dt_rank must be positive", k));
        if (N_ <= 0 || N_ > vm_selective_max_state()) throw ConfigError(format("part '%s': state (%d) must be within 1..%d", k, N_, vm_selective_max_state()));
        if (K_ < 1 || K_ > 64) throw ConfigError(format("part '%s': conv (%d) must be within 1..64", k, K_));
    }

    WeightTable weight_specs() const override {
        WeightTable t;
        t["in"].shape = {2ll * C_, hidden_};
        t["conv"].shape = {C_, K_};
        t["conv.b"].shape = {C_};
        t["x"].shape = {R_ + 2ll * N_, C_};
        t["dt"].shape = {C_, R_};
        t["dt.b"].shape = {C_};
        t["A_log"].shape = {C_, N_};
        t["D"].shape = {C_};
        t["o"].shape = {hidden_, C_};
        return t;
    }

    void bind(const Weights& w, BindContext& bc) override {
        in_.bind({&w.at("in")}, bc);
        x_.bind({&w.at("x")}, bc, 8);
        dt_.bind({&w.at("dt")}, bc);
        out_.bind({&w.at("o")}, bc);
        taps_ = bc.upload(w.at("conv"), DType::F32);
        conv_b_ = bc.upload(w.at("conv.b"), DType::F32);
        dt_b_ = bc.upload(w.at("dt.b"), DType::F32);
        A2_ = bc.upload_mapped(w.at("A_log"), [](float v) { return static_cast<float>(-std::exp(static_cast<double>(v)) * 1.4426950408889634074); });
        D_ = bc.upload(w.at("D"), DType::F32);
    }

    bool graph_safe() const override { return true; }        // slots and token offsets are read on the device

    CacheNeed cache_need() const override {
        CacheNeed n;                                          // kind None: no keys, no values
        n.state_floats = static_cast<int>(vm_selective_state_floats(C_, N_, K_));
        return n;
    }

    void forward(StepContext& ctx, const void* x, void* out) override {
        const DType act = ctx.act_dtype;
        void* proj = ctx.take_tokens(2ll * C_, act);
        project(ctx, in_, x, proj);
        const void* z = static_cast<const char*>(proj) + static_cast<size_t>(C_) * dtype_size(act);
        void* u = ctx.take_tokens(C_, act);
        ops::short_conv_silu(proj, 2 * C_, 0, fp(taps_), fp(conv_b_), C_ * N_, ctx, C_, K_, u);
        const int ldr = static_cast<int>(x_.out_features);   // (filled up to a multiple of eight)
        float* r = static_cast<float*>(ctx.take_tokens(ldr, DType::F32));
        project_f32(ctx, x_, u, r);
        void* y = ctx.take_tokens(C_, act);
        if (ctx.one_token_each) {
            ops::selective_step(u, r, ldr, dt_.weight, R_, z, 2 * C_, fp(dt_b_), fp(A2_), fp(D_), ctx, y, C_, N_);
        } else {
            void* low = ctx.take_tokens(R_, act);
            ops::take_columns(r, ldr, 0, low, R_, ctx);
            float* dt = static_cast<float*>(ctx.take_tokens(C_, DType::F32));
            project_f32(ctx, dt_, low, dt);
            ctx.give(low);
            ops::selective_scan(u, dt, C_, r, ldr, R_, z, 2 * C_, fp(dt_b_), fp(A2_), fp(D_), ctx, y, C_, N_);
            ctx.give(dt);
        }
        ctx.give(r);
        ctx.give(u);
        ctx.give(proj);
        project(ctx, out_, y, out);
        ctx.give(y);
    }

private:
    static const float* fp(const DeviceTensor& t) { return static_cast<const float*>(t.ptr); }
    int hidden_ = 0, C_ = 0, R_ = 0, N_ = 0, K_ = 4;
    Linear in_, x_, dt_, out_;
    DeviceTensor taps_, conv_b_, dt_b_, A2_, D_;
};

namespace {
RegisterPart reg("mixer", "selective_scan", [](const json::Value& a) { return std::make_shared<SelectiveScan>(a); });
}  // namespace

}  // namespace vmb
