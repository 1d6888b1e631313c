// Kernels of a layer whose sublayers read the residual stream itself and whose norm sits on the sublayer's OUTPUT:
//
//   a short causal convolution over time on every channel of what a sublayer reads, added to it:
//       out_t = h_t + sum_j taps[:, j] * h_(t - K + 1 + j)        (zeros before the sequence's start)
//     with the last K - 1 inputs of every sequence kept in a float32 state area from step to step;
//   h += rmsnorm(y) * w, the residual sum of a normed sublayer output;
//   the same sum followed by the next sublayer's norm, for layers with a norm on both sides of every sublayer;
//   the polynomial activation  a N(z) + b N(z^2) + c N(z^3) + e, N = division of a token's row by its root mean square;
//   rotation of a slice of every head's row (rotary positions on a part of the head), copied to another layout;
//   multiplication by the sigmoid of a gate.
//
// The residual stream is float32; everything here computes in float32 and rounds once on the way out.
#include <cstdint>

#include "common.cuh"

namespace {

// ------------------------------------------------------------------------------------------------ convolution on the input
// grid (T); a block walks the channels of one token.  state [max_slots, state_stride] float32; this convolution's K - 1 kept
// rows of `hid` channels start at state_offset: row i holds the input at position p0 - (K - 1) + i, p0 the step's first position
// of the sequence.
template <typename T>
__global__ void input_conv_kernel(const float* __restrict__ h, const float* __restrict__ taps, const float* __restrict__ state, long long state_stride,
                                  int state_offset, const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                                  const int* __restrict__ cu_tokens, const int* __restrict__ slots, T* __restrict__ out, int hid, int K) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t = blockIdx.x;
    const int seq = seq_of_token[t];
    const int first = cu_tokens[seq];                    // the sequence's first token of this step
    const int in_step = t - first;                       // tokens of the sequence before this one in the step
    const float* kept = state + (size_t)slots[seq] * state_stride + state_offset;
    (void)positions;
    for (int c = threadIdx.x; c < hid; c += blockDim.x) {
        const float* w = taps + (size_t)c * K;
        float acc = h[(size_t)t * hid + c] * (1.0f + w[K - 1]);
        for (int j = 0; j < K - 1; ++j) {
            const int back = K - 1 - j;                  // how many tokens before t
            const float v = back <= in_step ? h[(size_t)(t - back) * hid + c] : kept[(size_t)(K - 1 - back + in_step) * hid + c];
            acc = fmaf(w[j], v, acc);
        }
        out[(size_t)t * hid + c] = vm_from_float<T>(acc);
    }
}

// The same for bfloat16 outputs and hid % 4 == 0: a thread makes four neighbouring channels of one token with 16-byte loads (the rows of
// earlier tokens come out of L1 / L2: the step's rows are read from memory once).  KT: the number of taps when it is 2, 3 or 4 (their
// 4 x K weights are K 16-byte loads), 0: any number (scalar loads of the weights).
template <int KT>
__global__ void __launch_bounds__(256)
input_conv_vec_kernel(const float* __restrict__ h, const float* __restrict__ taps, const float* __restrict__ state, long long state_stride,
                      int state_offset, const int* __restrict__ seq_of_token, const int* __restrict__ cu_tokens, const int* __restrict__ slots,
                      __nv_bfloat16* __restrict__ out, int hid, int K_any, long long n_vec) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= n_vec) return;
    const int K = KT ? KT : K_any;
    const int per = hid >> 2;
    const int t = (int)(idx / per), c = (int)(idx - (long long)t * per) << 2;
    const int seq = seq_of_token[t];
    const int in_step = t - cu_tokens[seq];
    const float* kept = state + (size_t)slots[seq] * state_stride + state_offset;
    float tw[KT ? 4 * KT : 4];
    if (KT) {
        const float4* w4 = reinterpret_cast<const float4*>(taps + (size_t)c * K);
#pragma unroll
        for (int q = 0; q < (KT ? KT : 1); ++q) {
            const float4 v = w4[q];
            tw[4 * q] = v.x; tw[4 * q + 1] = v.y; tw[4 * q + 2] = v.z; tw[4 * q + 3] = v.w;
        }
    }
    const float4 x = *reinterpret_cast<const float4*>(h + (size_t)t * hid + c);
    float4 acc;
    if (KT) {
        acc.x = x.x * (1.0f + tw[0 * KT + KT - 1]); acc.y = x.y * (1.0f + tw[1 * KT + KT - 1]);
        acc.z = x.z * (1.0f + tw[2 * KT + KT - 1]); acc.w = x.w * (1.0f + tw[3 * KT + KT - 1]);
    } else {
        acc.x = x.x * (1.0f + taps[(size_t)c * K + K - 1]); acc.y = x.y * (1.0f + taps[(size_t)(c + 1) * K + K - 1]);
        acc.z = x.z * (1.0f + taps[(size_t)(c + 2) * K + K - 1]); acc.w = x.w * (1.0f + taps[(size_t)(c + 3) * K + K - 1]);
    }
#pragma unroll
    for (int j = 0; j < (KT ? KT - 1 : 64); ++j) {
        if (!KT && j >= K - 1) break;
        const int back = K - 1 - j;
        const float* src = back <= in_step ? h + (size_t)(t - back) * hid + c : kept + (size_t)(K - 1 - back + in_step) * hid + c;
        const float4 v = *reinterpret_cast<const float4*>(src);
        if (KT) {
            acc.x = fmaf(tw[0 * KT + j], v.x, acc.x); acc.y = fmaf(tw[1 * KT + j], v.y, acc.y);
            acc.z = fmaf(tw[2 * KT + j], v.z, acc.z); acc.w = fmaf(tw[3 * KT + j], v.w, acc.w);
        } else {
            acc.x = fmaf(taps[(size_t)c * K + j], v.x, acc.x); acc.y = fmaf(taps[(size_t)(c + 1) * K + j], v.y, acc.y);
            acc.z = fmaf(taps[(size_t)(c + 2) * K + j], v.z, acc.z); acc.w = fmaf(taps[(size_t)(c + 3) * K + j], v.w, acc.w);
        }
    }
    const __nv_bfloat162 o01 = __floats2bfloat162_rn(acc.x, acc.y), o23 = __floats2bfloat162_rn(acc.z, acc.w);
    uint2 o;
    o.x = *reinterpret_cast<const unsigned*>(&o01); o.y = *reinterpret_cast<const unsigned*>(&o23);
    *reinterpret_cast<uint2*>(out + (size_t)t * hid + c) = o;
}

// Many tokens, 2 to 4 taps: a thread makes four neighbouring channels of RUN consecutive tokens and carries the K - 1 earlier rows along in
// registers, so every row of the step is loaded once per thread that needs it as a halo and once as the token itself (K - 1 + RUN loads
// for RUN tokens).  Where the next token belongs to another sequence the carried rows are fetched anew (from the step or the kept rows).
template <int KT, int RUN>
__global__ void __launch_bounds__(256)
input_conv_run_kernel(const float* __restrict__ h, const float* __restrict__ taps, const float* __restrict__ state, long long state_stride,
                      int state_offset, const int* __restrict__ seq_of_token, const int* __restrict__ cu_tokens, const int* __restrict__ slots,
                      __nv_bfloat16* __restrict__ out, int hid, int T, long long n_vec) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= n_vec) return;
    const int per = hid >> 2;
    const int g = (int)(idx / per), c = (int)(idx - (long long)g * per) << 2;
    float tw[4 * KT];
    {
        const float4* w4 = reinterpret_cast<const float4*>(taps + (size_t)c * KT);
#pragma unroll
        for (int q = 0; q < KT; ++q) {
            const float4 v = w4[q];
            tw[4 * q] = v.x; tw[4 * q + 1] = v.y; tw[4 * q + 2] = v.z; tw[4 * q + 3] = v.w;
        }
    }
    float4 win[KT - 1];                      // win[j]: the input KT - 1 - j tokens back
    int seq_before = -1;
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
        const int t = g * RUN + i;
        if (t >= T) break;
        const int seq = seq_of_token[t];
        if (seq != seq_before) {
            const int in_step = t - cu_tokens[seq];
            const float* kept = state + (size_t)slots[seq] * state_stride + state_offset;
#pragma unroll
            for (int j = 0; j < KT - 1; ++j) {
                const int back = KT - 1 - j;
                const float* src = back <= in_step ? h + (size_t)(t - back) * hid + c : kept + (size_t)(KT - 1 - back + in_step) * hid + c;
                win[j] = *reinterpret_cast<const float4*>(src);
            }
            seq_before = seq;
        }
        const float4 x = *reinterpret_cast<const float4*>(h + (size_t)t * hid + c);
        float4 acc;
        acc.x = x.x * (1.0f + tw[0 * KT + KT - 1]); acc.y = x.y * (1.0f + tw[1 * KT + KT - 1]);
        acc.z = x.z * (1.0f + tw[2 * KT + KT - 1]); acc.w = x.w * (1.0f + tw[3 * KT + KT - 1]);
#pragma unroll
        for (int j = 0; j < KT - 1; ++j) {
            acc.x = fmaf(tw[0 * KT + j], win[j].x, acc.x); acc.y = fmaf(tw[1 * KT + j], win[j].y, acc.y);
            acc.z = fmaf(tw[2 * KT + j], win[j].z, acc.z); acc.w = fmaf(tw[3 * KT + j], win[j].w, acc.w);
        }
        const __nv_bfloat162 o01 = __floats2bfloat162_rn(acc.x, acc.y), o23 = __floats2bfloat162_rn(acc.z, acc.w);
        uint2 o;
        o.x = *reinterpret_cast<const unsigned*>(&o01); o.y = *reinterpret_cast<const unsigned*>(&o23);
        *reinterpret_cast<uint2*>(out + (size_t)t * hid + c) = o;
#pragma unroll
        for (int j = 0; j + 1 < KT - 1; ++j) win[j] = win[j + 1];
        win[KT - 2] = x;
    }
}

// grid (B, ceil(hid / threads)); a thread owns one channel of one sequence and moves its K - 1 kept inputs on by the step's tokens.
// Row i of the new state is the input n - (K - 1) + i tokens into the step, or, before the step, row i + n of the old state; rows are
// written in ascending order, so a row is read before it is overwritten.
__global__ void input_conv_keep_kernel(const float* __restrict__ h, float* __restrict__ state, long long state_stride, int state_offset,
                                       const int* __restrict__ cu_tokens, const int* __restrict__ slots, int hid, int K) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int seq = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= hid) return;
    const int first = cu_tokens[seq], n = cu_tokens[seq + 1] - first;
    float* kept = state + (size_t)slots[seq] * state_stride + state_offset;
    for (int i = 0; i < K - 1; ++i) {
        const int at = n - (K - 1) + i;
        float v;
        if (at >= 0) v = h[(size_t)(first + at) * hid + c];
        else v = kept[(size_t)(i + n) * hid + c];
        kept[(size_t)i * hid + c] = v;
    }
}

// one token per sequence: convolution and kept inputs in one pass (a thread owns its channel's kept inputs)
template <typename T>
__global__ void input_conv_step_kernel(const float* __restrict__ h, const float* __restrict__ taps, float* __restrict__ state, long long state_stride,
                                       int state_offset, const int* __restrict__ slots, T* __restrict__ out, int hid, int K) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int seq = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= hid) return;
    float* kept = state + (size_t)slots[seq] * state_stride + state_offset;
    const float* w = taps + (size_t)c * K;
    const float x = h[(size_t)seq * hid + c];
    float acc = x * (1.0f + w[K - 1]);
    for (int j = 0; j < K - 1; ++j) {
        const float v = kept[(size_t)j * hid + c];
        acc = fmaf(w[j], v, acc);
        if (j > 0) kept[(size_t)(j - 1) * hid + c] = v;
    }
    if (K > 1) kept[(size_t)(K - 2) * hid + c] = x;
    out[(size_t)seq * hid + c] = vm_from_float<T>(acc);
}

// ------------------------------------------------------------------------------------------------ h += rmsnorm(y) * w
// one block per token; y float32 or T, rows of ld elements
template <typename Y>
__global__ void norm_residual_kernel(float* __restrict__ h, const Y* __restrict__ y, long long ld, const float* __restrict__ w, int hid, float eps) {
    __shared__ float red[32];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t = blockIdx.x;
    const Y* yr = y + (size_t)t * ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < hid; i += blockDim.x) {
        const float v = vm_to_float(yr[i]);
        ss += v * v;
    }
    ss = vm_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)hid + eps);
    for (int i = threadIdx.x; i < hid; i += blockDim.x) h[(size_t)t * hid + i] += vm_to_float(yr[i]) * inv * w[i];      // (the row comes out of L1 again)
}

// The same for bfloat16 y with hid % 4 == 0 and ld % 4 == 0: a warp per token, 8-byte loads of y (its second pass finds the row in L1),
// 16-byte updates of h; no block-wide barrier.
constexpr int NR_WARPS = 4;
__global__ void __launch_bounds__(NR_WARPS * 32)
norm_residual_vec_kernel(float* __restrict__ h, const __nv_bfloat16* __restrict__ y, long long ld, const float* __restrict__ w, int T, int hid, float eps) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t = blockIdx.x * NR_WARPS + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (t >= T) return;
    const uint2* yr = reinterpret_cast<const uint2*>(y + (size_t)t * ld);
    const int n4 = hid >> 2;
    float ss = 0.f;
    for (int i = lane; i < n4; i += 32) {
        const uint2 d = yr[i];
        const __nv_bfloat162 d01 = *reinterpret_cast<const __nv_bfloat162*>(&d.x), d23 = *reinterpret_cast<const __nv_bfloat162*>(&d.y);
        const float a = __low2float(d01), b = __high2float(d01), c = __low2float(d23), e = __high2float(d23);
        ss += a * a + b * b + c * c + e * e;
    }
    ss = vm_warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)hid + eps);
    float4* hr = reinterpret_cast<float4*>(h + (size_t)t * hid);
    const float4* w4 = reinterpret_cast<const float4*>(w);
    for (int i = lane; i < n4; i += 32) {
        const uint2 d = yr[i];
        const __nv_bfloat162 d01 = *reinterpret_cast<const __nv_bfloat162*>(&d.x), d23 = *reinterpret_cast<const __nv_bfloat162*>(&d.y);
        const float4 ww = w4[i];
        float4 v = hr[i];
        v.x += __low2float(d01) * inv * ww.x; v.y += __high2float(d01) * inv * ww.y;
        v.z += __low2float(d23) * inv * ww.z; v.w += __high2float(d23) * inv * ww.w;
        hr[i] = v;
    }
}

// The same sum for steps of one token per sequence, followed by the NEXT sublayer's input convolution on the row just made (a thread owns
// its channel through both): h += rmsnorm(y) * w ; out = h + conv(h) with the kept inputs moved on.  grid (B, ceil(hid / blockDim)): every
// block sums the squares of the token's whole row (a few KB out of L2) and then makes its own blockDim channels, so that a wide row is
// spread over several SMs instead of walked by one block.
template <typename Y, typename T>
__global__ void norm_residual_conv_step_kernel(float* __restrict__ h, const Y* __restrict__ y, long long ld, const float* __restrict__ w, int hid, float eps,
                                               const float* __restrict__ taps, float* __restrict__ state, long long state_stride, int state_offset,
                                               const int* __restrict__ slots, T* __restrict__ out, int K) {
    __shared__ float red[32];
    vm_pdl_launch_dependents();
    const int t = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
    const bool mine = c < hid;
    // weights are constants: they may be read before the wait on the kernel that makes y
    const float* tw = taps + (size_t)(mine ? c : 0) * K;
    const float wc = mine ? w[c] : 0.f, last = tw[K - 1];
    vm_pdl_wait();
    float* kept = state + (size_t)slots[t] * state_stride + state_offset;
    const Y* yr = y + (size_t)t * ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < hid; i += blockDim.x) {
        const float v = vm_to_float(yr[i]);
        ss += v * v;
    }
    ss = vm_block_sum(ss, red);
    if (!mine) return;
    const float inv = 1.0f / sqrtf(ss / (float)hid + eps);
    const float x = h[(size_t)t * hid + c] + vm_to_float(yr[c]) * inv * wc;
    h[(size_t)t * hid + c] = x;
    float acc = x * (1.0f + last);
    for (int j = 0; j < K - 1; ++j) {
        const float v = kept[(size_t)j * hid + c];
        acc = fmaf(tw[j], v, acc);
        if (j > 0) kept[(size_t)(j - 1) * hid + c] = v;
    }
    if (K > 1) kept[(size_t)(K - 2) * hid + c] = x;
    out[(size_t)t * hid + c] = vm_from_float<T>(acc);
}

// ------------------------------------------------------------------------------------------------ h += rmsnorm(y + bias) * w_out;  out = rmsnorm(h) * w_in
// A layer with a norm on both sides of its sublayers: the sum of one sublayer and the read of the next in one pass, one block per token.
// bias float32 [hid] or null.  `rows` (null: all): block i makes row rows[i] of h and y into row i of out, and h stays as it is.
__device__ __forceinline__ float4 ns_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ns_load4(const __nv_bfloat16* p) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void ns_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void ns_store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 r;
    r.x = *reinterpret_cast<const unsigned*>(&a);
    r.y = *reinterpret_cast<const unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
}

// rows of 4 n values: a thread keeps RUNS runs of four values of its row in registers (hid <= 4 * RUNS * blockDim)
template <typename T, int RUNS>
__global__ void __launch_bounds__(256)
norm_sum_norm_vec_kernel(float* __restrict__ h, const T* __restrict__ y, const float* __restrict__ bias, const float* __restrict__ w_out, float eps_out,
                         const float* __restrict__ w_in, float eps_in, T* __restrict__ out, const int* __restrict__ rows, int hid) {
    __shared__ float red[32];
    vm_pdl_launch_dependents();
    float4 wo[RUNS], wi[RUNS], x[RUNS], s[RUNS];
#pragma unroll
    for (int c = 0; c < RUNS; ++c) {                     // (weights are constants: they may be read before the wait)
        const int i = (threadIdx.x + c * blockDim.x) * 4;
        wo[c] = wi[c] = x[c] = s[c] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i >= hid) continue;
        wo[c] = ns_load4(w_out + i);
        wi[c] = ns_load4(w_in + i);
        if (bias) x[c] = ns_load4(bias + i);
    }
    vm_pdl_wait();
    const size_t t = rows ? rows[blockIdx.x] : blockIdx.x;
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < RUNS; ++c) {
        const int i = (threadIdx.x + c * blockDim.x) * 4;
        if (i >= hid) continue;
        const float4 v = ns_load4(y + t * hid + i);
        s[c] = ns_load4(h + t * hid + i);
        x[c].x += v.x; x[c].y += v.y; x[c].z += v.z; x[c].w += v.w;
        ss += x[c].x * x[c].x + x[c].y * x[c].y + x[c].z * x[c].z + x[c].w * x[c].w;
    }
    ss = vm_block_sum(ss, red);
    const float fo = 1.0f / sqrtf(ss / (float)hid + eps_out);
    float st = 0.f;
#pragma unroll
    for (int c = 0; c < RUNS; ++c) {
        const int i = (threadIdx.x + c * blockDim.x) * 4;
        s[c].x += x[c].x * fo * wo[c].x; s[c].y += x[c].y * fo * wo[c].y; s[c].z += x[c].z * fo * wo[c].z; s[c].w += x[c].w * fo * wo[c].w;
        if (i < hid && !rows) ns_store4(h + t * hid + i, s[c]);
        st += s[c].x * s[c].x + s[c].y * s[c].y + s[c].z * s[c].z + s[c].w * s[c].w;
    }
    st = vm_block_sum(st, red);
    const float fi = 1.0f / sqrtf(st / (float)hid + eps_in);
#pragma unroll
    for (int c = 0; c < RUNS; ++c) {
        const int i = (threadIdx.x + c * blockDim.x) * 4;
        if (i >= hid) continue;
        ns_store4(out + (size_t)blockIdx.x * hid + i, make_float4(s[c].x * fi * wi[c].x, s[c].y * fi * wi[c].y, s[c].z * fi * wi[c].z, s[c].w * fi * wi[c].w));
    }
}

// any width; the row is walked three times (it comes out of L1 again)
template <typename T>
__global__ void norm_sum_norm_kernel(float* __restrict__ h, const T* __restrict__ y, const float* __restrict__ bias, const float* __restrict__ w_out,
                                     float eps_out, const float* __restrict__ w_in, float eps_in, T* __restrict__ out, const int* __restrict__ rows, int hid) {
    __shared__ float red[32];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const size_t t = rows ? rows[blockIdx.x] : blockIdx.x;
    const T* yr = y + t * hid;
    float* hr = h + t * hid;
    float ss = 0.f;
    for (int i = threadIdx.x; i < hid; i += blockDim.x) {
        const float v = vm_to_float(yr[i]) + (bias ? bias[i] : 0.f);
        ss += v * v;
    }
    ss = vm_block_sum(ss, red);
    const float fo = 1.0f / sqrtf(ss / (float)hid + eps_out);
    float st = 0.f;
    for (int i = threadIdx.x; i < hid; i += blockDim.x) {
        const float v = hr[i] + (vm_to_float(yr[i]) + (bias ? bias[i] : 0.f)) * fo * w_out[i];
        st += v * v;
    }
    st = vm_block_sum(st, red);
    const float fi = 1.0f / sqrtf(st / (float)hid + eps_in);
    for (int i = threadIdx.x; i < hid; i += blockDim.x) {
        const float v = hr[i] + (vm_to_float(yr[i]) + (bias ? bias[i] : 0.f)) * fo * w_out[i];
        if (!rows) hr[i] = v;
        out[(size_t)blockIdx.x * hid + i] = vm_from_float<T>(v * fi * w_in[i]);
    }
}

template <typename T>
int launch_norm_sum_norm(float* h, const T* y, const float* bias, const float* w_out, float eps_out, const float* w_in, float eps_in, T* out, const int* rows,
                         int n, int hid, cudaStream_t stream) {
    const uintptr_t at = (uintptr_t)h | (uintptr_t)y | (uintptr_t)bias | (uintptr_t)w_out | (uintptr_t)w_in | (uintptr_t)out;
    if (hid % 4 == 0 && at % 16 == 0 && hid <= 4096) {
        const int threads = hid >= 1024 ? 256 : (hid >= 512 ? 128 : 64);
        const int runs = (hid / 4 + threads - 1) / threads;
#define VM_NSN(R_) \
    vm_launch_pdl(norm_sum_norm_vec_kernel<T, R_>, dim3(n), dim3(threads), 0, stream, h, y, bias, w_out, eps_out, w_in, eps_in, out, rows, hid)
        if (runs <= 1) VM_NSN(1);
        else if (runs <= 2) VM_NSN(2);
        else VM_NSN(4);
#undef VM_NSN
    } else {
        vm_launch_pdl(norm_sum_norm_kernel<T>, dim3(n), dim3(hid >= 512 ? 256 : 128), 0, stream, h, y, bias, w_out, eps_out, w_in, eps_in, out, rows, hid);
    }
    return vm_launch_status();
}

// ------------------------------------------------------------------------------------------------ two sublayers on one input, joined
// h += sa (ca a + ca2 a2) + sb b, value by value: a (and a2) what the mixer left, b the feed-forward's result, sa and sb [hid] float32.
// a2 and b may be null, sa and sb too (1).  copy (activation dtype, may be null) receives the new h.
template <typename T>
__global__ void scaled_sum_vec_kernel(float* __restrict__ h, const T* __restrict__ a, float ca, const T* __restrict__ a2, float ca2, const float* __restrict__ sa,
                                      const T* __restrict__ b, const float* __restrict__ sb, T* __restrict__ copy, long long n4, int hid4) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n4; i += (long long)gridDim.x * blockDim.x) {
        const int col = 4 * (int)(i % hid4);
        float4 v = ns_load4(h + 4 * i), x = ns_load4(a + 4 * i);
        x.x *= ca; x.y *= ca; x.z *= ca; x.w *= ca;
        if (a2) {
            const float4 y = ns_load4(a2 + 4 * i);
            x.x = fmaf(ca2, y.x, x.x); x.y = fmaf(ca2, y.y, x.y); x.z = fmaf(ca2, y.z, x.z); x.w = fmaf(ca2, y.w, x.w);
        }
        const float4 s = sa ? ns_load4(sa + col) : one;
        x.x *= s.x; x.y *= s.y; x.z *= s.z; x.w *= s.w;
        if (b) {
            const float4 y = ns_load4(b + 4 * i), w = sb ? ns_load4(sb + col) : one;
            x.x = fmaf(w.x, y.x, x.x); x.y = fmaf(w.y, y.y, x.y); x.z = fmaf(w.z, y.z, x.z); x.w = fmaf(w.w, y.w, x.w);
        }
        v.x += x.x; v.y += x.y; v.z += x.z; v.w += x.w;
        ns_store4(h + 4 * i, v);
        if (copy) ns_store4(copy + 4 * i, v);
    }
}

template <typename T>
__global__ void scaled_sum_kernel(float* __restrict__ h, const T* __restrict__ a, float ca, const T* __restrict__ a2, float ca2, const float* __restrict__ sa,
                                  const T* __restrict__ b, const float* __restrict__ sb, T* __restrict__ copy, long long n, int hid) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const int col = (int)(i % hid);
        float x = ca * vm_to_float(a[i]);
        if (a2) x = fmaf(ca2, vm_to_float(a2[i]), x);
        if (sa) x *= sa[col];
        if (b) x = fmaf(sb ? sb[col] : 1.f, vm_to_float(b[i]), x);
        const float v = h[i] + x;
        h[i] = v;
        if (copy) copy[i] = vm_from_float<T>(v);
    }
}

template <typename T>
int launch_scaled_sum(float* h, const T* a, float ca, const T* a2, float ca2, const float* sa, const T* b, const float* sb, T* copy, int T_, int hid,
                      cudaStream_t stream) {
    const uintptr_t at = (uintptr_t)h | (uintptr_t)a | (uintptr_t)a2 | (uintptr_t)sa | (uintptr_t)b | (uintptr_t)sb | (uintptr_t)copy;
    const bool vec = hid % 4 == 0 && at % 16 == 0;
    const long long n = (long long)T_ * hid / (vec ? 4 : 1), want = (n + 255) / 256;
    const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16));
    if (vec) vm_launch_pdl(scaled_sum_vec_kernel<T>, grid, dim3(256), 0, stream, h, a, ca, a2, ca2, sa, b, sb, copy, n, hid / 4);
    else vm_launch_pdl(scaled_sum_kernel<T>, grid, dim3(256), 0, stream, h, a, ca, a2, ca2, sa, b, sb, copy, n, hid);
    return vm_launch_status();
}

// ------------------------------------------------------------------------------------------------ a token's own row, gated
// out[t, i] = gelu_tanh(z[t, i]) * table[token_t, off + i]; z float32 [T, ldz], table rows of ld_table values in W.  A token outside the
// table reads its first row (the embedding, which reads the same token, reports it).
__device__ __forceinline__ float gtr_gelu(float v) {      // 0.5 v (1 + tanh(u)) = v sigmoid(2 u)
    return v / (1.0f + expf(-1.5957691216057308f * (v + 0.044715f * v * v * v)));
}

// four neighbouring columns a thread
template <typename W, typename T>
__global__ void gated_token_rows_vec_kernel(const float* __restrict__ z, int ldz, const int* __restrict__ tokens, const W* __restrict__ table, long long ld_table,
                                            int off, int vocab, T* __restrict__ out, int n, int total4) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total4) return;
    const int t = i / (n / 4), c = 4 * (i - t * (n / 4)), id = tokens[t];
    const float4 v = ns_load4(z + (size_t)t * ldz + c), e = ns_load4(table + (size_t)(id >= 0 && id < vocab ? id : 0) * ld_table + off + c);
    ns_store4(out + (size_t)t * n + c, make_float4(gtr_gelu(v.x) * e.x, gtr_gelu(v.y) * e.y, gtr_gelu(v.z) * e.z, gtr_gelu(v.w) * e.w));
}

template <typename W, typename T>
__global__ void gated_token_rows_kernel(const float* __restrict__ z, int ldz, const int* __restrict__ tokens, const W* __restrict__ table, long long ld_table,
                                        int off, int vocab, T* __restrict__ out, int n, long long total) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / n;
        const int c = (int)(i - t * n), id = tokens[t];
        const float v = z[t * ldz + c], e = vm_to_float(table[(size_t)(id >= 0 && id < vocab ? id : 0) * ld_table + off + c]);
        out[i] = vm_from_float<T>(gtr_gelu(v) * e);
    }
}

// ------------------------------------------------------------------------------------------------ polynomial activation with unit-rms powers
// one block per token; z [T, n] in Z (float32 or the activation dtype), out in T
template <typename Z, typename T>
__global__ void polynorm_kernel(const Z* z, const float* __restrict__ coef, T* out, int n, float eps) {      // (z may be out)
    __shared__ float red[32];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t = blockIdx.x;
    const Z* zr = z + (size_t)t * n;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = vm_to_float(zr[i]), v2 = v * v;
        s2 += v2;
        s4 += v2 * v2;
        s6 += v2 * v2 * v2;
    }
    s2 = vm_block_sum(s2, red);
    s4 = vm_block_sum(s4, red);
    s6 = vm_block_sum(s6, red);
    const float a = coef[0] / sqrtf(s2 / (float)n + eps), b = coef[1] / sqrtf(s4 / (float)n + eps), c = coef[2] / sqrtf(s6 / (float)n + eps),
                e = coef[3];
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = vm_to_float(zr[i]);
        out[(size_t)t * n + i] = vm_from_float<T>(fmaf(v, fmaf(v, fmaf(v, c, b), a), e));
    }
}

// The same in bfloat16 with n % 8 == 0: 16-byte loads and stores, the three sums reduced together.  (z may be out.)
__global__ void __launch_bounds__(256) polynorm_vec_kernel(const __nv_bfloat16* z, const float* __restrict__ coef, __nv_bfloat16* out, int n, float eps) {
    __shared__ float red[3][8];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const uint4* zr = reinterpret_cast<const uint4*>(z + (size_t)t * n);
    uint4* orow = reinterpret_cast<uint4*>(out + (size_t)t * n);
    const int n8 = n >> 3;
    float s2 = 0.f, s4 = 0.f, s6 = 0.f;
    for (int i = threadIdx.x; i < n8; i += 256) {
        const uint4 d = zr[i];
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&d);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float a = __low2float(p[k]), b = __high2float(p[k]), a2 = a * a, b2 = b * b;
            s2 += a2 + b2;
            s4 += a2 * a2 + b2 * b2;
            s6 += a2 * a2 * a2 + b2 * b2 * b2;
        }
    }
    s2 = vm_warp_sum(s2); s4 = vm_warp_sum(s4); s6 = vm_warp_sum(s6);
    if (lane == 0) { red[0][warp] = s2; red[1][warp] = s4; red[2][warp] = s6; }
    __syncthreads();
    s2 = s4 = s6 = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) { s2 += red[0][k]; s4 += red[1][k]; s6 += red[2][k]; }
    const float a = coef[0] / sqrtf(s2 / (float)n + eps), b = coef[1] / sqrtf(s4 / (float)n + eps), c = coef[2] / sqrtf(s6 / (float)n + eps),
                e = coef[3];
    for (int i = threadIdx.x; i < n8; i += 256) {
        const uint4 d = zr[i];
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&d);
        uint4 o;
        __nv_bfloat162* q = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            const float u = __low2float(p[k]), v = __high2float(p[k]);
            q[k] = __floats2bfloat162_rn(fmaf(u, fmaf(u, fmaf(u, c, b), a), e), fmaf(v, fmaf(v, fmaf(v, c, b), a), e));
        }
        orow[i] = o;
    }
}

// ------------------------------------------------------------------------------------------------ rotation of a slice of every head
// dst[t, h, dst_off + i] = rotated src[t, h, src_off + i], i < width: the first rotary_dim values turn by the token's position (pairs by
// `pairing`), the rest pass.  One thread per (token, head, pair or passing value).
template <typename T>
__global__ void rotate_slice_kernel(const T* __restrict__ src, long long src_ld, int src_head, int src_off, T* __restrict__ dst, long long dst_ld,
                                    int dst_head, int dst_off, const int* __restrict__ positions, const float* __restrict__ inv_freq, int rotary_dim,
                                    int pairing, int width, int H, int n_tokens) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int half = rotary_dim / 2, per = half + (width - rotary_dim);
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)n_tokens * H * per) return;
    const int i = (int)(idx % per);
    const int hh = (int)((idx / per) % H);
    const int t = (int)(idx / ((long long)per * H));
    const T* s = src + (size_t)t * src_ld + (size_t)hh * src_head + src_off;
    T* d = dst + (size_t)t * dst_ld + (size_t)hh * dst_head + dst_off;
    if (i >= half) {
        const int k = rotary_dim + (i - half);
        d[k] = s[k];
        return;
    }
    const int ia = pairing == VM_PAIR_INTERLEAVED ? 2 * i : i, ib = pairing == VM_PAIR_INTERLEAVED ? 2 * i + 1 : i + half;
    const float ang = (float)positions[t] * inv_freq[i];
    float sn, cs;
    sincosf(ang, &sn, &cs);
    const float u = vm_to_float(s[ia]), v = vm_to_float(s[ib]);
    d[ia] = vm_from_float<T>(u * cs - v * sn);
    d[ib] = vm_from_float<T>(v * cs + u * sn);
}

// ------------------------------------------------------------------------------------------------ x *= sigmoid(gate)
template <typename T>
__global__ void sigmoid_gate_kernel(T* __restrict__ x, const float* __restrict__ gate, long long gate_ld, int cols, long long n) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / cols;
        const int c = (int)(i - t * cols);
        const float g = gate[t * gate_ld + c];
        x[i] = vm_from_float<T>(vm_to_float(x[i]) / (1.0f + expf(-g)));
    }
}

// bfloat16, cols % 4 == 0, gate rows 16-byte aligned: four values per thread
__global__ void __launch_bounds__(256) sigmoid_gate_vec_kernel(__nv_bfloat16* __restrict__ x, const float* __restrict__ gate, long long gate_ld, int cols,
                                                               long long n_vec) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int per = cols >> 2;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n_vec; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / per;
        const int c = (int)(i - t * per) << 2;
        const float4 g = *reinterpret_cast<const float4*>(gate + t * gate_ld + c);
        uint2* px = reinterpret_cast<uint2*>(x + t * cols + c);
        const uint2 d = *px;
        const __nv_bfloat162 d01 = *reinterpret_cast<const __nv_bfloat162*>(&d.x), d23 = *reinterpret_cast<const __nv_bfloat162*>(&d.y);
        const __nv_bfloat162 o01 = __floats2bfloat162_rn(__low2float(d01) / (1.0f + expf(-g.x)), __high2float(d01) / (1.0f + expf(-g.y)));
        const __nv_bfloat162 o23 = __floats2bfloat162_rn(__low2float(d23) / (1.0f + expf(-g.z)), __high2float(d23) / (1.0f + expf(-g.w)));
        uint2 o;
        o.x = *reinterpret_cast<const unsigned*>(&o01); o.y = *reinterpret_cast<const unsigned*>(&o23);
        *px = o;
    }
}

}  // namespace

// h float32 [T, hid]; taps float32 [hid, K]; out [T, hid] in the activation dtype.  The kept inputs of every sequence of the step are moved on
// (after the convolution has read them): h must still hold the step's inputs.  one_token_each: token s is sequence s's only one.
VM_API int vm_input_conv(const float* h, const float* taps, float* state, long long state_stride, int state_offset, const int* positions,
                         const int* seq_of_token, const int* cu_tokens, const int* slots, void* out, int T, int B, int hid, int K, int one_token_each,
                         int act_dtype, cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    if (hid <= 0 || K < 1 || K > 64 || (K > 1 && (!state || state_offset < 0 || state_offset + (long long)(K - 1) * hid > state_stride)))
        return VM_ERR_BAD_ARG;
    if (act_dtype != VM_F32 && act_dtype != VM_BF16) return VM_ERR_UNSUPPORTED;
    const int threads = hid >= 512 ? 256 : 128;
    if (one_token_each) {
        if (T != B) return VM_ERR_BAD_ARG;
        const dim3 grid(B, (hid + threads - 1) / threads);
        if (act_dtype == VM_F32)
            vm_launch_pdl(input_conv_step_kernel<float>, grid, dim3(threads), 0, stream, h, taps, state, state_stride, state_offset, slots, (float*)out, hid, K);
        else
            vm_launch_pdl(input_conv_step_kernel<__nv_bfloat16>, grid, dim3(threads), 0, stream, h, taps, state, state_stride, state_offset, slots,
                          (__nv_bfloat16*)out, hid, K);
        return vm_launch_status();
    }
    const bool aligned = hid % 4 == 0 && state_stride % 4 == 0 && state_offset % 4 == 0 && ((uintptr_t)h | (uintptr_t)taps | (uintptr_t)state) % 16 == 0 &&
                         (uintptr_t)out % 8 == 0;
    if (act_dtype == VM_BF16 && aligned && K >= 2 && K <= 4 && T >= 64) {
        constexpr int RUN = 4;
        const long long n_vec = (long long)((T + RUN - 1) / RUN) * (hid >> 2);
        const dim3 grid((unsigned)((n_vec + 255) / 256));
#define VM_CONV_RUN(KT)                                                                                                                                   \
    vm_launch_pdl(input_conv_run_kernel<KT, RUN>, grid, dim3(256), 0, stream, h, taps, (const float*)state, state_stride, state_offset, seq_of_token, cu_tokens, \
                  slots, (__nv_bfloat16*)out, hid, T, n_vec)
        if (K == 2) VM_CONV_RUN(2);
        else if (K == 3) VM_CONV_RUN(3);
        else VM_CONV_RUN(4);
#undef VM_CONV_RUN
    } else if (act_dtype == VM_BF16 && aligned) {
        const long long n_vec = (long long)T * (hid >> 2);
        const dim3 grid((unsigned)((n_vec + 255) / 256));
#define VM_CONV_VEC(KT)                                                                                                                              \
    vm_launch_pdl(input_conv_vec_kernel<KT>, grid, dim3(256), 0, stream, h, taps, (const float*)state, state_stride, state_offset, seq_of_token, cu_tokens, \
                  slots, (__nv_bfloat16*)out, hid, K, n_vec)
        if (K == 2) VM_CONV_VEC(2);
        else if (K == 3) VM_CONV_VEC(3);
        else if (K == 4) VM_CONV_VEC(4);
        else VM_CONV_VEC(0);
#undef VM_CONV_VEC
    } else if (act_dtype == VM_F32)
        vm_launch_pdl(input_conv_kernel<float>, dim3(T), dim3(threads), 0, stream, h, taps, (const float*)state, state_stride, state_offset, positions,
                      seq_of_token, cu_tokens, slots, (float*)out, hid, K);
    else
        vm_launch_pdl(input_conv_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, h, taps, (const float*)state, state_stride, state_offset,
                      positions, seq_of_token, cu_tokens, slots, (__nv_bfloat16*)out, hid, K);
    int st = vm_launch_status();
    if (st || K == 1) return st;
    vm_launch_pdl(input_conv_keep_kernel, dim3(B, (hid + threads - 1) / threads), dim3(threads), 0, stream, h, state, state_stride, state_offset, cu_tokens,
                  slots, hid, K);
    return vm_launch_status();
}

// h float32 [T, hid] += rmsnorm(y) * w; y [T, ld] float32 (y_dtype VM_F32) or bfloat16
VM_API int vm_norm_residual_add(float* h, const void* y, long long ld, int y_dtype, const float* w, int T, int hid, float eps, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (hid <= 0 || ld < hid) return VM_ERR_BAD_ARG;
    const int threads = hid >= 512 ? 256 : 128;
    const size_t smem = 0;
    if (y_dtype == VM_BF16 && T > 32 && hid % 4 == 0 && ld % 4 == 0 && ((uintptr_t)h | (uintptr_t)w) % 16 == 0 && (uintptr_t)y % 8 == 0) {
        vm_launch_pdl(norm_residual_vec_kernel, dim3((T + NR_WARPS - 1) / NR_WARPS), dim3(NR_WARPS * 32), 0, stream, h, (const __nv_bfloat16*)y, ld, w, T, hid,
                      eps);
        return vm_launch_status();
    }
    if (y_dtype == VM_F32) vm_launch_pdl(norm_residual_kernel<float>, dim3(T), dim3(threads), smem, stream, h, (const float*)y, ld, w, hid, eps);
    else if (y_dtype == VM_BF16)
        vm_launch_pdl(norm_residual_kernel<__nv_bfloat16>, dim3(T), dim3(threads), smem, stream, h, (const __nv_bfloat16*)y, ld, w, hid, eps);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}

// h float32 [T, hid] += rmsnorm(y + bias) * w_out; out [T, hid] = rmsnorm(h) * w_in.  y and out in act_dtype, bias float32 [hid] or null.
// With `rows` (int32 [n]) only those n rows are made, into rows 0 .. n of out, and h is not written.
VM_API int vm_norm_sum_norm(float* h, const void* y, const float* bias, const float* w_out, float eps_out, const float* w_in, float eps_in, void* out,
                            const int* rows, int n, int hid, int act_dtype, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (hid <= 0 || !w_out || !w_in) return VM_ERR_BAD_ARG;
    if (act_dtype == VM_F32) return launch_norm_sum_norm<float>(h, (const float*)y, bias, w_out, eps_out, w_in, eps_in, (float*)out, rows, n, hid, stream);
    if (act_dtype == VM_BF16)
        return launch_norm_sum_norm<__nv_bfloat16>(h, (const __nv_bfloat16*)y, bias, w_out, eps_out, w_in, eps_in, (__nv_bfloat16*)out, rows, n, hid, stream);
    return VM_ERR_UNSUPPORTED;
}

VM_API int vm_scaled_sum(float* h, const void* a, float ca, const void* a2, float ca2, const float* sa, const void* b, const float* sb, void* copy, int T, int hid,
                         int act_dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (hid <= 0 || !a) return VM_ERR_BAD_ARG;
    if (act_dtype == VM_F32)
        return launch_scaled_sum<float>(h, (const float*)a, ca, (const float*)a2, ca2, sa, (const float*)b, sb, (float*)copy, T, hid, stream);
    if (act_dtype == VM_BF16)
        return launch_scaled_sum<__nv_bfloat16>(h, (const __nv_bfloat16*)a, ca, (const __nv_bfloat16*)a2, ca2, sa, (const __nv_bfloat16*)b, sb,
                                                (__nv_bfloat16*)copy, T, hid, stream);
    return VM_ERR_UNSUPPORTED;
}

VM_API int vm_gated_token_rows(const float* z, int ldz, const int* tokens, const void* table, int table_dtype, long long ld_table, int off, int vocab, void* out,
                               int n, int T, int act_dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (n <= 0 || ldz < n || off < 0 || ld_table < off + n || vocab <= 0) return VM_ERR_BAD_ARG;
    const long long total = (long long)T * n, want = (total + 255) / 256;
    const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16));
    const uintptr_t at = (uintptr_t)z | (uintptr_t)table | (uintptr_t)out;
    const bool vec = n % 4 == 0 && ldz % 4 == 0 && ld_table % 4 == 0 && off % 4 == 0 && at % 16 == 0 && total < (1ll << 31);
    const int total4 = (int)(total / 4);
#define VM_GTR(W, T_) \
    if (vec) vm_launch_pdl(gated_token_rows_vec_kernel<W, T_>, dim3((total4 + 127) / 128), dim3(128), 0, stream, z, ldz, tokens, (const W*)table, ld_table, off, \
                           vocab, (T_*)out, n, total4); \
    else vm_launch_pdl(gated_token_rows_kernel<W, T_>, grid, dim3(256), 0, stream, z, ldz, tokens, (const W*)table, ld_table, off, vocab, (T_*)out, n, total)
    if (table_dtype == VM_F32 && act_dtype == VM_F32) { VM_GTR(float, float); }
    else if (table_dtype == VM_F32 && act_dtype == VM_BF16) { VM_GTR(float, __nv_bfloat16); }
    else if (table_dtype == VM_BF16 && act_dtype == VM_BF16) { VM_GTR(__nv_bfloat16, __nv_bfloat16); }
    else return VM_ERR_UNSUPPORTED;
#undef VM_GTR
    return vm_launch_status();
}

// One token per sequence (token s is sequence s's): h += rmsnorm(y) * w, then out = h + conv(h) as vm_input_conv does for such a step,
// the kept inputs at state_offset moved on.  y and out in act_dtype (y_dtype VM_F32: y float32).
VM_API int vm_norm_residual_conv_step(float* h, const void* y, long long ld, int y_dtype, const float* w, int B, int hid, float eps, const float* taps,
                                      float* state, long long state_stride, int state_offset, const int* slots, void* out, int K, int act_dtype,
                                      cudaStream_t stream) {
    if (B <= 0) return 0;
    if (hid <= 0 || ld < hid || K < 1 || K > 64 || (K > 1 && (!state || state_offset < 0 || state_offset + (long long)(K - 1) * hid > state_stride)))
        return VM_ERR_BAD_ARG;
    const int threads = hid >= 512 ? 256 : 128;
    const size_t smem = 0;
    const dim3 grid(B, (hid + threads - 1) / threads);
    if (y_dtype == VM_F32 && act_dtype == VM_F32)
        vm_launch_pdl(norm_residual_conv_step_kernel<float, float>, grid, dim3(threads), smem, stream, h, (const float*)y, ld, w, hid, eps, taps, state,
                      state_stride, state_offset, slots, (float*)out, K);
    else if (y_dtype == VM_F32 && act_dtype == VM_BF16)
        vm_launch_pdl(norm_residual_conv_step_kernel<float, __nv_bfloat16>, grid, dim3(threads), smem, stream, h, (const float*)y, ld, w, hid, eps, taps,
                      state, state_stride, state_offset, slots, (__nv_bfloat16*)out, K);
    else if (y_dtype == VM_BF16 && act_dtype == VM_BF16)
        vm_launch_pdl(norm_residual_conv_step_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(threads), smem, stream, h, (const __nv_bfloat16*)y, ld, w,
                      hid, eps, taps, state, state_stride, state_offset, slots, (__nv_bfloat16*)out, K);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}

// out[t, :] = a N(z) + b N(z^2) + c N(z^3) + e over the n values of a token; coef float32 [4] = a, b, c, e; z in z_dtype, out in act_dtype
VM_API int vm_polynorm(const void* z, int z_dtype, const float* coef, void* out, int T, int n, float eps, int act_dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (n <= 0) return VM_ERR_BAD_ARG;
    const int threads = n >= 1024 ? 512 : (n >= 512 ? 256 : 128);
    if (z_dtype == VM_F32 && act_dtype == VM_F32)
        vm_launch_pdl(polynorm_kernel<float, float>, dim3(T), dim3(threads), 0, stream, (const float*)z, coef, (float*)out, n, eps);
    else if (z_dtype == VM_F32 && act_dtype == VM_BF16)
        vm_launch_pdl(polynorm_kernel<float, __nv_bfloat16>, dim3(T), dim3(threads), 0, stream, (const float*)z, coef, (__nv_bfloat16*)out, n, eps);
    else if (z_dtype == VM_BF16 && act_dtype == VM_BF16 && n % 8 == 0 && ((uintptr_t)z | (uintptr_t)out) % 16 == 0)
        vm_launch_pdl(polynorm_vec_kernel, dim3(T), dim3(256), 0, stream, (const __nv_bfloat16*)z, coef, (__nv_bfloat16*)out, n, eps);
    else if (z_dtype == VM_BF16 && act_dtype == VM_BF16)
        vm_launch_pdl(polynorm_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(T), dim3(threads), 0, stream, (const __nv_bfloat16*)z, coef, (__nv_bfloat16*)out, n,
                      eps);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}

// rows of H heads: src [T, src_ld] with a head every src_head elements, the slice at src_off; dst likewise (src == dst with equal
// layouts: in place).  The slice's first rotary_dim of `width` values are rotated.
VM_API int vm_rotate_slice(const void* src, long long src_ld, int src_head, int src_off, void* dst, long long dst_ld, int dst_head, int dst_off,
                           const int* positions, const float* inv_freq, int rotary_dim, int pairing, int width, int H, int T, int act_dtype,
                           cudaStream_t stream) {
    if (T <= 0 || width <= 0) return 0;
    if (H <= 0 || rotary_dim < 0 || rotary_dim % 2 || rotary_dim > width || (rotary_dim > 0 && !inv_freq)) return VM_ERR_BAD_ARG;
    const long long n = (long long)T * H * (rotary_dim / 2 + width - rotary_dim);
    const int blocks = (int)((n + 255) / 256);
    if (act_dtype == VM_F32)
        vm_launch_pdl(rotate_slice_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)src, src_ld, src_head, src_off, (float*)dst, dst_ld,
                      dst_head, dst_off, positions, inv_freq, rotary_dim, pairing, width, H, T);
    else if (act_dtype == VM_BF16)
        vm_launch_pdl(rotate_slice_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)src, src_ld, src_head, src_off,
                      (__nv_bfloat16*)dst, dst_ld, dst_head, dst_off, positions, inv_freq, rotary_dim, pairing, width, H, T);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}

// x [T, cols] (activation dtype) *= sigmoid(gate [T, gate_ld] float32, its first `cols` columns)
VM_API int vm_sigmoid_gate(void* x, const float* gate, long long gate_ld, int T, int cols, int act_dtype, cudaStream_t stream) {
    if (T <= 0 || cols <= 0) return 0;
    const long long n = (long long)T * cols;
    const long long want = (n + 255) / 256;
    const int blocks = (int)(want < 148 * 16 ? want : 148 * 16);
    if (act_dtype == VM_BF16 && cols % 4 == 0 && gate_ld % 4 == 0 && (uintptr_t)gate % 16 == 0 && (uintptr_t)x % 8 == 0) {
        const long long n_vec = n >> 2, want_vec = (n_vec + 255) / 256;
        vm_launch_pdl(sigmoid_gate_vec_kernel, dim3((unsigned)(want_vec < 148 * 16 ? want_vec : 148 * 16)), dim3(256), 0, stream, (__nv_bfloat16*)x, gate,
                      gate_ld, cols, n_vec);
        return vm_launch_status();
    }
    if (act_dtype == VM_F32) vm_launch_pdl(sigmoid_gate_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)x, gate, gate_ld, cols, n);
    else if (act_dtype == VM_BF16)
        vm_launch_pdl(sigmoid_gate_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (__nv_bfloat16*)x, gate, gate_ld, cols, n);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}
