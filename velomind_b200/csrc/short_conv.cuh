// The short causal convolution over time on every channel, with bias and SiLU, in front of a state-space recurrence; the inputs of a
// sequence's last K - 1 tokens are kept in its state area, float32 [K - 1, C] at conv_off.  Shared by the state-space mixers' files.
#pragma once
#include "common.cuh"

namespace {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// grid (channel tiles, tokens): a thread per (token, channel).  u: columns [u_col, u_col + C) of proj [T, ld].
template <typename T>
__global__ void conv_silu_kernel(const T* __restrict__ proj, int ld, int u_col, const float* __restrict__ taps, const float* __restrict__ bias,
                                 const float* __restrict__ state, int state_floats, int conv_off, const int* __restrict__ positions,
                                 const int* __restrict__ seq_of_token, const int* __restrict__ cu_tokens, const int* __restrict__ slots, int n_tokens,
                                 int C, int K, T* __restrict__ out) {
    const int t = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int seq = seq_of_token[t];
    const int local = t - cu_tokens[seq];                  // place of the token among its sequence's new tokens
    const float* kept = state + (size_t)slots[seq] * state_floats + conv_off;      // [K - 1, C]: inputs of the K - 1 tokens before this step
    float acc = bias ? bias[c] : 0.f;
    for (int k = 0; k < K; ++k) {
        const int back = K - 1 - k;                        // tap k reads the input `back` tokens ago
        float u;
        if (local - back >= 0) u = vm_to_float(proj[(size_t)(t - back) * ld + u_col + c]);
        else u = kept[(size_t)(K - 1 + local - back) * C + c];
        acc = fmaf(taps[(size_t)c * K + k], u, acc);
    }
    out[(size_t)t * C + c] = vm_from_float<T>(silu_f(acc));
}

// Two neighbouring channels a thread (one load of both), CONV_TOK tokens one after another with the K - 1 earlier inputs carried in registers.
// The same sum in the same order as above.
constexpr int CONV_TOK = 8;
__device__ __forceinline__ float2 conv_load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 conv_load2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void conv_store2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void conv_store2(__nv_bfloat16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }

template <typename T, int K>
__global__ void __launch_bounds__(128)
conv_silu_pairs_kernel(const T* __restrict__ proj, int ld, int u_col, const float* __restrict__ taps, const float* __restrict__ bias,
                       const float* __restrict__ state, int state_floats, int conv_off, const int* __restrict__ seq_of_token, const int* __restrict__ cu_tokens,
                       const int* __restrict__ slots, int n_tokens, int C, T* __restrict__ out) {
    const int c = 2 * (blockIdx.x * blockDim.x + threadIdx.x), t0 = blockIdx.y * CONV_TOK;
    if (c >= C) return;
    float2 w[K], u[K];                                     // taps; u[K - 1] the current token's input, u[K - 1 - b] that of b tokens ago
#pragma unroll
    for (int k = 0; k < K; ++k) w[k] = make_float2(taps[(size_t)c * K + k], taps[(size_t)(c + 1) * K + k]);
    const float2 b2 = bias ? make_float2(bias[c], bias[c + 1]) : make_float2(0.f, 0.f);
    const T* base = proj + u_col + c;
    float2 fresh[CONV_TOK];                                // (all loads before the first use)
#pragma unroll
    for (int i = 0; i < CONV_TOK; ++i) fresh[i] = t0 + i < n_tokens ? conv_load2(base + (size_t)(t0 + i) * ld) : make_float2(0.f, 0.f);
    int seq = -1;
#pragma unroll
    for (int i = 0; i < CONV_TOK; ++i) {
        const int t = t0 + i;
        if (t >= n_tokens) break;
        const int sq = seq_of_token[t];
        if (sq != seq) {                                   // the first token here, or another sequence's first one: the inputs before it
            seq = sq;
            const int local = t - cu_tokens[sq];
            const float* kept = state + (size_t)slots[sq] * state_floats + conv_off;
#pragma unroll
            for (int back = 1; back < K; ++back) {
                if (local - back >= 0) u[K - 1 - back] = conv_load2(base + (size_t)(t - back) * ld);
                else u[K - 1 - back] = make_float2(kept[(size_t)(K - 1 + local - back) * C + c], kept[(size_t)(K - 1 + local - back) * C + c + 1]);
            }
        }
        u[K - 1] = fresh[i];
        float2 acc = b2;
#pragma unroll
        for (int k = 0; k < K; ++k) {
            acc.x = fmaf(w[k].x, u[k].x, acc.x);
            acc.y = fmaf(w[k].y, u[k].y, acc.y);
        }
        conv_store2(out + (size_t)t * C + c, make_float2(__fdividef(acc.x, 1.0f + __expf(-acc.x)), __fdividef(acc.y, 1.0f + __expf(-acc.y))));
#pragma unroll
        for (int k = 0; k + 1 < K; ++k) u[k] = u[k + 1];
    }
}

// A block per sequence, a thread per channel: the last K - 1 inputs after this step (older ones move up, new ones come in).
template <typename T>
__global__ void conv_keep_kernel(const T* __restrict__ proj, int ld, int u_col, float* __restrict__ state, int state_floats, int conv_off,
                                 const int* __restrict__ cu_tokens, const int* __restrict__ slots, int C, int K) {
    const int seq = blockIdx.x;
    const int t0 = cu_tokens[seq], n = cu_tokens[seq + 1] - t0;
    if (n <= 0) return;
    float* kept = state + (size_t)slots[seq] * state_floats + conv_off;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        // new row j holds the input at local place n - (K - 1) + j; a negative place is old row j + n
        for (int j = 0; j < K - 1; ++j) {                  // ascending j reads only rows >= j: nothing it still needs is overwritten
            const int local = n - (K - 1) + j;
            kept[(size_t)j * C + c] = local >= 0 ? vm_to_float(proj[(size_t)(t0 + local) * ld + u_col + c]) : kept[(size_t)(j + n) * C + c];
        }
    }
}


// One new token per sequence (token s belongs to sequence s): the convolution and its memory in one pass; a thread per (sequence, channel).
template <typename T>
__global__ void conv_step_kernel(const T* __restrict__ proj, int ld, int u_col, const float* __restrict__ taps, const float* __restrict__ bias,
                                 float* __restrict__ state, int state_floats, int conv_off, const int* __restrict__ slots, int B, int C, int K,
                                 T* __restrict__ out) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (long long)B * C) return;
    const int seq = (int)(i / C), c = (int)(i - (long long)seq * C);
    float* kept = state + (size_t)slots[seq] * state_floats + conv_off;
    const float u = vm_to_float(proj[(size_t)seq * ld + u_col + c]);
    float acc = fmaf(taps[(size_t)c * K + K - 1], u, bias ? bias[c] : 0.f);
    for (int j = 0; j < K - 1; ++j) {
        const float v = kept[(size_t)j * C + c];
        acc = fmaf(taps[(size_t)c * K + j], v, acc);
        if (j > 0) kept[(size_t)(j - 1) * C + c] = v;      // the memory moves up by one token
    }
    if (K > 1) kept[(size_t)(K - 2) * C + c] = u;
    out[(size_t)seq * C + c] = vm_from_float<T>(silu_f(acc));
}

// the convolution of a step: one launch for steps of one token per sequence, else one for the outputs and one for the kept inputs
template <typename T>
int launch_short_conv(const void* proj, int ld, int u_col, const float* taps, const float* bias, float* state, int state_floats, int conv_off,
                      const int* positions, const int* seq_of_token, const int* cu_tokens, const int* slots, int one_token_each, int T_, int B, int C, int K,
                      void* out, cudaStream_t stream) {
    if (one_token_each) {
        const long long n = (long long)T_ * C;
        vm_launch_pdl(conv_step_kernel<T>, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, stream, (const T*)proj, ld, u_col, taps, bias, state, state_floats,
                      conv_off, slots, B, C, K, (T*)out);
    } else {
        if (T_ > 65535) return VM_ERR_UNSUPPORTED;
        const bool pairs = C % 2 == 0 && ld % 2 == 0 && u_col % 2 == 0 && (((uintptr_t)proj | (uintptr_t)out) & (2 * sizeof(T) - 1)) == 0;
#define VM_CONV(K_)                                                                                                                          \
    if (pairs && K == K_)                                                                                                                    \
        conv_silu_pairs_kernel<T, K_><<<dim3((C / 2 + 127) / 128, (T_ + CONV_TOK - 1) / CONV_TOK), 128, 0, stream>>>(                          \
            (const T*)proj, ld, u_col, taps, bias, state, state_floats, conv_off, seq_of_token, cu_tokens, slots, T_, C, (T*)out);
        VM_CONV(2)
        else VM_CONV(3)
        else VM_CONV(4)
#undef VM_CONV
        else conv_silu_kernel<T><<<dim3((C + 255) / 256, T_), 256, 0, stream>>>((const T*)proj, ld, u_col, taps, bias, state, state_floats, conv_off, positions,
                                                                                seq_of_token, cu_tokens, slots, T_, C, K, (T*)out);
        if (K > 1)
            conv_keep_kernel<T><<<dim3(B, (C + 255) / 256), 256, 0, stream>>>((const T*)proj, ld, u_col, state, state_floats, conv_off, cu_tokens, slots, C, K);
    }
    return vm_launch_status();
}

}  // namespace
