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
        conv_silu_kernel<T><<<dim3((C + 255) / 256, T_), 256, 0, stream>>>((const T*)proj, ld, u_col, taps, bias, state, state_floats, conv_off, positions,
                                                                           seq_of_token, cu_tokens, slots, T_, C, K, (T*)out);
        if (K > 1)
            conv_keep_kernel<T><<<dim3(B, (C + 255) / 256), 256, 0, stream>>>((const T*)proj, ld, u_col, state, state_floats, conv_off, cu_tokens, slots, C, K);
    }
    return vm_launch_status();
}

}  // namespace
