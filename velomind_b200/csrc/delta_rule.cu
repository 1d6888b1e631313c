// The gated delta rule: a matrix memory per sequence and head that forgets, corrects what it holds under a key, and is read by a query.
//
//     S <- g_t S ;   u_t = beta_t (v_t - S^T k_t) ;   S <- S + k_t u_t^T ;   o_t = S^T q_t          S [Dk, Dv] float32
//
// H heads of values read G heads of queries and keys (head h: number h / (H / G)).  What enters it, from the layer's projections
// (float32 rows [q: G Dk | k: G Dk | v: H Dv | ...]):
//     every channel of q, k, v passes a causal convolution over time (taps [C, K], the last one weighs the token itself) and SiLU;
//     q and k become unit vectors per head, x / sqrt(sum x^2 + 1e-6), and q is multiplied by q_scale;
//     beta = sigmoid(b),  log g = -exp(A_log) softplus(a + dt_bias)         one number per token and head, b and a being projected too.
// Everything here is float32 (sums of log decays float64).
//
// A sequence keeps S [H, Dk, Dv] and the K - 1 last projected rows of C = 2 G Dk + H Dv channels.  The kept rows are there twice: a step
// that starts at place p reads copy p & 1, and the copy of the place it leaves off at is written, so that in a step of one token no block
// overwrites what another still reads.
//
// Three ways to run it:
//   a step of one token per sequence: ONE kernel from the projections to the gated, normed heads (delta_step_kernel);
//   small pieces and odd sizes: the preparation, then token by token with the memory in registers (delta_scan_kernel);
//   prompts: the preparation, then 64 tokens at a time (below).
#include <cstdint>

#include "common.cuh"

namespace {

constexpr float UNIT_EPS = 1e-6f;

__device__ __forceinline__ float dr_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float dr_softplus(float x) { return x > 0.f ? x + log1pf(expf(-x)) : log1pf(expf(x)); }

// the convolution of channel c at token t (`in_step` tokens of its sequence lie before it in this step); kept: the step's copy of the kept rows
__device__ __forceinline__ float dr_conv(const float* __restrict__ proj, int ld, const float* __restrict__ taps, int K, const float* kept, int C, size_t t,
                                         int in_step, int c) {
    float v = 0.f;
    for (int j = 0; j < K; ++j) {
        const int back = K - 1 - j;
        const float u = back <= in_step ? proj[(t - back) * ld + c] : kept[(size_t)(K - 1 - back + in_step) * C + c];
        v = fmaf(taps[(size_t)c * K + j], u, v);
    }
    return v;
}

// ------------------------------------------------------------------------------------------------ preparation
// grid (ceil(T / PT), 2 G + H + 1): a block makes one head of q, k or v of PT neighbouring tokens; the last one their beta and log g.
// rows float32 [T, C]: q | k | v as the recurrence reads them; gates float32 [T, 2 H]: beta, then log g.
constexpr int PT = 8, PREP_THREADS = 256;

__global__ void __launch_bounds__(PREP_THREADS)
delta_prepare_kernel(const float* __restrict__ proj, int ld, int b_off, int a_off, const float* __restrict__ taps, int K, const float* __restrict__ state,
                     long long state_stride, int kept_offset, const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                     const int* __restrict__ cu_tokens, const int* __restrict__ slots, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                     float q_scale, float* __restrict__ rows, float* __restrict__ gates, int T, int H, int G, int Dk, int Dv) {
    extern __shared__ float vals[];          // [PT][Dk]
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t0 = blockIdx.x * PT, unit = blockIdx.y, C = 2 * G * Dk + H * Dv;
    if (unit == 2 * G + H) {
        for (int i = threadIdx.x; i < PT * H; i += blockDim.x) {
            const int t = t0 + i / H, h = i % H;
            if (t >= T) break;
            const float b = proj[(size_t)t * ld + b_off + h], a = proj[(size_t)t * ld + a_off + h];
            gates[(size_t)t * 2 * H + h] = 1.0f / (1.0f + expf(-b));
            gates[(size_t)t * 2 * H + H + h] = -expf(A_log[h]) * dr_softplus(a + dt_bias[h]);
        }
        return;
    }
    const bool is_qk = unit < 2 * G;
    const int D = is_qk ? Dk : Dv, col = is_qk ? unit * Dk : 2 * G * Dk + (unit - 2 * G) * Dv;
    for (int i = threadIdx.x; i < PT * D; i += blockDim.x) {
        const int tt = i / D, c = col + (i - tt * D), t = t0 + tt;
        if (t >= T) break;
        const int seq = seq_of_token[t], in_step = t - cu_tokens[seq];
        const float* kept = state + (size_t)slots[seq] * state_stride + kept_offset + (size_t)((positions[t] - in_step) & 1) * (K - 1) * C;
        const float v = dr_silu(dr_conv(proj, ld, taps, K, kept, C, t, in_step, c));
        if (is_qk) vals[i] = v;
        else rows[(size_t)t * C + c] = v;
    }
    if (!is_qk) return;
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float scale = unit < G ? q_scale : 1.0f;
    for (int tt = warp; tt < PT && t0 + tt < T; tt += PREP_THREADS / 32) {
        float ss = 0.f;
        for (int i = lane; i < D; i += 32) ss += vals[tt * D + i] * vals[tt * D + i];
        ss = vm_warp_sum(ss);
        const float f = scale / sqrtf(ss + UNIT_EPS);
        for (int i = lane; i < D; i += 32) rows[(size_t)(t0 + tt) * C + col + i] = vals[tt * D + i] * f;
    }
}

// The same for heads of a multiple of four values and up to four taps: a warp makes one head of RUN neighbouring tokens, a lane four (or NQ
// times four) neighbouring channels, with the K - 1 rows before the token carried along in registers, so that every row is loaded once and a
// halo of K - 1 rows per run.  Warps of neighbouring heads lie side by side: they read neighbouring parts of the same rows.
constexpr int RUN = 8;
__device__ __forceinline__ float4 dr_fma4(float4 a, float4 b, float4 c) { return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w)); }

template <int K, int NQ>
__global__ void __launch_bounds__(PREP_THREADS)
delta_prepare_run_kernel(const float* __restrict__ proj, int ld, int b_off, int a_off, const float* __restrict__ taps, const float* __restrict__ state,
                         long long state_stride, int kept_offset, const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                         const int* __restrict__ cu_tokens, const int* __restrict__ slots, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                         float q_scale, float* __restrict__ rows, float* __restrict__ gates, int T, int H, int G, int Dk, int Dv) {
    vm_pdl_launch_dependents();
    const int units = 2 * G + H + 1, C = 2 * G * Dk + H * Dv, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * (PREP_THREADS / 32) + (threadIdx.x >> 5);
    const int run = (int)(item / units), unit = (int)(item - (long long)run * units), t0 = run * RUN;
    if (t0 >= T) return;
    if (unit == 2 * G + H) {                              // beta and log g of the run's tokens
        vm_pdl_wait();
        for (int i = lane; i < RUN * H; i += 32) {
            const int t = t0 + i / H, h = i % H;
            if (t >= T) break;
            const float b = proj[(size_t)t * ld + b_off + h], a = proj[(size_t)t * ld + a_off + h];
            gates[(size_t)t * 2 * H + h] = 1.0f / (1.0f + expf(-b));
            gates[(size_t)t * 2 * H + H + h] = -expf(A_log[h]) * dr_softplus(a + dt_bias[h]);
        }
        return;
    }
    const bool is_qk = unit < 2 * G;
    const int D = is_qk ? Dk : Dv, col = is_qk ? unit * Dk : 2 * G * Dk + (unit - 2 * G) * Dv;
    float4 w[NQ][K];                                      // w[.][j]: tap j of the lane's four channels
#pragma unroll
    for (int n = 0; n < NQ; ++n) {
        const int c = 4 * (lane + 32 * n);
        const float* tp = taps + (size_t)(col + (c < D ? c : 0)) * K;
#pragma unroll
        for (int j = 0; j < K; ++j) w[n][j] = make_float4(tp[j], tp[K + j], tp[2 * K + j], tp[3 * K + j]);
    }
    vm_pdl_wait();
    const float scale = unit < G ? q_scale : 1.0f;
    float4 win[NQ][K > 1 ? K - 1 : 1];                    // win[.][j]: the projected row K - 1 - j places back
    int seq_before = -1;
    for (int t = t0; t < min(t0 + RUN, T); ++t) {
        const int seq = seq_of_token[t];
        if (K > 1 && seq != seq_before) {
            const int in_step = t - cu_tokens[seq];
            const float* kept = state + (size_t)slots[seq] * state_stride + kept_offset + (size_t)((positions[t] - in_step) & 1) * (K - 1) * C;
#pragma unroll
            for (int n = 0; n < NQ; ++n) {
                const int c = 4 * (lane + 32 * n);
#pragma unroll
                for (int j = 0; j < K - 1; ++j) {
                    const int back = K - 1 - j;
                    const float* src = back <= in_step ? proj + (size_t)(t - back) * ld : kept + (size_t)(K - 1 - back + in_step) * C;
                    win[n][j] = c < D ? *reinterpret_cast<const float4*>(src + col + c) : make_float4(0.f, 0.f, 0.f, 0.f);
                }
            }
            seq_before = seq;
        }
        float4 y[NQ];
        float ss = 0.f;
#pragma unroll
        for (int n = 0; n < NQ; ++n) {
            const int c = 4 * (lane + 32 * n);
            const float4 x = c < D ? *reinterpret_cast<const float4*>(proj + (size_t)t * ld + col + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int j = 0; j < K - 1; ++j) v = dr_fma4(w[n][j], win[n][j], v);
            v = dr_fma4(w[n][K - 1], x, v);
#pragma unroll
            for (int j = 0; j + 1 < K - 1; ++j) win[n][j] = win[n][j + 1];
            if (K > 1) win[n][K > 1 ? K - 2 : 0] = x;
            y[n] = make_float4(dr_silu(v.x), dr_silu(v.y), dr_silu(v.z), dr_silu(v.w));
            if (c < D) ss += y[n].x * y[n].x + y[n].y * y[n].y + y[n].z * y[n].z + y[n].w * y[n].w;
        }
        float f = 1.0f;
        if (is_qk) f = scale / sqrtf(vm_warp_sum(ss) + UNIT_EPS);
#pragma unroll
        for (int n = 0; n < NQ; ++n) {
            const int c = 4 * (lane + 32 * n);
            if (c < D) *reinterpret_cast<float4*>(rows + (size_t)t * C + col + c) = make_float4(y[n].x * f, y[n].y * f, y[n].z * f, y[n].w * f);
        }
    }
}

// grid (B, slices of the channels): the kept rows of a sequence move on by the step's tokens, from the copy of its first place to the copy
// of the place behind its last token (they may be the same one: a thread owns its channel and reads before it writes)
constexpr int MAX_TAPS = 16;
__global__ void delta_keep_rows_kernel(const float* __restrict__ proj, int ld, int C, int K, float* __restrict__ state, long long state_stride, int kept_offset,
                                       const int* __restrict__ positions, const int* __restrict__ cu_tokens, const int* __restrict__ slots) {
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int seq = blockIdx.x, first = cu_tokens[seq], n = cu_tokens[seq + 1] - first;
    if (n <= 0) return;
    const int p0 = positions[first];
    float* base = state + (size_t)slots[seq] * state_stride + kept_offset;
    const float* from = base + (size_t)(p0 & 1) * (K - 1) * C;
    float* to = base + (size_t)((p0 + n) & 1) * (K - 1) * C;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        float nw[MAX_TAPS];
        for (int j = 0; j < K - 1; ++j) {
            const int d = K - 1 - j;                      // row j holds the token d places before the next step
            nw[j] = d <= n ? proj[(size_t)(first + n - d) * ld + c] : from[(size_t)(j + n) * C + c];
        }
        for (int j = 0; j < K - 1; ++j) to[(size_t)j * C + c] = nw[j];
    }
}

// ------------------------------------------------------------------------------------------------ token by token
// grid (sequences, heads, slices of 32 value columns): warp w holds the memory's rows w NR .. w NR + NR, a lane a column.  With the memory
// S before the token, S^T k and S^T q are summed together: u = beta (v - g S^T k) and o = g S^T q + (q . k) u.
constexpr int SCAN_WARPS = 8, SCAN_COLS = 32;

template <int NR>
__global__ void __launch_bounds__(SCAN_WARPS * 32)
delta_scan_kernel(const float* __restrict__ rows, const float* __restrict__ gates, float* __restrict__ state, long long state_stride, int state_offset,
                  const int* __restrict__ cu_tokens, const int* __restrict__ slots, float* __restrict__ o, int H, int G, int Dk, int Dv) {
    extern __shared__ float sm[];            // q [Dk], k [Dk], parts of S^T k and of S^T q [warps, columns] each, parts of q . k [warps]
    float* qs = sm;
    float* ks = qs + Dk;
    float* part_k = ks + Dk;
    float* part_q = part_k + SCAN_WARPS * SCAN_COLS;
    float* part_qk = part_q + SCAN_WARPS * SCAN_COLS;
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, g = h / (H / G), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int col = blockIdx.z * SCAN_COLS + lane, C = 2 * G * Dk + H * Dv;
    const int first = cu_tokens[seq], n = cu_tokens[seq + 1] - first;
    if (n <= 0) return;
    const bool live = col < Dv;
    float* S = state + (size_t)slots[seq] * state_stride + state_offset + (size_t)h * Dk * Dv;
    float s[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) {
        const int i = warp * NR + r;
        s[r] = (live && i < Dk) ? S[(size_t)i * Dv + col] : 0.f;
    }
    for (int i0 = 0; i0 < n; ++i0) {
        const size_t t = (size_t)first + i0;
        const float* row = rows + t * C;
        __syncthreads();                     // the token before is done with q, k and the parts
        for (int i = threadIdx.x; i < Dk; i += blockDim.x) {
            qs[i] = row[(size_t)g * Dk + i];
            ks[i] = row[(size_t)(G + g) * Dk + i];
        }
        __syncthreads();
        float ak = 0.f, aq = 0.f, qk = 0.f;
#pragma unroll
        for (int r = 0; r < NR; ++r) {
            const int i = warp * NR + r;
            if (i < Dk) {
                ak = fmaf(s[r], ks[i], ak);
                aq = fmaf(s[r], qs[i], aq);
                qk = fmaf(qs[i], ks[i], qk);
            }
        }
        part_k[warp * SCAN_COLS + lane] = ak;
        part_q[warp * SCAN_COLS + lane] = aq;
        if (lane == 0) part_qk[warp] = qk;
        __syncthreads();
        ak = aq = qk = 0.f;
#pragma unroll
        for (int w = 0; w < SCAN_WARPS; ++w) {
            ak += part_k[w * SCAN_COLS + lane];
            aq += part_q[w * SCAN_COLS + lane];
            qk += part_qk[w];
        }
        const float beta = gates[t * 2 * H + h], keep = expf(gates[t * 2 * H + H + h]);
        const float v = live ? row[(size_t)2 * G * Dk + (size_t)h * Dv + col] : 0.f;
        const float u = beta * (v - keep * ak);
#pragma unroll
        for (int r = 0; r < NR; ++r) {
            const int i = warp * NR + r;
            if (i < Dk) s[r] = fmaf(ks[i], u, keep * s[r]);
        }
        if (warp == 0 && live) o[t * ((size_t)H * Dv) + (size_t)h * Dv + col] = fmaf(qk, u, keep * aq);
    }
#pragma unroll
    for (int r = 0; r < NR; ++r) {
        const int i = warp * NR + r;
        if (live && i < Dk) S[(size_t)i * Dv + col] = s[r];
    }
}

// ------------------------------------------------------------------------------------------------ one token per sequence
// grid (sequences, heads): convolution, unit vectors, gates, the memory's step, the head's norm and its SiLU gate.  The memory is read and
// written once, four neighbouring columns of a row per thread; thread (row group, column quad) owns rows rg, rg + RG, ...
constexpr int STEP_THREADS = 512;

template <typename T, int NR>
__global__ void __launch_bounds__(STEP_THREADS)
delta_step_kernel(const float* __restrict__ proj, int ld, int g_off, int b_off, int a_off, const float* __restrict__ taps, int K, float* __restrict__ state,
                  long long state_stride, int state_offset, int kept_offset, const int* __restrict__ positions, const int* __restrict__ slots,
                  const float* __restrict__ A_log, const float* __restrict__ dt_bias, const float* __restrict__ norm_w, float eps, float q_scale,
                  T* __restrict__ out, int H, int G, int Dk, int Dv) {
    extern __shared__ __align__(16) float sm[];          // q [Dk], k [Dk], v [Dv], u [Dv], parts [2][RG][Dv]
    __shared__ float red[32], scal[5];                   // 1 / |q| (times q_scale), 1 / |k|, q . k of the raw rows, beta, g
    float* qs = sm;
    float* ks = qs + Dk;
    float* vs = ks + Dk;
    float* us = vs + Dv;
    float* part = us + Dv;
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, per = H / G, g = h / per, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int Q = Dv >> 2, RG = STEP_THREADS / Q, quad = tid % Q, rg = tid / Q, C = 2 * G * Dk + H * Dv;
    float* mine = state + (size_t)slots[seq] * state_stride;
    float* S = mine + state_offset + (size_t)h * Dk * Dv;
    float4 s[NR];
    const bool owner = rg < RG;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int r = rg + i * RG;
        s[i] = owner && r < Dk ? *reinterpret_cast<const float4*>(S + (size_t)r * Dv + 4 * quad) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int pos = positions[seq];
    const float* kept = mine + kept_offset + (size_t)(pos & 1) * (K - 1) * C;
    float* next = mine + kept_offset + (size_t)((pos + 1) & 1) * (K - 1) * C;
    for (int i = tid; i < 2 * Dk + Dv; i += STEP_THREADS) {
        const bool is_v = i >= 2 * Dk;
        const int c = is_v ? 2 * G * Dk + h * Dv + (i - 2 * Dk) : (i < Dk ? g * Dk + i : (G + g) * Dk + (i - Dk));
        const float x = proj[(size_t)seq * ld + c];
        const float* w = taps + (size_t)c * K;
        const bool moves = is_v || h % per == 0;         // the first head of a group moves its shared query and key rows on
        float v = 0.f;
        for (int j = 0; j < K - 1; ++j) {
            const float u = kept[(size_t)j * C + c];
            v = fmaf(w[j], u, v);
            if (moves && j > 0) next[(size_t)(j - 1) * C + c] = u;
        }
        if (moves && K > 1) next[(size_t)(K - 2) * C + c] = x;
        qs[i] = dr_silu(fmaf(w[K - 1], x, v));           // (q, k and v lie one behind the other)
    }
    __syncthreads();
    if (warp < 3) {                                      // warp 0: |q|^2, warp 1: |k|^2, warp 2: q . k
        const float* a = warp == 1 ? ks : qs;
        const float* b = warp == 0 ? qs : ks;
        float v = 0.f;
        for (int i = lane; i < Dk; i += 32) v = fmaf(a[i], b[i], v);
        v = vm_warp_sum(v);
        if (lane == 0) scal[warp] = warp == 2 ? v : (warp == 0 ? q_scale : 1.0f) / sqrtf(v + UNIT_EPS);
    } else if (warp == 3 && lane == 0) {
        const float* row = proj + (size_t)seq * ld;
        scal[3] = 1.0f / (1.0f + expf(-row[b_off + h]));
        scal[4] = expf(-expf(A_log[h]) * dr_softplus(row[a_off + h] + dt_bias[h]));
    }
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int r = rg + i * RG;
        if (owner && r < Dk) {
            const float k = ks[r], q = qs[r];
            ak.x = fmaf(s[i].x, k, ak.x); ak.y = fmaf(s[i].y, k, ak.y); ak.z = fmaf(s[i].z, k, ak.z); ak.w = fmaf(s[i].w, k, ak.w);
            aq.x = fmaf(s[i].x, q, aq.x); aq.y = fmaf(s[i].y, q, aq.y); aq.z = fmaf(s[i].z, q, aq.z); aq.w = fmaf(s[i].w, q, aq.w);
        }
    }
    if (owner) {
        *reinterpret_cast<float4*>(part + (size_t)rg * Dv + 4 * quad) = ak;
        *reinterpret_cast<float4*>(part + (size_t)(RG + rg) * Dv + 4 * quad) = aq;
    }
    __syncthreads();
    const float fq = scal[0], fk = scal[1], qk = scal[2] * scal[0] * scal[1], beta = scal[3], keep = scal[4];
    float o = 0.f;
    if (tid < Dv) {
        float sk = 0.f, sq = 0.f;
        for (int r = 0; r < RG; ++r) {
            sk += part[(size_t)r * Dv + tid];
            sq += part[(size_t)(RG + r) * Dv + tid];
        }
        const float u = beta * (vs[tid] - keep * sk * fk);
        us[tid] = u;
        o = fmaf(qk, u, keep * sq * fq);
    }
    const float ss = vm_block_sum(o * o, red);           // (its barriers also make u visible)
    if (tid < Dv) {
        const float gate = proj[(size_t)seq * ld + g_off + (size_t)h * Dv + tid];
        out[((size_t)seq * H + h) * Dv + tid] = vm_from_float<T>(o / sqrtf(ss / (float)Dv + eps) * norm_w[tid] * dr_silu(gate));
    }
    if (!owner) return;
    const float4 u = *reinterpret_cast<const float4*>(us + 4 * quad);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int r = rg + i * RG;
        if (r < Dk) {
            const float k = ks[r] * fk;
            float4 x = s[i];
            x.x = fmaf(k, u.x, keep * x.x); x.y = fmaf(k, u.y, keep * x.y); x.z = fmaf(k, u.z, keep * x.z); x.w = fmaf(k, u.w, keep * x.w);
            *reinterpret_cast<float4*>(S + (size_t)r * Dv + 4 * quad) = x;
        }
    }
}

// ------------------------------------------------------------------------------------------------ prompts, 64 tokens at a time
// Inside a chunk let b_t be the running sum of log g.  The corrections u solve a unit lower triangular system,
//     (I + A) u = beta v - (beta exp(b) k) S_start,     A[t][s] = beta_t exp(b_t - b_s) (k_t . k_s)  for s < t
// so with W = (I + A)^-1 (beta exp(b) k) and U = (I + A)^-1 (beta v), both free of S_start,
//     u = U - W S_start
//     S_end = exp(b_last) S_start + sum_t (exp(b_last - b_t) k_t) u_t^T
//     o_t   = exp(b_t) S_start^T q_t + sum_(s <= t) exp(b_t - b_s) (q_t . k_s) u_s
// and every exponent is <= 0.  Three passes: `local` makes W and U of all chunks of all sequences and heads at once (forward
// substitution, a column per thread, in registers); `carry` walks each sequence's chunks (a block per 16 columns of the memory), leaves
// every chunk's S_start and turns U into u; `finish`, parallel again, makes the outputs.
constexpr int CH = 64, CP = CH + 4, CTHREADS = 256, CCOLS = 16;

// floats of scratch per chunk and head: W^T [Dk, 64], u [64, Dv], S_start [Dk, Dv], exp(b_t) [64], exp(b_last - b_t) [64]
__host__ __device__ inline long long dr_chunk_floats(int Dk, int Dv) { return (long long)Dk * CH + (long long)CH * Dv + (long long)Dk * Dv + 2 * CH; }

__device__ __forceinline__ bool dr_chunk_of(int chunk, const int* __restrict__ cu_tokens, int B, int& start, int& len) {
    int before = 0;
    for (int b = 0; b < B; ++b) {
        const int n = cu_tokens[b + 1] - cu_tokens[b], nc = (n + CH - 1) / CH;
        if (chunk < before + nc) {
            const int c = chunk - before;
            start = cu_tokens[b] + c * CH;
            len = min(CH, n - c * CH);
            return true;
        }
        before += nc;
    }
    return false;
}

// rows of one head, channel-major: xT[i][t] = rows[start + t][col + i], zeros from `len` on.  Groups of eight tokens by four 16-byte runs
// of channels per warp: whole sectors from memory, few bank conflicts on the way into shared memory.
__device__ __forceinline__ void dr_load_T(const float* __restrict__ rows, int C, int col, int start, int len, int Dk, float* xT) {
    const int runs = (Dk / 4 + 3) / 4;                   // groups of four 16-byte runs
    for (int idx = threadIdx.x; idx < CH * 4 * runs; idx += CTHREADS) {
        const int t = (idx & 7) + 8 * ((idx >> 5) & 7), i = (((idx >> 3) & 3) + 4 * (idx >> 8)) * 4;
        if (i >= Dk) continue;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (t < len) v = *reinterpret_cast<const float4*>(rows + (size_t)(start + t) * C + col + i);
        xT[(i + 0) * CP + t] = v.x; xT[(i + 1) * CP + t] = v.y; xT[(i + 2) * CP + t] = v.z; xT[(i + 3) * CP + t] = v.w;
    }
}

// running sums of the chunk's log decays, float64 (warp 0 only; the caller synchronises)
__device__ __forceinline__ void dr_running_sums(const float* __restrict__ gates, int start, int len, int h, int H, double* b) {
    if (threadIdx.x >= 32) return;
    const int lane = threadIdx.x;
    const double x0 = 2 * lane < len ? (double)gates[(size_t)(start + 2 * lane) * 2 * H + H + h] : 0.0;
    const double x1 = 2 * lane + 1 < len ? (double)gates[(size_t)(start + 2 * lane + 1) * 2 * H + H + h] : 0.0;
    double run = x0 + x1;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
        const double y = __shfl_up_sync(0xffffffffu, run, d);
        if (lane >= d) run += y;
    }
    b[2 * lane] = run - x1;
    b[2 * lane + 1] = run;
}

// part[half][s * 64 + t] = sum over half of the channels of a_t[i] c_s[i], tiles of 8 tokens t by 4 tokens s that reach the diagonal or below
__device__ __forceinline__ void dr_tri_products(const float* aT, const float* cT, int Dk, float* part) {
    const int item = threadIdx.x;
    if (item >= 144) return;
    const int half = item / 72, r = item % 72;
    int tt = 0;
    while ((tt + 1) * (tt + 2) <= r) ++tt;               // row tile tt has 2 tt + 2 column tiles
    const int t0 = 8 * tt, s0 = 4 * (r - tt * (tt + 1));
    const int i_end = half ? Dk : Dk / 2;
    float acc[4][8] = {};
    for (int i = half ? Dk / 2 : 0; i < i_end; ++i) {
        const float4 a0 = *reinterpret_cast<const float4*>(aT + i * CP + t0), a1 = *reinterpret_cast<const float4*>(aT + i * CP + t0 + 4);
        const float4 c4 = *reinterpret_cast<const float4*>(cT + i * CP + s0);
        const float a[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w}, c[4] = {c4.x, c4.y, c4.z, c4.w};
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 8; ++y) acc[x][y] = fmaf(c[x], a[y], acc[x][y]);
    }
    float* p = part + half * CH * CH;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        *reinterpret_cast<float4*>(p + (s0 + x) * CH + t0) = make_float4(acc[x][0], acc[x][1], acc[x][2], acc[x][3]);
        *reinterpret_cast<float4*>(p + (s0 + x) * CH + t0 + 4) = make_float4(acc[x][4], acc[x][5], acc[x][6], acc[x][7]);
    }
}

// grid (chunks, heads)
__global__ void __launch_bounds__(CTHREADS, 2)
delta_local_kernel(const float* __restrict__ rows, const float* __restrict__ gates, const int* __restrict__ cu_tokens, int B, float* __restrict__ scratch, int H,
                   int G, int Dk, int Dv) {
    extern __shared__ __align__(16) float sm[];
    float* kT = sm;                          // [Dk][CP]
    float* part = kT + (size_t)Dk * CP;      // [2][64][64]; then A, transposed, in the first half
    __shared__ double b[CH];
    __shared__ float beta[CH], beta_eb[CH];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    int start, len;
    if (!dr_chunk_of(blockIdx.x, cu_tokens, B, start, len)) return;
    const int h = blockIdx.y, g = h / (H / G), tid = threadIdx.x, C = 2 * G * Dk + H * Dv;
    dr_load_T(rows, C, (G + g) * Dk, start, len, Dk, kT);
    dr_running_sums(gates, start, len, h, H, b);
    if (tid >= 64 && tid < 128) beta[tid - 64] = tid - 64 < len ? gates[(size_t)(start + tid - 64) * 2 * H + h] : 0.f;
    __syncthreads();
    dr_tri_products(kT, kT, Dk, part);
    __syncthreads();
    for (int idx = tid; idx < CH * CH; idx += CTHREADS) {
        const int s = idx / CH, t = idx % CH;
        part[idx] = t > s ? beta[t] * expf((float)(b[t] - b[s])) * (part[idx] + part[CH * CH + idx]) : 0.f;
    }
    float* W = scratch + ((size_t)blockIdx.x * H + h) * dr_chunk_floats(Dk, Dv);
    float* U = W + (size_t)Dk * CH;
    float* eb = U + (size_t)CH * Dv + (size_t)Dk * Dv;
    if (tid < CH) {
        const float e = expf((float)b[tid]);
        beta_eb[tid] = beta[tid] * e;
        eb[tid] = e;
        eb[CH + tid] = tid < len ? expf((float)(b[len - 1] - b[tid])) : 0.f;
    }
    __syncthreads();
    for (int col = tid; col < Dk + Dv; col += CTHREADS) {
        float x[CH];
        if (col < Dk) {
#pragma unroll
            for (int t = 0; t < CH; t += 4) {
                const float4 k = *reinterpret_cast<const float4*>(kT + col * CP + t);
                x[t] = beta_eb[t] * k.x;
                x[t + 1] = beta_eb[t + 1] * k.y;
                x[t + 2] = beta_eb[t + 2] * k.z;
                x[t + 3] = beta_eb[t + 3] * k.w;
            }
        } else {
            const float* v = rows + (size_t)start * C + 2 * G * Dk + (size_t)h * Dv + (col - Dk);
#pragma unroll
            for (int t = 0; t < CH; ++t) x[t] = t < len ? beta[t] * v[(size_t)t * C] : 0.f;
        }
        // forward substitution: as soon as x_s is known it leaves every later row
#pragma unroll
        for (int s = 0; s < CH - 1; ++s) {
#pragma unroll
            for (int t = (s + 1) / 4 * 4; t < CH; t += 4) {
                const float4 a = *reinterpret_cast<const float4*>(part + s * CH + t);
                if (t > s) x[t] = fmaf(-a.x, x[s], x[t]);
                if (t + 1 > s) x[t + 1] = fmaf(-a.y, x[s], x[t + 1]);
                if (t + 2 > s) x[t + 2] = fmaf(-a.z, x[s], x[t + 2]);
                x[t + 3] = fmaf(-a.w, x[s], x[t + 3]);
            }
        }
        if (col < Dk) {
#pragma unroll
            for (int t = 0; t < CH; t += 4) *reinterpret_cast<float4*>(W + (size_t)col * CH + t) = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
        } else {
#pragma unroll
            for (int t = 0; t < CH; ++t) U[(size_t)t * Dv + (col - Dk)] = x[t];
        }
    }
}

__device__ __forceinline__ void dr_copy16(float* smem, const float* gmem, bool pred) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = pred ? 16 : 0;                       // 0 source bytes: the destination is zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(bytes));
}

// grid (sequences, heads, slices of 16 value columns).  STAGES: chunks whose W and keys are in flight or in use at once.
template <int STAGES>
__global__ void __launch_bounds__(CTHREADS)
delta_carry_kernel(const float* __restrict__ rows, float* __restrict__ state, long long state_stride, int state_offset, const int* __restrict__ cu_tokens,
                   const int* __restrict__ slots, float* __restrict__ scratch, int H, int G, int Dk, int Dv) {
    extern __shared__ __align__(16) float sm[];
    float* Ws = sm;                                        // [STAGES][Dk][64]
    float* Ks = Ws + (size_t)STAGES * Dk * CH;             // [STAGES][64][Dk]
    float* Ss = Ks + (size_t)STAGES * Dk * CH;             // [Dk][16]
    float* ud = Ss + (size_t)Dk * CCOLS;                   // [64][16]: u_t exp(b_last - b_t)
    float* part = ud + CH * CCOLS;                         // [4][64][16]
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int seq = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * CCOLS, g = h / (H / G), tid = threadIdx.x, C = 2 * G * Dk + H * Dv;
    int first = 0;
    for (int b = 0; b < seq; ++b) first += (cu_tokens[b + 1] - cu_tokens[b] + CH - 1) / CH;
    const int t_first = cu_tokens[seq], n = cu_tokens[seq + 1] - t_first, nc = (n + CH - 1) / CH;
    if (nc <= 0) return;
    const size_t chunk_floats = (size_t)dr_chunk_floats(Dk, Dv);
    auto chunk = [&](int c) { return scratch + ((size_t)(first + c) * H + h) * chunk_floats; };
    auto load = [&](int c, int stage) {
        const float* W = chunk(c);
        float* w = Ws + (size_t)stage * Dk * CH;
        float* k = Ks + (size_t)stage * Dk * CH;
        const int start = t_first + c * CH, len = min(CH, n - c * CH), per = Dk / 4;
        for (int i = tid; i < Dk * CH / 4; i += CTHREADS) dr_copy16(w + 4 * i, W + 4 * i, true);
        for (int i = tid; i < CH * per; i += CTHREADS) {
            const int t = i / per, x = (i - t * per) * 4;
            dr_copy16(k + t * Dk + x, rows + (size_t)(start + (t < len ? t : 0)) * C + (size_t)(G + g) * Dk + x, t < len);
        }
        asm volatile("cp.async.commit_group;\n" ::);
    };
    float* S = state + (size_t)slots[seq] * state_stride + state_offset + (size_t)h * Dk * Dv;
    for (int i = tid; i < Dk * CCOLS; i += CTHREADS) {
        const int r = i / CCOLS, j = j0 + i % CCOLS;
        Ss[i] = j < Dv ? S[(size_t)r * Dv + j] : 0.f;
    }
    load(0, 0);
    const int warp = tid >> 5, lane = tid & 31;
    for (int c = 0; c < nc; ++c) {
        const int stage = STAGES == 2 ? c & 1 : 0, len = min(CH, n - c * CH);
        if (STAGES == 2 && c + 1 < nc) {
            load(c + 1, stage ^ 1);
            asm volatile("cp.async.wait_group 1;\n" ::);
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::);
        }
        float* Wg = chunk(c);
        float* U = Wg + (size_t)Dk * CH;
        float* Sg = U + (size_t)CH * Dv;
        const float* eb = Sg + (size_t)Dk * Dv;
        // what the second half of this chunk needs of global memory, asked for now: four values of U per thread and their factors
        float uu[4], ed[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = tid + x * CTHREADS, t = i / CCOLS, j = j0 + i % CCOLS;
            uu[x] = t < len && j < Dv ? U[(size_t)t * Dv + j] : 0.f;
            ed[x] = eb[CH + t];
        }
        const float e_last = eb[len - 1];
        __syncthreads();
        const float* w = Ws + (size_t)stage * Dk * CH;
        const float* k = Ks + (size_t)stage * Dk * CH;
        for (int i = tid; i < Dk * CCOLS; i += CTHREADS) {
            const int j = j0 + i % CCOLS;
            if (j < Dv) Sg[(size_t)(i / CCOLS) * Dv + j] = Ss[i];
        }
        {   // W S: tiles of 4 tokens x 4 columns, the channels dealt out to four pairs of warps
            const int split = warp >> 1, t0 = ((warp & 1) * 8 + (lane >> 2)) * 4, c0 = (lane & 3) * 4;
            float acc[4][4] = {};
            for (int i = split; i < Dk; i += 4) {
                const float4 a4 = *reinterpret_cast<const float4*>(w + i * CH + t0), s4 = *reinterpret_cast<const float4*>(Ss + i * CCOLS + c0);
                const float a[4] = {a4.x, a4.y, a4.z, a4.w}, s[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(a[x], s[y], acc[x][y]);
            }
#pragma unroll
            for (int x = 0; x < 4; ++x)
                *reinterpret_cast<float4*>(part + ((size_t)split * CH + t0 + x) * CCOLS + c0) = make_float4(acc[x][0], acc[x][1], acc[x][2], acc[x][3]);
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int i = tid + x * CTHREADS, t = i / CCOLS, j = j0 + i % CCOLS;
            const float u = uu[x] - (part[i] + part[CH * CCOLS + i] + part[2 * CH * CCOLS + i] + part[3 * CH * CCOLS + i]);
            if (t < len && j < Dv) U[(size_t)t * Dv + j] = u;
            ud[i] = t < len ? u * ed[x] : 0.f;
        }
        __syncthreads();
        // S <- exp(b_last) S + K^T ud: tiles of 4 channels x 2 columns
        for (int item = tid; item < (Dk / 4) * (CCOLS / 2); item += CTHREADS) {
            const int i0 = (item / (CCOLS / 2)) * 4, c0 = (item % (CCOLS / 2)) * 2;
            float acc[4][2] = {};
#pragma unroll 8
            for (int t = 0; t < CH; ++t) {
                const float4 k4 = *reinterpret_cast<const float4*>(k + t * Dk + i0);
                const float2 u2 = *reinterpret_cast<const float2*>(ud + t * CCOLS + c0);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    acc[x][0] = fmaf(kk[x], u2.x, acc[x][0]);
                    acc[x][1] = fmaf(kk[x], u2.y, acc[x][1]);
                }
            }
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                float2* d = reinterpret_cast<float2*>(Ss + (i0 + x) * CCOLS + c0);
                float2 v = *d;
                v.x = fmaf(e_last, v.x, acc[x][0]);
                v.y = fmaf(e_last, v.y, acc[x][1]);
                *d = v;
            }
        }
        __syncthreads();                                   // (S is complete; this stage's buffers may be filled again)
        if (STAGES == 1 && c + 1 < nc) load(c + 1, 0);
    }
    for (int i = tid; i < Dk * CCOLS; i += CTHREADS) {
        const int j = j0 + i % CCOLS;
        if (j < Dv) S[(size_t)(i / CCOLS) * Dv + j] = Ss[i];
    }
}

// grid (chunks, heads): o [T, H Dv]
__global__ void __launch_bounds__(CTHREADS, 2)
delta_finish_kernel(const float* __restrict__ rows, const float* __restrict__ gates, const int* __restrict__ cu_tokens, int B, const float* __restrict__ scratch,
                    float* __restrict__ o, int H, int G, int Dk, int Dv) {
    extern __shared__ __align__(16) float sm[];
    float* qT = sm;                          // [Dk][CP]
    float* kT = qT + (size_t)Dk * CP;        // [Dk][CP]; then 64 columns of S_start [Dk][64]
    float* part = kT + (size_t)Dk * CP;      // [2][64][64]; then the weighted scores, transposed, and 64 columns of u
    __shared__ double b[CH];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    int start, len;
    if (!dr_chunk_of(blockIdx.x, cu_tokens, B, start, len)) return;
    const int h = blockIdx.y, g = h / (H / G), tid = threadIdx.x, C = 2 * G * Dk + H * Dv;
    dr_load_T(rows, C, g * Dk, start, len, Dk, qT);
    dr_load_T(rows, C, (G + g) * Dk, start, len, Dk, kT);
    dr_running_sums(gates, start, len, h, H, b);
    __syncthreads();
    dr_tri_products(qT, kT, Dk, part);
    __syncthreads();
    for (int idx = tid; idx < CH * CH; idx += CTHREADS) {
        const int s = idx / CH, t = idx % CH;
        part[idx] = t >= s ? expf((float)(b[t] - b[s])) * (part[idx] + part[CH * CH + idx]) : 0.f;
    }
    __syncthreads();
    const float* U = scratch + ((size_t)blockIdx.x * H + h) * dr_chunk_floats(Dk, Dv) + (size_t)Dk * CH;
    const float* Sg = U + (size_t)CH * Dv;
    float* us = part + CH * CH;              // [64][64]
    const int t0 = (tid >> 4) * 4, c0 = (tid & 15) * 4;
    float ebt[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) ebt[x] = expf((float)b[t0 + x]);
    for (int j0 = 0; j0 < Dv; j0 += 64) {
        const int width4 = min(64, Dv - j0) / 4;
        for (int idx = tid; idx < Dk * 16; idx += CTHREADS) {
            const int i = idx >> 4, q = idx & 15;
            *reinterpret_cast<float4*>(kT + i * 64 + 4 * q) =
                q < width4 ? *reinterpret_cast<const float4*>(Sg + (size_t)i * Dv + j0 + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        for (int idx = tid; idx < CH * 16; idx += CTHREADS) {
            const int t = idx >> 4, q = idx & 15;
            *reinterpret_cast<float4*>(us + t * 64 + 4 * q) =
                t < len && q < width4 ? *reinterpret_cast<const float4*>(U + (size_t)t * Dv + j0 + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        __syncthreads();
        if (t0 < len && (tid & 15) < width4) {
            float acc[4][4] = {};
#pragma unroll 4
            for (int i = 0; i < Dk; ++i) {
                const float4 q4 = *reinterpret_cast<const float4*>(qT + i * CP + t0), s4 = *reinterpret_cast<const float4*>(kT + i * 64 + c0);
                const float q[4] = {q4.x, q4.y, q4.z, q4.w}, s[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(q[x], s[y], acc[x][y]);
            }
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int y = 0; y < 4; ++y) acc[x][y] *= ebt[x];
            const int s_end = min(t0 + 4, len);
            for (int s = 0; s < s_end; ++s) {
                const float4 p4 = *reinterpret_cast<const float4*>(part + s * CH + t0), u4 = *reinterpret_cast<const float4*>(us + s * 64 + c0);
                const float p[4] = {p4.x, p4.y, p4.z, p4.w}, u[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
                for (int x = 0; x < 4; ++x)
#pragma unroll
                    for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(p[x], u[y], acc[x][y]);
            }
#pragma unroll
            for (int x = 0; x < 4; ++x)
                if (t0 + x < len)
                    *reinterpret_cast<float4*>(o + (size_t)(start + t0 + x) * H * Dv + (size_t)h * Dv + j0 + c0) =
                        make_float4(acc[x][0], acc[x][1], acc[x][2], acc[x][3]);
        }
        __syncthreads();
    }
}

size_t local_smem(int Dk) { return ((size_t)Dk * CP + 2 * CH * CH) * sizeof(float); }
size_t finish_smem(int Dk) { return ((size_t)2 * Dk * CP + 2 * CH * CH) * sizeof(float); }
size_t carry_smem(int Dk, int stages) { return ((size_t)stages * 2 * Dk * CH + (size_t)Dk * CCOLS + CH * CCOLS + 4 * CH * CCOLS) * sizeof(float); }
constexpr size_t SMEM_MAX = 220 * 1024;

template <typename K>
cudaError_t allow_smem(K kernel, size_t bytes) {
    return bytes > 48 * 1024 ? cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) : cudaSuccess;
}

bool sizes_ok(int H, int G, int Dk, int Dv, int K) { return H > 0 && G > 0 && H % G == 0 && Dk > 0 && Dv > 0 && K >= 1 && K <= MAX_TAPS; }

}  // namespace

// float32 words a sequence keeps: the memories, then two copies of the K - 1 last projected rows
VM_API int vm_delta_state_floats(int H, int G, int Dk, int Dv, int K) { return H * Dk * Dv + 2 * (K - 1) * (2 * G * Dk + H * Dv); }

// 1 if vm_delta_step takes these sizes
VM_API int vm_delta_step_fits(int Dk, int Dv) {
    if (Dv % 4 || Dv > 256 || Dk <= 0) return 0;
    const int RG = STEP_THREADS / (Dv / 4);
    return (Dk + RG - 1) / RG <= 16 ? 1 : 0;
}

// tokens per chunk of vm_delta_chunks for these sizes (0: it does not take them), and the float32 words of scratch it wants
VM_API int vm_delta_chunk_tokens(int Dk, int Dv) {
    if (Dk <= 0 || Dv <= 0 || Dk % 4 || Dv % 4) return 0;
    return local_smem(Dk) <= SMEM_MAX && finish_smem(Dk) <= SMEM_MAX && carry_smem(Dk, 1) <= SMEM_MAX ? CH : 0;
}
VM_API long long vm_delta_scratch_floats(int n_chunks, int H, int Dk, int Dv) { return (long long)n_chunks * H * dr_chunk_floats(Dk, Dv); }

// proj float32 [T, ld]: columns [0, G Dk) q, [G Dk, 2 G Dk) k, [2 G Dk, C) v, beta's logits at b_off and the decay's at a_off ([H] each);
// taps float32 [C, K]; state [slot, state_stride] with this mixer's words at state_offset.  rows float32 [T, C], gates float32 [T, 2 H].
// The kept rows move on (second launch, K > 1).
VM_API int vm_delta_prepare(const float* proj, int ld, int b_off, int a_off, const float* taps, int K, float* state, long long state_stride, int state_offset,
                            const int* positions, const int* seq_of_token, const int* cu_tokens, const int* slots, const float* A_log, const float* dt_bias,
                            float q_scale, float* rows, float* gates, int T, int B, int H, int G, int Dk, int Dv, cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    if (!sizes_ok(H, G, Dk, Dv, K) || !state) return VM_ERR_BAD_ARG;
    const size_t smem = (size_t)PT * Dk * sizeof(float);
    if (smem > 96 * 1024 || 2 * G + H + 1 > 65535) return VM_ERR_UNSUPPORTED;
    const int kept = state_offset + H * Dk * Dv, C = 2 * G * Dk + H * Dv;
    const int widest = Dk > Dv ? Dk : Dv;
    if (Dk % 4 == 0 && Dv % 4 == 0 && widest <= 256 && K <= 4 && ld % 4 == 0 && state_stride % 4 == 0 && kept % 4 == 0 &&
        ((uintptr_t)proj | (uintptr_t)rows | (uintptr_t)state) % 16 == 0) {
        const long long warps = (long long)((T + RUN - 1) / RUN) * (2 * G + H + 1);
        const dim3 grid((unsigned)((warps + PREP_THREADS / 32 - 1) / (PREP_THREADS / 32)));
#define DR_PREP(K_, NQ_)                                                                                                                                      \
    vm_launch_pdl(delta_prepare_run_kernel<K_, NQ_>, grid, dim3(PREP_THREADS), 0, stream, proj, ld, b_off, a_off, taps, (const float*)state, state_stride, kept, \
                  positions, seq_of_token, cu_tokens, slots, A_log, dt_bias, q_scale, rows, gates, T, H, G, Dk, Dv)
#define DR_PREP_K(NQ_)                   \
    do {                                 \
        if (K == 1) DR_PREP(1, NQ_);     \
        else if (K == 2) DR_PREP(2, NQ_); \
        else if (K == 3) DR_PREP(3, NQ_); \
        else DR_PREP(4, NQ_);            \
    } while (0)
        if (widest <= 128) DR_PREP_K(1);
        else DR_PREP_K(2);
#undef DR_PREP_K
#undef DR_PREP
    } else {
        const cudaError_t e = allow_smem(delta_prepare_kernel, smem);
        if (e != cudaSuccess) return (int)e;
        vm_launch_pdl(delta_prepare_kernel, dim3((T + PT - 1) / PT, 2 * G + H + 1), dim3(PREP_THREADS), smem, stream, proj, ld, b_off, a_off, taps, K,
                      (const float*)state, state_stride, kept, positions, seq_of_token, cu_tokens, slots, A_log, dt_bias, q_scale, rows, gates, T, H, G, Dk, Dv);
    }
    const int st = vm_launch_status();
    if (st || K <= 1) return st;
    const int slices = (C + 255) / 256;
    vm_launch_pdl(delta_keep_rows_kernel, dim3(B, slices > 16 ? 16 : slices), dim3(256), 0, stream, proj, ld, C, K, state, state_stride, kept, positions, cu_tokens,
                  slots);
    return vm_launch_status();
}

// token by token over the prepared rows; o float32 [T, H Dv]
VM_API int vm_delta_scan(const float* rows, const float* gates, float* state, long long state_stride, int state_offset, const int* cu_tokens, const int* slots,
                         float* o, int T, int B, int H, int G, int Dk, int Dv, cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    if (!sizes_ok(H, G, Dk, Dv, 1) || !state) return VM_ERR_BAD_ARG;
    if (Dk > SCAN_WARPS * 64 || H > 65535) return VM_ERR_UNSUPPORTED;
    const dim3 grid(B, H, (Dv + SCAN_COLS - 1) / SCAN_COLS), block(SCAN_WARPS * 32);
    const size_t smem = ((size_t)2 * Dk + 2 * SCAN_WARPS * SCAN_COLS + SCAN_WARPS) * sizeof(float);
    const int per = (Dk + SCAN_WARPS - 1) / SCAN_WARPS;
#define DR_SCAN(NR) vm_launch_pdl(delta_scan_kernel<NR>, grid, block, smem, stream, rows, gates, state, state_stride, state_offset, cu_tokens, slots, o, H, G, Dk, Dv)
    if (per <= 4) DR_SCAN(4);
    else if (per <= 8) DR_SCAN(8);
    else if (per <= 16) DR_SCAN(16);
    else if (per <= 32) DR_SCAN(32);
    else DR_SCAN(64);
#undef DR_SCAN
    return vm_launch_status();
}

// one token per sequence (token s is sequence s's): from the projections (with the SiLU gate's H Dv columns at g_off) to
// out [B, H Dv] = o / rms(o) * norm_w * silu(gate) in the activation dtype; memory and kept rows move on
VM_API int vm_delta_step(const float* proj, int ld, int g_off, int b_off, int a_off, const float* taps, int K, float* state, long long state_stride,
                         int state_offset, const int* positions, const int* slots, const float* A_log, const float* dt_bias, const float* norm_w, float eps,
                         float q_scale, void* out, int B, int H, int G, int Dk, int Dv, int act_dtype, cudaStream_t stream) {
    if (B <= 0) return 0;
    if (!sizes_ok(H, G, Dk, Dv, K) || !state) return VM_ERR_BAD_ARG;
    if (!vm_delta_step_fits(Dk, Dv) || state_stride % 4 || state_offset % 4 || H > 65535) return VM_ERR_UNSUPPORTED;
    const int RG = STEP_THREADS / (Dv / 4), per = (Dk + RG - 1) / RG, kept = state_offset + H * Dk * Dv;
    const int pad = (4 - (2 * Dk) % 4) % 4;
    if (pad) return VM_ERR_UNSUPPORTED;                   // (16-byte loads of v and u behind q and k in shared memory)
    const size_t smem = ((size_t)2 * Dk + 2 * Dv + (size_t)2 * RG * Dv) * sizeof(float);
#define DR_STEP(T_, NR)                                                                                                                                    \
    vm_launch_pdl(delta_step_kernel<T_, NR>, dim3(B, H), dim3(STEP_THREADS), smem, stream, proj, ld, g_off, b_off, a_off, taps, K, state, state_stride, state_offset, \
                  kept, positions, slots, A_log, dt_bias, norm_w, eps, q_scale, (T_*)out, H, G, Dk, Dv)
#define DR_STEP_ROWS(T_)                     \
    do {                                     \
        if (per <= 1) DR_STEP(T_, 1);        \
        else if (per <= 2) DR_STEP(T_, 2);   \
        else if (per <= 4) DR_STEP(T_, 4);   \
        else if (per <= 8) DR_STEP(T_, 8);   \
        else DR_STEP(T_, 16);                \
    } while (0)
    if (act_dtype == VM_F32) DR_STEP_ROWS(float);
    else if (act_dtype == VM_BF16) DR_STEP_ROWS(__nv_bfloat16);
    else return VM_ERR_UNSUPPORTED;
#undef DR_STEP_ROWS
#undef DR_STEP
    return vm_launch_status();
}

// prompts: three launches over the prepared rows; n_chunks: the step's chunks of vm_delta_chunk_tokens tokens, summed over its sequences
VM_API int vm_delta_chunks(const float* rows, const float* gates, float* state, long long state_stride, int state_offset, const int* cu_tokens, const int* slots,
                           float* o, float* scratch, int n_chunks, int T, int B, int H, int G, int Dk, int Dv, cudaStream_t stream) {
    if (T <= 0 || B <= 0 || n_chunks <= 0) return 0;
    if (!sizes_ok(H, G, Dk, Dv, 1) || !state || !scratch) return VM_ERR_BAD_ARG;
    if (!vm_delta_chunk_tokens(Dk, Dv) || H > 65535) return VM_ERR_UNSUPPORTED;
    const int stages = carry_smem(Dk, 2) <= SMEM_MAX ? 2 : 1;
    cudaError_t e = allow_smem(delta_local_kernel, local_smem(Dk));
    if (e == cudaSuccess) e = allow_smem(delta_finish_kernel, finish_smem(Dk));
    if (e == cudaSuccess) e = stages == 2 ? allow_smem(delta_carry_kernel<2>, carry_smem(Dk, 2)) : allow_smem(delta_carry_kernel<1>, carry_smem(Dk, 1));
    if (e != cudaSuccess) return (int)e;
    vm_launch_pdl(delta_local_kernel, dim3(n_chunks, H), dim3(CTHREADS), local_smem(Dk), stream, rows, gates, cu_tokens, B, scratch, H, G, Dk, Dv);
    int st = vm_launch_status();
    if (st) return st;
    const dim3 grid(B, H, (Dv + CCOLS - 1) / CCOLS);
    if (stages == 2)
        vm_launch_pdl(delta_carry_kernel<2>, grid, dim3(CTHREADS), carry_smem(Dk, 2), stream, rows, state, state_stride, state_offset, cu_tokens, slots, scratch, H, G,
                      Dk, Dv);
    else
        vm_launch_pdl(delta_carry_kernel<1>, grid, dim3(CTHREADS), carry_smem(Dk, 1), stream, rows, state, state_stride, state_offset, cu_tokens, slots, scratch, H, G,
                      Dk, Dv);
    st = vm_launch_status();
    if (st) return st;
    vm_launch_pdl(delta_finish_kernel, dim3(n_chunks, H), dim3(CTHREADS), finish_smem(Dk), stream, rows, gates, cu_tokens, B, (const float*)scratch, o, H, G, Dk, Dv);
    return vm_launch_status();
}
