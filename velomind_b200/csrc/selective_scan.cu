// A selective state-space mixer in the manner of the first Mamba: a recurrence of `N` state values per channel with an input-dependent
// step size, behind a short causal convolution (short_conv.cuh).
//
//   r_t            = W_x x_t, columns [0, R) | B [N] | C [N]            (a product of the caller's)
//   dt_t,c         = softplus(W_dt[c, :] r_t[0, R) + b_c)
//   S_t[c, n]      = exp(dt_t,c A[c, n]) S_(t-1)[c, n] + dt_t,c x_t,c B_t,n          A < 0, given as A log2(e)
//   y_t,c          = sum_n S_t[c, n] C_t,n + D_c x_t,c;   out_t,c = y_t,c silu(z_t,c)
//
// What a sequence keeps (float32, in its slot's state area, from the pointer given): S [channels, N], then the convolution's last K - 1
// inputs [K - 1, channels].  Step sizes, decays, the state and the sums over it are float32 whatever the activation dtype.
//
// Four lanes (a quad) share a channel; lane q of the quad holds the states n = 4 V (i / V) + V q + i % V, V of them side by side, so that
// the quad's reads of B and C from shared memory lie side by side.
//
// Prompts.  Tokens come through shared memory sixteen at a time, asked for several stages ahead.  A block first works out the step sizes of
// the next sixteen (each thread four of them), then runs the recurrence over the current sixteen without a branch or a barrier; after every
// four tokens the quad exchanges its partial sums of y so that each lane ends up with one token's, and finishes those outputs at the end.  One pass over the tokens suffices where a step has enough channels and
// sequences; else the tokens are cut into pieces that run side by side: a first pass leaves what every piece adds to the state and the sum of
// its step sizes, a second one carries the state from piece to piece, a third one repeats the pieces from the right start.
//
// Decode steps.  One launch: the step size's dot product, the state's update and the gated output.
#include "short_conv.cuh"

namespace {

constexpr int SS_THREADS = 64;                 // 16 channels
constexpr int SS_CH = SS_THREADS / 4;
constexpr int SS_TT = 16;                      // tokens per stage
constexpr int SS_STAGES = 4;                   // stages of shared memory: a stage's rows are asked for 48 tokens ahead

__device__ __forceinline__ float ss_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// log(1 + e^z) = max(z, 0) + log1p(e^-|z|) without a branch: with u = e^-|z| in (0, 1] and w = u / (2 + u) <= 1/3,
// log1p(u) = 2 atanh(w) = 2 (w + w^3 / 3 + w^5 / 5 + ...); seven terms leave less than 1e-8 of the sum.
__device__ __forceinline__ float ss_softplus(float z) {
    const float u = expf(-fabsf(z));
    const float w = __fdividef(u, 2.0f + u), w2 = w * w;
    float a = fmaf(w2, 1.0f / 13.0f, 1.0f / 11.0f);
    a = fmaf(w2, a, 1.0f / 9.0f);
    a = fmaf(w2, a, 1.0f / 7.0f);
    a = fmaf(w2, a, 1.0f / 5.0f);
    a = fmaf(w2, a, 1.0f / 3.0f);
    a = fmaf(w2, a, 1.0f);
    return fmaf(2.0f * w, a, fmaxf(z, 0.0f));
}
// z sigmoid(z) without a branch
__device__ __forceinline__ float ss_silu(float z) { return __fdividef(z, 1.0f + expf(-z)); }

// states of lane q: index i -> n
template <int V> __device__ __forceinline__ int ss_state_of(int q, int i) { return (i / V) * 4 * V + q * V + i % V; }

// V values from shared memory, side by side
template <int V> __device__ __forceinline__ void ss_load(const float* p, float* v);
template <> __device__ __forceinline__ void ss_load<4>(const float* p, float* v) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
template <> __device__ __forceinline__ void ss_load<2>(const float* p, float* v) {
    const float2 f = *reinterpret_cast<const float2*>(p);
    v[0] = f.x; v[1] = f.y;
}

// 16 bytes to shared memory (zeros where there is nothing to read)
__device__ __forceinline__ void ss_copy16(void* smem, const void* gmem, bool in) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = in ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(gmem), "r"(bytes));
}

// the piece a block works on: sequence, first token, tokens.  Pieces are cut at multiples of `piece` new tokens of their sequence.
__device__ __forceinline__ bool ss_where(const int* __restrict__ cu_tokens, int B, int piece, int at, int& seq, int& t0, int& len) {
    for (seq = 0; seq < B; ++seq) {
        const int a = cu_tokens[seq], b = cu_tokens[seq + 1];
        const int np = (b - a + piece - 1) / piece;
        if (at < np) { t0 = a + at * piece; len = min(piece, b - t0); return true; }
        at -= np;
    }
    return false;
}

struct ScanParams {
    const void* x;              // [T, C] the convolved inputs (activation dtype)
    const float* dt;            // [T, ldt] the step sizes before bias and softplus
    const float* r;             // [T, ldr] with B at column b_col and C behind it
    const void* z;              // the gate, [T, ldz] from its first column on (activation dtype)
    const float *dt_bias, *A2, *D;
    float* state;               // S of slot s at state + s * state_stride
    long long state_stride;
    float* pieces;              // [n_pieces, C, N]: what a piece adds to the state, later the state it starts from
    float* dt_sums;             // [n_pieces, C]
    const int *cu_tokens, *slots;
    void* out;                  // [T, C] (activation dtype)
    int ldt, ldr, b_col, ldz, B, C, N, piece;
    int vec;                    // rows may be copied 16 bytes at a time
};

enum { SS_WHOLE = 0, SS_ADDS = 1, SS_FROM_START = 2 };

template <typename T, int NPT> constexpr int ss_stage_bytes() { return SS_TT * (2 * 4 * NPT * 4 + SS_CH * 4 + 2 * SS_CH * (int)sizeof(T)); }

template <typename T, int NPT, int MODE>
__global__ void __launch_bounds__(SS_THREADS) selective_scan_kernel(const ScanParams p) {
    constexpr int V = NPT % 4 == 0 ? 4 : 2;
    constexpr int NP = 4 * NPT;                               // states with padding
    constexpr int STAGE = ss_stage_bytes<T, NPT>();
    __shared__ float2 sdt[2][SS_TT * SS_CH];                  // (dt, dt x)
    extern __shared__ __align__(16) unsigned char ss_smem[];  // per stage: B | C [TT][2 NP], dt [TT][CH], x [TT][CH], z [TT][CH]
    int seq, t0, len;
    if (!ss_where(p.cu_tokens, p.B, p.piece, blockIdx.y, seq, t0, len)) return;
    const int tid = threadIdx.x, q = tid & 3, ch = tid >> 2;
    const int c0 = blockIdx.x * SS_CH, c = c0 + ch;
    const bool live = c < p.C;
    const int cc = live ? c : p.C - 1;                        // (idle quads store nothing)
    auto at = [&](int stage) { return ss_smem + (size_t)(stage % SS_STAGES) * STAGE; };
    if (NP > p.N)                                             // padded states read zeros
        for (int i = tid; i < SS_STAGES * SS_TT * 2 * NP; i += SS_THREADS) {
            const int row = i / (2 * NP), col = i - row * 2 * NP;
            if (col % NP >= p.N) reinterpret_cast<float*>(at(row / SS_TT))[(row % SS_TT) * 2 * NP + col] = 0.f;
        }
    // tokens [base, base + TT) of the piece into a stage
    auto load = [&](int base) {
        unsigned char* sm = at(base / SS_TT);
        float* bc = reinterpret_cast<float*>(sm);
        float* dts = bc + SS_TT * 2 * NP;
        T* xs = reinterpret_cast<T*>(dts + SS_TT * SS_CH);
        T* zs = xs + SS_TT * SS_CH;
        constexpr int E = 16 / (int)sizeof(T);                // values per 16 bytes
        constexpr int WIDE = MODE == SS_ADDS ? 1 : 2;
        if (p.vec) {
#pragma unroll
            for (int i = tid; i < SS_TT * WIDE * NPT; i += SS_THREADS) {      // (a padded row of B or C has NPT runs of four)
                const int k = i / (WIDE * NPT), j = i - k * WIDE * NPT, half = j / NPT, n = 4 * (j - half * NPT);
                const bool in = base + k < len;
                if (n < p.N) ss_copy16(bc + k * 2 * NP + half * NP + n, p.r + (size_t)(t0 + (in ? base + k : 0)) * p.ldr + p.b_col + half * p.N + n, in);
            }
#pragma unroll
            for (int i = tid; i < SS_TT * (SS_CH / 4); i += SS_THREADS) {
                const int k = i / (SS_CH / 4), j = 4 * (i - k * (SS_CH / 4));
                const bool in = base + k < len && c0 + j < p.C;
                ss_copy16(dts + k * SS_CH + j, p.dt + (size_t)(t0 + (in ? base + k : 0)) * p.ldt + (in ? c0 + j : 0), in);
            }
#pragma unroll
            for (int i = tid; i < SS_TT * (SS_CH / E); i += SS_THREADS) {
                const int k = i / (SS_CH / E), j = E * (i - k * (SS_CH / E));
                const bool in = base + k < len && c0 + j < p.C;
                const size_t row = (size_t)(t0 + (in ? base + k : 0));
                ss_copy16(xs + k * SS_CH + j, static_cast<const T*>(p.x) + row * p.C + (in ? c0 + j : 0), in);
                if (MODE != SS_ADDS) ss_copy16(zs + k * SS_CH + j, static_cast<const T*>(p.z) + row * p.ldz + (in ? c0 + j : 0), in);
            }
            return;
        }
        for (int i = tid; i < SS_TT * 2 * p.N; i += SS_THREADS) {
            const int k = i / (2 * p.N), j = i - k * 2 * p.N, half = j >= p.N, n = j - half * p.N;
            bc[k * 2 * NP + half * NP + n] = base + k < len ? p.r[(size_t)(t0 + base + k) * p.ldr + p.b_col + half * p.N + n] : 0.f;
        }
        for (int i = tid; i < SS_TT * SS_CH; i += SS_THREADS) {
            const int k = i / SS_CH, j = i - k * SS_CH;
            const bool in = base + k < len && c0 + j < p.C;
            const size_t row = (size_t)(t0 + base + k);
            dts[i] = in ? p.dt[row * p.ldt + c0 + j] : 0.f;
            xs[i] = in ? static_cast<const T*>(p.x)[row * p.C + c0 + j] : vm_from_float<T>(0.f);
            zs[i] = in && MODE != SS_ADDS ? static_cast<const T*>(p.z)[row * p.ldz + c0 + j] : vm_from_float<T>(0.f);
        }
    };
#pragma unroll
    for (int k = 0; k < SS_STAGES - 1; ++k) {
        if (k * SS_TT < len) load(k * SS_TT);
        asm volatile("cp.async.commit_group;\n" ::);
    }
    float A2[NPT], s[NPT];
    float* S = p.state + (size_t)p.slots[seq] * p.state_stride + (size_t)cc * p.N;
    float* piece_S = MODE == SS_WHOLE ? nullptr : p.pieces + ((size_t)blockIdx.y * p.C + cc) * p.N;
    const float* start = MODE == SS_WHOLE ? S : (MODE == SS_FROM_START ? piece_S : nullptr);
#pragma unroll
    for (int i = 0; i < NPT; ++i) {
        const int n = ss_state_of<V>(q, i);
        A2[i] = n < p.N ? p.A2[(size_t)cc * p.N + n] : 0.f;
        s[i] = start && n < p.N ? start[n] : 0.f;
    }
    const float skip = MODE == SS_ADDS ? 0.f : p.D[cc];
    float dt_sum = 0.f;
    T* og = static_cast<T*>(p.out) + cc;

    // step sizes of a stage's tokens for the block's channels; 0 past the end (the state then stays as it is)
    const int my_ch = tid & (SS_CH - 1), my_c = min(c0 + my_ch, p.C - 1);
    const float bias = p.dt_bias[my_c];
    auto steps = [&](int base) {
        const float* bc = reinterpret_cast<const float*>(at(base / SS_TT));
        const float* dts = bc + SS_TT * 2 * NP;
        const T* xs = reinterpret_cast<const T*>(dts + SS_TT * SS_CH);
        float2* out = sdt[(base / SS_TT) & 1];
#pragma unroll
        for (int j = 0; j < SS_TT * SS_CH / SS_THREADS; ++j) {
            const int k = (tid + j * SS_THREADS) / SS_CH;
            const float dt = base + k < len ? ss_softplus(dts[k * SS_CH + my_ch] + bias) : 0.f;
            out[k * SS_CH + my_ch] = make_float2(dt, dt * vm_to_float(xs[k * SS_CH + my_ch]));
        }
    };
    asm volatile("cp.async.wait_group %0;\n" ::"n"(SS_STAGES - 2));
    __syncthreads();
    steps(0);
    for (int base = 0; base < len; base += SS_TT) {
        asm volatile("cp.async.wait_group %0;\n" ::"n"(SS_STAGES - 3));
        __syncthreads();                                      // the next stage and this one's step sizes are there; the stage before is read by all
        if (base + (SS_STAGES - 1) * SS_TT < len) load(base + (SS_STAGES - 1) * SS_TT);
        asm volatile("cp.async.commit_group;\n" ::);
        if (base + SS_TT < len) steps(base + SS_TT);
        const float* bc = reinterpret_cast<const float*>(at(base / SS_TT));
        const float2* step = sdt[(base / SS_TT) & 1] + ch;
        float done[SS_TT / 4];                                // y of this lane's token of every four
#pragma unroll
        for (int g = 0; g < SS_TT; g += 4) {
            float part[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 d = step[(g + k) * SS_CH];
                if (MODE == SS_ADDS) dt_sum += d.x;
                const float* row = bc + (g + k) * 2 * NP;
                float y = 0.f;
#pragma unroll
                for (int i = 0; i < NPT; i += V) {
                    float b[V], cv[V];
                    ss_load<V>(row + ss_state_of<V>(q, i), b);
                    if (MODE != SS_ADDS) ss_load<V>(row + NP + ss_state_of<V>(q, i), cv);
#pragma unroll
                    for (int j = 0; j < V; ++j) {
                        s[i + j] = fmaf(ss_exp2(d.x * A2[i + j]), s[i + j], d.y * b[j]);
                        if (MODE != SS_ADDS) y = fmaf(s[i + j], cv[j], y);
                    }
                }
                part[k] = y;
            }
            if (MODE != SS_ADDS) {
                // lane q gets the sum over the quad of part[q]
                const bool up = q & 2, odd = q & 1;
                const float a0 = up ? part[2] : part[0], a1 = up ? part[3] : part[1];
                const float s0 = up ? part[0] : part[2], s1 = up ? part[1] : part[3];
                const float b0 = a0 + __shfl_xor_sync(0xffffffffu, s0, 2), b1 = a1 + __shfl_xor_sync(0xffffffffu, s1, 2);
                const float mine = odd ? b1 : b0, other = odd ? b0 : b1;
                done[g / 4] = mine + __shfl_xor_sync(0xffffffffu, other, 1);
            }
        }
        if (MODE != SS_ADDS) {
            const T* xs = reinterpret_cast<const T*>(bc + SS_TT * 2 * NP + SS_TT * SS_CH) + ch;
            const T* zs = xs + SS_TT * SS_CH;
#pragma unroll
            for (int g = 0; g < SS_TT; g += 4) {
                const float y = fmaf(skip, vm_to_float(xs[(g + q) * SS_CH]), done[g / 4]);
                if (base + g + q < len && live) og[(size_t)(t0 + base + g + q) * p.C] = vm_from_float<T>(y * ss_silu(vm_to_float(zs[(g + q) * SS_CH])));
            }
        }
    }
    asm volatile("cp.async.wait_all;\n" ::);
    float* keep = MODE == SS_WHOLE ? S : (MODE == SS_ADDS ? piece_S : nullptr);
    if (keep && live) {
#pragma unroll
        for (int i = 0; i < NPT; ++i) {
            const int n = ss_state_of<V>(q, i);
            if (n < p.N) keep[n] = s[i];
        }
    }
    if (MODE == SS_ADDS && live && q == 0) p.dt_sums[(size_t)blockIdx.y * p.C + c] = dt_sum;
}

// grid (ceil(C N / 256), sequences): a thread carries one state value through its sequence's pieces
__global__ void selective_carry_kernel(const ScanParams p) {
    const int seq = blockIdx.y;
    const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x, CN = (long long)p.C * p.N;
    if (e >= CN) return;
    int first = 0;
    for (int b = 0; b < seq; ++b) first += (p.cu_tokens[b + 1] - p.cu_tokens[b] + p.piece - 1) / p.piece;
    const int np = (p.cu_tokens[seq + 1] - p.cu_tokens[seq] + p.piece - 1) / p.piece;
    if (np <= 0) return;
    const int c = (int)(e / p.N);
    const float A2 = p.A2[e];
    float* S = p.state + (size_t)p.slots[seq] * p.state_stride + e;
    float cur = *S;
    for (int k0 = 0; k0 < np; k0 += 4) {
        float add[4], dts[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {                         // (four pieces' values are fetched before the first store)
            const bool in = k0 + k < np;
            add[k] = in ? p.pieces[(size_t)(first + k0 + k) * CN + e] : 0.f;
            dts[k] = in ? p.dt_sums[(size_t)(first + k0 + k) * p.C + c] : 0.f;
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            if (k0 + k >= np) break;
            p.pieces[(size_t)(first + k0 + k) * CN + e] = cur;      // the state at this piece's start
            cur = fmaf(ss_exp2(dts[k] * A2), cur, add[k]);
        }
    }
    *S = cur;
}

// ------------------------------------------------------------------------------------------------ decode steps
// dot product of R values of a weight row with float32 values in shared memory, by a quad (each lane its share)
__device__ __forceinline__ float quad_dot(const float* __restrict__ w, const float* x, int R, int q, bool vec) {
    float a = 0.f;
    if (vec) {
        for (int i = 4 * q; i < R; i += 16) {
            const float4 f = *reinterpret_cast<const float4*>(w + i);
            a = fmaf(f.x, x[i], fmaf(f.y, x[i + 1], fmaf(f.z, x[i + 2], fmaf(f.w, x[i + 3], a))));
        }
    } else {
        for (int i = q; i < R; i += 4) a = fmaf(w[i], x[i], a);
    }
    return a;
}
__device__ __forceinline__ float quad_dot(const __nv_bfloat16* __restrict__ w, const float* x, int R, int q, bool vec) {
    float a = 0.f;
    if (vec) {
#pragma unroll 4
        for (int i = 8 * q; i < R; i += 32) {
            const uint4 u = *reinterpret_cast<const uint4*>(w + i);
            const unsigned v[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v[k]));
                a = fmaf(f.x, x[i + 2 * k], fmaf(f.y, x[i + 2 * k + 1], a));
            }
        }
    } else {
        for (int i = q; i < R; i += 4) a = fmaf(__bfloat162float(w[i]), x[i], a);
    }
    return a;
}

constexpr int STEP_THREADS = 128;

// grid (ceil(C / 32), sequences); token s is sequence s's.  r rows [rank | B | C].
template <typename T, typename W>
__global__ void __launch_bounds__(STEP_THREADS)
selective_step_kernel(const T* __restrict__ x, const float* __restrict__ r, int ldr, const W* __restrict__ w_dt, int R, const T* __restrict__ z, int ldz,
                      const float* __restrict__ dt_bias, const float* __restrict__ A2, const float* __restrict__ D, float* __restrict__ state,
                      long long state_stride, const int* __restrict__ slots, T* __restrict__ out, int C, int N, int vec_dt, int vec_n) {
    extern __shared__ __align__(16) float sr[];              // [R + 2 N]
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int seq = blockIdx.y, q = threadIdx.x & 3, c = blockIdx.x * (STEP_THREADS / 4) + (threadIdx.x >> 2);
    for (int i = threadIdx.x; i < R + 2 * N; i += STEP_THREADS) sr[i] = r[(size_t)seq * ldr + i];
    __syncthreads();
    const bool live = c < C;
    const int cc = live ? c : C - 1;
    float dt = quad_dot(w_dt + (size_t)cc * R, sr, R, q, vec_dt != 0);
    dt += __shfl_xor_sync(0xffffffffu, dt, 1);
    dt += __shfl_xor_sync(0xffffffffu, dt, 2);
    dt = softplus_f(dt + dt_bias[cc]);
    const float xv = vm_to_float(x[(size_t)seq * C + cc]), dx = dt * xv;
    float* S = state + (size_t)slots[seq] * state_stride + (size_t)cc * N;
    const float* a2 = A2 + (size_t)cc * N;
    const float *sB = sr + R, *sC = sB + N;
    float y = 0.f;
    if (vec_n) {
        for (int n = 4 * q; n < N; n += 16) {
            float4 s = *reinterpret_cast<float4*>(S + n);
            const float4 a = *reinterpret_cast<const float4*>(a2 + n);
            s.x = fmaf(ss_exp2(dt * a.x), s.x, dx * sB[n]);
            s.y = fmaf(ss_exp2(dt * a.y), s.y, dx * sB[n + 1]);
            s.z = fmaf(ss_exp2(dt * a.z), s.z, dx * sB[n + 2]);
            s.w = fmaf(ss_exp2(dt * a.w), s.w, dx * sB[n + 3]);
            y = fmaf(s.x, sC[n], fmaf(s.y, sC[n + 1], fmaf(s.z, sC[n + 2], fmaf(s.w, sC[n + 3], y))));
            if (live) *reinterpret_cast<float4*>(S + n) = s;
        }
    } else {
        for (int n = q; n < N; n += 4) {
            const float s = fmaf(ss_exp2(dt * a2[n]), S[n], dx * sB[n]);
            y = fmaf(s, sC[n], y);
            if (live) S[n] = s;
        }
    }
    y += __shfl_xor_sync(0xffffffffu, y, 1);
    y += __shfl_xor_sync(0xffffffffu, y, 2);
    if (q == 0 && live) out[(size_t)seq * C + c] = vm_from_float<T>(fmaf(D[c], xv, y) * silu_f(vm_to_float(z[(size_t)seq * ldz + c])));
}

template <typename T, int MODE>
int launch_scan_mode(const ScanParams& p, int n_pieces, cudaStream_t stream) {
    const dim3 grid((p.C + SS_CH - 1) / SS_CH, n_pieces);
#define VM_SEL(NPT)                                                                             \
    if (p.N <= 4 * NPT) {                                                                       \
        constexpr int smem = SS_STAGES * ss_stage_bytes<T, NPT>();                              \
        static bool raised = false;                                                             \
        if (smem > 32 * 1024 && !raised) {                                                      \
            cudaError_t e = cudaFuncSetAttribute(selective_scan_kernel<T, NPT, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); \
            if (e != cudaSuccess) return (int)e;                                                \
            raised = true;                                                                      \
        }                                                                                       \
        selective_scan_kernel<T, NPT, MODE><<<grid, SS_THREADS, smem, stream>>>(p);             \
        return vm_launch_status();                                                              \
    }
    VM_SEL(2) VM_SEL(4) VM_SEL(6) VM_SEL(8) VM_SEL(12) VM_SEL(16) VM_SEL(32)
#undef VM_SEL
    return VM_ERR_UNSUPPORTED;
}

template <typename T>
int launch_scan(const ScanParams& p, int n_pieces, cudaStream_t stream) {
    if (!p.pieces) return launch_scan_mode<T, SS_WHOLE>(p, n_pieces, stream);
    int st = launch_scan_mode<T, SS_ADDS>(p, n_pieces, stream);
    if (st) return st;
    selective_carry_kernel<<<dim3((unsigned)(((long long)p.C * p.N + 255) / 256), p.B), 256, 0, stream>>>(p);
    st = vm_launch_status();
    if (st) return st;
    return launch_scan_mode<T, SS_FROM_START>(p, n_pieces, stream);
}

}  // namespace

VM_API long long vm_selective_state_floats(int C, int N, int K) { return (long long)C * N + (long long)(K - 1) * C; }
VM_API long long vm_selective_scratch_floats(int n_pieces, int C, int N) { return (long long)n_pieces * C * (N + 1); }
VM_API int vm_selective_max_state() { return 128; }

// out [T, C] = silu(bias + conv(columns [u_col, u_col + C) of proj)); the kept inputs lie in `state` (slot s at state + s * state_floats) at
// conv_off
VM_API int vm_short_conv_silu(const void* proj, int ld, int u_col, const float* taps, const float* bias, float* state, int state_floats, int conv_off,
                              const int* positions, const int* seq_of_token, const int* cu_tokens, const int* slots, int one_token_each, int T, int B, int C,
                              int K, void* out, int act_dtype, cudaStream_t stream) {
    if (T <= 0 || B <= 0) return 0;
    if (C <= 0 || K < 1 || K > 64 || ld < u_col + C || !state || (one_token_each && T != B)) return VM_ERR_BAD_ARG;
    if (act_dtype == VM_F32)
        return launch_short_conv<float>(proj, ld, u_col, taps, bias, state, state_floats, conv_off, positions, seq_of_token, cu_tokens, slots, one_token_each, T,
                                        B, C, K, out, stream);
    if (act_dtype == VM_BF16)
        return launch_short_conv<__nv_bfloat16>(proj, ld, u_col, taps, bias, state, state_floats, conv_off, positions, seq_of_token, cu_tokens, slots,
                                                one_token_each, T, B, C, K, out, stream);
    return VM_ERR_UNSUPPORTED;
}

// Prompts.  x [T, C] and z (rows of ldz) in the activation dtype, dt float32 [T, ldt] before bias and softplus, r float32 [T, ldr] with B and C
// (N columns each) from b_col on.  scratch null: one pass, a block per 16 channels and sequence (`piece` is then not read); else
// vm_selective_scratch_floats(n_pieces, ...) floats with n_pieces = sum over the sequences of ceil(new tokens / piece).
VM_API int vm_selective_scan(const void* x, const float* dt, int ldt, const float* r, int ldr, int b_col, const void* z, int ldz, const float* dt_bias,
                             const float* A2, const float* D, float* state, long long state_stride, const int* cu_tokens, const int* slots, void* out,
                             float* scratch, int piece, int n_pieces, int B, int C, int N, int act_dtype, cudaStream_t stream) {
    if (B <= 0 || n_pieces <= 0) return 0;
    if (C <= 0 || N <= 0 || ldt < C || ldz < C || ldr < b_col + 2 * N || !state || state_stride < (long long)C * N || (scratch && piece <= 0)) return VM_ERR_BAD_ARG;
    if (n_pieces > 65535 || B > 65535) return VM_ERR_UNSUPPORTED;
    ScanParams p{};
    p.x = x; p.dt = dt; p.r = r; p.z = z; p.dt_bias = dt_bias; p.A2 = A2; p.D = D; p.state = state; p.state_stride = state_stride;
    p.pieces = scratch; p.dt_sums = scratch ? scratch + (size_t)n_pieces * C * N : nullptr;
    p.cu_tokens = cu_tokens; p.slots = slots; p.out = out;
    p.ldt = ldt; p.ldr = ldr; p.b_col = b_col; p.ldz = ldz; p.B = B; p.C = C; p.N = N;
    p.piece = scratch ? piece : 0x3fffffff;
    const int e16 = act_dtype == VM_F32 ? 4 : 8;              // values of the activation dtype in 16 bytes
    const uintptr_t bases = (uintptr_t)x | (uintptr_t)dt | (uintptr_t)r | (uintptr_t)z;
    p.vec = bases % 16 == 0 && C % e16 == 0 && ldz % e16 == 0 && ldt % 4 == 0 && ldr % 4 == 0 && b_col % 4 == 0 && N % 4 == 0 ? 1 : 0;
    if (act_dtype == VM_F32) return launch_scan<float>(p, n_pieces, stream);
    if (act_dtype == VM_BF16) return launch_scan<__nv_bfloat16>(p, n_pieces, stream);
    return VM_ERR_UNSUPPORTED;
}

// One token per sequence.  r rows [rank | B | C], w_dt [C, rank] in w_dtype.
VM_API int vm_selective_step(const void* x, const float* r, int ldr, const void* w_dt, int w_dtype, int rank, const void* z, int ldz, const float* dt_bias,
                             const float* A2, const float* D, float* state, long long state_stride, const int* slots, void* out, int B, int C, int N,
                             int act_dtype, cudaStream_t stream) {
    if (B <= 0) return 0;
    if (C <= 0 || N <= 0 || rank <= 0 || ldz < C || ldr < rank + 2 * N || !state || state_stride < (long long)C * N) return VM_ERR_BAD_ARG;
    const size_t smem = (size_t)(rank + 2 * N) * sizeof(float);
    if (B > 65535 || smem > 48 * 1024) return VM_ERR_UNSUPPORTED;
    const dim3 grid((C + STEP_THREADS / 4 - 1) / (STEP_THREADS / 4), B);
    const int per16 = w_dtype == VM_F32 ? 4 : 8;
    const int vec_dt = rank % per16 == 0 && ((uintptr_t)w_dt & 15) == 0 ? 1 : 0;
    const int vec_n = N % 4 == 0 && state_stride % 4 == 0 && (((uintptr_t)state | (uintptr_t)A2) & 15) == 0 ? 1 : 0;
#define VM_STEP(T, W)                                                                                                                                     \
    vm_launch_pdl(selective_step_kernel<T, W>, grid, dim3(STEP_THREADS), smem, stream, (const T*)x, r, ldr, (const W*)w_dt, rank, (const T*)z, ldz, dt_bias, \
                  A2, D, state, state_stride, slots, (T*)out, C, N, vec_dt, vec_n)
    if (act_dtype == VM_F32 && w_dtype == VM_F32) VM_STEP(float, float);
    else if (act_dtype == VM_BF16 && w_dtype == VM_F32) VM_STEP(__nv_bfloat16, float);
    else if (act_dtype == VM_BF16 && w_dtype == VM_BF16) VM_STEP(__nv_bfloat16, __nv_bfloat16);
    else return VM_ERR_UNSUPPORTED;
#undef VM_STEP
    return vm_launch_status();
}

// dst [T, n] (activation dtype) = columns [col, col + n) of src float32 [T, ld]
namespace {
template <typename T>
__global__ void take_columns_kernel(const float* __restrict__ src, int ld, int col, T* __restrict__ dst, int n, long long total) {
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / n;
        dst[i] = vm_from_float<T>(src[t * ld + col + (i - t * n)]);
    }
}
}  // namespace
VM_API int vm_take_columns(const float* src, int ld, int col, void* dst, int n, int T, int act_dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (n <= 0 || col < 0 || ld < col + n) return VM_ERR_BAD_ARG;
    const long long total = (long long)T * n, want = (total + 255) / 256;
    const int blocks = (int)(want < 148 * 8 ? want : 148 * 8);
    if (act_dtype == VM_F32) take_columns_kernel<float><<<blocks, 256, 0, stream>>>(src, ld, col, (float*)dst, n, total);
    else if (act_dtype == VM_BF16) take_columns_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>(src, ld, col, (__nv_bfloat16*)dst, n, total);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}
