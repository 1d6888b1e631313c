// The two norms of a latent-attention layer and the cache write of its key/value latent, one launch.
//
// A latent-attention layer projects its input down twice: to a query latent and to a key/value latent.  Both are
// RMS-normed with a learned scale.  The query latent goes on to the query up-projection; the key/value latent is all the
// layer remembers of a token: one row per token in the paged cache (a group with one "head" of the latent's size and no
// second row), from which keys and values are made again, or, with the up-projections moved to the query's and the
// output's side, never made at all.
//
// Input: the down projections' float32 result [T, ld]: columns [0, q_rank) the query latent, [q_rank, q_rank + kv_rank) the
// key/value latent (absent for a layer that reads another layer's latents).  Statistics in float32.  One block per token.
//
// A layer with rotary positions keeps `rot_dim` more values per token behind the latent: columns [q_rank + kv_rank, q_rank +
// kv_rank + rot_dim) of the input, not normed, one key part that all heads share; its first `rotary_dim` values are turned by the
// token's position (angle and its sine and cosine in float32) before they are written.  A cache row then has kv_rank + rot_dim values.
#include "common.cuh"

template <typename T>
__global__ void latent_norm_write_kernel(const float* __restrict__ down, int ld, int q_rank, int kv_rank, const float* __restrict__ wq,
                                         const float* __restrict__ wkv, float eps, T* __restrict__ cq, const int* __restrict__ positions,
                                         const int* __restrict__ seq_of_token, const int* __restrict__ block_table, int max_blocks,
                                         T* __restrict__ pages, int n_pages, int rot_dim, int rotary_dim, const float* __restrict__ inv_freq,
                                         int pairing, int* __restrict__ err) {
    __shared__ float red[32];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t = blockIdx.x;
    const float* row = down + (size_t)t * ld;
    {
        float ss = 0.f;
        for (int i = threadIdx.x; i < q_rank; i += blockDim.x) ss += row[i] * row[i];
        ss = vm_block_sum(ss, red);
        const float inv = 1.0f / sqrtf(ss / (float)q_rank + eps);
        for (int i = threadIdx.x; i < q_rank; i += blockDim.x) cq[(size_t)t * q_rank + i] = vm_from_float<T>(row[i] * inv * wq[i]);
    }
    if (!pages) return;
    const float* lat = row + q_rank;
    float ss = 0.f;
    for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) ss += lat[i] * lat[i];
    ss = vm_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)kv_rank + eps);
    const int pos = positions[t], seq = seq_of_token[t];
    const int blk = pos / VM_PAGE_TOKENS;
    const int page = blk < max_blocks ? block_table[(size_t)seq * max_blocks + blk] : -1;
    if (page < 0 || page >= n_pages) {
        if (threadIdx.x == 0 && err) atomicExch(err, VM_ERRWORD_CACHE_WRITE);
        return;
    }
    T* dst = pages + ((size_t)page * VM_PAGE_TOKENS + (pos % VM_PAGE_TOKENS)) * (kv_rank + rot_dim);
    for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) dst[i] = vm_from_float<T>(lat[i] * inv * wkv[i]);
    const float* kr = lat + kv_rank;
    const int half = rotary_dim / 2;
    for (int i = threadIdx.x; i < half + (rot_dim - rotary_dim); i += blockDim.x) {
        if (i >= half) {                                   // behind the rotated values: as projected
            const int k = rotary_dim + (i - half);
            dst[kv_rank + k] = vm_from_float<T>(kr[k]);
            continue;
        }
        const int ia = pairing == VM_PAIR_INTERLEAVED ? 2 * i : i, ib = pairing == VM_PAIR_INTERLEAVED ? 2 * i + 1 : i + half;
        float sn, cs;
        sincosf((float)pos * inv_freq[i], &sn, &cs);
        const float u = kr[ia], v = kr[ib];
        dst[kv_rank + ia] = vm_from_float<T>(u * cs - v * sn);
        dst[kv_rank + ib] = vm_from_float<T>(v * cs + u * sn);
    }
}

// pages [n_pages, VM_PAGE_TOKENS, kv_rank + rot_dim]; inv_freq float32 [rotary_dim / 2]
VM_API int vm_latent_rope_norm_write(const float* down, int ld, int q_rank, int kv_rank, const float* wq, const float* wkv, float eps, void* cq,
                                     const int* positions, const int* seq_of_token, const int* block_table, int max_blocks, void* pages,
                                     int n_pages, int rot_dim, int rotary_dim, const float* inv_freq, int pairing, int T, int act_dtype, int* err,
                                     cudaStream_t stream) {
    if (T <= 0) return 0;
    if (q_rank <= 0 || kv_rank <= 0 || rot_dim < 0 || ld < q_rank + (pages ? kv_rank + rot_dim : 0)) return VM_ERR_BAD_ARG;
    if (rotary_dim < 0 || rotary_dim % 2 || rotary_dim > rot_dim || (rotary_dim > 0 && !inv_freq)) return VM_ERR_BAD_ARG;
    const int widest = q_rank > kv_rank ? q_rank : kv_rank;
    const int threads = widest >= 512 ? 256 : 128;
    if (act_dtype == VM_F32)
        vm_launch_pdl(latent_norm_write_kernel<float>, dim3(T), dim3(threads), 0, stream, down, ld, q_rank, kv_rank, wq, wkv, eps, (float*)cq, positions,
                      seq_of_token, block_table, max_blocks, (float*)pages, n_pages, rot_dim, rotary_dim, inv_freq, pairing, err);
    else if (act_dtype == VM_BF16)
        vm_launch_pdl(latent_norm_write_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, down, ld, q_rank, kv_rank, wq, wkv, eps,
                      (__nv_bfloat16*)cq, positions, seq_of_token, block_table, max_blocks, (__nv_bfloat16*)pages, n_pages, rot_dim, rotary_dim, inv_freq,
                      pairing, err);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}

VM_API int vm_latent_norm_write(const float* down, int ld, int q_rank, int kv_rank, const float* wq, const float* wkv, float eps, void* cq,
                                const int* positions, const int* seq_of_token, const int* block_table, int max_blocks, void* pages,
                                int n_pages, int T, int act_dtype, int* err, cudaStream_t stream) {
    return vm_latent_rope_norm_write(down, ld, q_rank, kv_rank, wq, wkv, eps, cq, positions, seq_of_token, block_table, max_blocks, pages, n_pages, 0, 0,
                                     nullptr, VM_PAIR_HALF_SPLIT, T, act_dtype, err, stream);
}

// A layer whose queries come straight from its input (no query latent): the projections' float32 row is
//     [ heads x (dim unrotated | rot_dim) queries | kv_rank latent | rot_dim shared key part | ... ]
// One launch rounds the unrotated query parts into q [T, heads * dim], turns the rotated ones into their place behind each head's room of
// q_far [T, heads * (kv_rank + rot_dim)] (the room in front is the up-projected query's), norms the latent, turns the key part and writes the
// cache row.  A token's angles are computed once for all heads.
template <typename T>
__global__ void latent_direct_kernel(const float* __restrict__ proj, int ld, int H, int D, int R, int kv_rank, const float* __restrict__ wkv, float eps,
                                     T* __restrict__ q, T* __restrict__ q_far, const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                                     const int* __restrict__ block_table, int max_blocks, T* __restrict__ pages, int n_pages, int rotary_dim,
                                     const float* __restrict__ inv_freq, int pairing, int* __restrict__ err) {
    extern __shared__ float angles[];        // cosines, then sines, [rotary_dim / 2] each
    __shared__ float red[32];
    vm_pdl_launch_dependents();
    vm_pdl_wait();
    const int t = blockIdx.x, pos = positions[t], half = rotary_dim / 2, Dq = D + R, far = kv_rank + R;
    const float* row = proj + (size_t)t * ld;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf((float)pos * inv_freq[i], &sn, &cs);
        angles[i] = cs;
        angles[half + i] = sn;
    }
    for (int i = threadIdx.x; i < H * D; i += blockDim.x) {
        const int h = i / D;
        q[(size_t)t * H * D + i] = vm_from_float<T>(row[h * Dq + (i - h * D)]);
    }
    const float* lat = row + H * Dq;
    float ss = 0.f;
    if (pages)
        for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) ss += lat[i] * lat[i];
    ss = vm_block_sum(ss, red);              // (its barriers also make the angles visible)
    T* dst = nullptr;
    if (pages) {
        const int blk = pos / VM_PAGE_TOKENS;
        const int page = blk < max_blocks ? block_table[(size_t)seq_of_token[t] * max_blocks + blk] : -1;
        if (page >= 0 && page < n_pages) dst = pages + ((size_t)page * VM_PAGE_TOKENS + (pos % VM_PAGE_TOKENS)) * far;
        else if (threadIdx.x == 0 && err) atomicExch(err, VM_ERRWORD_CACHE_WRITE);
    }
    if (dst) {
        const float inv = 1.0f / sqrtf(ss / (float)kv_rank + eps);
        for (int i = threadIdx.x; i < kv_rank; i += blockDim.x) dst[i] = vm_from_float<T>(lat[i] * inv * wkv[i]);
    }
    const int per = half + (R - rotary_dim);
    for (int i = threadIdx.x; i < (H + 1) * per; i += blockDim.x) {      // a pair (or a passing value) of a head, or of the shared key part (h = H)
        const int h = i / per, j = i - h * per;
        const float* x = h < H ? row + h * Dq + D : lat + kv_rank;
        T* y = h < H ? q_far + (size_t)t * H * far + (size_t)h * far + kv_rank : (dst ? dst + kv_rank : nullptr);
        if (!y) continue;
        if (j >= half) {
            const int k = rotary_dim + (j - half);
            y[k] = vm_from_float<T>(x[k]);
            continue;
        }
        const int ia = pairing == VM_PAIR_INTERLEAVED ? 2 * j : j, ib = pairing == VM_PAIR_INTERLEAVED ? 2 * j + 1 : j + half;
        const float cs = angles[j], sn = angles[half + j], u = x[ia], v = x[ib];
        y[ia] = vm_from_float<T>(u * cs - v * sn);
        y[ib] = vm_from_float<T>(v * cs + u * sn);
    }
}

VM_API int vm_latent_direct(const float* proj, int ld, int H, int D, int R, int kv_rank, const float* wkv, float eps, void* q, void* q_far,
                            const int* positions, const int* seq_of_token, const int* block_table, int max_blocks, void* pages, int n_pages,
                            int rotary_dim, const float* inv_freq, int pairing, int T, int act_dtype, int* err, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (H <= 0 || D <= 0 || R < 0 || kv_rank <= 0 || ld < H * (D + R) + (pages ? kv_rank + R : 0)) return VM_ERR_BAD_ARG;
    if (rotary_dim < 0 || rotary_dim % 2 || rotary_dim > R || (rotary_dim > 0 && !inv_freq)) return VM_ERR_BAD_ARG;
    const int threads = H * (D + R) >= 1024 ? 256 : 128;
    const size_t smem = (size_t)rotary_dim * sizeof(float);
    if (smem > 40 * 1024) return VM_ERR_UNSUPPORTED;
    if (act_dtype == VM_F32)
        vm_launch_pdl(latent_direct_kernel<float>, dim3(T), dim3(threads), smem, stream, proj, ld, H, D, R, kv_rank, wkv, eps, (float*)q, (float*)q_far, positions,
                      seq_of_token, block_table, max_blocks, (float*)pages, n_pages, rotary_dim, inv_freq, pairing, err);
    else if (act_dtype == VM_BF16)
        vm_launch_pdl(latent_direct_kernel<__nv_bfloat16>, dim3(T), dim3(threads), smem, stream, proj, ld, H, D, R, kv_rank, wkv, eps, (__nv_bfloat16*)q,
                      (__nv_bfloat16*)q_far, positions, seq_of_token, block_table, max_blocks, (__nv_bfloat16*)pages, n_pages, rotary_dim, inv_freq, pairing, err);
    else return VM_ERR_UNSUPPORTED;
    return vm_launch_status();
}
