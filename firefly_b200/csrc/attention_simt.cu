// Plain attention over the paged cache: one block per (query token, q head), scalar
// 32-bit arithmetic throughout.  It serves the true 32-bit path and stands beside
// the tensor-core kernel as its reference.  Any head size up to 512, any block
// size, any group size; prefill portions and decode tokens alike, since every
// query is described only by its sequence and absolute position.
//
// Formula as in the reference's decode kernel (src/kernels/attention.cu:291-447):
// s_j = (q.k_j)/sqrt(d) in 32-bit, running max and sum, o = sum p_j v_j / l, q head
// h reading kv head h / (nq/nkv) (:304).  Unlike the reference's prefill kernel
// (:173, mask on indices local to the portion) keys are taken from the cache by
// absolute position, 0..pos, or the last `window` of them.
//
// A bias by distance may be taken off the scores: `dist_bias` [nq, bias_len] floats, entry (h, i - j) for query
// position i and key position j (null: none).  The caller makes the table as long as the window, so every
// visible key has an entry; a key further away than the table counts as masked.
//
// A warp takes every 4th key starting at the first visible one, so the order of
// additions for a query depends only on its position and window, never on how the
// tokens were cut into steps or what else is in the batch.
#include "common.cuh"
#include <math_constants.h>

// Planes of a cache page: 2 (keys, then values) or, compiled with -DFF_KV_PLANES=1, one plane whose rows are
// keys and values at once (a mixer that caches one vector per token and reads values from its key rows).
#ifndef FF_KV_PLANES
#define FF_KV_PLANES 2
#endif

namespace ff {

constexpr int ATT_WARPS = 4;
constexpr int ATT_MAX_D = 512;
constexpr int ATT_PER_LANE = ATT_MAX_D / 32;

template <typename T>
__global__ void paged_attention_simt_kernel(
    const T* q, int q_stride, const T* cache,
    const int* __restrict__ block_table, int max_blocks, const int* __restrict__ token_seq,
    const int* __restrict__ positions, T* __restrict__ out, int out_stride, int nq, int nkv, int d,
    int block_size, int num_blocks, float scale, int window, const float* __restrict__ dist_bias, int bias_len,
    float softcap, const float* __restrict__ sink, int* __restrict__ status) {
    pdl_prologue();
    q = pdl_fresh(q);              // the kernel in front writes the finished heads and this step's cache rows
    cache = pdl_fresh(cache);
    __shared__ float s_m[ATT_WARPS], s_l[ATT_WARPS];
    __shared__ float s_acc[ATT_WARPS][ATT_MAX_D];
    const int t = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int kh = h / (nq / nkv);
    const int seq = token_seq[t], pos = positions[t];
    int kv_begin = first_visible_key(pos, window);
    const int kv_end = pos + 1;
    const float* bias_row = dist_bias ? dist_bias + (size_t)h * bias_len : nullptr;
    if (bias_row && kv_begin < pos - bias_len + 1) kv_begin = pos - bias_len + 1;

    float qr[ATT_PER_LANE], acc[ATT_PER_LANE];
    const T* qrow = q + (size_t)t * q_stride + (size_t)h * d;
#pragma unroll
    for (int jj = 0; jj < ATT_PER_LANE; ++jj) {
        const int i = lane + 32 * jj;
        qr[jj] = i < d ? to_float(qrow[i]) : 0.f;
        acc[jj] = 0.f;
    }
    // a sink (one more entry in the head's denominator, of this score and without a value) is taken in by the first warp
    float m = sink && warp == 0 ? sink[h] : -CUDART_INF_F, l = sink && warp == 0 ? 1.f : 0.f;
    const int* bt = block_table + (size_t)seq * max_blocks;
    for (int j = kv_begin + warp; j < kv_end; j += ATT_WARPS) {
        const int page = bt[j / block_size];
        if (page < 0 || page >= num_blocks) {
            if (lane == 0) atomicExch(status, 4);
            break;
        }
        const T* krow = cache + ((((size_t)page * FF_KV_PLANES) * nkv + kh) * block_size + j % block_size) * d;
        const T* vrow = krow + (size_t)(FF_KV_PLANES - 1) * nkv * block_size * d;
        float part = 0.f;
#pragma unroll
        for (int jj = 0; jj < ATT_PER_LANE; ++jj) {
            const int i = lane + 32 * jj;
            if (i < d) part += qr[jj] * to_float(krow[i]);
        }
        float s = warp_sum(part) * scale;
        if (softcap != 0.f) s = softcap * tanhf(s / softcap);      // a cap on the scaled score
        if (bias_row) s -= bias_row[pos - j];
        const float m_new = fmaxf(m, s);
        const float corr = expf(m - m_new);
        const float p = expf(s - m_new);
        l = l * corr + p;
#pragma unroll
        for (int jj = 0; jj < ATT_PER_LANE; ++jj) {
            const int i = lane + 32 * jj;
            if (i < d) acc[jj] = acc[jj] * corr + p * to_float(vrow[i]);
        }
        m = m_new;
    }
    if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
#pragma unroll
    for (int jj = 0; jj < ATT_PER_LANE; ++jj) {
        const int i = lane + 32 * jj;
        if (i < d) s_acc[warp][i] = acc[jj];
    }
    __syncthreads();
    float M = s_m[0];
#pragma unroll
    for (int w = 1; w < ATT_WARPS; ++w) M = fmaxf(M, s_m[w]);
    float wgt[ATT_WARPS], L = 0.f;
#pragma unroll
    for (int w = 0; w < ATT_WARPS; ++w) {
        wgt[w] = s_m[w] == -CUDART_INF_F ? 0.f : expf(s_m[w] - M);
        L += wgt[w] * s_l[w];
    }
    T* orow = out + (size_t)t * out_stride + (size_t)h * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < ATT_WARPS; ++w) o += wgt[w] * s_acc[w][i];
        orow[i] = from_float<T>(o / L);
    }
}

}  // namespace ff

using namespace ff;

FF_EXPORT int ff_paged_attention_simt(const void* q, int dtype, int q_stride, const void* cache,
                                      const int* block_table, int max_blocks, const int* token_seq,
                                      const int* positions, void* out, int out_stride, int T, int nq,
                                      int nkv, int d, int block_size, int num_blocks, float scale,
                                      int window, const float* dist_bias, int bias_len, float softcap, const float* sink, int* status,
                                      cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || d > ATT_MAX_D) return FF_ERR_UNSUPPORTED;
    if (nkv <= 0 || nq % nkv || (dist_bias && bias_len <= 0)) return FF_ERR_BAD_ARG;
    dim3 grid(T, nq);
    if (dtype == 0)
        FF_LAUNCH((paged_attention_simt_kernel<float>), grid, ATT_WARPS * 32, 0, stream, 
            (const float*)q, q_stride, (const float*)cache, block_table, max_blocks, token_seq,
            positions, (float*)out, out_stride, nq, nkv, d, block_size, num_blocks, scale, window, dist_bias, bias_len, softcap, sink, status);
    else if (dtype == 1)
        FF_LAUNCH((paged_attention_simt_kernel<bf16>), grid, ATT_WARPS * 32, 0, stream, 
            (const bf16*)q, q_stride, (const bf16*)cache, block_table, max_blocks, token_seq,
            positions, (bf16*)out, out_stride, nq, nkv, d, block_size, num_blocks, scale, window, dist_bias, bias_len, softcap, sink, status);
    else
        return FF_ERR_BAD_ARG;
    FF_LAUNCH_CHECK();
    return 0;
}
