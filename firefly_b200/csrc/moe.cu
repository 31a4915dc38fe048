// Routed experts: the router's choice, the plan that sorts a step's tokens by expert, the
// grouped products over the experts' stacked matrices, and the weighted sum back into the
// 32-bit residual.  Nothing here is read by the host: counts, offsets and the list of row
// tiles stay on the device, and the grouped products are launched for the largest number of
// tiles a step of that many tokens can have (blocks past the real count leave at once), so a
// step with routed experts can be captured into a CUDA graph.
//
//   s = softmax(z) over all experts (32-bit).  Experts form `groups` equal groups of
//   neighbours; a group's score is its largest s; only experts of the `keep` best groups may
//   be chosen; of those the `top` with the largest s are; weights = s / (sum of chosen s + 1e-20).
//   expert(h) = W_down (g * sigmoid(1.702 g) * (u + 1)),  g = min(W_gate h, limit),
//   u = clamp(W_up h, -limit, limit).
// Other forms by parameter: SiLU experts, experts without a gate (W_down relu(W_up h)^2), and weights that multiply an
// expert's input instead of its output (applied to the first product's 32-bit result, which is linear in the input).
//
// A row of a grouped product is one (token, choice) pair; its result is a plain dot product
// per output in a fixed order over K, so it does not depend on which other rows share its tile.
#include "moe.cuh"
#include <math_constants.h>

namespace ff {

constexpr int MOE_BM = 64, MOE_BN = 64, MOE_BK = 16;

// (value, index) arg-max over a warp; the lowest index wins ties
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, i, o);
        if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
    }
}

// One warp per token; z + bias (bias may be null) are the logits.  score 0: s = softmax(z) over all experts; 1: s =
// sigmoid(z); 2: s = z, and the weights are the softmax over the chosen experts' logits alone.  The choice uses
// c = s + correction (correction may be null); a group's score is its largest c (group_score 0) or the sum of
// its two largest (1); experts of closed groups count as minus infinity (c may be negative); the weights are the
// chosen experts' s, divided by their sum (+ 1e-20) when `renorm`.  Ties go to the lowest index.
// z rows are z_stride floats apart (further columns may follow the experts' logits).
__global__ void moe_route_kernel(const float* z, int z_stride, const float* __restrict__ bias, const float* __restrict__ correction, int T, int E, int top,
                                 int groups, int keep, int score, int group_score, int renorm,
                                 int* __restrict__ ids, float* __restrict__ wts) {
    pdl_prologue();
    z = pdl_fresh(z);
    extern __shared__ float sh[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * (blockDim.x >> 5) + warp;
    if (t >= T) return;
    float* s = sh + (size_t)warp * (2 * E + 2 * groups);
    float* a = s + E;              // choice scores; minus infinity when closed or taken
    float* gs = a + E;
    float* g_open = gs + groups;
    const float* zr = z + (size_t)t * z_stride;
    float mx = -CUDART_INF_F;
    for (int e = lane; e < E; e += 32) {
        s[e] = zr[e] + (bias ? bias[e] : 0.f);
        mx = fmaxf(mx, s[e]);
    }
    if (score == 0) {
        mx = warp_max(mx);
        float sum = 0.f;
        for (int e = lane; e < E; e += 32) { const float p = expf(s[e] - mx); s[e] = p; sum += p; }
        sum = warp_sum(sum);
        __syncwarp();
        for (int e = lane; e < E; e += 32) s[e] = s[e] / sum;
    } else if (score == 1) {
        for (int e = lane; e < E; e += 32) s[e] = 1.0f / (1.0f + expf(-s[e]));
    }
    __syncwarp();
    const int per = E / groups;
    for (int g = lane; g < groups; g += 32) {
        float m1 = -CUDART_INF_F, m2 = -CUDART_INF_F;
        for (int e = g * per; e < (g + 1) * per; ++e) {
            const float c = s[e] + (correction ? correction[e] : 0.f);
            if (c > m1) { m2 = m1; m1 = c; } else if (c > m2) m2 = c;
        }
        gs[g] = (group_score == 1 && per > 1) ? m1 + m2 : m1;
        g_open[g] = 0.f;
    }
    __syncwarp();
    for (int k = 0; k < keep; ++k) {
        float bv = -CUDART_INF_F;
        int bi = 0x7fffffff;
        for (int g = lane; g < groups; g += 32)
            if (g_open[g] == 0.f && (bi == 0x7fffffff || gs[g] > bv)) { bv = gs[g]; bi = g; }
        warp_argmax(bv, bi);
        if (lane == 0 && bi < groups) g_open[bi] = 1.f;
        __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
        a[e] = g_open[e / per] != 0.f ? s[e] + (correction ? correction[e] : 0.f) : -CUDART_INF_F;
    __syncwarp();
    float total = 0.f, largest = -CUDART_INF_F;
    for (int k = 0; k < top; ++k) {
        float bv = -CUDART_INF_F;
        int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32)
            if (a[e] > bv) { bv = a[e]; bi = e; }
        warp_argmax(bv, bi);
        if (bi >= E) bi = 0;                   // cannot happen: top <= keep * per open experts with finite scores
        const float w = s[bi];
        total += w;
        largest = fmaxf(largest, w);
        if (lane == 0) { ids[(size_t)t * top + k] = bi; wts[(size_t)t * top + k] = w; a[bi] = -CUDART_INF_F; }
        __syncwarp();
    }
    if (score == 2) {
        total = 0.f;
        for (int k = lane; k < top; k += 32) total += expf(wts[(size_t)t * top + k] - largest);
        total = warp_sum(total);
        for (int k = lane; k < top; k += 32) wts[(size_t)t * top + k] = expf(wts[(size_t)t * top + k] - largest) / total;
    } else if (renorm) {
        const float inv = 1.0f / (total + 1e-20f);
        __syncwarp();
        for (int k = lane; k < top; k += 32) wts[(size_t)t * top + k] *= inv;
    }
}

// Rows sorted by expert, by one block or by a cluster of them (each takes a run of the entries; they share their counts
// through distributed shared memory).  seg[e] .. seg[e+1] are expert e's rows; row_of[entry] is the row of
// (token, choice) = entry; src_tok[row] its token; the row tiles of row_tile rows (64 for the plain grouped kernel, 128 for
// the tensor-core one) are listed as (expert, first row) with their count in n_tiles.
// `wts` (or null): row_w[row] becomes the weight of the row's (token, choice).
constexpr int PLAN_THREADS = 1024, PLAN_BLOCKS = 8, PLAN_U = 8;
__global__ void __launch_bounds__(PLAN_THREADS)
moe_plan_kernel(const int* ids, const float* wts, float* __restrict__ row_w, int entries, int top, int E, int row_tile, int* __restrict__ seg,
                int* __restrict__ row_of, int* __restrict__ src_tok, int* __restrict__ tile_expert, int* __restrict__ tile_row0,
                int* __restrict__ n_tiles) {
    pdl_prologue();
    ids = pdl_fresh(ids);
    wts = pdl_fresh(wts);
    extern __shared__ int shi[];
    int* counts = shi;                // of this block's entries
    int* total = shi + E;
    int* cursor = total + E;          // next free row of an expert for this block
    const int rank = blockIdx.z, blocks = gridDim.z, tid = threadIdx.x;
    const int per = (entries + blocks - 1) / blocks, lo = min(entries, rank * per), hi = min(entries, lo + per);
    for (int e = tid; e < E; e += PLAN_THREADS) counts[e] = 0;
    __syncthreads();
    for (int i0 = lo + tid; i0 < hi; i0 += PLAN_THREADS * PLAN_U) {       // several entries' loads in flight at once
        int e[PLAN_U];
#pragma unroll
        for (int u = 0; u < PLAN_U; ++u) e[u] = i0 + u * PLAN_THREADS < hi ? ids[i0 + u * PLAN_THREADS] : -1;
#pragma unroll
        for (int u = 0; u < PLAN_U; ++u)
            if (e[u] >= 0) atomicAdd(&counts[e[u]], 1);
    }
    __syncthreads();
    if (blocks > 1) cluster_sync_all();
    for (int e = tid; e < E; e += PLAN_THREADS) {
        int all = 0, before = 0;
        if (blocks > 1) {
            const uint32_t addr = (uint32_t)__cvta_generic_to_shared(counts + e);
            for (int r = 0; r < blocks; ++r) {
                const int c = __float_as_int(ld_peer_smem(addr, (uint32_t)r));
                if (r < rank) before += c;
                all += c;
            }
        } else {
            all = counts[e];
        }
        total[e] = all;
        cursor[e] = before;
    }
    __syncthreads();
    if (tid < 32) {                   // running sums over the experts: rows and row tiles
        int rows0 = 0, tiles0 = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + tid, c = e < E ? total[e] : 0, nt = (c + row_tile - 1) / row_tile;
            int rs = c, ts = nt;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int a = __shfl_up_sync(0xffffffffu, rs, o), b = __shfl_up_sync(0xffffffffu, ts, o);
                if (tid >= o) { rs += a; ts += b; }
            }
            const int first = rows0 + rs - c;
            if (e < E) {
                cursor[e] += first;
                if (rank == 0) {
                    seg[e] = first;
                    for (int k = 0, at = tiles0 + ts - nt; k < nt; ++k) { tile_expert[at + k] = e; tile_row0[at + k] = first + k * row_tile; }
                }
            }
            rows0 += __shfl_sync(0xffffffffu, rs, 31);
            tiles0 += __shfl_sync(0xffffffffu, ts, 31);
        }
        if (rank == 0 && tid == 0) { seg[E] = rows0; n_tiles[0] = tiles0; }
    }
    __syncthreads();
    for (int i0 = lo + tid; i0 < hi; i0 += PLAN_THREADS * PLAN_U) {
        int e[PLAN_U];
        float w[PLAN_U];
#pragma unroll
        for (int u = 0; u < PLAN_U; ++u) {
            const int i = i0 + u * PLAN_THREADS;
            e[u] = i < hi ? ids[i] : -1;
            w[u] = wts && i < hi ? wts[i] : 0.f;
        }
#pragma unroll
        for (int u = 0; u < PLAN_U; ++u) {
            if (e[u] < 0) continue;
            const int i = i0 + u * PLAN_THREADS, row = atomicAdd(&cursor[e[u]], 1);
            row_of[i] = row;
            src_tok[row] = i / top;
            if (wts) row_w[row] = w[u];
        }
    }
    if (blocks > 1) cluster_sync_all();      // a peer may still be reading this block's counts
}

// out rows = A rows x B[e]^T for the row tile's expert e.  B: [E, N, K] row-major.
// MOE_GATEUP: two B matrices (gate and up, [E, N, K] each), A rows gathered from x by src_tok, and
// out[row, n] = clamped_glu(gate, up) in type T.  MOE_UP: one B matrix, gathered rows, out = relu(up)^2 in type T.
// MOE_DOWN: A = rows of `a` in place, out 32-bit.  `row_w` (or null; not MOE_DOWN): a row's products are multiplied by
// row_w[row] in front of the activation, which is a weight on the expert's input.
template <typename T, int KIND>
__global__ void __launch_bounds__(256) moe_grouped_kernel(
    const T* a, const int* src_tok, const T* __restrict__ b0, const T* __restrict__ b1,
    const int* seg, const int* tile_expert, const int* tile_row0,
    const int* n_tiles, const float* row_w, void* __restrict__ out, int N, int K, float limit, int act) {
    constexpr bool GATEUP = KIND == MOE_GATEUP, GATHER = KIND != MOE_DOWN;
    pdl_prologue();
    a = pdl_fresh(a); src_tok = pdl_fresh(src_tok); seg = pdl_fresh(seg);       // made by the kernels in front
    row_w = pdl_fresh(row_w);
    tile_expert = pdl_fresh(tile_expert); tile_row0 = pdl_fresh(tile_row0); n_tiles = pdl_fresh(n_tiles);
    if ((int)blockIdx.y >= n_tiles[0]) return;
    __shared__ float As[MOE_BK][MOE_BM + 1];
    __shared__ float Bs[GATEUP ? 2 : 1][MOE_BK][MOE_BN + 1];
    __shared__ int s_src[MOE_BM];
    const int e = tile_expert[blockIdx.y], row0 = tile_row0[blockIdx.y];
    const int rows = min(MOE_BM, seg[e + 1] - row0);
    const int n0 = blockIdx.x * MOE_BN;
    const int tid = threadIdx.x, ty = tid >> 4, tx = tid & 15;
    if (tid < MOE_BM) s_src[tid] = tid < rows ? (GATHER ? src_tok[row0 + tid] : row0 + tid) : -1;
    __syncthreads();
    const T* B0 = b0 + (size_t)e * N * K;
    const T* B1 = GATEUP ? b1 + (size_t)e * N * K : nullptr;
    float acc0[4][4] = {}, acc1[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += MOE_BK) {
        for (int idx = tid; idx < MOE_BM * MOE_BK; idx += 256) {
            const int r = idx / MOE_BK, kk = idx - r * MOE_BK;
            const int src = s_src[r];
            As[kk][r] = (src >= 0 && k0 + kk < K) ? to_float(a[(size_t)src * K + k0 + kk]) : 0.f;
        }
        for (int idx = tid; idx < MOE_BN * MOE_BK; idx += 256) {
            const int n = idx / MOE_BK, kk = idx - n * MOE_BK;
            const bool ok = n0 + n < N && k0 + kk < K;
            Bs[0][kk][n] = ok ? to_float(B0[(size_t)(n0 + n) * K + k0 + kk]) : 0.f;
            if (GATEUP) Bs[1][kk][n] = ok ? to_float(B1[(size_t)(n0 + n) * K + k0 + kk]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < MOE_BK; ++kk) {
            float av[4], bv[4], cv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) av[i] = As[kk][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; ++j) { bv[j] = Bs[0][kk][tx * 4 + j]; if (GATEUP) cv[j] = Bs[1][kk][tx * 4 + j]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    acc0[i][j] += av[i] * bv[j];
                    if (GATEUP) acc1[i][j] += av[i] * cv[j];
                }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = ty * 4 + i;
        if (r >= rows) continue;
        const float wr = GATHER && row_w ? row_w[row0 + r] : 1.0f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= N) continue;
            if (GATEUP) ((T*)out)[(size_t)(row0 + r) * N + n] = from_float<T>(clamped_glu(acc0[i][j] * wr, acc1[i][j] * wr, limit, act));
            else if (KIND == MOE_UP) ((T*)out)[(size_t)(row0 + r) * N + n] = from_float<T>(relu2(acc0[i][j] * wr));
            else ((float*)out)[(size_t)(row0 + r) * N + n] = acc0[i][j];
        }
    }
}

// y[t, f] = clamped_glu(gu[t, f], gu[t, F + f])
template <typename T>
__global__ void clamped_glu_kernel(const T* gu, T* __restrict__ y, int F, float limit, size_t total) {
    pdl_prologue();
    gu = pdl_fresh(gu);
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= total) return;
    const size_t t = idx / F;
    const int f = (int)(idx - t * F);
    y[idx] = from_float<T>(clamped_glu(to_float(gu[t * 2 * F + f]), to_float(gu[t * 2 * F + F + f]), limit));
}

// The same for bfloat16 with F % 8 == 0 and 16-byte aligned rows: eight columns a thread and group, two groups in flight.
__global__ void clamped_glu_vec8_kernel(const bf16* gu, bf16* __restrict__ y, int F, float limit, size_t groups) {
    pdl_prologue();
    gu = pdl_fresh(gu);
    const size_t step = (size_t)gridDim.x * blockDim.x;
    const int per = F / 8;
    size_t idx[2] = {(size_t)blockIdx.x * blockDim.x + threadIdx.x, 0};
    idx[1] = idx[0] + step;
    uint4 g[2], u[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        if (idx[k] >= groups) continue;
        const size_t t = idx[k] / per;
        const bf16* row = gu + t * 2 * F + (idx[k] - t * per) * 8;
        g[k] = *reinterpret_cast<const uint4*>(row);
        u[k] = *reinterpret_cast<const uint4*>(row + F);
    }
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        if (idx[k] >= groups) continue;
        const bf16* a = reinterpret_cast<const bf16*>(&g[k]);
        const bf16* b = reinterpret_cast<const bf16*>(&u[k]);
        uint4 o;
        bf16* c = reinterpret_cast<bf16*>(&o);
#pragma unroll
        for (int j = 0; j < 8; ++j) c[j] = __float2bfloat16_rn(clamped_glu_fast(__bfloat162float(a[j]), __bfloat162float(b[j]), limit, 0));
        *reinterpret_cast<uint4*>(y + idx[k] * 8) = o;
    }
}

// residual[t,:] (+)= mult * (sum_k wts[t,k] * rows[row_of[t*top+k],:] + gate * shared[t,:]); wts null: the weights are
// in the rows already; shared_z (or null): gate = sigmoid(shared_z[t * z_stride]), else 1; add 0: the residual is written.
__global__ void moe_combine_kernel(float* __restrict__ residual, const float* rows,
                                   const int* row_of, const float* wts,
                                   const float* shared, const float* shared_z, int z_stride, float mult, int add, int top,
                                   int W) {
    pdl_prologue();
    rows = pdl_fresh(rows); row_of = pdl_fresh(row_of); wts = pdl_fresh(wts); shared = pdl_fresh(shared);
    shared_z = pdl_fresh(shared_z);
    const int t = blockIdx.x;
    const float gate = shared_z ? 1.0f / (1.0f + expf(-shared_z[(size_t)t * z_stride])) : 1.0f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        float acc = 0.f;
        for (int k = 0; k < top; ++k)
            acc += (wts ? wts[(size_t)t * top + k] : 1.0f) * rows[(size_t)row_of[(size_t)t * top + k] * W + i];
        if (shared) acc += gate * shared[(size_t)t * W + i];
        residual[(size_t)t * W + i] = (add ? residual[(size_t)t * W + i] : 0.f) + mult * acc;
    }
}

}  // namespace ff

using namespace ff;

// rows of a row tile: of the tensor-core kernel (bfloat16, K % 8 == 0) or of the plain one
FF_EXPORT int ff_moe_row_tile(int tensor_cores) { return tensor_cores ? GROUPED_TC_ROWS : MOE_BM; }

FF_EXPORT int ff_moe_route(const float* z, int z_stride, const float* bias, const float* correction, int T, int E, int top, int groups, int keep,
                           int score, int group_score, int renorm, int* ids, float* wts, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (E <= 0 || z_stride < E || top <= 0 || top > E || groups <= 0 || E % groups || keep <= 0 || keep > groups ||
        top > keep * (E / groups))
        return FF_ERR_BAD_ARG;
    const int warps = 4;
    const size_t smem = (size_t)warps * (2 * E + 2 * groups) * sizeof(float);
    if (smem > 48 * 1024) return FF_ERR_UNSUPPORTED;
    FF_LAUNCH(moe_route_kernel, (T + warps - 1) / warps, warps * 32, smem, stream, z, z_stride, bias, correction, T, E, top, groups, keep, score,
              group_score, renorm, ids, wts);
    FF_LAUNCH_CHECK();
    return 0;
}

FF_EXPORT int ff_moe_plan(const int* ids, const float* wts, float* row_w, int entries, int top, int E, int row_tile, int* seg, int* row_of,
                          int* src_tok, int* tile_expert, int* tile_row0, int* n_tiles, cudaStream_t stream) {
    if (entries <= 0) return 0;
    if ((row_tile != MOE_BM && row_tile != GROUPED_TC_ROWS) || (wts && !row_w)) return FF_ERR_BAD_ARG;
    const size_t smem = (size_t)3 * E * sizeof(int);
    if (smem > 48 * 1024) return FF_ERR_UNSUPPORTED;
    const int blocks = entries >= 4096 ? PLAN_BLOCKS : 1;
    const int rc = launch_kernel_cluster(moe_plan_kernel, dim3(1, 1, blocks), dim3(PLAN_THREADS), smem, stream, blocks, ids, wts, row_w,
                                         entries, top, E, row_tile, seg, row_of, src_tok, tile_expert, tile_row0, n_tiles);
    if (rc) return rc;
    FF_LAUNCH_CHECK();
    return 0;
}

FF_EXPORT int ff_moe_grouped(const void* a, const int* src_tok, const void* b0, const void* b1, int dtype, int kind,
                             const int* seg, const int* tile_expert, const int* tile_row0, const int* n_tiles,
                             const float* row_w, void* out, int max_tiles, int N, int K, float limit, int act,
                             cudaStream_t stream) {
    if (max_tiles <= 0) return 0;
    if (kind < MOE_DOWN || kind > MOE_UP || (kind == MOE_GATEUP && !b1)) return FF_ERR_BAD_ARG;
    dim3 grid((N + MOE_BN - 1) / MOE_BN, max_tiles);
#define FF_MOE(T, KIND)                                                                                            \
    FF_LAUNCH((moe_grouped_kernel<T, KIND>), grid, 256, 0, stream, (const T*)a, src_tok, (const T*)b0, (const T*)b1, seg, \
              tile_expert, tile_row0, n_tiles, row_w, out, N, K, limit, act)
#define FF_MOE_KIND(T)                                                                                             \
    do {                                                                                                           \
        if (kind == MOE_GATEUP) FF_MOE(T, MOE_GATEUP);                                                             \
        else if (kind == MOE_UP) FF_MOE(T, MOE_UP);                                                                \
        else FF_MOE(T, MOE_DOWN);                                                                                  \
    } while (0)
    if (dtype == 0) FF_MOE_KIND(float);
    else if (dtype == 1) FF_MOE_KIND(bf16);
    else return FF_ERR_BAD_ARG;
#undef FF_MOE_KIND
#undef FF_MOE
    FF_LAUNCH_CHECK();
    return 0;
}

FF_EXPORT int ff_clamped_glu(const void* gu, void* y, int dtype, int T, int F, float limit, cudaStream_t stream) {
    const size_t total = (size_t)T * F;
    if (total == 0) return 0;
    if (dtype == 1 && F % 8 == 0 && (((uintptr_t)gu | (uintptr_t)y) & 15) == 0) {
        const size_t groups = total / 8;
        FF_LAUNCH(clamped_glu_vec8_kernel, (unsigned)((groups + 511) / 512), 256, 0, stream, (const bf16*)gu, (bf16*)y, F, limit, groups);
        FF_LAUNCH_CHECK();
        return 0;
    }
    const unsigned blocks = (unsigned)((total + 255) / 256);
    if (dtype == 0) FF_LAUNCH((clamped_glu_kernel<float>), blocks, 256, 0, stream, (const float*)gu, (float*)y, F, limit, total);
    else if (dtype == 1) FF_LAUNCH((clamped_glu_kernel<bf16>), blocks, 256, 0, stream, (const bf16*)gu, (bf16*)y, F, limit, total);
    else return FF_ERR_BAD_ARG;
    FF_LAUNCH_CHECK();
    return 0;
}

FF_EXPORT int ff_moe_combine(float* residual, const float* rows, const int* row_of, const float* wts,
                             const float* shared, const float* shared_z, int z_stride, float mult, int add, int T,
                             int top, int W, cudaStream_t stream) {
    if (T <= 0) return 0;
    FF_LAUNCH(moe_combine_kernel, T, W >= 1024 ? 256 : 128, 0, stream, residual, rows, row_of, wts, shared,
              shared_z, z_stride, mult, add, top, W);
    FF_LAUNCH_CHECK();
    return 0;
}
