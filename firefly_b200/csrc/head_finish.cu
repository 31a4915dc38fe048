// Finishing a step's query and key heads from the raw projection, and writing keys and values into the paged cache.
//
// In the order in which they are applied, each of them optional:
//   `bias`         (float [(nq + 2 nkv) d] in the row's layout) added to q, k and v in 32-bit;
//   `q_w`, `k_w`   (float [d]) an RMS norm of every q / k head over its `norm_dim` elements with this weight; with
//                  `norm_all` (float [nq d] / [nkv d]) one norm over all q heads together and one over all k heads, each head
//                  counting `norm_dim` elements;
//   rotation       of the first `rdims` elements of every q and k head (pairs (i, i + rdims/2), or (2i, 2i + 1) with
//                  `interleaved`; angle = position * f_i, cos and sin times `mag`);
//   `normalize`    q and k divided by their root mean square over `norm_dim` elements (no weight);
//   temperature    q times 1 + temp_coef ln(floor((position + 1) / temp_every) + 1)   (temp_every 0: none).
// q goes back in place, k and v into their page.  `value_is_key`: a row is q heads | k heads only, and the value is the
// key as projected (before its norm).
//
// The frequencies come as a 64-bit table (a scaled rotation changes the table, not this kernel); the angle is
// formed and reduced in double, so cos and sin are right to 32-bit rounding at any position.  Heads are laid out
// with `d` elements each; a head whose true size is smaller than d has zeros behind it (its matrix rows are zero), so
// sums over d are sums over the head.
#include "common.cuh"

namespace ff {

struct HeadFinish {
    int width, nq, nkv, d, norm_dim;
    float eps;
    const double* freq;
    int rdims;
    float mag;
    const int* positions;
    const int* token_seq;
    const int* block_table;
    int max_blocks, block_size, num_blocks;
    int* status;
    int interleaved, normalize;
    const float* bias;
    const float* q_w;
    const float* k_w;
    float temp_coef;
    int temp_every;
    int value_is_key;
    int T;
    int norm_all;
};

// Any type and size: one block a token, one warp a head.
template <typename T>
__global__ void head_finish_kernel(T* __restrict__ qkv, T* __restrict__ cache /*[blocks, 2, nkv, block, d]*/, HeadFinish A) {
    pdl_prologue();
    extern __shared__ float sh[];           // cos[half], sin[half], then one head of d floats per warp
    const int t = blockIdx.x, d = A.d, nq = A.nq, nkv = A.nkv, rdims = A.rdims;
    const int half = rdims / 2;
    const int pos = A.positions[t];
    float* s_cos = sh;
    float* s_sin = sh + half;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        double sn, cs;
        sincos((double)pos * A.freq[i], &sn, &cs);
        s_cos[i] = (float)cs * A.mag;
        s_sin[i] = (float)sn * A.mag;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    float* hbuf = sh + 2 * half + (size_t)warp * d;
    T* row = qkv + (size_t)t * A.width;
    T* krow = nullptr;
    T* vrow = nullptr;
    if (nkv > 0) {
        const int page = pos >= 0 && pos / A.block_size < A.max_blocks
                             ? A.block_table[(size_t)A.token_seq[t] * A.max_blocks + pos / A.block_size] : -1;
        if (page < 0 || page >= A.num_blocks) {
            if (threadIdx.x == 0) atomicExch(A.status, 2);
        } else {
            krow = cache + (((size_t)page * 2) * nkv * A.block_size + pos % A.block_size) * d;
            vrow = krow + (size_t)nkv * A.block_size * d;
        }
    }
    const float temp = A.temp_every > 0 ? query_temperature(pos, A.temp_coef, A.temp_every) : 1.0f;
    const int heads = nq + (A.value_is_key ? nkv : 2 * nkv);
    float inv_q = 1.f, inv_k = 1.f;          // norm_all: 1 / root mean square of all q heads, of all k heads
    if (A.norm_all) {
        __shared__ float scratch[32];
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x; i < (nq + nkv) * d; i += blockDim.x) {
            const float v = to_float(row[i]) + (A.bias ? A.bias[i] : 0.f);
            if (i < nq * d) sq += v * v;
            else sk += v * v;
        }
        inv_q = 1.0f / sqrtf(block_sum(sq, scratch) / (float)(nq * A.norm_dim) + A.eps);
        if (nkv > 0) inv_k = 1.0f / sqrtf(block_sum(sk, scratch) / (float)(nkv * A.norm_dim) + A.eps);
        __syncthreads();                     // q is rewritten in place below
    }
    for (int h = warp; h < heads; h += nwarps) {
        T* src = row + (size_t)h * d;
        const float* brow = A.bias ? A.bias + (size_t)h * d : nullptr;
        const bool is_k = h >= nq && h < nq + nkv;
        if (h >= nq + nkv || (is_k && A.value_is_key)) {     // a value: copied as it is (plus its bias)
            if (vrow) {
                T* dst = vrow + (size_t)(h - nq - (is_k ? 0 : nkv)) * A.block_size * d;
                if (brow)
                    for (int i = lane; i < d; i += 32) dst[i] = from_float<T>(to_float(src[i]) + brow[i]);
                else
                    for (int i = lane; i < d; i += 32) dst[i] = src[i];
            }
            if (!is_k) continue;
        }
        const float* w = is_k ? A.k_w : A.q_w;
        float ss = 0.f;
        for (int i = lane; i < d; i += 32) {
            const float v = to_float(src[i]) + (brow ? brow[i] : 0.f);
            hbuf[i] = v;
            ss += v * v;
        }
        if (w) {
            const float inv = A.norm_all ? (is_k ? inv_k : inv_q) : 1.0f / sqrtf(warp_sum(ss) / (float)A.norm_dim + A.eps);
            if (A.norm_all) w += (size_t)(is_k ? h - nq : h) * d;
            for (int i = lane; i < d; i += 32) hbuf[i] = hbuf[i] * inv * w[i];
        }
        __syncwarp();
        // element i after the rotation: its partner and the sign of the sine term depend on the pairing
        auto turned = [&](int i) -> float {
            float v = hbuf[i];
            if (i >= rdims) return v;
            if (A.interleaved) {
                const int f = i >> 1;
                return (i & 1) ? v * s_cos[f] + hbuf[i - 1] * s_sin[f] : v * s_cos[f] - hbuf[i + 1] * s_sin[f];
            }
            return i < half ? v * s_cos[i] - hbuf[i + half] * s_sin[i] : v * s_cos[i - half] + hbuf[i - half] * s_sin[i - half];
        };
        float inv = 1.0f;
        if (A.normalize) {
            float sr = 0.f;
            for (int i = lane; i < d; i += 32) { const float v = turned(i); sr += v * v; }
            sr = warp_sum(sr);
            inv = 1.0f / sqrtf(sr / (float)A.norm_dim + A.eps);
        }
        if (!is_k) inv *= temp;
        T* dst = is_k ? (krow ? krow + (size_t)(h - nq) * A.block_size * d : nullptr) : src;
        if (dst)
            for (int i = lane; i < d; i += 32) dst[i] = from_float<T>(turned(i) * inv);
        __syncwarp();
    }
}

// The same for bfloat16 with sizes in steps of 8 and 16-byte aligned rows.  A lane holds eight neighbouring elements
// of a head, P (a power of two, >= d / 8) lanes a head, 32 / P heads a warp and pass; a pair's other half comes from
// the lane that holds it, sums over a head are shuffles inside its P lanes.  A block takes HFV_TOK tokens (their
// angles in shared memory) and its warps the heads of all of them, HFV_U passes with their loads in flight together.
constexpr int HFV_TOK = 4, HFV_THREADS = 256, HFV_U = 4;

template <int P, bool ALL>
__global__ void __launch_bounds__(HFV_THREADS) head_finish_vec_kernel(bf16* __restrict__ qkv, bf16* __restrict__ cache, HeadFinish A) {
    extern __shared__ float sh[];                             // [HFV_TOK][2][half]
    __shared__ int s_page[HFV_TOK];
    __shared__ float s_temp[HFV_TOK];
    __shared__ float s_part[HFV_TOK][2][2], s_inv[HFV_TOK][2];
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int t0 = blockIdx.x * HFV_TOK, nt = min(HFV_TOK, A.T - t0);
    const int d = A.d, nq = A.nq, nkv = A.nkv, half = A.rdims / 2;
    // positions, pages and angles do not depend on the kernel in front
    for (int idx = threadIdx.x; idx < nt * half; idx += HFV_THREADS) {
        const int u = idx / half, i = idx - u * half;
        double sn, cs;
        sincos((double)A.positions[t0 + u] * A.freq[i], &sn, &cs);
        sh[(u * 2) * half + i] = (float)cs * A.mag;
        sh[(u * 2 + 1) * half + i] = (float)sn * A.mag;
    }
    if ((int)threadIdx.x < nt) {
        const int t = t0 + threadIdx.x, pos = A.positions[t];
        s_temp[threadIdx.x] = A.temp_every > 0 ? query_temperature(pos, A.temp_coef, A.temp_every) : 1.0f;
        int page = -1;
        if (nkv > 0 && pos >= 0 && pos / A.block_size < A.max_blocks)
            page = A.block_table[(size_t)A.token_seq[t] * A.max_blocks + pos / A.block_size];
        if (page >= A.num_blocks) page = -1;
        s_page[threadIdx.x] = page;
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    __syncthreads();
    if (nkv > 0 && (int)threadIdx.x < nt && s_page[threadIdx.x] < 0) atomicExch(A.status, 2);
    constexpr int HPW = 32 / P;                               // heads a warp takes in one pass
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = HFV_THREADS / 32;
    const int sub = lane % P, e0 = sub * 8;
    const bool in_head = e0 < d;
    const int heads = nq + (A.value_is_key ? nkv : 2 * nkv);
    const int items = nt * heads;                             // (token, head) pairs of the block
    const int passes = (items + HPW - 1) / HPW;
    const bool turns = e0 < A.rdims;
    if constexpr (ALL) {
        // sums over all q heads and over all k heads: two warps a token, each every other group of 32 x 8 elements; the
        // rows are read again below (from the cache then)
        static_assert(HFV_TOK * 2 == HFV_THREADS / 32, "two warps a token");
        const int tl = warp >> 1, part = warp & 1;
        float s[2] = {0.f, 0.f};
        if (tl < nt) {
            const bf16* row = qkv + (size_t)(t0 + tl) * A.width;
            const int nq8 = nq * d / 8, all8 = (nq + nkv) * d / 8;
#pragma unroll 4
            for (int c = part * 32 + lane; c < all8; c += 64) {
                const uint4 raw = *reinterpret_cast<const uint4*>(row + (size_t)c * 8);
                const bf16* rb = reinterpret_cast<const bf16*>(&raw);
                float ss = 0.f;
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const float v = __bfloat162float(rb[j]) + (A.bias ? A.bias[c * 8 + j] : 0.f);
                    ss += v * v;
                }
                if (c < nq8) s[0] += ss;
                else s[1] += ss;
            }
        }
        s[0] = warp_sum(s[0]);
        s[1] = warp_sum(s[1]);
        if (lane == 0) { s_part[tl][part][0] = s[0]; s_part[tl][part][1] = s[1]; }
        __syncthreads();
        if ((int)threadIdx.x < HFV_TOK * 2) {
            const int u = threadIdx.x >> 1, kind = threadIdx.x & 1, n = (kind ? nkv : nq) * A.norm_dim;
            s_inv[u][kind] = 1.0f / sqrtf((s_part[u][0][kind] + s_part[u][1][kind]) / (float)max(n, 1) + A.eps);
        }
        __syncthreads();
    }
    const int hl = half / 8;                                  // lanes a half of the rotated elements takes
    const bool upper = turns && !A.interleaved && e0 >= half;
    for (int p0 = warp; p0 < passes; p0 += nwarps * HFV_U) {
        uint4 raw[HFV_U];
#pragma unroll
        for (int u = 0; u < HFV_U; ++u) {
            const int item = (p0 + u * nwarps) * HPW + lane / P;
            raw[u] = make_uint4(0u, 0u, 0u, 0u);
            if (item < items && in_head)
                raw[u] = *reinterpret_cast<const uint4*>(qkv + (size_t)(t0 + item / heads) * A.width + (size_t)(item % heads) * d + e0);
        }
#pragma unroll
        for (int u = 0; u < HFV_U; ++u) {
            if (p0 + u * nwarps >= passes) break;             // the same for the whole warp
            const int item = (p0 + u * nwarps) * HPW + lane / P;
            const bool live = item < items && in_head;
            const int tl = item < items ? item / heads : 0, h = item < items ? item % heads : 0;
            const bool is_k = h >= nq && h < nq + nkv, is_v = h >= nq + nkv;
            float v[8];
            const bf16* rb = reinterpret_cast<const bf16*>(&raw[u]);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = __bfloat162float(rb[j]);
            if (A.bias && live) {
                const float* b = A.bias + (size_t)h * d + e0;
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] += b[j];
            }
            const int pos = A.positions[t0 + tl];
            const int page = s_page[tl];
            bf16* krow = nkv > 0 && page >= 0 ? cache + (((size_t)page * 2) * nkv * A.block_size + pos % A.block_size) * d : nullptr;
            auto put = [&](bf16* dst) {
                uint4 ov;
                bf16* o = reinterpret_cast<bf16*>(&ov);
#pragma unroll
                for (int j = 0; j < 8; ++j) o[j] = __float2bfloat16_rn(v[j]);
                *reinterpret_cast<uint4*>(dst + e0) = ov;
            };
            if (live && krow && (is_v || (is_k && A.value_is_key)))
                put(krow + (size_t)(nkv + h - nq - (is_v ? nkv : 0)) * A.block_size * d);
            // values stay in the shuffles below with the rest of their warp
            const float* w = is_v ? nullptr : (is_k ? A.k_w : A.q_w);
            if constexpr (ALL) {
                if (w && live) {
                    const float inv = s_inv[tl][is_k ? 1 : 0];
                    const float4* wh = reinterpret_cast<const float4*>(w + (size_t)(is_k ? h - nq : h) * d + e0);
                    const float4 w0 = wh[0], w1 = wh[1];
                    v[0] *= inv * w0.x; v[1] *= inv * w0.y; v[2] *= inv * w0.z; v[3] *= inv * w0.w;
                    v[4] *= inv * w1.x; v[5] *= inv * w1.y; v[6] *= inv * w1.z; v[7] *= inv * w1.w;
                }
            } else if (A.q_w || A.k_w) {
                float ss = 0.f;
#pragma unroll
                for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
#pragma unroll
                for (int o = P / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
                if (w && live) {
                    const float inv = 1.0f / sqrtf(ss / (float)A.norm_dim + A.eps);
#pragma unroll
                    for (int j = 0; j < 8; ++j) v[j] = v[j] * inv * w[e0 + j];
                }
            }
            if (half > 0) {
                const float* cs = sh + (tl * 2) * half;
                const float* sn = cs + half;
                if (A.interleaved) {
                    if (turns) {
#pragma unroll
                        for (int j = 0; j < 8; j += 2) {
                            const float a = v[j], b = v[j + 1], c = cs[e0 / 2 + j / 2], s = sn[e0 / 2 + j / 2];
                            v[j] = a * c - b * s;
                            v[j + 1] = b * c + a * s;
                        }
                    }
                } else {
                    const int other = turns ? (upper ? lane - hl : lane + hl) : lane;
                    const int f0 = upper ? e0 - half : e0;
#pragma unroll
                    for (int j = 0; j < 8; ++j) {
                        const float b = __shfl_sync(0xffffffffu, v[j], other);
                        if (turns) v[j] = upper ? v[j] * cs[f0 + j] + b * sn[f0 + j] : v[j] * cs[f0 + j] - b * sn[f0 + j];
                    }
                }
            }
            float mul = is_k || is_v ? 1.0f : s_temp[tl];
            if (A.normalize) {
                float ss = 0.f;
#pragma unroll
                for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
#pragma unroll
                for (int o = P / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
                mul *= 1.0f / sqrtf(ss / (float)A.norm_dim + A.eps);
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] *= mul;
            if (live && !is_v) {
                if (!is_k) put(qkv + (size_t)(t0 + tl) * A.width + (size_t)h * d);
                else if (krow) put(krow + (size_t)(h - nq) * A.block_size * d);
            }
        }
    }
}

}  // namespace ff

using namespace ff;

FF_EXPORT int ff_head_finish(void* qkv, int dtype, int width, int T, int nq, int nkv, int d, int norm_dim, float eps,
                             const double* freq, int rdims, float mag, const int* positions, const int* token_seq,
                             const int* block_table, int max_blocks, int block_size, int num_blocks, void* cache,
                             int* status, int interleaved, int normalize, const float* bias, const float* q_w,
                             const float* k_w, float temp_coef, int temp_every, int value_is_key, int norm_all, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (rdims < 0 || rdims % 2 || rdims > d || norm_dim <= 0 || norm_dim > d || d > 1024) return FF_ERR_BAD_ARG;
    const int heads = nq + (value_is_key ? nkv : 2 * nkv);
    if (width < heads * d || (norm_all && (!q_w || (nkv > 0 && !k_w)))) return FF_ERR_BAD_ARG;
    HeadFinish A{width, nq, nkv, d, norm_dim, eps, freq, rdims, mag, positions, token_seq, block_table, max_blocks, block_size,
                 num_blocks, status, interleaved, normalize, bias, q_w, k_w, temp_coef, temp_every, value_is_key, T, norm_all};
    const bool pairs_fit = rdims % 8 == 0 && (interleaved || (rdims / 2) % 8 == 0);
    if (dtype == 1 && d % 8 == 0 && d <= 256 && width % 8 == 0 && pairs_fit && (((uintptr_t)qkv | (uintptr_t)cache) & 15) == 0 &&
        (!norm_all || (((uintptr_t)q_w | (uintptr_t)k_w) & 15) == 0)) {
        const size_t smem = (size_t)HFV_TOK * rdims * sizeof(float);
        const unsigned blocks = (unsigned)((T + HFV_TOK - 1) / HFV_TOK);
#define FF_HFV(P)                                                                                                       \
    do {                                                                                                                \
        if (norm_all) FF_LAUNCH((head_finish_vec_kernel<P, true>), blocks, HFV_THREADS, smem, stream, (bf16*)qkv, (bf16*)cache, A); \
        else FF_LAUNCH((head_finish_vec_kernel<P, false>), blocks, HFV_THREADS, smem, stream, (bf16*)qkv, (bf16*)cache, A); \
    } while (0)
        if (d <= 32) FF_HFV(4);
        else if (d <= 64) FF_HFV(8);
        else if (d <= 128) FF_HFV(16);
        else FF_HFV(32);
#undef FF_HFV
        FF_LAUNCH_CHECK();
        return 0;
    }
    const int threads = heads >= 4 ? 128 : 32 * (heads > 0 ? heads : 1);
    const size_t smem = ((size_t)rdims + (size_t)(threads / 32) * d) * sizeof(float);
    if (dtype == 0) FF_LAUNCH((head_finish_kernel<float>), T, threads, smem, stream, (float*)qkv, (float*)cache, A);
    else if (dtype == 1) FF_LAUNCH((head_finish_kernel<bf16>), T, threads, smem, stream, (bf16*)qkv, (bf16*)cache, A);
    else return FF_ERR_BAD_ARG;
    FF_LAUNCH_CHECK();
    return 0;
}
