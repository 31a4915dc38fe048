// The seam between two parts of a model whose residual is several streams side by side (hyper-connections), in one pass
// over a token's rows.  With the S streams x_1 .. x_S in front of it:
//
//   x_t  <- sum_s mix[s, t] x_s + out_w[t] y       what the part in front adds, all streams at once from the old ones
//   u     = sum_s in_w[s] x_s                      what the next part reads (in_w null: the plain sum)
//   out   = norm(u)                                (u - mean) / sqrt(var + eps) * w + b with `center`, else
//                                                  u / sqrt(mean(u^2) + eps) * w (+ b);  w null: out = u
//
// y is a tensor, or the weighted sum of a token's rows of a grouped product (routed experts) plus a shared row, formed
// here; or there is none yet (the first part of a model), and only u and the norm are formed.  `same`: src is one row a
// token, and every stream equals it (the embedding output).  dst null: the new streams are used for u and not kept.
// Everything is 32-bit; y may be bfloat16, out is in the activation type.
#include "common.cuh"

namespace ff {

enum { Y_NONE = 0, Y_FLOAT = 1, Y_BF16 = 2, Y_ROUTED = 3 };
constexpr int SEAM_MAX_STREAMS = 32;        // of the form for any number of streams
constexpr int SEAM_FIXED_STREAMS = 8;       // up to here a build of its own for each number

struct SeamArgs {
    const float* src;
    float* dst;
    const void* y;
    const float* rows;
    const int* row_of;
    const float* wts;
    const float* shared;
    const float* mix;
    const float* out_w;
    const float* in_w;
    const float* w;
    const float* b;
    float eps;
    int center;
    void* out;
    const int* row_idx;
    int W, kind, top, same, out_bf16;
    int n_in;                  // numbers in in_w
};

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(bf16* p, float4 v) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}
__device__ __forceinline__ float4 zero4() { return make_float4(0.f, 0.f, 0.f, 0.f); }
__device__ __forceinline__ void add4(float4& a, float c, float4 v) {
    a.x = fmaf(c, v.x, a.x); a.y = fmaf(c, v.y, a.y); a.z = fmaf(c, v.z, a.z); a.w = fmaf(c, v.w, a.w);
}

// What the kernels in front of this one have written, as seen behind the wait.
struct SeamData {
    const float* src;
    float* dst;
    const void* y;
    const float* rows;
    const int* row_of;
    const float* wts;
    const float* shared;
    __device__ explicit SeamData(const SeamArgs& A)
        : src(pdl_fresh(A.src)), dst(pdl_fresh(A.dst)), y(pdl_fresh((const char*)A.y)), rows(pdl_fresh(A.rows)),
          row_of(pdl_fresh(A.row_of)), wts(pdl_fresh(A.wts)), shared(pdl_fresh(A.shared)) {}
};

// W % 4 == 0 and W <= 4 * IT * threads: u stays in registers, every input is read once.
template <int S, int IT>
__global__ void __launch_bounds__(1024) stream_seam_vec_kernel(SeamArgs A) {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    __shared__ float scratch[32];
    __shared__ float s_c[S * S + 2 * S];                      // mix [from][to], out, in
    const int W = A.W;
    // these weights do not depend on the kernel in front
    for (int i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {
        float c = 0.f;
        if (i < S * S) c = A.kind != Y_NONE ? A.mix[i] : 0.f;
        else if (i < S * S + S) c = A.kind != Y_NONE ? A.out_w[i - S * S] : 0.f;
        else if (S == 1 && A.n_in > 1) {                      // equal streams read at once: one row times the sum of the weights
            for (int q = 0; q < A.n_in; ++q) c += A.in_w ? A.in_w[q] : 1.0f;
        } else c = A.in_w ? A.in_w[i - S * S - S] : 1.0f;
        s_c[i] = c;
    }
    const float* mix = s_c;
    const float* ow = s_c + S * S;
    const float* iw = ow + S;
    __syncthreads();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const size_t r = blockIdx.x, t = A.row_idx ? A.row_idx[r] : blockIdx.x;
    const SeamData d(A);
    const float* src = d.src + t * W * (A.same ? 1 : S);
    float* dst = d.dst ? d.dst + t * W * S : nullptr;
    float4 u[IT];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < IT; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        u[k] = zero4();
        if (i >= W) continue;
        float4 x[S];
        if (A.same) {
            const float4 v = ld4(src + i);
#pragma unroll
            for (int s = 0; s < S; ++s) x[s] = v;
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) x[s] = ld4(src + (size_t)s * W + i);
        }
        if (A.kind == Y_NONE) {
#pragma unroll
            for (int s = 0; s < S; ++s) add4(u[k], iw[s], x[s]);
        } else {
            float4 y = zero4();
            if (A.kind == Y_BF16) y = ld4((const bf16*)d.y + t * W + i);
            else if (A.kind == Y_FLOAT) y = ld4((const float*)d.y + t * W + i);
            else {
                for (int c = 0; c < A.top; ++c)
                    add4(y, d.wts[t * A.top + c], ld4(d.rows + (size_t)d.row_of[t * A.top + c] * W + i));
                if (d.shared) add4(y, 1.0f, ld4(d.shared + t * W + i));
            }
#pragma unroll
            for (int q = 0; q < S; ++q) {
                float4 n = zero4();
#pragma unroll
                for (int s = 0; s < S; ++s) add4(n, mix[s * S + q], x[s]);
                add4(n, ow[q], y);
                if (dst) st4(dst + (size_t)q * W + i, n);
                add4(u[k], iw[q], n);
            }
        }
        sum += (u[k].x + u[k].y) + (u[k].z + u[k].w);
    }
    float mean = 0.f, inv = 1.f;
    if (A.w) {
        if (A.center) mean = block_sum(sum, scratch) / (float)W;
        float sq = 0.f;
#pragma unroll
        for (int k = 0; k < IT; ++k) {
            if ((int)(threadIdx.x + k * blockDim.x) * 4 >= W) continue;
            const float a = u[k].x - mean, b = u[k].y - mean, c = u[k].z - mean, e = u[k].w - mean;
            sq += (a * a + b * b) + (c * c + e * e);
        }
        inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)W + A.eps);
    }
#pragma unroll
    for (int k = 0; k < IT; ++k) {
        const int i = (threadIdx.x + k * blockDim.x) * 4;
        if (i >= W) continue;
        float4 v = u[k];
        if (A.w) {
            const float4 g = ld4(A.w + i), c = A.b ? ld4(A.b + i) : zero4();
            v = make_float4((v.x - mean) * inv * g.x + c.x, (v.y - mean) * inv * g.y + c.y,
                            (v.z - mean) * inv * g.z + c.z, (v.w - mean) * inv * g.w + c.w);
        }
        if (A.out_bf16) st4((bf16*)A.out + r * W + i, v);
        else st4((float*)A.out + r * W + i, v);
    }
}

// Any width and up to SEAM_MAX_STREAMS streams: one element a step, u in shared memory.
__global__ void stream_seam_kernel(SeamArgs A, int S) {
    pdl_prologue();
    extern __shared__ float u_row[];
    __shared__ float scratch[32];
    const int W = A.W;
    const size_t r = blockIdx.x, t = A.row_idx ? A.row_idx[r] : blockIdx.x;
    const SeamData d(A);
    const float* src = d.src + t * W * (A.same ? 1 : S);
    float* dst = d.dst ? d.dst + t * W * S : nullptr;
    float sum = 0.f;
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
        float x[SEAM_MAX_STREAMS];
        for (int s = 0; s < S; ++s) x[s] = src[A.same ? i : (size_t)s * W + i];
        float y = 0.f, u = 0.f;
        if (A.kind == Y_BF16) y = __bfloat162float(((const bf16*)d.y)[t * W + i]);
        else if (A.kind == Y_FLOAT) y = ((const float*)d.y)[t * W + i];
        else if (A.kind == Y_ROUTED) {
            for (int c = 0; c < A.top; ++c)
                y = fmaf(d.wts[t * A.top + c], d.rows[(size_t)d.row_of[t * A.top + c] * W + i], y);
            if (d.shared) y += d.shared[t * W + i];
        }
        for (int q = 0; q < S; ++q) {
            float n = x[q];
            if (A.kind != Y_NONE) {
                n = 0.f;
                for (int s = 0; s < S; ++s) n = fmaf(A.mix[s * S + q], x[s], n);
                n = fmaf(A.out_w[q], y, n);
                if (dst) dst[(size_t)q * W + i] = n;
            }
            u = fmaf(A.in_w ? A.in_w[q] : 1.0f, n, u);
        }
        u_row[i] = u;
        sum += u;
    }
    float mean = 0.f, inv = 1.f;
    if (A.w) {
        if (A.center) mean = block_sum(sum, scratch) / (float)W;
        float sq = 0.f;
        for (int i = threadIdx.x; i < W; i += blockDim.x) { const float v = u_row[i] - mean; sq += v * v; }
        inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)W + A.eps);
    }
    for (int i = threadIdx.x; i < W; i += blockDim.x) {          // a thread reads back its own elements
        float v = u_row[i];
        if (A.w) v = (v - mean) * inv * A.w[i] + (A.b ? A.b[i] : 0.f);
        if (A.out_bf16) ((bf16*)A.out)[r * W + i] = __float2bfloat16_rn(v);
        else ((float*)A.out)[r * W + i] = v;
    }
}

template <int S>
static int seam_vec(const SeamArgs& A, int rows, cudaStream_t stream) {
    const int groups = A.W / 4;
    if (rows <= 256 && A.W <= 4096) {                         // few rows: more threads a row, each with less to wait for
        const int threads = ((groups + 31) / 32) * 32;
        FF_LAUNCH((stream_seam_vec_kernel<S, 1>), rows, threads, 0, stream, A);
    } else if (A.W <= 2048) {
        const int threads = (((groups + 1) / 2 + 31) / 32) * 32;
        FF_LAUNCH((stream_seam_vec_kernel<S, 2>), rows, threads, 0, stream, A);
    } else {
        const int threads = (((groups + 3) / 4 + 31) / 32) * 32;
        FF_LAUNCH((stream_seam_vec_kernel<S, 4>), rows, threads, 0, stream, A);
    }
    FF_LAUNCH_CHECK();
    return 0;
}

}  // namespace ff

using namespace ff;

FF_EXPORT int ff_stream_seam_max_streams() { return SEAM_MAX_STREAMS; }

// y_kind: 0 none, 1 float32 y, 2 bfloat16 y, 3 routed rows (rows, row_of, wts, top, shared or null).  `rows_out` is the
// number of rows of `out` (row_idx: their tokens, else 0, 1, ...).
FF_EXPORT int ff_stream_seam(const float* src, float* dst, const void* y, int y_kind, const float* rows, const int* row_of,
                             const float* wts, int top, const float* shared, const float* mix, const float* out_w,
                             const float* in_w, const float* w, const float* b, float eps, int center, void* out,
                             int out_dtype, const int* row_idx, int rows_out, int S, int W, int same, cudaStream_t stream) {
    if (rows_out <= 0) return 0;
    if (!src || !out || S <= 0 || W <= 0 || y_kind < Y_NONE || y_kind > Y_ROUTED || out_dtype < 0 || out_dtype > 1)
        return FF_ERR_BAD_ARG;
    if (y_kind != Y_NONE && (!mix || !out_w)) return FF_ERR_BAD_ARG;
    if ((y_kind == Y_FLOAT || y_kind == Y_BF16) && !y) return FF_ERR_BAD_ARG;
    if (y_kind == Y_ROUTED && (!rows || !row_of || !wts || top <= 0)) return FF_ERR_BAD_ARG;
    if (dst && (row_idx || y_kind == Y_NONE || (same && dst == src))) return FF_ERR_BAD_ARG;
    SeamArgs A{src, dst, y, rows, row_of, wts, shared, mix, out_w, in_w, w, b, eps, center, out, row_idx, W, y_kind, top, same, out_dtype, S};
    const bool aligned = (((uintptr_t)src | (uintptr_t)dst | (uintptr_t)y | (uintptr_t)rows | (uintptr_t)shared | (uintptr_t)w |
                           (uintptr_t)b | (uintptr_t)out) & 15) == 0;
    if (aligned && W % 4 == 0 && W <= 16384 && S <= SEAM_FIXED_STREAMS) {
        switch (same && y_kind == Y_NONE ? 1 : S) {
            case 1: return seam_vec<1>(A, rows_out, stream);
            case 2: return seam_vec<2>(A, rows_out, stream);
            case 3: return seam_vec<3>(A, rows_out, stream);
            case 4: return seam_vec<4>(A, rows_out, stream);
            case 5: return seam_vec<5>(A, rows_out, stream);
            case 6: return seam_vec<6>(A, rows_out, stream);
            case 7: return seam_vec<7>(A, rows_out, stream);
            default: return seam_vec<8>(A, rows_out, stream);
        }
    }
    const size_t smem = (size_t)W * sizeof(float);
    if (S > SEAM_MAX_STREAMS || smem > 200 * 1024) return FF_ERR_UNSUPPORTED;
    if (smem > 48 * 1024) FF_SMEM_LIMIT(stream_seam_kernel, 200 * 1024);
    FF_LAUNCH(stream_seam_kernel, rows_out, W >= 1024 ? 256 : 128, smem, stream, A, S);
    FF_LAUNCH_CHECK();
    return 0;
}
