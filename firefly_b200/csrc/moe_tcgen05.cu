// The grouped products of routed experts on the fifth-generation tensor cores.
//
// A block takes one tile of 128 rows of one expert (the plan's row tiles, see moe.cu) and BC rows of the expert's
// matrices.  The rows are the M operand of tcgen05.mma and the matrices' rows its N operand; the accumulator
// [128 rows][BC] is in tensor memory.  For the first product the rows are tokens' activations picked by `src_tok`: four
// at a time by TMA gather, one gather a lane (a tile with fewer rows asks for that many only: what lies in shared memory
// beyond them only makes accumulator rows that nobody reads).  The experts' matrices are stacked, so that a box of
// weight rows is a plain 2D tile of one tall matrix.  With gate and up a tile's first half is gate rows and its second
// half the same rows of up: the pair of a column is in one thread's accumulator row, and the epilogue applies the
// activation there.  Two blocks share an SM, one's epilogue under the other's main loop.
//
// A result is a dot product over K in a fixed order, whatever shares its tile.  Every wait on an mbarrier is bounded:
// after about a second the kernel records an error code, lets its copies land, frees its tensor memory and returns.
#include "tcgen05.cuh"
#include "moe.cuh"

namespace ff {

constexpr int GM = GROUPED_TC_ROWS;   // rows of a row tile (MMA M)
constexpr int GROUPED_THREADS = 192;  // a warp for the loads, one for the MMAs, four for the epilogue

template <int BC> struct GroupedCfg {
    static constexpr int A_BYTES = GM * BK * 2;
    static constexpr int B_BYTES = BC * BK * 2;
    static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
    static constexpr int STAGES = (108 * 1024) / STAGE_BYTES;          // two blocks an SM
    static constexpr size_t SMEM = (size_t)STAGES * STAGE_BYTES + 1024 /* alignment slack */ + 256 /* barriers */;
};

struct GroupedArgs {
    const int* src_tok;
    const int* seg;
    const int* tile_expert;
    const int* tile_row0;
    const int* n_tiles;
    const float* row_w;
    void* out;
    int N, K;
    float limit;
    int act;
    int* status;
};

__device__ __forceinline__ void tma_gather4(bool issue, uint32_t dst, const CUtensorMap* map, int x, const int (&r)[4], uint32_t bar) {
    asm volatile("{\n\t.reg .pred q;\n\tsetp.ne.b32 q, %8, 0;\n\t"
                 "@q cp.async.bulk.tensor.2d.shared::cluster.global.tile::gather4.mbarrier::complete_tx::bytes "
                 "[%0], [%1, {%3, %4, %5, %6, %7}], [%2];\n\t}"
                 ::"r"(dst), "l"(map), "r"(bar), "r"(x), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"((uint32_t)issue) : "memory");
}

template <int KIND, int BC>
__global__ void __launch_bounds__(GROUPED_THREADS)
moe_grouped_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b0,
                      const __grid_constant__ CUtensorMap map_b1, const GroupedArgs a) {
    using Cfg = GroupedCfg<BC>;
    constexpr int STAGES = Cfg::STAGES;
    constexpr bool GATHER = KIND != MOE_DOWN;
    constexpr int COLS = KIND == MOE_GATEUP ? BC / 2 : BC;             // output columns of a block
    extern __shared__ unsigned char smem_raw[];
    unsigned char* tiles = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint64_t* bars = reinterpret_cast<uint64_t*>(tiles + (size_t)STAGES * Cfg::STAGE_BYTES);
    // bars[0..S) full, bars[S..2S) empty, bars[2S] accumulator ready
    __shared__ uint32_t s_tmem_base;
    __shared__ int s_abort;
    const int warp = __shfl_sync(0xffffffffu, (int)(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;
    const bool issue = lane == 0;

    // the plan comes from the kernel in front: nothing can be asked for before it is there
    grid_dependency_wait();
    const int* seg = pdl_fresh(a.seg);
    if ((int)blockIdx.y >= *pdl_fresh(a.n_tiles)) return;
    const int e = pdl_fresh(a.tile_expert)[blockIdx.y], row0 = pdl_fresh(a.tile_row0)[blockIdx.y];
    const int rows = min(GM, seg[e + 1] - row0);
    const int n0 = blockIdx.x * COLS;
    const int n_iters = (a.K + BK - 1) / BK;

    if (threadIdx.x == 0) {
        s_abort = 0;
        for (int i = 0; i < 2 * STAGES + 1; ++i) mbar_init(smem_addr(&bars[i]), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_addr(&s_tmem_base)), "r"((uint32_t)BC) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = s_tmem_base;
    volatile int* abort_flag = &s_abort;
    // only now: a kernel that starts early must not take tensor memory that this block still waits for
    grid_launch_dependents();

    if (warp == 0) {
        // ------------------------------------------------ producer: TMA loads --
        int src[4];
        const int groups = (rows + 3) >> 2;                            // gathers of four rows that the tile needs
        if (GATHER) {
            const int* st = pdl_fresh(a.src_tok);
#pragma unroll
            for (int j = 0; j < 4; ++j) src[j] = st[row0 + min(4 * lane + j, rows - 1)];
        }
        const uint32_t bytes = Cfg::B_BYTES + (GATHER ? (uint32_t)groups * 4 * BK * 2 : (uint32_t)Cfg::A_BYTES);
        int issued = 0;
        for (int it = 0; it < n_iters; ++it) {
            const int s = it % STAGES;
            if (it >= STAGES &&
                !__all_sync(0xffffffffu, mbar_wait(smem_addr(&bars[STAGES + s]), ((it / STAGES) & 1) ^ 1, a.status, abort_flag, 111)))
                break;
            const uint32_t full = smem_addr(&bars[s]);
            const uint32_t sa = smem_addr(tiles + (size_t)s * Cfg::STAGE_BYTES), sb = sa + Cfg::A_BYTES;
            mbar_expect_tx(issue, full, bytes);
            __syncwarp();
            if (KIND == MOE_GATEUP) {
                tma_load_2d(issue, sb, &map_b0, it * BK, e * a.N + n0, full);
                tma_load_2d(issue, sb + Cfg::B_BYTES / 2, &map_b1, it * BK, e * a.N + n0, full);
            } else {
                tma_load_2d(issue, sb, &map_b0, it * BK, e * a.N + n0, full);
            }
            if (GATHER) tma_gather4(lane < groups, sa + lane * 4 * BK * 2, &map_a, it * BK, src, full);
            else tma_load_2d(issue, sa, &map_a, it * BK, row0, full);
            issued = it + 1;
        }
        if (*abort_flag) {
            // let the copies that are still in flight land before the block's memory goes away
            for (int it = max(0, issued - STAGES); it < issued; ++it) {
                const unsigned long long start = clock64();
                while (!mbar_try_wait(smem_addr(&bars[it % STAGES]), (it / STAGES) & 1))
                    if (clock64() - start > WAIT_LIMIT_CYCLES) break;
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------ MMA issuer ----------
        const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BC >> 3) << 17) | ((uint32_t)(GM >> 4) << 24);
        for (int it = 0; it < n_iters; ++it) {
            const int s = it % STAGES;
            if (!__all_sync(0xffffffffu, mbar_wait(smem_addr(&bars[s]), (it / STAGES) & 1, a.status, abort_flag, 112))) break;
            tc_fence_after();
            const uint32_t sa = smem_addr(tiles + (size_t)s * Cfg::STAGE_BYTES), sb = sa + Cfg::A_BYTES;
#pragma unroll
            for (int k = 0; k < BK / UMMA_K; ++k)
                tc_mma_bf16(issue, tmem_base, smem_desc_sw128(sa + k * UMMA_K * 2), smem_desc_sw128(sb + k * UMMA_K * 2), idesc,
                            (it > 0 || k > 0) ? 1u : 0u);
            tc_commit(issue, smem_addr(&bars[STAGES + s]));            // stage free when these MMAs have read it
            __syncwarp();
        }
        tc_commit(issue, smem_addr(&bars[2 * STAGES]));                // accumulator complete
    } else {
        // ------------------------------------------------ epilogue: one accumulator row a thread --
        const int quad = warp & 3;                                     // this warp's 32 lanes of tensor memory
        const int r = quad * 32 + lane;
        const bool live = r < rows;
        const float wr = KIND != MOE_DOWN && a.row_w && live ? pdl_fresh(a.row_w)[row0 + r] : 1.0f;
        const bool ok = __all_sync(0xffffffffu, mbar_wait(smem_addr(&bars[2 * STAGES]), 0, a.status, abort_flag, 113)) && !*abort_flag;
        tc_fence_after();
        const uint32_t acc = tmem_base + ((uint32_t)(quad * 32) << 16);
        const int cols = min(COLS, a.N - n0);
        if (__all_sync(0xffffffffu, ok) && quad * 32 < rows) {          // the same for the whole warp: the loads are warp-wide
            const bool vec = (a.N & (KIND == MOE_DOWN ? 3 : 7)) == 0;  // 16-byte stores stay aligned
#pragma unroll 1
            for (int c0 = 0; c0 < cols; c0 += 16) {
                float v[16];
                tc_ld16(acc + c0, v);
                if constexpr (KIND == MOE_GATEUP) {
                    float u[16];
                    tc_ld16(acc + BC / 2 + c0, u);
#pragma unroll
                    for (int i = 0; i < 16; ++i) v[i] = clamped_glu_fast(v[i] * wr, u[i] * wr, a.limit, a.act);
                } else if constexpr (KIND == MOE_UP) {
#pragma unroll
                    for (int i = 0; i < 16; ++i) v[i] = relu2(v[i] * wr);
                }
                if (!live) continue;
                const size_t o = (size_t)(row0 + r) * a.N + n0 + c0;
                if constexpr (KIND == MOE_DOWN) {
                    float* dst = (float*)a.out + o;
                    if (vec && c0 + 16 <= cols) {
#pragma unroll
                        for (int i = 0; i < 4; ++i)
                            reinterpret_cast<float4*>(dst)[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (c0 + i < cols) dst[i] = v[i];
                    }
                } else {
                    bf16* dst = (bf16*)a.out + o;
                    if (vec && c0 + 16 <= cols) {
                        uint32_t w[8];
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            __nv_bfloat162 p = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
                            w[i] = *reinterpret_cast<uint32_t*>(&p);
                        }
                        reinterpret_cast<uint4*>(dst)[0] = make_uint4(w[0], w[1], w[2], w[3]);
                        reinterpret_cast<uint4*>(dst)[1] = make_uint4(w[4], w[5], w[6], w[7]);
                    } else {
#pragma unroll
                        for (int i = 0; i < 16; ++i)
                            if (c0 + i < cols) dst[i] = __float2bfloat16_rn(v[i]);
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        __syncwarp();
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"((uint32_t)BC) : "memory");
    }
}

template <int KIND, int BC>
static int grouped_launch(const CUtensorMap& ma, const CUtensorMap& mb0, const CUtensorMap& mb1, const GroupedArgs& a, int max_tiles,
                          cudaStream_t stream) {
    constexpr int COLS = KIND == MOE_GATEUP ? BC / 2 : BC;
    FF_SMEM_LIMIT((moe_grouped_tc_kernel<KIND, BC>), GroupedCfg<BC>::SMEM);
    dim3 grid((a.N + COLS - 1) / COLS, max_tiles);
    FF_LAUNCH((moe_grouped_tc_kernel<KIND, BC>), grid, GROUPED_THREADS, GroupedCfg<BC>::SMEM, stream, ma, mb0, mb1, a);
    FF_LAUNCH_CHECK();
    return 0;
}

}  // namespace ff

using namespace ff;

// a: bfloat16 [a_rows, K] (kind MOE_DOWN: the sorted rows themselves; else the tokens' rows, picked by src_tok).
// b0, b1: bfloat16 [E, N, K].  The plan's row tiles have 128 rows.  wide: 256 weight rows a block instead of 128.
FF_EXPORT int ff_moe_grouped_tc(const void* a, int a_rows, const int* src_tok, const void* b0, const void* b1, int E, int kind,
                                const int* seg, const int* tile_expert, const int* tile_row0, const int* n_tiles,
                                const float* row_w, void* out, int max_tiles, int N, int K, float limit, int act, int wide,
                                int* status, cudaStream_t stream) {
    if (max_tiles <= 0) return 0;
    if (kind < MOE_DOWN || kind > MOE_UP || (kind == MOE_GATEUP && !b1) || !status || a_rows <= 0 || E <= 0 || N <= 0 || K <= 0 || K % 8)
        return FF_ERR_BAD_ARG;
    if ((((uintptr_t)a | (uintptr_t)b0 | (uintptr_t)b1 | (uintptr_t)out) & 15) != 0 || (long long)E * N >= (1ll << 31) || max_tiles > 65535)
        return FF_ERR_BAD_ARG;
    const int bc = wide ? 256 : 128, box = kind == MOE_GATEUP ? bc / 2 : bc;
    CUtensorMap ma, mb0, mb1;
    int rc = make_map(a, a_rows, K, kind == MOE_DOWN ? GM : 1, &ma);       // a gather's box is one row high
    if (rc) return rc;
    rc = make_map(b0, E * N, K, box, &mb0);
    if (rc) return rc;
    mb1 = mb0;
    if (kind == MOE_GATEUP && (rc = make_map(b1, E * N, K, box, &mb1))) return rc;
    GroupedArgs g{src_tok, seg, tile_expert, tile_row0, n_tiles, row_w, out, N, K, limit, act, status};
#define FF_GROUPED(KIND) return wide ? grouped_launch<KIND, 256>(ma, mb0, mb1, g, max_tiles, stream) \
                                     : grouped_launch<KIND, 128>(ma, mb0, mb1, g, max_tiles, stream)
    if (kind == MOE_GATEUP) FF_GROUPED(MOE_GATEUP);
    if (kind == MOE_UP) FF_GROUPED(MOE_UP);
    FF_GROUPED(MOE_DOWN);
#undef FF_GROUPED
}
