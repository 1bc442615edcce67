// BF16 weights x bf16 activation rows on the 5th-generation tensor cores: the prefill form of linear_bf16.cuh.
//
// D[weight row][activation row] = W tile x X tile^T: TMEM lanes are weight rows, TMEM columns activation rows, so a warp's
// epilogue store is a run of consecutive outputs of one activation row. Both operands are K-major and come through TMA
// tensor maps (64 k = one 128-byte swizzled row per stage and row).
//
// Persistent CTA (static tile schedule, activation tiles fastest so that CTAs running together share weight tiles in L2):
//   warp 0     one lane posts the tensor copies of the stage ring
//   warp 1     one lane issues the MMAs and commits (stage barriers to the producer, accumulator barrier to the epilogue)
//   warps 2-5  epilogue: TMEM -> registers -> global; two accumulator sets, so it overlaps the next tile's MMAs
// NA = 2 keeps two 128-row weight tiles per activation tile: twice the rows of one matrix, or the same rows of gate and up,
// whose product act(gate) * up is then formed in the epilogue without a round trip.
// Every mbarrier wait is bounded; a wait that runs out raises the device flag and the CTA still frees its TMEM.
#include "linear_bf16.cuh"
#include "tensor_map.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr int BM = 128, BKE = 64;            // weight rows of one tile, k elements of a stage (128 bytes)
constexpr int A_BYTES = BM * BKE * 2;
constexpr int SMEM_BUDGET = 200 * 1024;
constexpr int EPI_WARPS = 4, TC_THREADS = (2 + EPI_WARPS) * 32;

template <int NA, int BN>
struct Shape {
    static constexpr int STAGE = NA * A_BYTES + BN * BKE * 2;
    static constexpr int STAGES = SMEM_BUDGET / STAGE < 8 ? SMEM_BUDGET / STAGE : 8;
    static constexpr int COLS = NA * BN;                            // TMEM columns of one accumulator set
    static constexpr int TMEM = 2 * COLS < 32 ? 32 : 2 * COLS;      // power of two by construction
    static constexpr int BARS = 2 * STAGES + 4;
    static constexpr int SMEM = STAGES * STAGE + BARS * 8 + 16 + 1024;   // the dynamic area is aligned to 1024 by hand
};

struct TcArgs {
    void* y; int ldy, y_group_stride;
    const float* scale; int scale_ld;
    const RowSegment* segs; const int32_t* n_segs;
    int w_rows, rows, groups, ksteps, x_group_stride;
    int m_tiles, n_tiles;                    // per group: ceil(w_rows / (128 or 256)), ceil(rows / BN); n_tiles unused with segments
    int a2_rows;                             // row offset of the second weight tile (0 with a separate up matrix)
    int* timeout_flag;
};

__device__ __forceinline__ uint64_t desc_sw128(uint32_t saddr) {      // K-major, 128-byte swizzle, 8-row groups 1024 B apart
    return (uint64_t) ((saddr & 0x3ffffu) >> 4) | (1ull << 16) | ((uint64_t) (1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void umma_bf16(uint32_t d, uint64_t a, uint64_t b, uint32_t idesc, uint32_t accumulate) {
    asm volatile("{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
                 "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
                 ::"r"(d), "l"(a), "l"(b), "r"(idesc), "r"(accumulate) : "memory");
}
__device__ __forceinline__ void umma_commit(uint64_t* bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(skd::smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void arrive(uint64_t* bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(skd::smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void tmem_ld32(uint32_t ta, float (&u)[32]) {
    uint32_t r[32];
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
        "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];\n\t"
        "tcgen05.wait::ld.sync.aligned;"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]),
          "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]),
          "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]),
          "=r"(r[30]), "=r"(r[31])
        : "r"(ta)
        : "memory");
#pragma unroll
    for (int i = 0; i < 32; ++i) u[i] = __uint_as_float(r[i]);
}

struct Tile { int group, col_group, m0, x_row, n_valid; };     // weight row inside the group, first activation row, valid rows of the tile

template <int NA, int BN>
__device__ __forceinline__ Tile tile_at(const TcArgs& a, int t) {
    Tile r;
    if (a.segs) {
        const RowSegment sg = a.segs[t / a.m_tiles];
        r.group = sg.group; r.col_group = 0; r.x_row = sg.start; r.n_valid = sg.count;
        r.m0 = t % a.m_tiles;
    } else {
        const int nt = t % a.n_tiles, q = t / a.n_tiles;
        r.group = r.col_group = q / a.m_tiles;
        r.m0 = q % a.m_tiles;
        r.x_row = nt * BN; r.n_valid = min(BN, a.rows - nt * BN);
    }
    r.m0 *= BM + a.a2_rows;                   // 128 rows per tile, 256 when the second weight tile continues the first
    return r;
}

template <int NA, int BN, int OUT>
__global__ void __launch_bounds__(TC_THREADS, 1)
gemm_bf16_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_a2, const __grid_constant__ CUtensorMap map_b,
                    const TcArgs a) {
    typedef Shape<NA, BN> S;
    constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t) (BN >> 3) << 17) | ((uint32_t) (BM >> 4) << 24);
    extern __shared__ uint8_t raw[];
    uint8_t* smem = raw + ((1024 - (skd::smem_u32(raw) & 1023)) & 1023);
    uint64_t* full = (uint64_t*) (smem + S::STAGES * S::STAGE);
    uint64_t* empty = full + S::STAGES;
    uint64_t* acc_full = empty + S::STAGES;
    uint64_t* acc_empty = acc_full + 2;
    uint32_t* tmem_slot = (uint32_t*) (acc_empty + 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    skd::pdl_launch_dependents();
    if (warp == 1) {
        if (lane == 0) {
            for (int s = 0; s < S::STAGES; ++s) { skd::mbar_init(full + s, 1); skd::mbar_init(empty + s, 1); }
            for (int b = 0; b < 2; ++b) { skd::mbar_init(acc_full + b, 1); skd::mbar_init(acc_empty + b, EPI_WARPS); }
            skd::mbar_fence_init();
        }
        __syncwarp();
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(skd::smem_u32(tmem_slot)), "r"(S::TMEM) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = *tmem_slot;
    skd::pdl_wait();
    const int total = a.m_tiles * (a.segs ? *a.n_segs : a.n_tiles * a.groups);

    if (warp == 0 && lane == 0) {
        // ---------------------------------------------- producer ----------------------------------------------
        int it = 0;                                             // stages posted so far
        bool ok = true;
        for (int t = blockIdx.x; t < total && ok; t += gridDim.x) {
            const Tile tl = tile_at<NA, BN>(a, t);
            const int wrow = tl.group * a.w_rows + tl.m0, xk = tl.col_group * a.x_group_stride;
            for (int k = 0; k < a.ksteps; ++k, ++it) {
                const int s = it % S::STAGES;
                if (it >= S::STAGES && !(ok = skd::mbar_wait_bounded(empty + s, ((it / S::STAGES) + 1) & 1, a.timeout_flag))) break;
                uint8_t* st = smem + s * S::STAGE;
                skd::mbar_expect_tx(full + s, S::STAGE);
                skd::tma_load_2d(st, &map_a, k * BKE, wrow, full + s);
                if (NA == 2) skd::tma_load_2d(st + A_BYTES, &map_a2, k * BKE, wrow + a.a2_rows, full + s);
                skd::tma_load_2d(st + NA * A_BYTES, &map_b, xk + k * BKE, tl.x_row, full + s);
            }
        }
        // copies still in flight must land before the CTA leaves: the last round of each posted stage
        for (int j = max(0, it - S::STAGES); j < it; ++j)
            if (!skd::mbar_wait_bounded(full + j % S::STAGES, (j / S::STAGES) & 1, a.timeout_flag)) break;
    } else if (warp == 1 && lane == 0) {
        // ---------------------------------------------- MMA issuer ----------------------------------------------
        int it = 0, n = 0;
        bool ok = true;
        for (int t = blockIdx.x; t < total && ok; t += gridDim.x, ++n) {
            const int set = n & 1;
            if (n >= 2 && !(ok = skd::mbar_wait_bounded(acc_empty + set, ((n >> 1) + 1) & 1, a.timeout_flag))) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t d = tmem + set * S::COLS;
            for (int k = 0; k < a.ksteps; ++k, ++it) {
                const int s = it % S::STAGES;
                if (!(ok = skd::mbar_wait_bounded(full + s, (it / S::STAGES) & 1, a.timeout_flag))) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t base = skd::smem_u32(smem + s * S::STAGE);
                const uint64_t da = desc_sw128(base), db = desc_sw128(base + NA * A_BYTES);
#pragma unroll
                for (int kk = 0; kk < BKE / 16; ++kk)             // a K = 16 step advances the start address by 32 bytes inside the swizzle atom
#pragma unroll
                    for (int i = 0; i < NA; ++i)
                        umma_bf16(d + i * BN, da + (uint64_t) ((i * A_BYTES + kk * 32) >> 4), db + (uint64_t) (kk * 2), IDESC, (k | kk) != 0);
                umma_commit(empty + s);
            }
            if (ok) umma_commit(acc_full + set);
        }
    } else if (warp >= 2) {
        // ---------------------------------------------- epilogue ----------------------------------------------
        const int quad = warp & 3;                               // TMEM lanes 32 * quad .. + 31 belong to this warp
        int n = 0;
        for (int t = blockIdx.x; t < total; t += gridDim.x, ++n) {
            const int set = n & 1;
            const Tile tl = tile_at<NA, BN>(a, t);
            int ok = skd::mbar_wait_bounded(acc_full + set, (n >> 1) & 1, a.timeout_flag) ? 1 : 0;
            ok = __all_sync(~0u, ok);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t src = tmem + set * S::COLS + ((uint32_t) (quad * 32) << 16);
            const int wr = tl.m0 + quad * 32 + lane;
#pragma unroll 1
            for (int c0 = 0; c0 < BN; c0 += 32) {
                if (c0 >= tl.n_valid) break;
                float u[32], v[32];
                tmem_ld32(src + c0, u);
                if (NA == 2) tmem_ld32(src + BN + c0, v);
                // lane j fetches the factor of column j once; a load per column in the loop below would serialise on its latency
                const float fl = a.scale && c0 + lane < tl.n_valid ? a.scale[(size_t) (tl.x_row + c0 + lane) * a.scale_ld + tl.col_group] : 1.0f;
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    const float f = __shfl_sync(~0u, fl, j);
                    if (c0 + j >= tl.n_valid) break;
                    const int r = tl.x_row + c0 + j;
                    const size_t at = (size_t) r * a.ldy + (size_t) tl.col_group * a.y_group_stride + wr;
                    if (lin_gated(OUT)) {
                        if (wr < a.w_rows) ((bf16*) a.y)[at] = __float2bfloat16_rn(skd::lin_gate<OUT>(u[j] * f) * (v[j] * f));
                    } else {
                        if (wr < a.w_rows) { if (OUT == LIN_OUT_F32) ((float*) a.y)[at] = u[j] * f; else ((bf16*) a.y)[at] = __float2bfloat16_rn(u[j] * f); }
                        if (NA == 2 && wr + BM < a.w_rows) { if (OUT == LIN_OUT_F32) ((float*) a.y)[at + BM] = v[j] * f; else ((bf16*) a.y)[at + BM] = __float2bfloat16_rn(v[j] * f); }
                    }
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) arrive(acc_empty + set);
        }
    }
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(S::TMEM) : "memory");
}

template <int NA, int BN, int OUT>
int32_t run_tc(const LinearArgs& l, cudaStream_t s) {
    typedef Shape<NA, BN> S;
    CUtensorMap ma, ma2, mb;
    const int64_t w_total = (int64_t) l.groups * l.w_rows;
    SK_TRY(tensor_map_rows(&ma, l.w, w_total, l.ldw, BM));
    if (lin_gated(OUT)) SK_TRY(tensor_map_rows(&ma2, l.w2, w_total, l.ldw, BM)); else ma2 = ma;
    SK_TRY(tensor_map_rows(&mb, (const bf16*) l.x, l.x_rows_alloc, l.ldx, BN));
    TcArgs a = {};
    a.y = l.y; a.ldy = l.ldy; a.y_group_stride = l.y_group_stride; a.scale = l.scale; a.scale_ld = l.scale_ld;
    a.segs = l.segs; a.n_segs = l.n_segs; a.w_rows = l.w_rows; a.rows = l.rows; a.groups = l.groups;
    a.ksteps = l.ldw / BKE; a.x_group_stride = l.x_group_stride;
    a.a2_rows = (NA == 2 && !lin_gated(OUT)) ? BM : 0;
    a.m_tiles = (l.w_rows + BM + a.a2_rows - 1) / (BM + a.a2_rows);
    a.n_tiles = (l.rows + BN - 1) / BN;
    a.timeout_flag = device_timeout_flag();
    const int64_t tiles = (int64_t) a.m_tiles * (l.segs ? l.max_segs : (int64_t) a.n_tiles * l.groups);
    SK_REQUIRE(tiles < (1ll << 30), "gemm_bf16_tc: too many tiles");
    SK_TRY(ensure_dynamic_smem((const void*) gemm_bf16_tc_kernel<NA, BN, OUT>, S::SMEM));
    const int grid = (int) std::min<int64_t>(tiles, sm_count());
    SK_CUDA(launch_pdl(gemm_bf16_tc_kernel<NA, BN, OUT>, dim3(grid), dim3(TC_THREADS), S::SMEM, s, ma, ma2, mb, a));
    return SKAINET_CUDA_OK;
}

template <int NA, int BN>
int32_t run_out(const LinearArgs& l, cudaStream_t s) {
    return l.out == LIN_OUT_ACT ? run_tc<NA, BN, LIN_OUT_ACT>(l, s) : run_tc<NA, BN, LIN_OUT_F32>(l, s);
}

}  // namespace

int32_t launch_gemm_bf16_tc(const LinearArgs& l, cudaStream_t s) {
    SK_REQUIRE(!l.f32_act && l.row_index == nullptr, "gemm_bf16_tc: bf16 rows in order only");
    const int rows = l.segs ? l.seg_rows : l.rows;
    // a segment's rows past its end belong to the next one: their columns are computed and not stored
    if (l.out == LIN_OUT_GEGLU) return rows <= 32 ? run_tc<2, 32, LIN_OUT_GEGLU>(l, s) : run_tc<2, 128, LIN_OUT_GEGLU>(l, s);
    if (l.out == LIN_OUT_SWIGLU) return rows <= 32 ? run_tc<2, 32, LIN_OUT_SWIGLU>(l, s) : run_tc<2, 128, LIN_OUT_SWIGLU>(l, s);
    if (rows <= 32) return run_out<1, 32>(l, s);
    const int64_t wide = (int64_t) ((l.w_rows + 2 * BM - 1) / (2 * BM)) * (l.segs ? l.max_segs : (int64_t) ((l.rows + 127) / 128) * l.groups);
    return l.w_rows > BM && wide * 5 >= (int64_t) sm_count() * 4 ? run_out<2, 128>(l, s) : run_out<1, 128>(l, s);
}

}  // namespace sk
