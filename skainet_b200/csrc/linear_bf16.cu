// Linears over BF16 weights (contract: linear_bf16.cuh).
//
//   linear_ring_kernel    up to 16 activation rows (decode): every weight byte is read once, through a ring of shared-memory
//                         stages filled by TMA; bound by the weight stream. The arithmetic is mma.sync: it only saves the CUDA
//                         cores the unpacking. K is permuted identically in both operands, so that a lane's 16-byte load
//                         (8 consecutive k of a row) is two k16 steps' worth of its A fragment.
//   linear_f32_kernel     fp32 activations, fp32 FMA: the 32-bit mode, every row count.
//   gemm_bf16_tc.cu       more rows: tcgen05.
#include "linear_bf16.cuh"
#include "tensor_map.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr int RG_WARPS = 8, RG_TILE = 16, RG_THREADS = (RG_WARPS + 1) * 32;
constexpr int RG_SMEM = 96 * 1024;       // ring and partial sums of two CTAs fit an SM

// MT weight matrices (gate and up), 16 rows of each per unit; a stage holds KB blocks of 64 k: [matrix][block][16 rows][128 bytes],
// the 16-byte chunks of a row XORed with the row (the copy engine's 128-byte swizzle). One copy instruction per matrix and stage:
// with one per row the stream was bound by the issue of the copies (1.9-3.2 TB/s).
template <int MT>
struct Ring {
    static constexpr int KB = MT == 1 ? 8 : 4, KC = KB * 64, MAT = KB * RG_TILE * 128, STAGE = MT * MAT;
    static constexpr int STAGES = (RG_SMEM - (MT - 1) * 16 * 1024) / STAGE;
};
template <int MT, int NB>
constexpr int ring_smem() { return Ring<MT>::STAGES * Ring<MT>::STAGE + 2 * RG_WARPS * MT * NB * RG_TILE * 8 * 4 + 2 * Ring<MT>::STAGES * 8 + 1024; }

// Persistent CTA; a unit is 16 output rows of one group (or of one segment's expert) over all of K. One producer warp streams
// the units' rows; eight consumer warps take every eighth k32 step of a stage, and their partial sums meet in shared memory in
// fixed order at the end of a unit. NB = tiles of 8 activation rows.
template <int NB, int OUT>
__global__ void __launch_bounds__(RG_THREADS, 2)
linear_ring_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_w2, const LinearArgs a, int* __restrict__ timeout_flag) {
    constexpr bool DUAL = lin_gated(OUT);
    constexpr int MT = DUAL ? 2 : 1;
    typedef Ring<MT> R;
    extern __shared__ uint8_t raw[];
    uint8_t* smem = raw + ((1024 - (skd::smem_u32(raw) & 1023)) & 1023);
    float* part = (float*) (smem + R::STAGES * R::STAGE);               // [2][warps][MT][NB][8 * 16]
    uint64_t* full = (uint64_t*) (part + 2 * RG_WARPS * MT * NB * RG_TILE * 8);
    uint64_t* empty = full + R::STAGES;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    skd::pdl_launch_dependents();
    if (threadIdx.x == 0) {
        for (int s = 0; s < R::STAGES; ++s) { skd::mbar_init(full + s, 1); skd::mbar_init(empty + s, RG_WARPS); }
        skd::mbar_fence_init();
    }
    __syncthreads();
    const int tiles = (a.w_rows + RG_TILE - 1) / RG_TILE, chunks = (a.ldw + R::KC - 1) / R::KC;
    const bool producer = warp == RG_WARPS;
    if (!producer || a.segs) skd::pdl_wait();        // weights do not depend on the predecessor: the ring fills before the wait
    const int units = tiles * (a.segs ? *a.n_segs : a.groups);

    if (producer) {
        if (lane != 0) return;
        int it = 0;
        bool ok = true;
        for (int u = blockIdx.x; u < units && ok; u += gridDim.x) {
            const int row = (a.segs ? a.segs[u / tiles].group : u / tiles) * a.w_rows + (u % tiles) * RG_TILE;
            for (int c = 0; c < chunks; ++c, ++it) {
                const int s = it % R::STAGES;
                if (it >= R::STAGES && !(ok = skd::mbar_wait_bounded(empty + s, ((it / R::STAGES) + 1) & 1, timeout_flag))) break;
                uint8_t* st = smem + s * R::STAGE;
                skd::mbar_expect_tx(full + s, R::STAGE);
                skd::tma_load_3d(st, &map_w, 0, row, c * R::KB, full + s);
                if (DUAL) skd::tma_load_3d(st + R::MAT, &map_w2, 0, row, c * R::KB, full + s);
            }
        }
        for (int j = max(0, it - R::STAGES); j < it; ++j)               // no copy outlives the CTA
            if (!skd::mbar_wait_bounded(full + j % R::STAGES, (j / R::STAGES) & 1, timeout_flag)) break;
        return;
    }
    bool ok = true;
    int it = 0, buf = 0;
    for (int u = blockIdx.x; u < units; u += gridDim.x, buf ^= 1) {
        int col_group = u / tiles, row0 = 0, n_rows = a.rows;
        if (a.segs) { const RowSegment sg = a.segs[u / tiles]; col_group = 0; row0 = sg.start; n_rows = sg.count; }
        const bf16* xp[NB];
        bool live[NB];
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int n = b * 8 + g;
            live[b] = n < n_rows;
            const int r = live[b] ? (a.row_index ? a.row_index[row0 + n] : row0 + n) : 0;
            xp[b] = (const bf16*) a.x + (size_t) r * a.ldx + (size_t) col_group * a.x_group_stride;
        }
        float acc[MT][NB][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int b = 0; b < NB; ++b)
#pragma unroll
                for (int i = 0; i < 4; ++i) acc[m][b][i] = 0.0f;
        // A warp takes k32 steps warp, warp + 8, .. of a stage: half h of block j, of whose eight 16-byte chunks lane t takes 2t + h,
        // so that the rows of a quarter-warp meet different banks. The activation's fragments are fetched a stage ahead.
        constexpr int PER = 2 * R::KB / RG_WARPS;
        const int h = warp & 1, kb0 = warp >> 1;
        uint4 xv[PER][NB], xn[PER][NB];
        auto load_x = [&](uint4 (&x)[PER][NB], int c) {
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                const int k = (c * R::KB + kb0 + p * (RG_WARPS / 2)) * 64 + (2 * t + h) * 8;
#pragma unroll
                for (int b = 0; b < NB; ++b) x[p][b] = live[b] && k < a.ldw ? *reinterpret_cast<const uint4*>(xp[b] + k) : make_uint4(0, 0, 0, 0);
            }
        };
        load_x(xn, 0);
        for (int c = 0; c < chunks; ++c, ++it) {
            const int s = it % R::STAGES;
#pragma unroll
            for (int p = 0; p < PER; ++p)
#pragma unroll
                for (int b = 0; b < NB; ++b) xv[p][b] = xn[p][b];
            if (c + 1 < chunks) load_x(xn, c + 1);
            ok = ok && skd::mbar_wait_bounded(full + s, (it / R::STAGES) & 1, timeout_flag);
            if (ok) {
                const uint8_t* st = smem + s * R::STAGE + g * 128 + (((2 * t + h) ^ g) << 4);       // rows g and g + 8 share the XOR
#pragma unroll
                for (int p = 0; p < PER; ++p) {
                    const uint8_t* bl = st + (kb0 + p * (RG_WARPS / 2)) * RG_TILE * 128;
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        const uint4 w0 = skd::lds128(bl + m * R::MAT), w1 = skd::lds128(bl + m * R::MAT + 8 * 128);
#pragma unroll
                        for (int b = 0; b < NB; ++b) {
                            skd::mma_bf16(acc[m][b], w0.x, w1.x, w0.y, w1.y, xv[p][b].x, xv[p][b].y);
                            skd::mma_bf16(acc[m][b], w0.z, w1.z, w0.w, w1.w, xv[p][b].z, xv[p][b].w);
                        }
                    }
                }
            }
            __syncwarp();
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(skd::smem_u32(empty + s)) : "memory");
        }
        float* pb = part + (size_t) buf * RG_WARPS * MT * NB * RG_TILE * 8;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int b = 0; b < NB; ++b) {      // acc[0], [1]: output row g, activation rows 2t, 2t+1; acc[2], [3]: output row g + 8
                float* p = pb + ((warp * MT + m) * NB + b) * RG_TILE * 8;
                p[(2 * t) * RG_TILE + g] = acc[m][b][0]; p[(2 * t + 1) * RG_TILE + g] = acc[m][b][1];
                p[(2 * t) * RG_TILE + g + 8] = acc[m][b][2]; p[(2 * t + 1) * RG_TILE + g + 8] = acc[m][b][3];
            }
        asm volatile("bar.sync 1, %0;" ::"n"(RG_WARPS * 32) : "memory");
        const int tile = (u % tiles) * RG_TILE;
        for (int i = threadIdx.x; i < NB * 8 * RG_TILE; i += RG_WARPS * 32) {
            const int o = i % RG_TILE, n = i / RG_TILE;
            if (n >= n_rows || tile + o >= a.w_rows) continue;
            float v = 0.0f, v2 = 0.0f;
#pragma unroll
            for (int w = 0; w < RG_WARPS; ++w) {
                v += pb[((w * MT) * NB + (n >> 3)) * RG_TILE * 8 + (n & 7) * RG_TILE + o];
                if (DUAL) v2 += pb[((w * MT + MT - 1) * NB + (n >> 3)) * RG_TILE * 8 + (n & 7) * RG_TILE + o];
            }
            const int r = row0 + n;
            if (a.scale) { const float f = a.scale[(size_t) r * a.scale_ld + col_group]; v *= f; v2 *= f; }
            const size_t at = (size_t) r * a.ldy + (size_t) col_group * a.y_group_stride + tile + o;
            if (OUT == LIN_OUT_F32) ((float*) a.y)[at] = v;
            else if (OUT == LIN_OUT_ACT) ((bf16*) a.y)[at] = __float2bfloat16_rn(v);
            else ((bf16*) a.y)[at] = __float2bfloat16_rn(skd::lin_gate<OUT>(v) * v2);
        }
    }
}

// 64 output rows x 32 activation rows per CTA, K in steps of 32 through shared memory; a thread owns 4 x 2 outputs.
constexpr int F_O = 64, F_N = 32, F_K = 32;
template <int OUT>
__global__ void __launch_bounds__(256)
linear_f32_kernel(const LinearArgs a) {
    constexpr bool DUAL = lin_gated(OUT);
    __shared__ float sx[F_N][F_K + 1], sw[DUAL ? 2 : 1][F_O][F_K + 1];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int o0 = blockIdx.x * F_O;
    int group = blockIdx.z, row0 = 0, n_rows = a.rows;
    const int nb0 = blockIdx.y * F_N;
    if (a.segs) {
        if ((int) blockIdx.z >= *a.n_segs) return;
        const RowSegment sg = a.segs[blockIdx.z];
        group = sg.group; row0 = sg.start; n_rows = sg.count;
        if (nb0 >= n_rows) return;
    }
    const size_t goff = (size_t) group * a.w_rows * a.ldw;
    const int col_group = a.segs ? 0 : group;
    const float* x = (const float*) a.x + (size_t) col_group * a.x_group_stride;
    const int to = threadIdx.x & 15, tn = threadIdx.x >> 4;      // outputs to + 16 i, rows tn + 16 j
    float acc[2][4][2] = {};
    for (int k0 = 0; k0 < a.ldw; k0 += F_K) {
        for (int i = threadIdx.x; i < F_N * F_K; i += 256) {
            const int n = i / F_K, k = i % F_K;
            float v = 0.0f;
            if (nb0 + n < n_rows) {
                const int r = row0 + nb0 + n;
                v = x[(size_t) (a.row_index ? a.row_index[r] : r) * a.ldx + k0 + k];
            }
            sx[n][k] = v;
        }
        for (int i = threadIdx.x; i < F_O * F_K; i += 256) {
            const int o = i / F_K, k = i % F_K;
            const bool in = o0 + o < a.w_rows;
            const size_t at = goff + (size_t) (o0 + o) * a.ldw + k0 + k;
            sw[0][o][k] = in ? __bfloat162float(a.w[at]) : 0.0f;
            if (DUAL) sw[DUAL ? 1 : 0][o][k] = in ? __bfloat162float(a.w2[at]) : 0.0f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < F_K; ++k) {
            const float x0 = sx[tn][k], x1 = sx[tn + 16][k];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float w = sw[0][to + 16 * i][k];
                acc[0][i][0] = fmaf(w, x0, acc[0][i][0]); acc[0][i][1] = fmaf(w, x1, acc[0][i][1]);
                if (DUAL) {
                    const float u = sw[DUAL ? 1 : 0][to + 16 * i][k];
                    acc[1][i][0] = fmaf(u, x0, acc[1][i][0]); acc[1][i][1] = fmaf(u, x1, acc[1][i][1]);
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int n = nb0 + tn + 16 * j;
        if (n >= n_rows) continue;
        const int r = row0 + n;
        const float f = a.scale ? a.scale[(size_t) r * a.scale_ld + col_group] : 1.0f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int o = o0 + to + 16 * i;
            if (o >= a.w_rows) continue;
            const float v = acc[0][i][j] * f;
            ((float*) a.y)[(size_t) r * a.ldy + (size_t) col_group * a.y_group_stride + o] = DUAL ? skd::lin_gate<OUT>(v) * (acc[1][i][j] * f) : v;
        }
    }
}

template <typename T>
__global__ void gather_rows_kernel(const T* __restrict__ src, const int32_t* __restrict__ index, T* __restrict__ dst, int ld) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const uint4* s = reinterpret_cast<const uint4*>(src + (size_t) index[blockIdx.x] * ld);
    uint4* d = reinterpret_cast<uint4*>(dst + (size_t) blockIdx.x * ld);
    const int n = ld * (int) sizeof(T) / 16;
    for (int i = threadIdx.x; i < n; i += blockDim.x) d[i] = s[i];
}

template <typename T>
__global__ void to_act_kernel(const float* __restrict__ x, int cols, T* __restrict__ out, int ld) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    for (int i = threadIdx.x; i < ld; i += blockDim.x)
        skd::store_act(out + (size_t) blockIdx.x * ld + i, i < cols ? x[(size_t) blockIdx.x * cols + i] : 0.0f);
}

template <int NB, int OUT>
int32_t run_ring(const LinearArgs& a, cudaStream_t s) {
    constexpr int bytes = ring_smem<lin_gated(OUT) ? 2 : 1, NB>();
    const int64_t units = (int64_t) ((a.w_rows + RG_TILE - 1) / RG_TILE) * (a.segs ? a.max_segs : a.groups);
    constexpr int KB = Ring<lin_gated(OUT) ? 2 : 1>::KB;
    CUtensorMap mw, mw2;
    SK_TRY(tensor_map_k_blocks(&mw, a.w, (int64_t) a.groups * a.w_rows, a.ldw, RG_TILE, KB));
    if (lin_gated(OUT)) SK_TRY(tensor_map_k_blocks(&mw2, a.w2, (int64_t) a.groups * a.w_rows, a.ldw, RG_TILE, KB)); else mw2 = mw;
    SK_TRY(ensure_dynamic_smem((const void*) linear_ring_kernel<NB, OUT>, bytes));
    const int64_t slots = (int64_t) sm_count() * (bytes <= 112 * 1024 ? 2 : 1);
    SK_CUDA(launch_pdl(linear_ring_kernel<NB, OUT>, dim3((unsigned) std::min<int64_t>(units, slots)), dim3(RG_THREADS), bytes, s, mw, mw2, a, device_timeout_flag()));
    return SKAINET_CUDA_OK;
}
template <int NB>
int32_t run_ring_out(const LinearArgs& a, cudaStream_t s) {
    if (a.out == LIN_OUT_SWIGLU) return run_ring<NB, LIN_OUT_SWIGLU>(a, s);
    if (a.out == LIN_OUT_GEGLU) return run_ring<NB, LIN_OUT_GEGLU>(a, s);
    return a.out == LIN_OUT_ACT ? run_ring<NB, LIN_OUT_ACT>(a, s) : run_ring<NB, LIN_OUT_F32>(a, s);
}
template <int OUT>
int32_t run_f32(const LinearArgs& a, cudaStream_t s) {
    const int rows = a.segs ? a.seg_rows : a.rows;
    const dim3 grid((a.w_rows + F_O - 1) / F_O, (rows + F_N - 1) / F_N, a.segs ? a.max_segs : a.groups);
    SK_CUDA(launch_pdl(linear_f32_kernel<OUT>, grid, dim3(256), 0, s, a));
    return SKAINET_CUDA_OK;
}

}  // namespace

int32_t launch_linear_bf16(const LinearArgs& a, cudaStream_t s) {
    if (a.rows <= 0 || a.w_rows <= 0) return SKAINET_CUDA_OK;
    SK_REQUIRE(a.ldw % 64 == 0 && a.ldx % 8 == 0 && a.x_group_stride % 8 == 0, "linear_bf16: leading dimensions %d, %d, %d", a.ldw, a.ldx, a.x_group_stride);
    SK_REQUIRE((a.segs ? a.max_segs : a.groups) <= 65535, "linear_bf16: more than 65535 groups or segments");
    if (a.f32_act) {
        SK_REQUIRE((a.segs ? a.seg_rows : a.rows) <= 65535 * F_N, "linear_bf16: too many rows");
        if (a.out == LIN_OUT_GEGLU) return run_f32<LIN_OUT_GEGLU>(a, s);
        return a.out == LIN_OUT_SWIGLU ? run_f32<LIN_OUT_SWIGLU>(a, s) : run_f32<LIN_OUT_F32>(a, s);
    }
    const int rows = a.segs ? a.seg_rows : a.rows;
    if (rows <= 8) return run_ring_out<1>(a, s);
    if (rows <= RING_MAX_ROWS) return run_ring_out<2>(a, s);
    return launch_gemm_bf16_tc(a, s);
}

int32_t launch_gather_rows(const void* src, const int32_t* index, void* dst, int rows, int ld, bool f32_act, cudaStream_t s) {
    if (rows <= 0) return SKAINET_CUDA_OK;
    if (f32_act) SK_CUDA(launch_pdl(gather_rows_kernel<float>, dim3(rows), dim3(128), 0, s, (const float*) src, index, (float*) dst, ld));
    else SK_CUDA(launch_pdl(gather_rows_kernel<bf16>, dim3(rows), dim3(128), 0, s, (const bf16*) src, index, (bf16*) dst, ld));
    return SKAINET_CUDA_OK;
}

int32_t launch_to_act(const float* x, int rows, int cols, void* out, int ld, bool f32_act, cudaStream_t s) {
    if (rows <= 0) return SKAINET_CUDA_OK;
    if (f32_act) SK_CUDA(launch_pdl(to_act_kernel<float>, dim3(rows), dim3(256), 0, s, x, cols, (float*) out, ld));
    else SK_CUDA(launch_pdl(to_act_kernel<bf16>, dim3(rows), dim3(256), 0, s, x, cols, (bf16*) out, ld));
    return SKAINET_CUDA_OK;
}

}  // namespace sk
