// Linears over BF16 weights (contract: linear_bf16.cuh).
//
//   linear_skinny_kernel  up to 16 activation rows (decode): every weight byte is read once, straight from HBM into the
//                         mma.sync A fragments; bound by the weight stream, the tensor instructions only save the CUDA
//                         cores the unpacking. K is permuted identically in both operands so that a lane's 16-byte load
//                         (8 consecutive k of a row) is two k16 steps' worth of its A fragment.
//   linear_f32_kernel     fp32 activations, fp32 FMA: the 32-bit mode, every row count.
//   gemm_bf16_tc.cu       more rows: tcgen05.
#include "linear_bf16.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr int SK_WARPS = 8, SK_TILE = 16;

// CTA = 16 output rows of one group (or one segment's expert); its eight warps take every eighth k32 step, then the partial
// sums meet in shared memory in fixed order. NB = tiles of 8 activation rows.
template <int NB, int OUT, int U>
__global__ void __launch_bounds__(SK_WARPS * 32)
linear_skinny_kernel(const LinearArgs a) {
    constexpr bool DUAL = OUT == LIN_OUT_SWIGLU;
    constexpr int MT = DUAL ? 2 : 1;
    __shared__ float part[SK_WARPS][MT][NB][SK_TILE * 8 + 4];
    skd::pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int tile = blockIdx.x * SK_TILE;
    const int steps = a.ldw >> 5;
    int group = blockIdx.y, row0 = 0, n_rows = a.rows;
    if (a.segs) {
        skd::pdl_wait();
        if ((int) blockIdx.y >= *a.n_segs) return;
        const RowSegment sg = a.segs[blockIdx.y];
        group = sg.group; row0 = sg.start; n_rows = sg.count;
    }
    const size_t goff = (size_t) group * a.w_rows * a.ldw;
    const bf16* wp[MT][2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const size_t off = goff + (size_t) min(tile + g + 8 * h, a.w_rows - 1) * a.ldw + 8 * t;
        wp[0][h] = a.w + off;
        if (DUAL) wp[MT - 1][h] = a.w2 + off;
    }
    uint4 wr[U][MT][2];
    auto load_w = [&](int st0) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int st = st0 + u * SK_WARPS;
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int h = 0; h < 2; ++h) wr[u][m][h] = st < steps ? skd::ld_stream(wp[m][h] + (size_t) st * 32) : make_uint4(0, 0, 0, 0);
        }
    };
    load_w(warp);                            // weights do not depend on the predecessor: in flight before the wait
    if (!a.segs) skd::pdl_wait();
    const bf16* xp[NB];
    bool live[NB];
#pragma unroll
    for (int b = 0; b < NB; ++b) {
        const int n = b * 8 + g;
        live[b] = n < n_rows;
        const int r = live[b] ? (a.row_index ? a.row_index[row0 + n] : row0 + n) : 0;
        xp[b] = (const bf16*) a.x + (size_t) r * a.ldx + (size_t) (a.segs ? 0 : group) * a.x_group_stride + 8 * t;
    }
    float acc[MT][NB][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[m][b][i] = 0.0f;
    for (int st0 = warp; st0 < steps; st0 += U * SK_WARPS) {
        if (st0 != warp) load_w(st0);
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int st = st0 + u * SK_WARPS;
            if (st >= steps) break;
#pragma unroll
            for (int b = 0; b < NB; ++b) {
                uint4 xv = make_uint4(0, 0, 0, 0);
                if (live[b]) xv = *reinterpret_cast<const uint4*>(xp[b] + (size_t) st * 32);
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    skd::mma_bf16(acc[m][b], wr[u][m][0].x, wr[u][m][1].x, wr[u][m][0].y, wr[u][m][1].y, xv.x, xv.y);
                    skd::mma_bf16(acc[m][b], wr[u][m][0].z, wr[u][m][1].z, wr[u][m][0].w, wr[u][m][1].w, xv.z, xv.w);
                }
            }
        }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int b = 0; b < NB; ++b) {      // acc[0], [1]: output row g, activation rows 2t, 2t+1; acc[2], [3]: output row g + 8
            float* p = part[warp][m][b];
            p[(2 * t) * SK_TILE + g] = acc[m][b][0]; p[(2 * t + 1) * SK_TILE + g] = acc[m][b][1];
            p[(2 * t) * SK_TILE + g + 8] = acc[m][b][2]; p[(2 * t + 1) * SK_TILE + g + 8] = acc[m][b][3];
        }
    __syncthreads();
    for (int i = threadIdx.x; i < NB * 8 * SK_TILE; i += SK_WARPS * 32) {
        const int o = i % SK_TILE, n = i / SK_TILE;
        if (n >= n_rows || tile + o >= a.w_rows) continue;
        float v = 0.0f, v2 = 0.0f;
#pragma unroll
        for (int w = 0; w < SK_WARPS; ++w) {
            v += part[w][0][n >> 3][(n & 7) * SK_TILE + o];
            if (DUAL) v2 += part[w][MT - 1][n >> 3][(n & 7) * SK_TILE + o];
        }
        const int r = row0 + n;
        if (a.scale) { const float f = a.scale[(size_t) r * a.scale_ld + (a.segs ? 0 : group)]; v *= f; v2 *= f; }
        const size_t at = (size_t) r * a.ldy + (size_t) (a.segs ? 0 : group) * a.y_group_stride + tile + o;
        if (OUT == LIN_OUT_F32) ((float*) a.y)[at] = v;
        else if (OUT == LIN_OUT_ACT) ((bf16*) a.y)[at] = __float2bfloat16_rn(v);
        else ((bf16*) a.y)[at] = __float2bfloat16_rn(skd::silu(v) * v2);
    }
}

// 64 output rows x 32 activation rows per CTA, K in steps of 32 through shared memory; a thread owns 4 x 2 outputs.
constexpr int F_O = 64, F_N = 32, F_K = 32;
template <int OUT>
__global__ void __launch_bounds__(256)
linear_f32_kernel(const LinearArgs a) {
    constexpr bool DUAL = OUT == LIN_OUT_SWIGLU;
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
            ((float*) a.y)[(size_t) r * a.ldy + (size_t) col_group * a.y_group_stride + o] = DUAL ? skd::silu(v) * (acc[1][i][j] * f) : v;
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

template <int NB, int OUT, int U>
int32_t run_skinny(const LinearArgs& a, cudaStream_t s) {
    const dim3 grid((a.w_rows + SK_TILE - 1) / SK_TILE, a.segs ? a.max_segs : a.groups);
    SK_CUDA(launch_pdl(linear_skinny_kernel<NB, OUT, U>, grid, dim3(SK_WARPS * 32), 0, s, a));
    return SKAINET_CUDA_OK;
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
        return a.out == LIN_OUT_SWIGLU ? run_f32<LIN_OUT_SWIGLU>(a, s) : run_f32<LIN_OUT_F32>(a, s);
    }
    const int rows = a.segs ? a.seg_rows : a.rows;
    if (rows <= 8) {
        if (a.out == LIN_OUT_SWIGLU) return run_skinny<1, LIN_OUT_SWIGLU, 4>(a, s);
        return a.out == LIN_OUT_ACT ? run_skinny<1, LIN_OUT_ACT, 8>(a, s) : run_skinny<1, LIN_OUT_F32, 8>(a, s);
    }
    if (rows <= SKINNY_MAX_ROWS) {
        if (a.out == LIN_OUT_SWIGLU) return run_skinny<2, LIN_OUT_SWIGLU, 4>(a, s);
        return a.out == LIN_OUT_ACT ? run_skinny<2, LIN_OUT_ACT, 8>(a, s) : run_skinny<2, LIN_OUT_F32, 8>(a, s);
    }
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
