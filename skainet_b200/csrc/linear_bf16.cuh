// Linears over BF16 weights: y[n][o] = sum_k x[n][k] * W[o][k] with 32-bit accumulation, plain, per group (one matrix per
// attention head) or per routed segment (one matrix per expert), with the epilogues a decoder step needs.
//
// Weights are row-major [rows][ld] with ld = bf16_ld(cols), a multiple of 64 whose tail is zero, so that every kernel can
// walk K in whole steps; activation rows have the same padding, and the owner of an activation buffer keeps its tail zero.
// Activations are bf16, or fp32 when the whole model runs in 32-bit (the weights then stay bf16, which fp32 holds exactly).
#pragma once
#include "common.cuh"

#include <cuda_bf16.h>

namespace sk {

typedef __nv_bfloat16 bf16;

constexpr int bf16_ld(int cols) { return (cols + 63) / 64 * 64; }

// A run of activation rows that share one weight matrix: rows [start, start + count) take matrix `group`.
struct RowSegment { int32_t group, start, count, pad; };

// fp32 rows | activation type | silu(W x) * (W2 x) | gelu(W x) * (W2 x), tanh form; the last two in the activation type
enum { LIN_OUT_F32 = 0, LIN_OUT_ACT = 1, LIN_OUT_SWIGLU = 2, LIN_OUT_GEGLU = 3 };
constexpr bool lin_gated(int out) { return out == LIN_OUT_SWIGLU || out == LIN_OUT_GEGLU; }

struct LinearArgs {
    const bf16 *w = nullptr, *w2 = nullptr;      // w2: the up matrix of the gated outputs
    int w_rows = 0;                              // output rows of one group
    int ldw = 0;                                 // padded K
    int groups = 1;                              // matrices stacked in w, [groups][w_rows][ldw]
    const void* x = nullptr;                     // activation rows
    int ldx = 0, x_group_stride = 0;             // elements; group g reads columns [g * x_group_stride, + ldw)
    int x_rows_alloc = 0;                        // rows the buffer behind x holds
    int rows = 0;
    void* y = nullptr;
    int ldy = 0, y_group_stride = 0;             // group g writes columns [g * y_group_stride, + w_rows)
    const float* scale = nullptr;                // optional factor of the products, scale[row * scale_ld + group]
    int scale_ld = 0;
    // routed form: segments in device memory instead of groups x rows; row_index maps a sorted row to its row in x (may be null)
    const RowSegment* segs = nullptr;
    const int32_t* n_segs = nullptr;
    int max_segs = 0, seg_rows = 0;              // bound on the number of segments and on their length
    const int32_t* row_index = nullptr;
    bool f32_act = false;
    int out = LIN_OUT_F32;
};

int32_t launch_linear_bf16(const LinearArgs& a, cudaStream_t s);

// Rows (plain and per-group) up to which the streaming kernel is used, and the segment length it takes.
constexpr int RING_MAX_ROWS = 16, RING_SEG_ROWS = 8;

// gemm_bf16_tc.cu
int32_t launch_gemm_bf16_tc(const LinearArgs& a, cudaStream_t s);
// dst[i][:] = src[index[i]][:] for i < rows; ld elements of the activation type per row (a multiple of 8)
int32_t launch_gather_rows(const void* src, const int32_t* index, void* dst, int rows, int ld, bool f32_act, cudaStream_t s);
// fp32 [rows][cols] -> activation rows [rows][ld], tail zeroed
int32_t launch_to_act(const float* x, int rows, int cols, void* out, int ld, bool f32_act, cudaStream_t s);

}  // namespace sk

#ifdef __CUDACC__
namespace skd {

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
// 0.5 z (1 + tanh(u)) = z / (1 + exp(-2u)), u = sqrt(2/pi) (z + 0.044715 z^3)
__device__ __forceinline__ float gelu_tanh(float z) { return z / (1.0f + expf(-1.5957691216057308f * z * (1.0f + 0.044715f * z * z))); }
template <int OUT> __device__ __forceinline__ float lin_gate(float v) { return OUT == sk::LIN_OUT_GEGLU ? gelu_tanh(v) : silu(v); }
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ void store_act(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void store_act(float* p, float v) { *p = v; }
__device__ __forceinline__ float load_act(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float load_act(const float* p) { return *p; }
__device__ __forceinline__ float bf16_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
// c += a (16 x 16, row major) * b (16 x 8)
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

}  // namespace skd
#endif
