// Gated linear recurrences: per head a state S [kdim][vdim] with one decay per token,
//
//   S <- g S + k u^T,   o = S^T q                                     q, k, v: short causal convolution over time, then silu
//
//   delta rule      q, k unit vectors (q times q_scale);  u = beta (v - (g S)^T k);  g = exp(-exp(A_log) softplus(a + dt_bias))
//   state space     u = dt v, o += D v;  dt = softplus(a + dt_bias);  g = exp(-exp(A_log) dt)          (Mamba-2: q = C, k = B, v = x)
//
// The two share layouts, the convolution, the state store and the kernels; a head reads the q and k of its group. Everything
// is fp32 except what the tile kernels of long prompts take as exact bf16 terms.
#pragma once
#include "linear_bf16.cuh"
#include "rowmap.cuh"

namespace sk {

constexpr int RECUR_MAX_KDIM = 512;

struct RecurGeom {
    int heads, groups;                     // value heads; query/key heads
    int kdim, vdim, taps;
    bool delta;
    constexpr int vld() const { return (vdim + 3) / 4 * 4; }
    constexpr int q_dim() const { return groups * kdim; }
    constexpr int v_dim() const { return heads * vdim; }
    constexpr int conv_dim() const { return 2 * q_dim() + v_dim(); }
    constexpr size_t state_size() const { return (size_t) heads * kdim * vld(); }      // floats of one sequence
    constexpr size_t tail_size() const { return (size_t) taps * conv_dim(); }
};

struct RecurArgs {
    RecurGeom g;
    const float* proj = nullptr;           // fp32 [row][proj_ld]
    int proj_ld = 0, conv_off = 0;         // the convolution's channels are columns conv_off .. conv_off + conv_dim
    int q_off = 0, k_off = 0, v_off = 0;   // channels, counted from conv_off
    int dt_off = 0, beta_off = 0;          // columns of the decay's and of beta's pre-activations, one per head
    const float *conv_w = nullptr, *conv_b = nullptr;     // [channel][taps], oldest input first; [channel] or null
    const float *a_log = nullptr, *dt_bias = nullptr, *d = nullptr;
    float q_scale = 1.0f;
    float* state = nullptr;                // [sequence][head][kdim][vld]
    float* tail = nullptr;                 // [sequence][taps][conv_dim]: the convolution's inputs, position p in slot p % taps
    float* out = nullptr;                  // [row][heads * vdim]
    int rows = 0, rows_alloc = 0;
    RowMap map = {nullptr, -1};            // seq < 0: one token of each of `rows` sequences; else `rows` tokens of one
    bool f32_act = false;
    // work buffers of the tile kernels, null when the model never runs them
    void* work = nullptr;
};

// A sequence at position 0 starts from a zero state and zero inputs whatever its store holds.
int32_t launch_recurrence(const RecurArgs& a, cudaStream_t s);

// Bytes of RecurArgs::work for passes of up to `rows` tokens; 0 when the tile kernels do not take the geometry.
size_t recur_work_bytes(const RecurGeom& g, int rows);

// recurrence_chunk.cu: `rows` tokens of one sequence
constexpr int RECUR_CHUNK_MIN_ROWS = 12;
int32_t launch_recur_chunks(const RecurArgs& a, cudaStream_t s);

}  // namespace sk

#ifdef __CUDACC__
namespace skd {

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// Input of convolution channel c at position p; rows of the pass start at position pos0 in row row0.
__device__ __forceinline__ float conv_input(const sk::RecurArgs& a, const float* tail, int row0, int pos0, int p, int c) {
    if (p < 0) return 0.0f;
    if (p >= pos0) return a.proj[(size_t) (row0 + p - pos0) * a.proj_ld + a.conv_off + c];
    return tail[(size_t) (p % a.g.taps) * a.g.conv_dim() + c];
}

}  // namespace skd
#endif
