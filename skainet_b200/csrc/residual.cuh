// What stands between the sublayers: residual sum and RMS norms of the sublayer outputs (one number, or one per coordinate),
// of the next sublayer's input, of a mixer's gated output, and the depth average over the earlier layers' results. Everything here is fp32; only the copy
// the next linear reads is narrowed.
#pragma once
#include "linear_bf16.cuh"
#include "rowmap.cuh"

namespace sk {

struct SublayerArgs {
    const float* y = nullptr;            // sublayer output [row][cols], or with slot_pos the sum of y[slot_pos[row * top + k]]
    const int32_t* slot_pos = nullptr;
    int top = 1;
    const float* base = nullptr;         // residual stream the sublayer read
    float gain = 1.0f, eps = 0.0f;
    int rows = 0, cols = 0;
    float* state = nullptr;              // base + norm(y); may alias base
    // depth average: with n_states > 0 x = sum_{j < n_states - 1} coef[j] * states[j] + coef[n_states - 1] * state
    const float* coef = nullptr;
    int n_states = 0;
    const float* states = nullptr;       // [n][state_stride]
    size_t state_stride = 0;
    float* x = nullptr;                  // the stream after the average (unused without one)
    void* act = nullptr;                 // the same in the activation type, [row][act_ld]
    int act_ld = 0;
    bool f32_act = false;
};
int32_t launch_sublayer(const SublayerArgs& a, cudaStream_t s);

// Embedding rows of a BF16 table: fp32 into x and state0, and the activation copy.
int32_t launch_embed_rows(const bf16* table, int ld, const int32_t* ids, int rows, int cols, int vocab, float* x, float* state0, void* act, int act_ld,
                          bool f32_act, cudaStream_t s);
// Norms on both sides of a sublayer, with a gain per coordinate:
//   x += norm(y) * post;  x += add (when given);  act = norm(x) * pre (when given)
struct SandwichArgs {
    const float *y = nullptr, *post = nullptr;   // sublayer output [row][cols]
    const float* add = nullptr;                  // [row][cols], a second summand of the stream
    const float* pre = nullptr;                  // gain of the next sublayer's norm; null: act is not written
    float* x = nullptr;                          // residual stream [row][cols]
    void* act = nullptr;
    int act_ld = 0;
    float eps = 0.0f;
    int rows = 0, cols = 0;
    bool f32_act = false;
};
int32_t launch_sandwich(const SandwichArgs& a, cudaStream_t s);

// x = table[id] * scale + sinusoid(position), sine and cosine of position * freq[i] in coordinates 2i and 2i + 1; x0 (may be
// null) takes a copy, act = norm(x) * pre.
struct EmbedPosArgs {
    const bf16* table = nullptr;
    int ld = 0, vocab = 0;
    const int32_t* ids = nullptr;
    float scale = 1.0f, eps = 0.0f;
    const double* freq = nullptr;                // [ceil(cols / 2)]
    RowMap map = {nullptr, -1};
    const float* pre = nullptr;
    float *x = nullptr, *x0 = nullptr;
    void* act = nullptr;
    int act_ld = 0, rows = 0, cols = 0;
    bool f32_act = false;
};
int32_t launch_embed_pos(const EmbedPosArgs& a, cudaStream_t s);

// y = o normed in parts of `part` columns, times gain, gated by silu(z), in the activation type.
//   gate_first: norm(o * silu(z)) * gain[column];  else norm(o) * gain[column % part] * silu(z)
struct GatedNormArgs {
    const float* o = nullptr;              // [row][cols]
    const float* z = nullptr;              // [row][z_ld]
    int z_ld = 0;
    const float* gain = nullptr;
    bool gate_first = false;
    int part = 0, cols = 0, rows = 0;
    float eps = 0.0f;
    void* act = nullptr;
    int act_ld = 0;
    bool f32_act = false;
};
int32_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s);

// act[i] = rmsnorm(x[index ? index[i] : i]) * gain[c] for i < rows
int32_t launch_row_norm(const float* x, const int32_t* index, int rows, int cols, const float* gain, float eps, void* act, int act_ld, bool f32_act, cudaStream_t s);
// act[i] = rmsnorm(x[index ? index[i] : i]) * gain for i < rows
int32_t launch_scalar_norm(const float* x, const int32_t* index, int rows, int cols, float gain, float eps, void* act, int act_ld, bool f32_act, cudaStream_t s);

}  // namespace sk
