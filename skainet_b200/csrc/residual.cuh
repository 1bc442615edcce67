// What stands between the sublayers of a design whose norms sit on the sublayer outputs: residual sum, one-number RMS norm,
// depth average over the earlier layers' results. Everything here is fp32; only the copy the next linear reads is narrowed.
#pragma once
#include "linear_bf16.cuh"

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
// act[i] = rmsnorm(x[index ? index[i] : i]) * gain for i < rows
int32_t launch_scalar_norm(const float* x, const int32_t* index, int rows, int cols, float gain, float eps, void* act, int act_ld, bool f32_act, cudaStream_t s);

}  // namespace sk
