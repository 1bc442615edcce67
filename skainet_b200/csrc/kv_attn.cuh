// Attention over per-head keys and values kept in a ring of positions: grouped query heads, keys and values of different
// sizes, projection biases, unit-rms queries and keys, a chunk mask, a softmax with a sink. No rotation.
//
//   q, k <- x / sqrt(mean(x^2) + eps) per head;   score = (q . k) * scale
//   position i sees j <= i of its own chunk (chunks of `chunk` positions counted from 0; 0: every j <= i)
//   weight_j = exp(score_j) / (exp(sink) + sum_j exp(score_j))
#pragma once
#include "linear_bf16.cuh"
#include "rowmap.cuh"

namespace sk {

struct KvGeom {
    int heads, kv_heads, dim, vdim;
    constexpr int kld() const { return (dim + 15) / 16 * 16; }       // key row and prepared query, zero tail
    constexpr int vcld() const { return (vdim + 15) / 16 * 16; }     // value row, zero tail
    constexpr int out_ld() const { return bf16_ld(heads * vdim); }
    constexpr int proj_rows() const { return (heads + kv_heads) * dim + kv_heads * vdim; }     // q | k | v
};

struct KvCache {                          // one layer's ring of `cap` positions per sequence and key/value head; position p in slot p % cap
    void *k = nullptr, *v = nullptr;      // [sequence][kv_head][cap][kld], [..][vcld], activation type
    int cap = 0;
};

struct KvAttnArgs {
    KvGeom g;
    float scale = 1.0f, eps = 0.0f;
    int chunk = 0;
    const float* proj = nullptr;          // fp32 [row][proj_ld]: q | k | v
    int proj_ld = 0;
    const float *bias = nullptr;          // q | k | v, or null
    const float *sink = nullptr;          // [heads], or null
    KvCache cache;
    void *q = nullptr, *out = nullptr;    // activation type: prepared queries [row][head][kld]; concatenated heads [row][out_ld]
    float* part = nullptr;                // key-split records, kv_part_floats() floats
    int rows = 0;
    RowMap map = {nullptr, -1};
    int kv_bound = 0;                     // bound on the sequence length after this step
    bool f32_act = false;
};

constexpr int KV_PART_RECORDS = 64 * 320;   // (row, head, split) records a split launch may use: [mixed values, vcld | maximum | sum]
inline size_t kv_part_floats(const KvGeom& g) { return (size_t) KV_PART_RECORDS * (g.vcld() + 2); }

// proj -> biases, norms, ring append, attention, concatenated heads in a.out.
int32_t launch_kv_attention(const KvAttnArgs& a, cudaStream_t s);

}  // namespace sk
