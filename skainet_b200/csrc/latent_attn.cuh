// Latent attention: keys and values of all heads are linear images of one small latent per token, so the cache holds the
// latent c (normalised) and a rotated key part shared by all heads, and nothing per head.
//
//   score(i, j, h) = ( q_h . (W_uk,h c_j) + qr_h . kr_j ) * scale = ( (W_uk,h^T q_h) . c_j + qr_h . kr_j ) * scale
//   out(i, h)      = W_uv,h ( sum_j p_ij c_j ) * sigmoid(gate_h)
//
// W_uk is folded into the query and W_uv applied to the mixed latent, in prompts and in decoding alike: attention then reads
// one [latent | rotated part] row per key for all heads, and a cached row is never expanded.
#pragma once
#include "linear_bf16.cuh"
#include "rowmap.cuh"

namespace sk {

constexpr int pad16(int n) { return (n + 15) / 16 * 16; }

struct LatentGeom {                       // what the buffers of a layer are laid out by
    int heads, dim, rot_dim, vdim, kv_rank;
    constexpr int dim_ld() const { return bf16_ld(dim); }                    // q, unrotated part: [row][head][dim_ld]
    constexpr int rank_ld() const { return bf16_ld(kv_rank); }               // mixed latent: [row][head][rank_ld]
    constexpr int rank_pad() const { return pad16(kv_rank); }
    constexpr int key_ld() const { return pad16(kv_rank) + pad16(rot_dim); } // cache row and folded query: [latent, zero tail | rotated part, zero tail]
    constexpr int out_ld() const { return bf16_ld(heads * vdim); }           // concatenated heads
    bool operator<(const LatentGeom& o) const {
        const int a[5] = {heads, dim, rot_dim, vdim, kv_rank}, b[5] = {o.heads, o.dim, o.rot_dim, o.vdim, o.kv_rank};
        for (int i = 0; i < 5; ++i) if (a[i] != b[i]) return a[i] < b[i];
        return false;
    }
};

struct LatentCache {                      // one layer's rows; a ring of `cap` positions per sequence
    void* rows = nullptr;                 // [sequences][cap][key_ld]
    int cap = 0;
};

struct LatentArgs {
    LatentGeom g;
    float scale = 1.0f, eps = 0.0f;
    int window = 0;                       // keys a query sees: itself and window - 1 before it
    const float* proj = nullptr;          // fp32 [row][proj_ld]: q (heads x [dim, rot_dim]) | latent, rotated part (owners only) | gates
    int proj_ld = 0, q_rows = 0;
    bool owner = true;                    // this layer computes and appends the latent
    const float *norm = nullptr;          // gain of the latent's norm
    const float *cos_t = nullptr, *sin_t = nullptr;    // [position][rot_dim / 2]
    LatentCache cache;
    void *qn = nullptr, *qf = nullptr, *mix = nullptr, *out = nullptr;   // activation-type buffers: unrotated q | folded q | mixed latent | gated heads
    float *gates = nullptr;               // sigmoid gates, [row][heads]
    float *part = nullptr;                // key-split records, [row][head][split][rank_pad + 2]
    const bf16 *uk_t = nullptr, *uv = nullptr;   // [heads][kv_rank][dim_ld], [heads][vdim][rank_ld]
    int rows = 0, rows_alloc = 0;
    RowMap map = {nullptr, -1};
    int kv_bound = 0;                     // bound on the sequence length after this step
    bool f32_act = false;
};

constexpr int LATENT_FUSED_ROWS = 4;      // rows up to which the folds of W_uk and W_uv run inside the kernels around attention
constexpr int LATENT_PART_RECORDS = 64 * 320;

// proj -> rotation, latent norm, cache append, gates, folded query, attention over the cache, gated heads in a.out.
int32_t launch_latent_attention(const LatentArgs& a, cudaStream_t s);
// dst[h][r][d] (ld bf16_ld(dim)) = src[h * dim + d][r] (ld bf16_ld(kv_rank)): W_uk per head, transposed
int32_t launch_transpose_heads(const bf16* src, bf16* dst, int heads, int dim, int kv_rank, cudaStream_t s);

}  // namespace sk
