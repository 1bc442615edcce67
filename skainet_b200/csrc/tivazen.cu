// The Tivazen design of the decoder runtime (contract: include/skainet_cuda_tivazen.h). Per layer
//
//   q | latent, key part | gates (one merged linear)  ->  latent attention (latent_attn.cuh)  ->  o  ->  x += norm(.)
//   gate, up -> silu * up -> down, or router -> experts on their rows  ->  x += norm(.)  ->  weighted sum of all states
//
// The residual stream and the states X_0 (embedding) .. X_L of the rows in flight are fp32; linears read a narrowed copy.
// Decode steps and prompt passes run the same body over rows; only the row map and the kernels the row count selects differ.
#include "decoder.cuh"
#include "latent_attn.cuh"
#include "linear_bf16.cuh"
#include "moe.cuh"
#include "residual.cuh"
#include "tma.cuh"
#include "../../include/skainet_cuda_tivazen.h"

#include <algorithm>
#include <cmath>
#include <map>
#include <set>
#include <tuple>
#include <vector>

namespace sk {

namespace {

constexpr int PREFILL_ROWS = 1024;       // rows of one prompt pass unless the configuration says otherwise

// Seeded noise in a sequence's cache rows; the zero tails stay zero.
template <typename T>
__global__ void fill_latent_kernel(T* rows, int cap, int key_ld, int rank, int rank_pad, int rot, uint64_t seed) {
    const int64_t n = (int64_t) cap * key_ld;
    for (int64_t i = blockIdx.x * (int64_t) blockDim.x + threadIdx.x; i < n; i += (int64_t) gridDim.x * blockDim.x) {
        const int c = (int) (i % key_ld);
        if (c >= rank && (c < rank_pad || c >= rank_pad + rot)) continue;
        uint64_t z = (seed + (uint64_t) i) * 0x9E3779B97F4A7C15ull;
        z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull; z ^= z >> 27;
        skd::store_act(rows + i, ((float) (z & 0xFFFF) / 32768.0f - 1.0f) * 1.7f);
    }
}

struct AttnBuffers { void *qn = nullptr, *qf = nullptr, *mix = nullptr, *out = nullptr; };

struct TvLayer {
    skainet_tivazen_layer c;
    int owner = 0;                        // layer whose cache is read
    LatentGeom geom;
    int q_rows = 0, proj_rows = 0;
    Weight *proj = nullptr, *uk = nullptr, *uv = nullptr, *o = nullptr, *router = nullptr, *gate = nullptr, *up = nullptr, *down = nullptr;
    float norm1 = 1.0f, norm2 = 1.0f;
    float *dkv_norm = nullptr, *depth = nullptr;
    LatentCache cache;
    const float *cos_t = nullptr, *sin_t = nullptr;
    AttnBuffers buf;
    void* hidden = nullptr;
};

const bf16* data(const Weight* w) { return (const bf16*) w->qs; }

struct Tivazen : Decoder {
    skainet_tivazen_config cfg;
    bool f32 = false;
    int act_size = 2, width_ld = 0, max_slots = 0;
    std::vector<TvLayer> layers;
    Weight *embed = nullptr, *head = nullptr;
    float final_norm = 1.0f;
    std::set<std::tuple<int, int, int>> missing;       // (layer, matrix | 100 + vector, expert) not set yet
    // per row in flight
    float *x = nullptr, *states = nullptr, *proj = nullptr, *gates = nullptr, *y = nullptr, *part = nullptr, *z = nullptr;
    void *act = nullptr, *act_sorted = nullptr, *act_final = nullptr;
    int32_t* want = nullptr;
    RouteBuffers route;

    ~Tivazen() override {
        for (auto& L : layers) for (Weight* w : {L.proj, L.uk, L.uv, L.o, L.router, L.gate, L.up, L.down}) if (w) weight_release(w);
        if (embed) weight_release(embed);
        if (head) weight_release(head);
    }

    int32_t create(const skainet_tivazen_layer* ls);
    int32_t body(int rows, RowMap map, int kv_bound, cudaStream_t s);
    int32_t feed_forward(TvLayer& L, int rows, cudaStream_t s);
    int32_t head_rows(const int32_t* index_dev, int n, cudaStream_t s);

    int32_t finalize() override {
        if (!missing.empty()) {
            const auto& k = *missing.begin();
            const int w = std::get<1>(k);
            set_error("tivazen_finalize: %d tensors missing, first: %s %d of layer %d, expert %d", (int) missing.size(), w >= 100 ? "vector" : "matrix", w % 100,
                      std::get<0>(k), std::get<2>(k));
            return SKAINET_CUDA_ERR_INVALID;
        }
        return SKAINET_CUDA_OK;
    }
    int32_t enqueue_decode(int batch, int kv_bound, cudaStream_t s) override {
        SK_TRY(body(batch, RowMap{pos, -1}, kv_bound, s));
        return head_rows(nullptr, batch, s);
    }
    int32_t enqueue_prompt(int rows, int seq, int kv_bound, cudaStream_t s) override { return body(rows, RowMap{pos, seq}, kv_bound, s); }
    int32_t enqueue_head(const int32_t* rows, int n, cudaStream_t s) override {
        SK_CUDA(cudaMemcpyAsync(want, rows, sizeof(int32_t) * n, cudaMemcpyHostToDevice, s));
        return head_rows(want, n, s);
    }
    int32_t fill_context(int seq, int n, uint64_t seed) override {
        (void) n;
        for (size_t i = 0; i < layers.size(); ++i) {
            TvLayer& L = layers[i];
            if (L.owner != (int) i) continue;
            const LatentGeom& g = L.geom;
            const size_t off = (size_t) seq * L.cache.cap * g.key_ld();
            const uint64_t sd = seed + 977ull * i + 31ull * seq;
            if (f32) fill_latent_kernel<float><<<592, 256, 0, stream>>>((float*) L.cache.rows + off, L.cache.cap, g.key_ld(), g.kv_rank, g.rank_pad(), g.rot_dim, sd);
            else fill_latent_kernel<bf16><<<592, 256, 0, stream>>>((bf16*) L.cache.rows + off, L.cache.cap, g.key_ld(), g.kv_rank, g.rank_pad(), g.rot_dim, sd);
        }
        SK_CUDA(cudaGetLastError());
        return SKAINET_CUDA_OK;
    }
    // Weights once (of a routed layer at most batch * top experts), the visible cache rows, the states of the depth averages.
    int64_t step_bytes(int batch) const override {
        int64_t bytes = head->packed_bytes + (int64_t) batch * d_model * 2;
        for (size_t i = 0; i < layers.size(); ++i) {
            const TvLayer& L = layers[i];
            for (const Weight* w : {L.proj, L.uk, L.uv, L.o, L.router}) if (w) bytes += w->packed_bytes;
            const int64_t mlp = L.gate ? L.gate->packed_bytes + L.up->packed_bytes + L.down->packed_bytes : 0;
            bytes += L.c.mlp == SKAINET_TV_MLP_MOE ? mlp / L.c.experts * std::min(L.c.experts, batch * L.c.top) : mlp;
            for (int b = 0; b < batch; ++b)
                bytes += (int64_t) std::min(L.c.window, host_pos[b] + 1) * L.geom.key_ld() * act_size + (int64_t) (i + 2) * d_model * 4;
        }
        return bytes;
    }
    const float* buffer(int which) const override {
        if (which == 0) return x;
        if (which == 1) return proj;
        return which >= 16 && which < 17 + (int) layers.size() ? states + (size_t) (which - 16) * max_rows * d_model : nullptr;
    }
};

int32_t Tivazen::create(const skainet_tivazen_layer* ls) {
    const size_t R = max_rows, A = act_size;
    std::map<LatentGeom, AttnBuffers> attn;
    std::map<std::pair<int, int>, void*> hidden;                       // (inner size, slots per row)
    std::map<std::pair<double, int>, std::pair<float*, float*>> rope;
    int max_proj = 0, max_heads = 0, max_experts = 0, max_rank = 0;
    auto matrix = [&](Weight** w, int rows, int cols) -> int32_t { return weight_alloc(SKAINET_ENC_BF16, rows, cols, w); };
    max_slots = max_rows;
    for (int i = 0; i < cfg.n_layers; ++i) if (ls[i].mlp == SKAINET_TV_MLP_MOE) max_slots = std::max(max_slots, max_rows * ls[i].top);
    for (int i = 0; i < cfg.n_layers; ++i) {
        TvLayer& L = layers[i];
        const skainet_tivazen_layer& c = L.c = ls[i];
        L.owner = c.kv_from < 0 ? i : c.kv_from;
        L.geom = LatentGeom{c.heads, c.dim, c.rot_dim, c.vdim, c.kv_rank};
        const LatentGeom& g = L.geom;
        const bool own = L.owner == i;
        L.q_rows = c.heads * (c.dim + c.rot_dim);
        L.proj_rows = L.q_rows + (own ? c.kv_rank + c.rot_dim : 0) + c.heads;
        SK_TRY(matrix(&L.proj, L.proj_rows, d_model)); SK_TRY(matrix(&L.uk, c.heads * c.kv_rank, c.dim)); SK_TRY(matrix(&L.uv, c.heads * c.vdim, c.kv_rank));
        SK_TRY(matrix(&L.o, d_model, c.heads * c.vdim));
        for (int w : {SKAINET_TV_Q, SKAINET_TV_UK, SKAINET_TV_UV, SKAINET_TV_G, SKAINET_TV_O}) missing.insert({i, w, 0});
        for (int v : {SKAINET_TV_NORM1, SKAINET_TV_DEPTH}) missing.insert({i, 100 + v, 0});
        if (own) {
            missing.insert({i, SKAINET_TV_DKV, 0}); missing.insert({i, 100 + SKAINET_TV_DKV_NORM, 0});
            SK_TRY(alloc(&L.dkv_norm, c.kv_rank));
            // a ring: the keys the first row of a pass still sees, and the pass's own rows, for the widest window that reads it
            int window = c.window;
            for (int j = i + 1; j < cfg.n_layers; ++j) if (ls[j].kv_from == i) window = std::max(window, ls[j].window);
            L.cache.cap = (int) std::min<int64_t>(max_seq, (int64_t) window - 1 + max_rows);
            SK_TRY(alloc(&L.cache.rows, (size_t) max_batch * L.cache.cap * g.key_ld() * A));
        } else L.cache = layers[L.owner].cache;
        SK_TRY(alloc(&L.depth, i + 2));
        if (c.mlp != SKAINET_TV_MLP_NONE) {
            const int E = c.mlp == SKAINET_TV_MLP_MOE ? c.experts : 1, slots = c.mlp == SKAINET_TV_MLP_MOE ? c.top : 1;
            SK_TRY(matrix(&L.gate, E * c.ff, d_model)); SK_TRY(matrix(&L.up, E * c.ff, d_model)); SK_TRY(matrix(&L.down, E * d_model, c.ff));
            for (int e = 0; e < E; ++e) for (int w : {SKAINET_TV_GATE, SKAINET_TV_UP, SKAINET_TV_DOWN}) missing.insert({i, w, e});
            missing.insert({i, 100 + SKAINET_TV_NORM2, 0});
            if (c.mlp == SKAINET_TV_MLP_MOE) { SK_TRY(matrix(&L.router, E, d_model)); missing.insert({i, SKAINET_TV_ROUTER, 0}); max_experts = std::max(max_experts, E); }
            void*& h = hidden[{c.ff, slots}];
            if (!h) SK_TRY(alloc(&h, R * slots * bf16_ld(c.ff) * A));
            L.hidden = h;
        }
        AttnBuffers& b = attn[g];
        if (!b.qn) {
            SK_TRY(alloc(&b.qn, R * c.heads * g.dim_ld() * A)); SK_TRY(alloc(&b.qf, R * c.heads * g.key_ld() * A));
            SK_TRY(alloc(&b.mix, R * c.heads * g.rank_ld() * A)); SK_TRY(alloc(&b.out, R * g.out_ld() * A));
        }
        L.buf = b;
        auto& t = rope[{c.rope_base, c.rot_dim}];
        if (!t.first) {                                   // rotation factors: angle = pos * base^(-2i/n) in double, rounded once
            const int half = c.rot_dim / 2;
            std::vector<float> cs((size_t) max_seq * half), sn(cs.size());
            for (int k = 0; k < half; ++k) {
                const double f = pow(c.rope_base, -2.0 * (double) k / (double) c.rot_dim);
                for (int p = 0; p < max_seq; ++p) { cs[(size_t) p * half + k] = (float) cos((double) p * f); sn[(size_t) p * half + k] = (float) sin((double) p * f); }
            }
            SK_TRY(alloc(&t.first, cs.size())); SK_TRY(alloc(&t.second, sn.size()));
            SK_CUDA(cudaMemcpy(t.first, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice));
            SK_CUDA(cudaMemcpy(t.second, sn.data(), sn.size() * 4, cudaMemcpyHostToDevice));
        }
        L.cos_t = t.first; L.sin_t = t.second;
        max_proj = std::max(max_proj, L.proj_rows); max_heads = std::max(max_heads, c.heads); max_rank = std::max(max_rank, g.rank_pad());
    }
    SK_TRY(matrix(&embed, vocab, d_model)); SK_TRY(matrix(&head, vocab, d_model));
    missing.insert({-1, SKAINET_TV_EMBED, 0}); missing.insert({-1, SKAINET_TV_HEAD, 0}); missing.insert({-1, 100 + SKAINET_TV_FINAL_NORM, 0});
    SK_TRY(alloc(&x, R * d_model)); SK_TRY(alloc(&states, R * d_model * (cfg.n_layers + 1))); SK_TRY(alloc(&proj, R * max_proj)); SK_TRY(alloc(&gates, R * max_heads));
    SK_TRY(alloc(&y, (size_t) max_slots * d_model)); SK_TRY(alloc(&part, (size_t) LATENT_PART_RECORDS * (max_rank + 2)));
    SK_TRY(alloc(&act, R * width_ld * A)); SK_TRY(alloc(&act_final, (size_t) logits_rows * width_ld * A)); SK_TRY(alloc(&want, logits_rows));
    if (max_experts) {
        SK_TRY(alloc(&act_sorted, (size_t) max_slots * width_ld * A)); SK_TRY(alloc(&z, R * max_experts));
        SK_TRY(alloc(&route.slot_expert, max_slots)); SK_TRY(alloc(&route.slot_weight, max_slots)); SK_TRY(alloc(&route.slot_pos, max_slots));
        SK_TRY(alloc(&route.sorted_row, max_slots)); SK_TRY(alloc(&route.sorted_weight, max_slots));
        SK_TRY(alloc(&route.segs, 2 * (size_t) max_slots + 1)); SK_TRY(alloc(&route.n_segs, 1));
    }
    return SKAINET_CUDA_OK;
}

// The layer's feed-forward of act: y[row][width], or y[sorted position][width] when routed.
int32_t Tivazen::feed_forward(TvLayer& L, int rows, cudaStream_t s) {
    const skainet_tivazen_layer& c = L.c;
    LinearArgs l;
    l.f32_act = f32; l.x = act; l.ldx = l.ldw = width_ld; l.x_rows_alloc = max_rows; l.rows = rows;
    if (c.mlp == SKAINET_TV_MLP_MOE) {
        l.w = data(L.router); l.w_rows = c.experts; l.y = z; l.ldy = c.experts;
        SK_TRY(launch_linear_bf16(l, s));
        // short runs stream their expert's weights past a few rows at a time, long ones go to the tensor-core tiles
        const int slots = rows * c.top, per = slots / c.experts;
        const int seg_rows = f32 ? 32 : per <= 4 ? RING_SEG_ROWS : per <= 24 ? 32 : 128;
        SK_TRY(launch_route(z, rows, c.experts, c.top, seg_rows, route, s));
        l.segs = route.segs; l.n_segs = route.n_segs; l.seg_rows = seg_rows; l.max_segs = route_max_segs(slots, c.experts, seg_rows);
        l.groups = c.experts; l.rows = slots; l.scale = route.sorted_weight; l.scale_ld = 1;      // the weight multiplies the expert's input
        if (f32 || seg_rows <= RING_MAX_ROWS) l.row_index = route.sorted_row;
        else {
            SK_TRY(launch_gather_rows(act, route.sorted_row, act_sorted, slots, width_ld, f32, s));
            l.x = act_sorted; l.x_rows_alloc = max_slots;
        }
    }
    l.w = data(L.gate); l.w2 = data(L.up); l.w_rows = c.ff; l.y = L.hidden; l.ldy = bf16_ld(c.ff); l.out = LIN_OUT_SWIGLU;
    SK_TRY(launch_linear_bf16(l, s));
    l.w = data(L.down); l.w2 = nullptr; l.w_rows = d_model; l.ldw = l.ldx = bf16_ld(c.ff); l.x = L.hidden; l.y = y; l.ldy = d_model; l.out = LIN_OUT_F32;
    l.x_rows_alloc = c.mlp == SKAINET_TV_MLP_MOE ? max_rows * c.top : max_rows;
    l.scale = nullptr; l.row_index = nullptr;
    return launch_linear_bf16(l, s);
}

int32_t Tivazen::body(int rows, RowMap map, int kv_bound, cudaStream_t s) {
    const size_t stride = (size_t) max_rows * d_model;
    SK_TRY(launch_embed_rows(data(embed), width_ld, cur_token, rows, d_model, vocab, x, states, act, width_ld, f32, s));
    for (size_t i = 0; i < layers.size(); ++i) {
        TvLayer& L = layers[i];
        const skainet_tivazen_layer& c = L.c;
        LinearArgs l;
        l.f32_act = f32; l.x_rows_alloc = max_rows; l.rows = rows;
        l.w = data(L.proj); l.w_rows = L.proj_rows; l.ldw = l.ldx = width_ld; l.x = act; l.y = proj; l.ldy = L.proj_rows;
        SK_TRY(launch_linear_bf16(l, s));
        LatentArgs a;
        a.g = L.geom; a.scale = c.scale; a.eps = cfg.eps; a.window = c.window; a.proj = proj; a.proj_ld = L.proj_rows; a.q_rows = L.q_rows;
        a.owner = L.owner == (int) i; a.norm = L.dkv_norm; a.cos_t = L.cos_t; a.sin_t = L.sin_t; a.cache = L.cache;
        a.qn = L.buf.qn; a.qf = L.buf.qf; a.mix = L.buf.mix; a.out = L.buf.out; a.gates = gates; a.part = part;
        a.uk_t = data(L.uk); a.uv = data(L.uv); a.rows = rows; a.rows_alloc = max_rows; a.map = map; a.kv_bound = kv_bound; a.f32_act = f32;
        SK_TRY(launch_latent_attention(a, s));
        l.w = data(L.o); l.w_rows = d_model; l.ldw = l.ldx = L.geom.out_ld(); l.x = L.buf.out; l.y = y; l.ldy = d_model;
        SK_TRY(launch_linear_bf16(l, s));
        SublayerArgs n;
        n.y = y; n.base = x; n.gain = L.norm1; n.eps = cfg.eps; n.rows = rows; n.cols = d_model; n.state = states + (i + 1) * stride;
        n.act = act; n.act_ld = width_ld; n.f32_act = f32;
        if (c.mlp != SKAINET_TV_MLP_NONE) {
            SK_TRY(launch_sublayer(n, s));
            SK_TRY(feed_forward(L, rows, s));
            n.base = n.state; n.gain = L.norm2;
            if (c.mlp == SKAINET_TV_MLP_MOE) { n.slot_pos = route.slot_pos; n.top = c.top; }
        }
        n.coef = L.depth; n.n_states = (int) i + 2; n.states = states; n.state_stride = stride; n.x = x;
        SK_TRY(launch_sublayer(n, s));
    }
    return SKAINET_CUDA_OK;
}

int32_t Tivazen::head_rows(const int32_t* index_dev, int n, cudaStream_t s) {
    SK_TRY(launch_scalar_norm(x, index_dev, n, d_model, final_norm, cfg.eps, act_final, width_ld, f32, s));
    LinearArgs l;
    l.f32_act = f32; l.x_rows_alloc = logits_rows; l.rows = n; l.w = data(head); l.w_rows = vocab; l.ldw = l.ldx = width_ld; l.x = act_final; l.y = logits; l.ldy = vocab;
    return launch_linear_bf16(l, s);
}

// Where a matrix of the checkpoint goes: destination, first row, and the shape it must have.
struct Slot { Weight* w = nullptr; int row0 = 0, rows = 0, cols = 0; };
Slot slot_of(Tivazen& m, int layer, int which, int expert) {
    Slot r;
    if (which == SKAINET_TV_EMBED || which == SKAINET_TV_HEAD) { r.w = which == SKAINET_TV_EMBED ? m.embed : m.head; r.rows = m.vocab; r.cols = m.d_model; return r; }
    TvLayer& L = m.layers[layer];
    const auto& c = L.c;
    const bool own = L.owner == layer;
    switch (which) {
        case SKAINET_TV_Q:   r.w = L.proj; r.rows = L.q_rows; r.cols = m.d_model; break;
        case SKAINET_TV_DKV: if (own) { r.w = L.proj; r.row0 = L.q_rows; r.rows = c.kv_rank + c.rot_dim; r.cols = m.d_model; } break;
        case SKAINET_TV_G:   r.w = L.proj; r.row0 = L.proj_rows - c.heads; r.rows = c.heads; r.cols = m.d_model; break;
        case SKAINET_TV_UK:  r.w = L.uk; r.rows = c.heads * c.dim; r.cols = c.kv_rank; break;
        case SKAINET_TV_UV:  r.w = L.uv; r.rows = c.heads * c.vdim; r.cols = c.kv_rank; break;
        case SKAINET_TV_O:   r.w = L.o; r.rows = m.d_model; r.cols = c.heads * c.vdim; break;
        case SKAINET_TV_ROUTER: r.w = L.router; r.rows = c.experts; r.cols = m.d_model; break;
        case SKAINET_TV_GATE: r.w = L.gate; r.row0 = expert * c.ff; r.rows = c.ff; r.cols = m.d_model; break;
        case SKAINET_TV_UP:   r.w = L.up; r.row0 = expert * c.ff; r.rows = c.ff; r.cols = m.d_model; break;
        case SKAINET_TV_DOWN: r.w = L.down; r.row0 = expert * m.d_model; r.rows = m.d_model; r.cols = c.ff; break;
        default: break;
    }
    return r;
}

}  // namespace

}  // namespace sk

using namespace sk;

extern "C" {

int32_t skainet_cuda_tivazen_create(const skainet_tivazen_config* cfg, const skainet_tivazen_layer* ls, skainet_model_t* out) {
    SK_REQUIRE(cfg && ls && out, "tivazen_create: null argument");
    *out = 0;
    const auto& c = *cfg;
    SK_REQUIRE(c.n_layers > 0 && c.width > 0 && c.vocab > 0, "tivazen_create: non-positive dimension");
    SK_REQUIRE(c.max_seq >= 1 && c.max_batch >= 1 && c.max_batch <= 4096 && c.prefill_rows >= 0 && c.prefill_rows <= 65535, "tivazen_create: max_seq %d, max_batch %d, prefill_rows %d", c.max_seq, c.max_batch, c.prefill_rows);
    for (int i = 0; i < c.n_layers; ++i) {
        const auto& l = ls[i];
        SK_REQUIRE(l.heads > 0 && l.heads <= LATENT_PART_RECORDS / LATENT_FUSED_ROWS && l.dim > 0 && l.vdim > 0 && l.kv_rank > 0, "tivazen_create: layer %d: bad attention sizes", i);
        SK_REQUIRE(l.rot_dim > 0 && l.rot_dim % 2 == 0, "tivazen_create: layer %d: rot_dim %d must be even", i, l.rot_dim);
        SK_REQUIRE(l.window >= 1 && l.rope_base > 0, "tivazen_create: layer %d: window %d, rope base %g", i, l.window, l.rope_base);
        SK_REQUIRE(l.mlp >= SKAINET_TV_MLP_NONE && l.mlp <= SKAINET_TV_MLP_MOE && (l.mlp == SKAINET_TV_MLP_NONE || l.ff > 0), "tivazen_create: layer %d: bad feed-forward", i);
        if (l.mlp == SKAINET_TV_MLP_MOE) SK_REQUIRE(l.experts >= 1 && l.experts <= ROUTE_MAX_EXPERTS && l.top >= 1 && l.top <= l.experts, "tivazen_create: layer %d: %d of %d experts", i, l.top, l.experts);
        if (l.kv_from >= 0) {
            SK_REQUIRE(l.kv_from < i && ls[l.kv_from].kv_from < 0, "tivazen_create: layer %d takes its cache from layer %d, which has none of its own before it", i, l.kv_from);
            const auto& o = ls[l.kv_from];
            SK_REQUIRE(o.kv_rank == l.kv_rank && o.rot_dim == l.rot_dim && o.rope_base == l.rope_base, "tivazen_create: layers %d and %d share a cache and differ in kv_rank or rotation", i, l.kv_from);
        }
    }
    SK_TRY(ensure_device());
    Tivazen* m = new Tivazen();
    m->cfg = c;
    m->f32 = c.act_f32 != 0; m->act_size = m->f32 ? 4 : 2;
    m->vocab = m->vocab_l = c.vocab; m->d_model = c.width; m->width_ld = bf16_ld(c.width); m->max_seq = c.max_seq; m->max_batch = c.max_batch;
    m->max_rows = std::max(c.max_batch, std::min(c.prefill_rows ? c.prefill_rows : PREFILL_ROWS, c.max_seq));
    m->layers.resize(c.n_layers);
    int32_t st = decoder_init(m);
    if (st == SKAINET_CUDA_OK) st = m->create(ls);
    if (st != SKAINET_CUDA_OK) { decoder_destroy(m); return st; }
    *out = decoder_handle(m);
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_tivazen_set_weight(skainet_model_t h, int32_t layer, int32_t which, int32_t expert, skainet_weight_t wh) {
    Tivazen* m = design_from_handle<Tivazen>(h, __func__);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    Weight* w = weight_from_handle(wh);
    if (!w) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(!m->finalized, "tivazen_set_weight: model already finalized");
    const bool model_level = which == SKAINET_TV_EMBED || which == SKAINET_TV_HEAD;
    SK_REQUIRE(model_level || (layer >= 0 && layer < m->cfg.n_layers), "tivazen_set_weight: layer %d out of range", layer);
    const bool routed = !model_level && m->layers[layer].c.mlp == SKAINET_TV_MLP_MOE && which >= SKAINET_TV_GATE;
    SK_REQUIRE(!routed || (expert >= 0 && expert < m->layers[layer].c.experts), "tivazen_set_weight: expert %d out of range", expert);
    const int e = routed ? expert : 0;
    const Slot t = slot_of(*m, layer, which, e);
    SK_REQUIRE(t.w != nullptr, "tivazen_set_weight: layer %d has no matrix %d", layer, which);
    SK_REQUIRE(w->enc == SKAINET_ENC_BF16 && w->rows == t.rows && w->cols == t.cols, "tivazen_set_weight: matrix %d of layer %d: encoding %d [%d, %d], model expects BF16 [%d, %d]",
               which, layer, w->enc, w->rows, w->cols, t.rows, t.cols);
    SK_TRY(set_thread_device(m->device));
    if (which == SKAINET_TV_UK) SK_TRY(launch_transpose_heads(data(w), (bf16*) t.w->qs, m->layers[layer].c.heads, m->layers[layer].c.dim, m->layers[layer].c.kv_rank, nullptr));
    else SK_CUDA(cudaMemcpy((bf16*) t.w->qs + (size_t) t.row0 * bf16_ld(t.cols), w->qs, (size_t) t.rows * bf16_ld(t.cols) * 2, cudaMemcpyDeviceToDevice));
    SK_CUDA(cudaStreamSynchronize(nullptr));
    m->missing.erase({model_level ? -1 : layer, which, e});
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_tivazen_set_vector(skainet_model_t h, int32_t layer, int32_t which, const float* v, int32_t n) {
    Tivazen* m = design_from_handle<Tivazen>(h, __func__);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(v != nullptr && !m->finalized, "tivazen_set_vector: null values or a finalized model");
    const bool model_level = which == SKAINET_TV_FINAL_NORM;
    SK_REQUIRE(model_level || (layer >= 0 && layer < m->cfg.n_layers), "tivazen_set_vector: layer %d out of range", layer);
    TvLayer* L = model_level ? nullptr : &m->layers[layer];
    float *host = nullptr, *dev = nullptr;
    int want = 1;
    switch (which) {
        case SKAINET_TV_FINAL_NORM: host = &m->final_norm; break;
        case SKAINET_TV_NORM1: host = &L->norm1; break;
        case SKAINET_TV_NORM2: if (L->c.mlp != SKAINET_TV_MLP_NONE) host = &L->norm2; break;
        case SKAINET_TV_DKV_NORM: dev = L->dkv_norm; want = L->c.kv_rank; break;
        case SKAINET_TV_DEPTH: dev = L->depth; want = layer + 2; break;
        default: break;
    }
    SK_REQUIRE(host || dev, "tivazen_set_vector: layer %d has no vector %d", layer, which);
    SK_REQUIRE(n == want, "tivazen_set_vector: vector %d of layer %d has %d values, model expects %d", which, layer, n, want);
    SK_TRY(set_thread_device(m->device));
    if (host) *host = v[0]; else SK_CUDA(cudaMemcpy(dev, v, sizeof(float) * n, cudaMemcpyHostToDevice));
    m->missing.erase({model_level ? -1 : layer, 100 + which, 0});
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_tivazen_synth(skainet_model_t h, uint64_t seed, float std) {
    Tivazen* m = design_from_handle<Tivazen>(h, __func__);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(!m->finalized, "tivazen_synth: model already finalized");
    SK_TRY(set_thread_device(m->device));
    uint64_t k = 0;
    auto fill = [&](Weight* w) -> int32_t { return w ? launch_synth(*w, seed + 1000003ull * ++k, std, 0, 0, 0, w->cols, nullptr) : SKAINET_CUDA_OK; };
    SK_TRY(fill(m->embed)); SK_TRY(fill(m->head));
    for (int i = 0; i < m->cfg.n_layers; ++i) {
        TvLayer& L = m->layers[i];
        for (Weight* w : {L.proj, L.uk, L.uv, L.o, L.router, L.gate, L.up, L.down}) SK_TRY(fill(w));
        const std::vector<float> ones(L.c.kv_rank, 1.0f);
        if (L.dkv_norm) SK_CUDA(cudaMemcpy(L.dkv_norm, ones.data(), sizeof(float) * L.c.kv_rank, cudaMemcpyHostToDevice));
        std::vector<float> depth(i + 2, 0.125f);
        depth.back() = 1.0f;
        SK_CUDA(cudaMemcpy(L.depth, depth.data(), sizeof(float) * depth.size(), cudaMemcpyHostToDevice));
    }
    m->missing.clear();
    SK_CUDA(cudaDeviceSynchronize());
    return SKAINET_CUDA_OK;
}

}  // extern "C"
