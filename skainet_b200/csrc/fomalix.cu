// The Fomalix design of the decoder runtime (contract: include/skainet_cuda_fomalix.h). Per layer run
//
//   act = norm1(x)                                         (left by the kernel before)
//   attention   q | k | v  (one merged linear)             ->  ring attention (kv_attn.cuh)               ->  o
//   delta rule  q | k | v | b | a | g                      ->  recurrence (recurrence.cuh)  ->  gated norm ->  o
//   Mamba-2     z | x | B | C | dt                         ->  recurrence                   ->  gated norm ->  o
//   x += norm1b(.), act = norm2(x)  ->  gate, up -> gelu * up -> down  ->  x += norm2b(.) [+ embedding output], act = next norm1(x)
//
// The looped span is unrolled into layer runs: what a sequence holds belongs to a run, the weights to a layer. The residual
// stream and all recurrent state are fp32; linears read a narrowed copy. Decode steps and prompt passes run the same body over
// rows; only the row map and the kernels the row count selects differ.
#include "decoder.cuh"
#include "kv_attn.cuh"
#include "linear_bf16.cuh"
#include "recurrence.cuh"
#include "residual.cuh"
#include "../../include/skainet_cuda_fomalix.h"

#include <algorithm>
#include <cmath>
#include <map>
#include <set>
#include <vector>

namespace sk {

namespace {

constexpr int PREFILL_ROWS = 1024;       // rows of one prompt pass unless the configuration says otherwise

// Where a matrix or vector of the checkpoint goes.
struct MatrixSlot { Weight* w = nullptr; int row0 = 0, rows = 0, cols = 0; };
struct VectorSlot { float* p = nullptr; int n = 0; };

struct FxLayer {
    skainet_fomalix_layer c;
    Weight *proj = nullptr, *o = nullptr, *gate = nullptr, *up = nullptr, *down = nullptr;
    int proj_rows = 0;
    KvGeom kv = {};
    RecurGeom rec = {};
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *bias = nullptr, *sink = nullptr, *conv = nullptr, *conv_b = nullptr,
          *a_log = nullptr, *dt_bias = nullptr, *d = nullptr, *mix_norm = nullptr;
    void *mixed = nullptr, *hidden = nullptr;        // activation rows: concatenated heads, feed-forward's inner values
    std::map<int, MatrixSlot> matrices;
    std::map<int, VectorSlot> vectors;

    bool attention() const { return c.type == SKAINET_FX_ATTENTION; }
    int inner() const { return c.heads * c.vdim; }
};

struct FxRun {                            // one pass through a layer
    int layer = 0;
    bool again = false;                   // the embedding output is added before it
    KvCache cache;
    float *state = nullptr, *tail = nullptr;
};

const bf16* data(const Weight* w) { return (const bf16*) w->qs; }

__global__ void fill_noise_kernel(float* f, bf16* h, int64_t n, float scale, uint64_t seed) {
    for (int64_t i = blockIdx.x * (int64_t) blockDim.x + threadIdx.x; i < n; i += (int64_t) gridDim.x * blockDim.x) {
        uint64_t z = (seed + (uint64_t) i) * 0x9E3779B97F4A7C15ull;
        z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull; z ^= z >> 27;
        const float v = ((float) (z & 0xFFFF) / 32768.0f - 1.0f) * scale;
        if (f) f[i] = v; else h[i] = __float2bfloat16_rn(v);
    }
}
// rows of ld elements of which the first n are noise
__global__ void clear_tails_kernel(float* f, bf16* h, int64_t rows, int n, int ld) {
    for (int64_t i = blockIdx.x * (int64_t) blockDim.x + threadIdx.x; i < rows * (ld - n); i += (int64_t) gridDim.x * blockDim.x) {
        const int64_t at = i / (ld - n) * ld + n + i % (ld - n);
        if (f) f[at] = 0.0f; else h[at] = __float2bfloat16_rn(0.0f);
    }
}

struct Fomalix : Decoder {
    skainet_fomalix_config cfg;
    bool f32 = false;
    int act_size = 2, width_ld = 0;
    std::vector<FxLayer> layers;
    std::vector<FxRun> runs;
    Weight *embed = nullptr, *head = nullptr;
    float* final_norm = nullptr;
    double* freq = nullptr;
    std::set<std::pair<int, int>> missing;            // (layer, matrix | 100 + vector) not set yet
    // per row in flight
    float *x = nullptr, *x0 = nullptr, *proj = nullptr, *y = nullptr, *rec_out = nullptr, *part = nullptr;
    void *act = nullptr, *act_final = nullptr, *q = nullptr, *work = nullptr;
    int32_t* want = nullptr;

    ~Fomalix() override {
        for (auto& L : layers) for (Weight* w : {L.proj, L.o, L.gate, L.up, L.down}) if (w) weight_release(w);
        if (embed) weight_release(embed);
        if (head) weight_release(head);
    }

    int32_t create(const skainet_fomalix_layer* ls);
    int32_t create_layer(int i, const skainet_fomalix_layer& c);
    int32_t body(int rows, RowMap map, int kv_bound, bool to_head, cudaStream_t s);
    int32_t mixer(FxLayer& L, FxRun& r, int rows, RowMap map, int kv_bound, cudaStream_t s);
    int32_t head_rows(int n, cudaStream_t s);

    int32_t finalize() override {
        if (!missing.empty()) {
            const auto& k = *missing.begin();
            set_error("fomalix_finalize: %d tensors missing, first: %s %d of layer %d", (int) missing.size(), k.second >= 100 ? "vector" : "matrix", k.second % 100, k.first);
            return SKAINET_CUDA_ERR_INVALID;
        }
        return SKAINET_CUDA_OK;
    }
    int32_t enqueue_decode(int batch, int kv_bound, cudaStream_t s) override {
        SK_TRY(body(batch, RowMap{pos, -1}, kv_bound, true, s));
        return head_rows(batch, s);
    }
    int32_t enqueue_prompt(int rows, int seq, int kv_bound, cudaStream_t s) override { return body(rows, RowMap{pos, seq}, kv_bound, false, s); }
    int32_t enqueue_head(const int32_t* rows, int n, cudaStream_t s) override {
        SK_CUDA(cudaMemcpyAsync(want, rows, sizeof(int32_t) * n, cudaMemcpyHostToDevice, s));
        SK_TRY(launch_row_norm(x, want, n, d_model, final_norm, cfg.eps, act_final, width_ld, f32, s));
        return head_rows(n, s);
    }
    int32_t fill_context(int seq, int n, uint64_t seed) override {
        (void) n;
        auto noise = [&](void* p, bool f, int64_t count, float scale, int tail_n, int ld) {
            fill_noise_kernel<<<592, 256, 0, stream>>>(f ? (float*) p : nullptr, f ? nullptr : (bf16*) p, count, scale, seed += 0x51ull);
            if (tail_n < ld) clear_tails_kernel<<<148, 256, 0, stream>>>(f ? (float*) p : nullptr, f ? nullptr : (bf16*) p, count / ld, tail_n, ld);
        };
        for (FxRun& r : runs) {
            const FxLayer& L = layers[r.layer];
            if (L.attention()) {
                const int64_t rows = (int64_t) L.kv.kv_heads * r.cache.cap;
                noise((char*) r.cache.k + (size_t) seq * rows * L.kv.kld() * act_size, f32, rows * L.kv.kld(), 1.7f, L.kv.dim, L.kv.kld());
                noise((char*) r.cache.v + (size_t) seq * rows * L.kv.vcld() * act_size, f32, rows * L.kv.vcld(), 1.7f, L.kv.vdim, L.kv.vcld());
            } else {
                noise(r.state + (size_t) seq * L.rec.state_size(), true, (int64_t) L.rec.state_size(), 0.1f, L.rec.vdim, L.rec.vld());
                noise(r.tail + (size_t) seq * L.rec.tail_size(), true, (int64_t) L.rec.tail_size(), 1.0f, 1, 1);
            }
        }
        SK_CUDA(cudaGetLastError());
        return SKAINET_CUDA_OK;
    }
    // Weights once per run, the visible keys and values, the recurrent state in and out.
    int64_t step_bytes(int batch) const override {
        int64_t bytes = head->packed_bytes + (int64_t) batch * d_model * 2;
        for (const FxRun& r : runs) {
            const FxLayer& L = layers[r.layer];
            for (const Weight* w : {L.proj, L.o, L.gate, L.up, L.down}) if (w) bytes += w->packed_bytes;
            for (int b = 0; b < batch; ++b) {
                const int64_t keys = L.c.chunk > 0 ? host_pos[b] % L.c.chunk + 1 : host_pos[b] + 1;
                bytes += L.attention() ? keys * L.kv.kv_heads * (L.kv.kld() + L.kv.vcld()) * act_size : (int64_t) (2 * L.rec.state_size() + L.rec.tail_size()) * 4;
            }
        }
        return bytes;
    }
    const float* buffer(int which) const override { return which == 0 ? x : which == 1 ? proj : nullptr; }
};

// Weights, vectors and where the checkpoint's tensors go.
int32_t Fomalix::create_layer(int i, const skainet_fomalix_layer& c) {
    FxLayer& L = layers[i];
    L.c = c;
    const int inner = L.inner(), qk = c.kv_heads * c.dim;
    auto matrix = [&](Weight** w, int rows, int cols) -> int32_t { return weight_alloc(SKAINET_ENC_BF16, rows, cols, w); };
    auto vec = [&](int which, float** p, int n) -> int32_t { SK_TRY(alloc(p, n)); L.vectors[which] = {*p, n}; return SKAINET_CUDA_OK; };
    int at = 0;
    std::vector<std::pair<int, int>> merged;                // (matrix, rows) of the merged projection
    SK_TRY(vec(SKAINET_FX_NORM1, &L.norm1, d_model)); SK_TRY(vec(SKAINET_FX_NORM1B, &L.norm1b, d_model));
    if (L.attention()) {
        L.kv = KvGeom{c.heads, c.kv_heads, c.dim, c.vdim};
        const int n[3] = {c.heads * c.dim, qk, c.kv_heads * c.vdim};
        SK_TRY(alloc(&L.bias, L.kv.proj_rows()));
        for (int j = 0; j < 3; ++j) { merged.push_back({SKAINET_FX_Q + j, n[j]}); L.vectors[SKAINET_FX_Q_BIAS + j] = {L.bias + at, n[j]}; at += n[j]; }
        SK_TRY(vec(SKAINET_FX_SINK, &L.sink, c.heads));
    } else {
        const bool delta = c.type == SKAINET_FX_DELTA;
        L.rec = RecurGeom{c.heads, c.kv_heads, c.dim, c.vdim, c.conv, delta};
        SK_TRY(alloc(&L.conv, (size_t) L.rec.conv_dim() * c.conv));
        SK_TRY(vec(SKAINET_FX_A_LOG, &L.a_log, c.heads)); SK_TRY(vec(SKAINET_FX_DT_BIAS, &L.dt_bias, c.heads));
        SK_TRY(vec(SKAINET_FX_MIX_NORM, &L.mix_norm, delta ? c.vdim : inner));
        if (delta) {
            merged = {{SKAINET_FX_Q, qk}, {SKAINET_FX_K, qk}, {SKAINET_FX_V, inner}, {SKAINET_FX_B, c.heads}, {SKAINET_FX_A, c.heads}, {SKAINET_FX_G, inner}};
            for (int j = 0; j < 3; ++j) { L.vectors[SKAINET_FX_Q_CONV + j] = {L.conv + (size_t) at * c.conv, merged[j].second * c.conv}; at += merged[j].second; }
        } else {
            merged = {{SKAINET_FX_IN, 2 * inner + 2 * qk + c.heads}};
            L.vectors[SKAINET_FX_CONV] = {L.conv, L.rec.conv_dim() * c.conv};
            SK_TRY(vec(SKAINET_FX_CONV_BIAS, &L.conv_b, L.rec.conv_dim())); SK_TRY(vec(SKAINET_FX_D, &L.d, c.heads));
        }
    }
    for (auto& m : merged) L.proj_rows += m.second;
    SK_TRY(matrix(&L.proj, L.proj_rows, d_model)); SK_TRY(matrix(&L.o, d_model, inner));
    at = 0;
    for (auto& m : merged) { L.matrices[m.first] = {L.proj, at, m.second, d_model}; at += m.second; }
    L.matrices[SKAINET_FX_O] = {L.o, 0, d_model, inner};
    if (c.ff) {
        SK_TRY(matrix(&L.gate, c.ff, d_model)); SK_TRY(matrix(&L.up, c.ff, d_model)); SK_TRY(matrix(&L.down, d_model, c.ff));
        L.matrices[SKAINET_FX_GATE] = {L.gate, 0, c.ff, d_model}; L.matrices[SKAINET_FX_UP] = {L.up, 0, c.ff, d_model}; L.matrices[SKAINET_FX_DOWN] = {L.down, 0, d_model, c.ff};
        SK_TRY(vec(SKAINET_FX_NORM2, &L.norm2, d_model)); SK_TRY(vec(SKAINET_FX_NORM2B, &L.norm2b, d_model));
    }
    for (auto& m : L.matrices) missing.insert({i, m.first});
    for (auto& v : L.vectors) missing.insert({i, 100 + v.first});
    return SKAINET_CUDA_OK;
}

int32_t Fomalix::create(const skainet_fomalix_layer* ls) {
    const size_t R = max_rows, A = act_size;
    std::map<int, void*> act_rows;                          // activation buffers by inner size: their zero tails differ
    auto rows_of = [&](int n, void** p) -> int32_t {
        void*& b = act_rows[n];
        if (!b) SK_TRY(alloc(&b, R * bf16_ld(n) * A));
        *p = b;
        return SKAINET_CUDA_OK;
    };
    size_t max_proj = 1, max_inner = 1, max_q = 0, max_part = 0, max_work = 0;
    for (int i = 0; i < cfg.n_layers; ++i) {
        SK_TRY(create_layer(i, ls[i]));
        FxLayer& L = layers[i];
        SK_TRY(rows_of(L.inner(), &L.mixed));
        if (L.c.ff) SK_TRY(rows_of(L.c.ff, &L.hidden));
        max_proj = std::max<size_t>(max_proj, L.proj_rows); max_inner = std::max<size_t>(max_inner, L.inner());
        if (L.attention()) { max_q = std::max<size_t>(max_q, R * L.c.heads * L.kv.kld()); max_part = std::max(max_part, kv_part_floats(L.kv)); }
        else if (!f32) max_work = std::max(max_work, recur_work_bytes(L.rec, max_rows));
    }
    for (int i = 0; i < cfg.n_layers; ++i) {
        if (i == cfg.loop_start)
            for (int t = 0; t < cfg.loop_times; ++t)
                for (int j = cfg.loop_start; j < cfg.loop_stop; ++j) { FxRun r; r.layer = j; r.again = t > 0 && j == cfg.loop_start; runs.push_back(r); }
        if (i >= cfg.loop_start && i < cfg.loop_stop) continue;
        FxRun r;
        r.layer = i;
        runs.push_back(r);
    }
    for (FxRun& r : runs) {
        const FxLayer& L = layers[r.layer];
        if (L.attention()) {            // a ring: the keys the first row of a pass still sees, and the pass's own rows
            r.cache.cap = L.c.chunk > 0 ? (int) std::min<int64_t>(max_seq, (int64_t) L.c.chunk - 1 + max_rows) : max_seq;
            SK_TRY(alloc(&r.cache.k, (size_t) max_batch * L.c.kv_heads * r.cache.cap * L.kv.kld() * A));
            SK_TRY(alloc(&r.cache.v, (size_t) max_batch * L.c.kv_heads * r.cache.cap * L.kv.vcld() * A));
        } else {
            SK_TRY(alloc(&r.state, max_batch * L.rec.state_size())); SK_TRY(alloc(&r.tail, max_batch * L.rec.tail_size()));
        }
    }
    SK_TRY(weight_alloc(SKAINET_ENC_BF16, vocab, d_model, &embed)); SK_TRY(weight_alloc(SKAINET_ENC_BF16, vocab, d_model, &head));
    SK_TRY(alloc(&final_norm, d_model));
    for (int k : {SKAINET_FX_EMBED, SKAINET_FX_HEAD, 100 + SKAINET_FX_FINAL_NORM}) missing.insert({-1, k});
    std::vector<double> f((d_model + 1) / 2);
    for (size_t k = 0; k < f.size(); ++k) f[k] = pow(10000.0, -2.0 * (double) k / (double) d_model);
    SK_TRY(alloc(&freq, f.size()));
    SK_CUDA(cudaMemcpy(freq, f.data(), sizeof(double) * f.size(), cudaMemcpyHostToDevice));
    SK_TRY(alloc(&x, R * d_model)); SK_TRY(alloc(&x0, R * d_model)); SK_TRY(alloc(&y, R * d_model)); SK_TRY(alloc(&proj, R * max_proj)); SK_TRY(alloc(&rec_out, R * max_inner));
    SK_TRY(alloc(&act, R * width_ld * A)); SK_TRY(alloc(&act_final, (size_t) logits_rows * width_ld * A)); SK_TRY(alloc(&want, logits_rows));
    SK_TRY(alloc(&q, max_q * A)); SK_TRY(alloc(&part, max_part)); SK_TRY(alloc(&work, max_work));
    return SKAINET_CUDA_OK;
}

// The run's mixer over act, up to the concatenated heads in L.mixed.
int32_t Fomalix::mixer(FxLayer& L, FxRun& r, int rows, RowMap map, int kv_bound, cudaStream_t s) {
    const skainet_fomalix_layer& c = L.c;
    if (L.attention()) {
        KvAttnArgs a;
        a.g = L.kv; a.scale = c.scale; a.eps = cfg.eps; a.chunk = c.chunk; a.proj = proj; a.proj_ld = L.proj_rows; a.bias = L.bias; a.sink = L.sink; a.cache = r.cache;
        a.q = q; a.out = L.mixed; a.part = part; a.rows = rows; a.map = map; a.kv_bound = kv_bound; a.f32_act = f32;
        return launch_kv_attention(a, s);
    }
    const int inner = L.inner(), qk = L.rec.q_dim();
    RecurArgs a;
    GatedNormArgs n;
    a.g = L.rec; a.proj = proj; a.proj_ld = L.proj_rows; a.conv_w = L.conv; a.conv_b = L.conv_b; a.a_log = L.a_log; a.dt_bias = L.dt_bias; a.d = L.d;
    a.state = r.state; a.tail = r.tail; a.out = rec_out; a.rows = rows; a.rows_alloc = max_rows; a.map = map; a.f32_act = f32; a.work = work;
    n.o = rec_out; n.z_ld = L.proj_rows; n.gain = L.mix_norm; n.cols = inner; n.rows = rows; n.eps = cfg.eps; n.act = L.mixed; n.act_ld = bf16_ld(inner); n.f32_act = f32;
    if (L.rec.delta) {
        a.q_off = 0; a.k_off = qk; a.v_off = 2 * qk; a.beta_off = 2 * qk + inner; a.dt_off = a.beta_off + c.heads;
        a.q_scale = 1.0f / sqrtf((float) c.dim);
        n.z = proj + a.dt_off + c.heads; n.part = c.vdim;
    } else {
        a.conv_off = inner; a.v_off = 0; a.k_off = inner; a.q_off = inner + qk; a.dt_off = 2 * inner + 2 * qk;
        n.z = proj; n.part = inner / c.norm_groups; n.gate_first = true;
    }
    SK_TRY(launch_recurrence(a, s));
    return launch_gated_norm(n, s);
}

int32_t Fomalix::body(int rows, RowMap map, int kv_bound, bool to_head, cudaStream_t s) {
    EmbedPosArgs e;
    e.table = data(embed); e.ld = width_ld; e.vocab = vocab; e.ids = cur_token; e.scale = cfg.embed_scale; e.eps = cfg.eps; e.freq = freq; e.map = map;
    e.pre = layers[runs[0].layer].norm1; e.x = x; e.x0 = cfg.loop_times > 1 ? x0 : nullptr; e.act = act; e.act_ld = width_ld; e.rows = rows; e.cols = d_model; e.f32_act = f32;
    SK_TRY(launch_embed_pos(e, s));
    for (size_t i = 0; i < runs.size(); ++i) {
        FxLayer& L = layers[runs[i].layer];
        LinearArgs l;
        l.f32_act = f32; l.x_rows_alloc = max_rows; l.rows = rows;
        l.w = data(L.proj); l.w_rows = L.proj_rows; l.ldw = l.ldx = width_ld; l.x = act; l.y = proj; l.ldy = L.proj_rows;
        SK_TRY(launch_linear_bf16(l, s));
        SK_TRY(mixer(L, runs[i], rows, map, kv_bound, s));
        l.w = data(L.o); l.w_rows = d_model; l.ldw = l.ldx = bf16_ld(L.inner()); l.x = L.mixed; l.y = y; l.ldy = d_model;
        SK_TRY(launch_linear_bf16(l, s));
        SandwichArgs n;
        n.y = y; n.post = L.norm1b; n.x = x; n.act = act; n.act_ld = width_ld; n.eps = cfg.eps; n.rows = rows; n.cols = d_model; n.f32_act = f32;
        if (L.c.ff) {
            n.pre = L.norm2;
            SK_TRY(launch_sandwich(n, s));
            l.w = data(L.gate); l.w2 = data(L.up); l.w_rows = L.c.ff; l.ldw = l.ldx = width_ld; l.x = act; l.y = L.hidden; l.ldy = bf16_ld(L.c.ff); l.out = LIN_OUT_GEGLU;
            SK_TRY(launch_linear_bf16(l, s));
            l.w = data(L.down); l.w2 = nullptr; l.w_rows = d_model; l.ldw = l.ldx = bf16_ld(L.c.ff); l.x = L.hidden; l.y = y; l.ldy = d_model; l.out = LIN_OUT_F32;
            SK_TRY(launch_linear_bf16(l, s));
            n.post = L.norm2b;
        }
        if (i + 1 < runs.size()) { n.pre = layers[runs[i + 1].layer].norm1; n.add = runs[i + 1].again ? x0 : nullptr; }
        else { n.pre = to_head ? final_norm : nullptr; n.act = act_final; }
        SK_TRY(launch_sandwich(n, s));
    }
    return SKAINET_CUDA_OK;
}

// Logits of the n normed rows in act_final.
int32_t Fomalix::head_rows(int n, cudaStream_t s) {
    LinearArgs l;
    l.f32_act = f32; l.x_rows_alloc = logits_rows; l.rows = n; l.w = data(head); l.w_rows = vocab; l.ldw = l.ldx = width_ld; l.x = act_final; l.y = logits; l.ldy = vocab;
    return launch_linear_bf16(l, s);
}

}  // namespace

}  // namespace sk

using namespace sk;

extern "C" {

int32_t skainet_cuda_fomalix_create(const skainet_fomalix_config* cfg, const skainet_fomalix_layer* ls, skainet_model_t* out) {
    SK_REQUIRE(cfg && ls && out, "fomalix_create: null argument");
    *out = 0;
    const auto& c = *cfg;
    SK_REQUIRE(c.n_layers > 0 && c.width > 0 && c.vocab > 0, "fomalix_create: non-positive dimension");
    SK_REQUIRE(c.max_seq >= 1 && c.max_batch >= 1 && c.max_batch <= 4096 && c.prefill_rows >= 0 && c.prefill_rows <= 65535, "fomalix_create: max_seq %d, max_batch %d, prefill_rows %d", c.max_seq, c.max_batch, c.prefill_rows);
    SK_REQUIRE(c.loop_start >= 0 && c.loop_start < c.loop_stop && c.loop_stop <= c.n_layers && c.loop_times >= 1, "fomalix_create: layers %d to %d of %d, %d times", c.loop_start, c.loop_stop, c.n_layers, c.loop_times);
    for (int i = 0; i < c.n_layers; ++i) {
        const auto& l = ls[i];
        SK_REQUIRE(l.type >= SKAINET_FX_ATTENTION && l.type <= SKAINET_FX_MAMBA2, "fomalix_create: layer %d: mixer type %d", i, l.type);
        SK_REQUIRE(l.heads > 0 && l.kv_heads > 0 && l.dim > 0 && l.vdim > 0 && l.ff >= 0, "fomalix_create: layer %d: bad sizes", i);
        SK_REQUIRE(l.heads % l.kv_heads == 0, "fomalix_create: layer %d: %d heads in %d groups", i, l.heads, l.kv_heads);
        SK_REQUIRE(l.type != SKAINET_FX_ATTENTION || l.chunk >= 0, "fomalix_create: layer %d: chunk %d", i, l.chunk);
        SK_REQUIRE(l.type == SKAINET_FX_ATTENTION || (l.conv >= 1 && l.dim <= RECUR_MAX_KDIM), "fomalix_create: layer %d: %d taps, key size %d (at most %d)", i, l.conv, l.dim, RECUR_MAX_KDIM);
        SK_REQUIRE(l.type != SKAINET_FX_MAMBA2 || (l.norm_groups >= 1 && (l.heads * l.vdim) % l.norm_groups == 0), "fomalix_create: layer %d: norm in %d parts", i, l.norm_groups);
    }
    SK_TRY(ensure_device());
    Fomalix* m = new Fomalix();
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

int32_t skainet_cuda_fomalix_set_weight(skainet_model_t h, int32_t layer, int32_t which, skainet_weight_t wh) {
    Fomalix* m = design_from_handle<Fomalix>(h, __func__);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    Weight* w = weight_from_handle(wh);
    if (!w) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(!m->finalized, "fomalix_set_weight: model already finalized");
    const bool model_level = which == SKAINET_FX_EMBED || which == SKAINET_FX_HEAD;
    SK_REQUIRE(model_level || (layer >= 0 && layer < m->cfg.n_layers), "fomalix_set_weight: layer %d out of range", layer);
    MatrixSlot t;
    if (model_level) t = {which == SKAINET_FX_EMBED ? m->embed : m->head, 0, m->vocab, m->d_model};
    else { auto it = m->layers[layer].matrices.find(which); if (it != m->layers[layer].matrices.end()) t = it->second; }
    SK_REQUIRE(t.w != nullptr, "fomalix_set_weight: layer %d has no matrix %d", layer, which);
    SK_REQUIRE(w->enc == SKAINET_ENC_BF16 && w->rows == t.rows && w->cols == t.cols, "fomalix_set_weight: matrix %d of layer %d: encoding %d [%d, %d], model expects BF16 [%d, %d]",
               which, layer, w->enc, w->rows, w->cols, t.rows, t.cols);
    SK_TRY(set_thread_device(m->device));
    SK_CUDA(cudaMemcpy((bf16*) t.w->qs + (size_t) t.row0 * bf16_ld(t.cols), w->qs, (size_t) t.rows * bf16_ld(t.cols) * 2, cudaMemcpyDeviceToDevice));
    SK_CUDA(cudaStreamSynchronize(nullptr));
    m->missing.erase({model_level ? -1 : layer, which});
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_fomalix_set_vector(skainet_model_t h, int32_t layer, int32_t which, const float* v, int32_t n) {
    Fomalix* m = design_from_handle<Fomalix>(h, __func__);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(v != nullptr && !m->finalized, "fomalix_set_vector: null values or a finalized model");
    const bool model_level = which == SKAINET_FX_FINAL_NORM;
    SK_REQUIRE(model_level || (layer >= 0 && layer < m->cfg.n_layers), "fomalix_set_vector: layer %d out of range", layer);
    VectorSlot t;
    if (model_level) t = {m->final_norm, m->d_model};
    else { auto it = m->layers[layer].vectors.find(which); if (it != m->layers[layer].vectors.end()) t = it->second; }
    SK_REQUIRE(t.p != nullptr, "fomalix_set_vector: layer %d has no vector %d", layer, which);
    SK_REQUIRE(n == t.n, "fomalix_set_vector: vector %d of layer %d has %d values, model expects %d", which, layer, n, t.n);
    SK_TRY(set_thread_device(m->device));
    SK_CUDA(cudaMemcpy(t.p, v, sizeof(float) * n, cudaMemcpyHostToDevice));
    m->missing.erase({model_level ? -1 : layer, 100 + which});
    return SKAINET_CUDA_OK;
}

int32_t skainet_cuda_fomalix_synth(skainet_model_t h, uint64_t seed, float std) {
    Fomalix* m = design_from_handle<Fomalix>(h, __func__);
    if (!m) return SKAINET_CUDA_ERR_HANDLE;
    SK_REQUIRE(!m->finalized, "fomalix_synth: model already finalized");
    SK_TRY(set_thread_device(m->device));
    uint64_t k = 0;
    auto fill = [&](Weight* w) -> int32_t { return w ? launch_synth(*w, seed + 1000003ull * ++k, std, 0, 0, 0, w->cols, nullptr) : SKAINET_CUDA_OK; };
    auto set = [&](float* p, int n, float v) -> int32_t {
        const std::vector<float> host(n, v);
        SK_CUDA(cudaMemcpy(p, host.data(), sizeof(float) * n, cudaMemcpyHostToDevice));
        return SKAINET_CUDA_OK;
    };
    SK_TRY(fill(m->embed)); SK_TRY(fill(m->head)); SK_TRY(set(m->final_norm, m->d_model, 1.0f));
    for (FxLayer& L : m->layers) {
        for (Weight* w : {L.proj, L.o, L.gate, L.up, L.down}) SK_TRY(fill(w));
        for (auto& v : L.vectors) {
            const int w = v.first;
            const bool gain = w <= SKAINET_FX_NORM2B || w == SKAINET_FX_MIX_NORM;
            SK_TRY(set(v.second.p, v.second.n, gain ? 1.0f : w == SKAINET_FX_A_LOG ? -2.0f : w == SKAINET_FX_DT_BIAS ? -2.0f : 0.0f));
        }
        if (!L.conv) continue;
        std::vector<float> taps((size_t) L.rec.conv_dim() * L.rec.taps, 0.25f);
        for (int ch = 0; ch < L.rec.conv_dim(); ++ch) taps[(size_t) (ch + 1) * L.rec.taps - 1] = 1.0f;
        SK_CUDA(cudaMemcpy(L.conv, taps.data(), sizeof(float) * taps.size(), cudaMemcpyHostToDevice));
    }
    m->missing.clear();
    SK_CUDA(cudaDeviceSynchronize());
    return SKAINET_CUDA_OK;
}

}  // extern "C"
