// Ring attention with a chunk mask and a sink (contract: kv_attn.cuh).
//
//   kv_prep_kernel       biases, unit-rms queries and keys, ring append (prompts; in a decode step the tile kernel does it).
//   kv_attn_tile_kernel  bf16: the MMA rows are (activation row, head) pairs that share a key/value head, so a staged key or value
//                        row serves the whole group. In prompts each of four warps owns 16 pairs and all read the same tile of 64
//                        keys; in a decode step four warps own the same 16 pairs and a quarter of the tile's keys each. Keys may
//                        be split over CTAs; kv_merge_kernel joins the parts in fixed order.
//   kv_attn_rows_kernel  fp32 FMA, one CTA per (row, head), any size: the 32-bit mode, and bf16 models whose heads are too large
//                        for the tile kernel.
#include "kv_attn.cuh"
#include "mma.cuh"
#include "tma.cuh"

#include <algorithm>
#include <climits>

namespace sk {

namespace {

constexpr float NEG_BIG = -1e30f;            // maximum over no key: finite, so differences stay defined

// First position that position i sees.
__device__ __forceinline__ int first_key(const KvAttnArgs& a, int i) { return a.chunk > 0 ? i / a.chunk * a.chunk : 0; }

// One warp prepares one vector of a row: u < heads a query, u < heads + kv_heads a key, else a value; put(i, x) stores coordinate i.
template <typename F>
__device__ __forceinline__ void prep_vector(const KvAttnArgs& a, int row, int u, int lane, F&& put) {
    const KvGeom& g = a.g;
    const bool is_v = u >= g.heads + g.kv_heads;
    const int n = is_v ? g.vdim : g.dim, off = is_v ? (g.heads + g.kv_heads) * g.dim + (u - g.heads - g.kv_heads) * g.vdim : u * g.dim;
    const float *p = a.proj + (size_t) row * a.proj_ld + off, *b = a.bias ? a.bias + off : nullptr;
    float r = 1.0f;
    if (!is_v) {
        float ss = 0.0f;
        for (int i = lane; i < n; i += 32) { const float v = p[i] + (b ? b[i] : 0.0f); ss = fmaf(v, v, ss); }
        r = 1.0f / sqrtf(skd::warp_sum(ss) / (float) n + a.eps);
    }
    for (int i = lane; i < n; i += 32) put(i, (p[i] + (b ? b[i] : 0.0f)) * r);
}
// Row of unit u >= heads in the ring.
template <typename T>
__device__ __forceinline__ T* cache_row(const KvAttnArgs& a, int row, int u) {
    const KvGeom& g = a.g;
    const bool is_v = u >= g.heads + g.kv_heads;
    const int slot = a.map.pos_of(row) % a.cache.cap, kh = u - g.heads - (is_v ? g.kv_heads : 0);
    const size_t at = ((size_t) a.map.seq_of(row) * g.kv_heads + kh) * a.cache.cap + slot;
    return is_v ? (T*) a.cache.v + at * g.vcld() : (T*) a.cache.k + at * g.kld();
}

template <typename T>
__global__ void __launch_bounds__(256) kv_prep_kernel(const KvAttnArgs a) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int units = a.g.heads + 2 * a.g.kv_heads, u = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (u >= units) return;
    T* dst = u < a.g.heads ? (T*) a.q + ((size_t) blockIdx.x * a.g.heads + u) * a.g.kld() : cache_row<T>(a, blockIdx.x, u);
    prep_vector(a, blockIdx.x, u, threadIdx.x & 31, [&](int i, float x) { skd::store_act(dst + i, x); });
}

constexpr int RK = 128;                      // keys of a tile = threads of a CTA
template <typename T>
__global__ void __launch_bounds__(RK) kv_attn_rows_kernel(const KvAttnArgs a) {
    const KvGeom& g = a.g;
    extern __shared__ float dyn[];           // q [kld] | mixed values [vcld]
    __shared__ float p[RK], sh[RK / 32];
    float *q = dyn, *acc = dyn + g.kld();
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int row = blockIdx.x, h = blockIdx.y, kh = h / (g.heads / g.kv_heads), t = threadIdx.x;
    const int pos = a.map.pos_of(row), lo = first_key(a, pos);
    const T* qp = (const T*) a.q + ((size_t) row * g.heads + h) * g.kld();
    const size_t base = ((size_t) a.map.seq_of(row) * g.kv_heads + kh) * a.cache.cap;
    for (int i = t; i < g.dim; i += RK) q[i] = skd::load_act(qp + i);
    for (int i = t; i < g.vdim; i += RK) acc[i] = 0.0f;
    float m = NEG_BIG, l = 0.0f;
    if (a.sink) { m = a.sink[h]; l = 1.0f; }
    __syncthreads();
    for (int j0 = lo; j0 <= pos; j0 += RK) {
        const int j = j0 + t, n = min(RK, pos + 1 - j0);
        float s = NEG_BIG;
        if (j <= pos) {
            const T* k = (const T*) a.cache.k + (base + j % a.cache.cap) * g.kld();
            s = 0.0f;
            for (int i = 0; i < g.dim; ++i) s = fmaf(q[i], skd::load_act(k + i), s);
            s *= a.scale;
        }
        float v = skd::warp_max(s);
        if ((t & 31) == 0) sh[t >> 5] = v;
        __syncthreads();
        v = m;
        for (int i = 0; i < RK / 32; ++i) v = fmaxf(v, sh[i]);
        const float fade = expf(m - v);
        m = v;
        p[t] = j <= pos ? expf(s - m) : 0.0f;
        float sum = skd::warp_sum(p[t]);
        __syncthreads();
        if ((t & 31) == 0) sh[t >> 5] = sum;
        __syncthreads();
        l *= fade;
        for (int i = 0; i < RK / 32; ++i) l += sh[i];
        for (int d = t; d < g.vdim; d += RK) {
            float o = acc[d] * fade;
            for (int i = 0; i < n; ++i) o = fmaf(p[i], skd::load_act((const T*) a.cache.v + (base + (j0 + i) % a.cache.cap) * g.vcld() + d), o);
            acc[d] = o;
        }
        __syncthreads();
    }
    for (int d = t; d < g.vdim; d += RK) skd::store_act((T*) a.out + (size_t) row * g.out_ld() + h * g.vdim + d, acc[d] / l);
}

constexpr float LOG2E = 1.4426950408889634f;
constexpr int TK = 64;                       // keys of a staged tile

__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// Widths up to 16 * KS (keys) and 8 * VN (values). DECODE: the activation rows of a CTA are one, its warps split the keys.
template <int KS, int VN, bool DECODE>
struct TileShape {
    static constexpr int WARPS = 4, ROWS = DECODE ? 16 : 64, KEYS = DECODE ? TK / WARPS : TK;   // pairs of a CTA, keys of a warp
    static constexpr int STAGES = DECODE ? 3 : 2;
    static constexpr bool Q_REGS = KS <= 8;                      // queries live in registers and pass through the last stage's key tile
    // rows are 16 bytes longer than the data: an odd number of 16-byte units, so ldmatrix rows meet different banks
    static __host__ __device__ int smem(int kld, int vcld) {
        const int tiles = ((Q_REGS ? 0 : ROWS * (kld + 8)) + STAGES * TK * (kld + 8 + vcld + 8)) * 2, merge = DECODE ? WARPS * 16 * (vcld + 2) * 4 : 0;
        return tiles > merge ? tiles : merge;
    }
};

template <int KS, int VN, bool DECODE>
__global__ void __launch_bounds__(TileShape<KS, VN, DECODE>::WARPS * 32)
kv_attn_tile_kernel(const KvAttnArgs a, int splits) {
    typedef TileShape<KS, VN, DECODE> S;
    extern __shared__ __align__(16) uint8_t raw[];
    const KvGeom g = a.g;
    const int kld = g.kld(), vcld = g.vcld(), klds = kld + 8, vlds = vcld + 8, ks_n = kld / 16, vn_n = vcld / 8;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, tq = lane & 3, group = g.heads / g.kv_heads;
    const int kh = blockIdx.y, split = blockIdx.z;
    // pairs [p0, p0 + ROWS) of this key/value head: row p / group, head p % group
    const int tiles_m = DECODE ? (group + 15) / 16 : 0;
    const int m_tile = DECODE ? (int) blockIdx.x % tiles_m : (int) (gridDim.x - 1 - blockIdx.x);          // the longest prompt tiles first
    const int row_base = DECODE ? (int) blockIdx.x / tiles_m : 0, p0 = m_tile * S::ROWS, pairs = DECODE ? group : a.rows * group;
    const uint32_t sk = skd::smem_u32(raw), sv = sk + S::STAGES * TK * klds * 2, sq = S::Q_REGS ? sk + (S::STAGES - 1) * TK * klds * 2 : sv + S::STAGES * TK * vlds * 2;
    skd::pdl_launch_dependents();
    if (!DECODE) skd::pdl_wait();                                 // positions and the ring's older rows were left by earlier steps
    const int seq = a.map.seq_of(row_base);
    const bf16* kc = (const bf16*) a.cache.k + ((size_t) seq * g.kv_heads + kh) * a.cache.cap * kld;
    const bf16* vc = (const bf16*) a.cache.v + ((size_t) seq * g.kv_heads + kh) * a.cache.cap * vcld;
    const int first_row = row_base + p0 / group, last_row = row_base + (min(pairs, p0 + S::ROWS) - 1) / group;
    const int pos_first = a.map.pos_of(first_row), pos_last = a.map.pos_of(last_row);
    const int lo = first_key(a, pos_first), lo_last = first_key(a, pos_last);
    int t0 = 0, t1 = (pos_last - lo) / TK + 1;
    if (splits > 1) { const int per = (t1 + splits - 1) / splits; t0 = min(t1, split * per); t1 = min(t1, t0 + per); }

    auto load_tile = [&](int t, int stage, int skip) {              // `skip`: a position that is not in the ring yet
        // a warp copies a key and its value at a time, a lane the same 16 bytes of each
        const int kch = kld / 8, both = kch + vcld / 8, j0 = lo + t * TK, slot0 = j0 % a.cache.cap, hole = skip - j0;
        for (int c = lane; c < both; c += 32) {
            const bool is_k = c < kch;
            const int ld = is_k ? kld : vcld, at = (is_k ? c : c - kch) * 8;
            const bf16* src = (is_k ? kc : vc) + at;
            uint32_t dst = is_k ? sk + ((stage * TK + warp) * klds + at) * 2 : sv + ((stage * TK + warp) * vlds + at) * 2;
            const uint32_t dst_step = S::WARPS * (is_k ? klds : vlds) * 2;
            if (slot0 + TK <= a.cache.cap) {
                src += (size_t) (slot0 + warp) * ld;
                const size_t src_step = (size_t) S::WARPS * ld;
#pragma unroll
                for (int r = 0; r < TK / S::WARPS; ++r, src += src_step, dst += dst_step)
                    if (!DECODE || warp + r * S::WARPS != hole) skd::cp16(dst, src);
            } else {
#pragma unroll 1
                for (int r = 0; r < TK / S::WARPS; ++r, dst += dst_step)
                    if (!DECODE || warp + r * S::WARPS != hole) skd::cp16(dst, src + (size_t) ((slot0 + warp + r * S::WARPS) % a.cache.cap) * ld);
            }
        }
    };
    // queries; rows past the last pair repeat it (prompts) or are zero, and are not stored
    if (!DECODE)
        for (int i = threadIdx.x; i < S::ROWS * (kld / 8); i += S::WARPS * 32) {
            const int r = i / (kld / 8), c = i % (kld / 8), p = min(p0 + r, pairs - 1);
            skd::cp16(sq + (r * klds + c * 8) * 2, (const bf16*) a.q + ((size_t) (row_base + p / group) * g.heads + kh * group + p % group) * kld + c * 8);
        }
    skd::cp_commit();
#pragma unroll
    for (int s = 0; s < S::STAGES - 1; ++s) { if (t0 + s < t1) load_tile(t0 + s, s, pos_last); skd::cp_commit(); }
    if (DECODE) {
        // the step's own vectors: biases and norms here, the new key and value into the ring and into the tile they belong to
        skd::pdl_wait();
        bf16* smem = (bf16*) raw;
        const int new_tile = (pos_last - lo) / TK, new_row = (pos_last - lo) % TK;
        const bool mine = new_tile >= t0 && new_tile < t1, staged = mine && new_tile < t0 + S::STAGES - 1;
        for (int u = warp; u < S::ROWS + 2; u += S::WARPS) {
            const int n = u == S::ROWS + 1 ? g.vdim : g.dim, np = u == S::ROWS + 1 ? vcld : kld;
            if (u < S::ROWS) {
                bf16* dst = smem + (sq - sk) / 2 + u * klds;
                for (int i = lane; i < np; i += 32) if (p0 + u >= pairs || i >= n) dst[i] = __float2bfloat16_rn(0.0f);
                if (p0 + u < pairs) prep_vector(a, row_base, kh * group + p0 + u, lane, [&](int i, float x) { dst[i] = __float2bfloat16_rn(x); });
            } else if (mine) {
                const int unit = g.heads + kh + (u == S::ROWS + 1 ? g.kv_heads : 0);
                bf16 *ring = cache_row<bf16>(a, row_base, unit), *dst = nullptr;
                if (staged) dst = u == S::ROWS ? smem + ((new_tile - t0) * TK + new_row) * klds : smem + (sv - sk) / 2 + ((new_tile - t0) * TK + new_row) * vlds;
                prep_vector(a, row_base, unit, lane, [&](int i, float x) { ring[i] = __float2bfloat16_rn(x); if (dst) dst[i] = __float2bfloat16_rn(x); });
                if (dst) for (int i = n + lane; i < np; i += 32) dst[i] = __float2bfloat16_rn(0.0f);
            }
        }
    }

    const int wr = DECODE ? 0 : warp * 16;                        // the warp's first pair
    int pos_r[2], lo_r[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        pos_r[i] = a.map.pos_of(row_base + min(p0 + wr + gr + 8 * i, pairs - 1) / group);
        lo_r[i] = first_key(a, pos_r[i]);
    }
    float o[VN][4];
#pragma unroll
    for (int n = 0; n < VN; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[n][i] = 0.0f;
    float m[2] = {NEG_BIG, NEG_BIG}, l[2] = {0.0f, 0.0f};
    uint32_t qf[S::Q_REGS ? KS : 1][4];
    const uint32_t q_at = sq + ((wr + (lane & 7) + ((lane >> 3) & 1) * 8) * klds + (lane >> 4) * 8) * 2;
    const int k0w = DECODE ? warp * S::KEYS : 0;                  // the warp's first key of a tile
    const uint32_t k_at = sk + ((k0w + (lane & 7) + (lane >> 4) * 8) * klds + ((lane >> 3) & 1) * 8) * 2;
    const uint32_t v_at = sv + ((k0w + (lane & 7) + ((lane >> 3) & 1) * 8) * vlds + (lane >> 4) * 8) * 2;
    const float sc2 = a.scale * LOG2E;
    if (S::Q_REGS) {
        if (!DECODE) skd::cp_wait<S::STAGES - 1>();
        __syncthreads();
#pragma unroll
        for (int k = 0; k < KS; ++k) if (k < ks_n) skd::ldsm4(qf[S::Q_REGS ? k : 0], q_at + k * 32);
    }
    constexpr int NK = S::KEYS / 8;

    for (int t = t0; t < t1; ++t) {
        const int stage = (t - t0) % S::STAGES;
        skd::cp_wait<S::STAGES - 2>();
        __syncthreads();
        if (t + S::STAGES - 1 < t1) load_tile(t + S::STAGES - 1, (t - t0 + S::STAGES - 1) % S::STAGES, INT_MIN / 2);
        skd::cp_commit();
        float c[NK][4];
#pragma unroll
        for (int n = 0; n < NK; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) c[n][i] = 0.0f;
#pragma unroll
        for (int k = 0; k < KS; ++k) {
            if (k >= ks_n) break;
            uint32_t qk[4];
            if (!S::Q_REGS) skd::ldsm4(qk, q_at + k * 32);
            const uint32_t* q = S::Q_REGS ? qf[S::Q_REGS ? k : 0] : qk;
#pragma unroll
            for (int n = 0; n < NK; n += 2) {
                uint32_t b[4];
                skd::ldsm4(b, k_at + ((stage * TK + n * 8) * klds + k * 16) * 2);
                skd::mma_bf16(c[n], q[0], q[1], q[2], q[3], b[0], b[1]);
                skd::mma_bf16(c[n + 1], q[0], q[1], q[2], q[3], b[2], b[3]);
            }
        }
        const int j0 = lo + t * TK + k0w;
        const bool whole = j0 >= lo_last && j0 + S::KEYS - 1 <= pos_first;
        float mx[2] = {m[0], m[1]};
        if (!whole)
#pragma unroll
            for (int n = 0; n < NK; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int j = j0 + n * 8 + tq * 2 + (i & 1);
                    if (j < lo_r[i >> 1] || j > pos_r[i >> 1]) c[n][i] = -INFINITY;
                }
#pragma unroll
        for (int n = 0; n < NK; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) { c[n][i] *= sc2; mx[i >> 1] = fmaxf(mx[i >> 1], c[n][i]); }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(~0u, mx[i], 1)); mx[i] = fmaxf(mx[i], __shfl_xor_sync(~0u, mx[i], 2));
            const float fade = ex2(m[i] - mx[i]);
            m[i] = mx[i];
            l[i] *= fade;
            if (__any_sync(~0u, fade != 1.0f))
#pragma unroll
                for (int n = 0; n < VN; ++n) { o[n][2 * i] *= fade; o[n][2 * i + 1] *= fade; }
        }
#pragma unroll
        for (int n = 0; n < NK; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) { c[n][i] = ex2(c[n][i] - m[i >> 1]); l[i >> 1] += c[n][i]; }
#pragma unroll
        for (int k = 0; k < NK / 2; ++k) {
            const uint32_t p[4] = {skd::pack_bf16(c[2 * k][0], c[2 * k][1]), skd::pack_bf16(c[2 * k][2], c[2 * k][3]), skd::pack_bf16(c[2 * k + 1][0], c[2 * k + 1][1]),
                                   skd::pack_bf16(c[2 * k + 1][2], c[2 * k + 1][3])};
#pragma unroll
            for (int n = 0; n < VN; n += 2) {
                if (n >= vn_n) break;
                uint32_t b[4];
                skd::ldsm4_t(b, v_at + ((stage * TK + k * 16) * vlds + n * 8) * 2);
                skd::mma_bf16(o[n], p[0], p[1], p[2], p[3], b[0], b[1]);
                skd::mma_bf16(o[n + 1], p[0], p[1], p[2], p[3], b[2], b[3]);
            }
        }
    }
    skd::cp_wait<0>();                                                 // the queries of a part without keys are still in flight
#pragma unroll
    for (int i = 0; i < 2; ++i) { l[i] += __shfl_xor_sync(~0u, l[i], 1); l[i] += __shfl_xor_sync(~0u, l[i], 2); }

    // Joins the sink, or leaves a record. `w` writes one pair's columns.
    auto finish = [&](int p, float mm, float ll, auto&& value, int d_first, int d_step, bool lead) {
        if (p >= pairs) return;
        const int row = row_base + p / group, h = kh * group + p % group;
        if (splits > 1) {
            float* rec = a.part + (((size_t) row * g.heads + h) * splits + split) * (vcld + 2);
            for (int d = d_first; d < vcld; d += d_step) value(d, [&](int at, float v) { rec[at] = v; });
            if (lead) { rec[vcld] = mm; rec[vcld + 1] = ll; }
            return;
        }
        float f = 1.0f, den = ll;
        if (a.sink) {
            const float s2 = a.sink[h] * LOG2E, top = fmaxf(mm, s2);
            f = exp2f(mm - top);
            den = ll * f + exp2f(s2 - top);
        }
        f /= den;
        bf16* out = (bf16*) a.out + (size_t) row * g.out_ld() + h * g.vdim;
        for (int d = d_first; d < g.vdim; d += d_step) value(d, [&](int at, float v) { if (at < g.vdim) out[at] = __float2bfloat16_rn(v * f); });
    };
    if (!DECODE) {
#pragma unroll
        for (int i = 0; i < 2; ++i)
            finish(p0 + wr + gr + 8 * i, m[i], l[i], [&](int d, auto&& put) {
                (void) d;
#pragma unroll
                for (int n = 0; n < VN; ++n) if (n < vn_n) { put(n * 8 + tq * 2, o[n][2 * i]); put(n * 8 + tq * 2 + 1, o[n][2 * i + 1]); }
            }, 0, 1 << 20, tq == 0);
    } else {
        // the warps' parts meet in shared memory: [warp][pair][vcld + 2]
        float* part = (float*) raw;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float* rec = part + (warp * 16 + gr + 8 * i) * (vcld + 2);
#pragma unroll
            for (int n = 0; n < VN; ++n) if (n < vn_n) { rec[n * 8 + tq * 2] = o[n][2 * i]; rec[n * 8 + tq * 2 + 1] = o[n][2 * i + 1]; }
            if (tq == 0) { rec[vcld] = m[i]; rec[vcld + 1] = l[i]; }
        }
        __syncthreads();
        for (int r = warp; r < 16 && p0 + r < pairs; r += S::WARPS) {
            float top = NEG_BIG, sum = 0.0f, f[S::WARPS];
#pragma unroll
            for (int w = 0; w < S::WARPS; ++w) top = fmaxf(top, part[(w * 16 + r) * (vcld + 2) + vcld]);
#pragma unroll
            for (int w = 0; w < S::WARPS; ++w) {
                const float* rec = part + (w * 16 + r) * (vcld + 2) + vcld;
                f[w] = exp2f(rec[0] - top);
                sum += rec[1] * f[w];
            }
            finish(p0 + r, top, sum, [&](int d, auto&& put) {
                float v = 0.0f;
#pragma unroll
                for (int w = 0; w < S::WARPS; ++w) v += part[(w * 16 + r) * (vcld + 2) + d] * f[w];
                put(d, v);
            }, lane, 32, lane == 0);
        }
    }
}

// One CTA per (row, head): its four warps take a quarter of the splits each; then the sink.
__global__ void __launch_bounds__(128) kv_merge_kernel(const KvAttnArgs a, int splits) {
    extern __shared__ float dyn[];                                // factors [splits] | sums [4][vcld]
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const KvGeom& g = a.g;
    const int row = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, vcld = g.vcld(), ld = vcld + 2;
    const float* rec = a.part + ((size_t) row * g.heads + h) * splits * ld;
    float *f = dyn, *sum = dyn + splits;
    // every warp forms the joint maximum and denominator; warp 0 leaves the factors
    float top = a.sink ? a.sink[h] * LOG2E : NEG_BIG, den = 0.0f;
    if (a.sink && lane == 0) den = 1.0f;
    const float s2 = top;
    for (int s = lane; s < splits; s += 32) top = fmaxf(top, rec[(size_t) s * ld + vcld]);
    top = skd::warp_max(top);
    den *= exp2f(s2 - top);
    for (int s = lane; s < splits; s += 32) {
        const float e = exp2f(rec[(size_t) s * ld + vcld] - top);
        if (warp == 0) f[s] = e;
        den = fmaf(rec[(size_t) s * ld + vcld + 1], e, den);
    }
    den = skd::warp_sum(den);
    __syncthreads();
    for (int d = 2 * lane; d < vcld; d += 64) {
        float2 v = make_float2(0.0f, 0.0f);
#pragma unroll 8
        for (int s = warp; s < splits; s += 4) {
            const float2 x = *reinterpret_cast<const float2*>(rec + (size_t) s * ld + d);
            v.x = fmaf(x.x, f[s], v.x); v.y = fmaf(x.y, f[s], v.y);
        }
        sum[warp * vcld + d] = v.x; sum[warp * vcld + d + 1] = v.y;
    }
    __syncthreads();
    for (int d = threadIdx.x; d < g.vdim; d += 128)
        ((bf16*) a.out)[(size_t) row * g.out_ld() + h * g.vdim + d] = __float2bfloat16_rn((sum[d] + sum[vcld + d] + sum[2 * vcld + d] + sum[3 * vcld + d]) / den);
}

// Pairs of a step's row reach no further than one row, so a decode step has a CTA row per sequence; prompts tile the pairs.
template <int KS, int VN, bool DECODE>
int32_t run_tile(const KvAttnArgs& a, cudaStream_t s) {
    typedef TileShape<KS, VN, DECODE> S;
    const KvGeom& g = a.g;
    const int group = g.heads / g.kv_heads, bytes = S::smem(g.kld(), g.vcld());
    const int mx = DECODE ? a.rows * ((group + 15) / 16) : (a.rows * group + S::ROWS - 1) / S::ROWS;
    const int seen = a.chunk > 0 ? std::min(a.kv_bound, a.chunk + (DECODE ? 0 : a.rows)) : a.kv_bound;
    const int64_t room = (int64_t) KV_PART_RECORDS / ((int64_t) a.rows * g.heads);
    const int tiles = (seen + TK - 1) / TK, base = mx * g.kv_heads, slots = sm_count() * std::max(1, std::min(3, 227 * 1024 / (bytes + 1024)));
    const int most = (int) std::max<int64_t>(1, std::min<int64_t>({(int64_t) tiles, room, (int64_t) (!DECODE && base * 2 > sm_count() ? 1 : 1024)}));
    // rounds of resident CTAs, each as long as its tiles and a fixed part of about three tiles; a merge costs about as much once
    int splits = 1;
    int64_t best = INT64_MAX;
    for (int k = 1; k <= most; ++k) {
        const int64_t cost = ((int64_t) base * k + slots - 1) / slots * ((tiles + k - 1) / k + 3) + (k > 1 ? 3 : 0);
        if (cost < best) { best = cost; splits = k; }
    }
    SK_TRY(ensure_dynamic_smem((const void*) kv_attn_tile_kernel<KS, VN, DECODE>, bytes));
    SK_CUDA(launch_pdl(kv_attn_tile_kernel<KS, VN, DECODE>, dim3(mx, g.kv_heads, splits), dim3(S::WARPS * 32), bytes, s, a, splits));
    if (splits > 1) SK_CUDA(launch_pdl(kv_merge_kernel, dim3(a.rows, g.heads), dim3(128), (splits + 4 * g.vcld()) * sizeof(float), s, a, splits));
    return SKAINET_CUDA_OK;
}
template <bool DECODE>
int32_t run_tile_size(const KvAttnArgs& a, cudaStream_t s) {
    const int n = std::max(a.g.kld(), a.g.vcld());
    if (n <= 64) return run_tile<4, 8, DECODE>(a, s);
    if (n <= 128) return run_tile<8, 16, DECODE>(a, s);
    return run_tile<16, 32, DECODE>(a, s);
}

template <typename T>
int32_t run_rows(const KvAttnArgs& a, cudaStream_t s) {
    const int bytes = (a.g.kld() + a.g.vcld()) * (int) sizeof(float);
    SK_TRY(ensure_dynamic_smem((const void*) kv_attn_rows_kernel<T>, bytes));
    SK_CUDA(launch_pdl(kv_attn_rows_kernel<T>, dim3(a.rows, a.g.heads), dim3(RK), bytes, s, a));
    return SKAINET_CUDA_OK;
}
template <typename T>
int32_t run_prep(const KvAttnArgs& a, cudaStream_t s) {
    SK_CUDA(launch_pdl(kv_prep_kernel<T>, dim3(a.rows, (a.g.heads + 2 * a.g.kv_heads + 7) / 8), dim3(256), 0, s, a));
    return SKAINET_CUDA_OK;
}

}  // namespace

int32_t launch_kv_attention(const KvAttnArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return SKAINET_CUDA_OK;
    if (a.f32_act) { SK_TRY(run_prep<float>(a, s)); return run_rows<float>(a, s); }
    const bool tiles = a.g.kld() <= 256 && a.g.vcld() <= 256;
    if (tiles && a.map.seq < 0) return run_tile_size<true>(a, s);
    SK_TRY(run_prep<bf16>(a, s));
    return tiles ? run_tile_size<false>(a, s) : run_rows<bf16>(a, s);
}

}  // namespace sk
