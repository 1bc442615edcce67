// Gated linear recurrences over prompts: chunks of 64 tokens as matrix products (contract: recurrence.cuh).
//
// With G_t the sum of the log decays of a chunk up to t, S the state before it, and all sums over the chunk's tokens,
//
//   u   state space: dt_t v_t;   delta rule: U = T W, W_t = beta_t (v_t - e^(G_t) S^T k_t), T = (I + A)^-1,
//                                A_ts = beta_t e^(G_t - G_s) (k_t . k_s) for s < t
//   o_t = e^(G_t) S^T q_t + sum_(s <= t) e^(G_t - G_s) (q_t . k_s) u_s
//   S  <- e^(G_end) S + sum_s e^(G_end - G_s) k_s u_s^T
//
//   recur_conv_kernel      convolution and silu in fp32, rounded to bf16; inverse lengths of q and k, step sizes, log decays.
//   recur_inverse_kernel   T of every chunk and head: column-wise substitution in fp32.
//   recur_scan_kernel      one CTA per head and 32 or 64 state columns walks the chunks; the state stays in registers (fp32).
//
// Exactness: q, k, v behind the convolution are bf16, everything after it is 32-bit. The tensor cores see fp32 factors as sums of
// three bf16 terms (24 bits); the lengths, decays and step sizes are applied outside the products, so q, k, v enter as one exact
// term and a product of an fp32 factor with one of them costs three MMAs, of two fp32 factors six. G is kept in double, so
// differences lose nothing to a strong decay earlier in the chunk.
#include "mma.cuh"
#include "recurrence.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr int CH = 64;                       // tokens of a chunk
constexpr int CONV_ROWS = 16;

int state_cols(const RecurGeom& g) { return !g.delta && g.vdim > 32 && g.kdim <= 128 ? 64 : 32; }

// Work buffers, all padded to whole chunks with zeros.
struct Work {
    bf16 *qk, *v, *inv;                      // [2 groups][rows][kp], [heads][rows][vp], [heads][chunk][3 terms][64][64]
    float *log_decay, *step, *length;        // [heads][rows], [heads][rows] (beta or dt), [2 groups][rows]
    int rows, kp, vp;
    size_t bytes;
};
Work layout(const RecurGeom& g, int rows, void* base) {
    Work w;
    w.rows = (rows + CH - 1) / CH * CH;
    w.kp = (g.kdim + 15) / 16 * 16;
    w.vp = (g.vdim + state_cols(g) - 1) / state_cols(g) * state_cols(g);
    size_t at = 0;
    auto take = [&](size_t bytes) { void* p = (char*) base + at; at += (bytes + 255) / 256 * 256; return p; };
    const size_t R = w.rows;
    w.qk = (bf16*) take(2 * g.groups * R * w.kp * 2);
    w.v = (bf16*) take(g.heads * R * w.vp * 2);
    w.inv = (bf16*) take(g.delta ? (size_t) g.heads * (R / CH) * 3 * CH * CH * 2 : 0);
    w.log_decay = (float*) take(g.heads * R * 4);
    w.step = (float*) take(g.heads * R * 4);
    w.length = (float*) take(2 * g.groups * R * 4);
    w.bytes = at;
    return w;
}

// grid: (16 rows, q or k vector of a group | v of a head)
__global__ void __launch_bounds__(256) recur_conv_kernel(const RecurArgs a, const Work w) {
    const RecurGeom& g = a.g;
    extern __shared__ float in[];                                   // [16 + taps - 1][n]
    const int u = blockIdx.y, row0 = blockIdx.x * CONV_ROWS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, T = g.taps;
    const bool is_v = u >= 2 * g.groups;
    const int h = u - 2 * g.groups, n = is_v ? g.vdim : g.kdim, np = is_v ? w.vp : w.kp;
    const int ch0 = is_v ? a.v_off + h * g.vdim : (u < g.groups ? a.q_off + u * g.kdim : a.k_off + (u - g.groups) * g.kdim);
    const float* tail = a.tail + (size_t) a.map.seq * g.tail_size();
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int pos0 = a.map.pos[a.map.seq];
    for (int r = warp; r < CONV_ROWS + T - 1; r += 8) {
        const int row = row0 + r - (T - 1);
        for (int c = lane; c < n; c += 32) in[r * n + c] = row < a.rows ? skd::conv_input(a, tail, 0, pos0, pos0 + row, ch0 + c) : 0.0f;
    }
    __syncthreads();
    bf16* out = is_v ? w.v + (size_t) h * w.rows * np : w.qk + (size_t) u * w.rows * np;
    for (int r = warp; r < CONV_ROWS; r += 8) {
        const int row = row0 + r;
        const bool live = row < a.rows;
        float ss = 0.0f;
        for (int c = lane; c < np; c += 32) {
            float y = 0.0f;
            if (live && c < n) {
                const float* wt = a.conv_w + (size_t) (ch0 + c) * T;
                y = a.conv_b ? a.conv_b[ch0 + c] : 0.0f;
                for (int j = 0; j < T; ++j) y = fmaf(wt[j], in[(r + j) * n + c], y);
                y = skd::silu(y);
            }
            const bf16 b = __float2bfloat16_rn(y);
            out[(size_t) row * np + c] = b;
            y = __bfloat162float(b);
            ss = fmaf(y, y, ss);
        }
        if (!is_v) {
            ss = skd::warp_sum(ss);
            if (lane == 0) w.length[(size_t) u * w.rows + row] = !live ? 0.0f : g.delta ? 1.0f / sqrtf(ss + 1e-6f) * (u < g.groups ? a.q_scale : 1.0f) : 1.0f;
        }
    }
    if (is_v && threadIdx.x < CONV_ROWS) {
        const int row = row0 + threadIdx.x;
        float ld = 0.0f, st = 0.0f;
        if (row < a.rows) {
            const float* p = a.proj + (size_t) row * a.proj_ld;
            const float dt = skd::softplus(p[a.dt_off + h] + a.dt_bias[h]);
            ld = -expf(a.a_log[h]) * dt;
            st = g.delta ? skd::sigmoid(p[a.beta_off + h]) : dt;
        }
        w.log_decay[(size_t) h * w.rows + row] = ld; w.step[(size_t) h * w.rows + row] = st;
    }
}

// The same for four taps and sizes that fill the tiles: a warp owns 128 channels (four per lane) of 16 rows and slides over them
// in registers. grid: (16 rows, groups of eight warps over q and k vectors | v channels | 32 heads' step sizes)
__global__ void __launch_bounds__(256) recur_conv4_kernel(const RecurArgs a, const Work w, int v_blocks) {
    const RecurGeom& g = a.g;
    const int unit = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, row0 = blockIdx.x * CONV_ROWS, qk_units = 2 * g.groups;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    if (unit >= qk_units + v_blocks) {
        const int h = (unit - qk_units - v_blocks) * 32 + lane;
        if (h >= g.heads) return;
        const float neg_a = -expf(a.a_log[h]), bias = a.dt_bias[h];
#pragma unroll 4
        for (int r = 0; r < CONV_ROWS; ++r) {
            const int row = row0 + r;
            float ld = 0.0f, st = 0.0f;
            if (row < a.rows) {
                const float* p = a.proj + (size_t) row * a.proj_ld;
                const float dt = skd::softplus(p[a.dt_off + h] + bias);
                ld = neg_a * dt;
                st = g.delta ? skd::sigmoid(p[a.beta_off + h]) : dt;
            }
            w.log_decay[(size_t) h * w.rows + row] = ld; w.step[(size_t) h * w.rows + row] = st;
        }
        return;
    }
    const bool is_v = unit >= qk_units;
    const int u = unit;                                             // q or k vector
    int ch, out_ld;
    bf16* out;
    bool live;
    if (is_v) {
        const int c = (unit - qk_units) * 128 + 4 * lane, h = c / g.vdim;
        live = c < g.v_dim();
        ch = a.v_off + c; out_ld = w.vp;
        out = w.v + (size_t) h * w.rows * w.vp + c % g.vdim;
    } else {
        live = 4 * lane < g.kdim;
        ch = (u < g.groups ? a.q_off + u * g.kdim : a.k_off + (u - g.groups) * g.kdim) + 4 * lane; out_ld = w.kp;
        out = w.qk + (size_t) u * w.rows * w.kp + 4 * lane;
    }
    const int pos0 = a.map.pos[a.map.seq];
    const float* tail = a.tail + (size_t) a.map.seq * g.tail_size();
    auto input = [&](int row) {
        if (!live || pos0 + row < 0 || row >= a.rows) return make_float4(0, 0, 0, 0);
        const float* p = row >= 0 ? a.proj + (size_t) row * a.proj_ld + a.conv_off + ch : tail + (size_t) ((pos0 + row) % 4) * g.conv_dim() + ch;
        return *reinterpret_cast<const float4*>(p);
    };
    float4 wt[4], bias = make_float4(0, 0, 0, 0);                   // taps of channel ch + i
#pragma unroll
    for (int i = 0; i < 4; ++i) wt[i] = live ? *reinterpret_cast<const float4*>(a.conv_w + (size_t) (ch + i) * 4) : make_float4(0, 0, 0, 0);
    if (live && a.conv_b) bias = make_float4(a.conv_b[ch], a.conv_b[ch + 1], a.conv_b[ch + 2], a.conv_b[ch + 3]);
    float4 x0 = input(row0 - 3), x1 = input(row0 - 2), x2 = input(row0 - 1);
#pragma unroll 8
    for (int r = 0; r < CONV_ROWS; ++r) {
        const int row = row0 + r;
        const float4 x3 = input(row);
        float4 y;
        y.x = skd::silu(fmaf(wt[0].w, x3.x, fmaf(wt[0].z, x2.x, fmaf(wt[0].y, x1.x, fmaf(wt[0].x, x0.x, bias.x)))));
        y.y = skd::silu(fmaf(wt[1].w, x3.y, fmaf(wt[1].z, x2.y, fmaf(wt[1].y, x1.y, fmaf(wt[1].x, x0.y, bias.y)))));
        y.z = skd::silu(fmaf(wt[2].w, x3.z, fmaf(wt[2].z, x2.z, fmaf(wt[2].y, x1.z, fmaf(wt[2].x, x0.z, bias.z)))));
        y.w = skd::silu(fmaf(wt[3].w, x3.w, fmaf(wt[3].z, x2.w, fmaf(wt[3].y, x1.w, fmaf(wt[3].x, x0.w, bias.w)))));
        x0 = x1; x1 = x2; x2 = x3;
        uint2 b = make_uint2(skd::pack_bf16(y.x, y.y), skd::pack_bf16(y.z, y.w));
        if (row >= a.rows) b = make_uint2(0, 0);
        if (live) *reinterpret_cast<uint2*>(out + (size_t) row * out_ld) = b;
        if (!is_v) {
            const float e0 = skd::bf16_lo(b.x), e1 = skd::bf16_hi(b.x), e2 = skd::bf16_lo(b.y), e3 = skd::bf16_hi(b.y);
            const float ss = skd::warp_sum(live ? fmaf(e0, e0, fmaf(e1, e1, fmaf(e2, e2, e3 * e3))) : 0.0f);
            if (lane == 0) w.length[(size_t) u * w.rows + row] = row >= a.rows ? 0.0f : g.delta ? 1.0f / sqrtf(ss + 1e-6f) * (u < g.groups ? a.q_scale : 1.0f) : 1.0f;
        }
    }
}

// Sums of the log decays up to every token of a chunk; lane l holds tokens 2l and 2l + 1.
__device__ __forceinline__ void decay_sums(float a, float b, int lane, double (&g)[2]) {
    double s = (double) a + (double) b;
    const double own = s;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const double v = __shfl_up_sync(~0u, s, o); if (lane >= o) s += v; }
    g[0] = s - own + (double) a;
    g[1] = s;
}

constexpr double MILD_DECAY = 50.0;          // a chunk's log decay up to which e^50 and e^-50 may be applied apart

constexpr int INV_LD = CH + 4;
// grid: (chunk, head); 128 threads
__global__ void __launch_bounds__(128) recur_inverse_kernel(const RecurArgs a, const Work w) {
    const RecurGeom& g = a.g;
    extern __shared__ __align__(16) uint8_t raw[];
    __shared__ double G[CH];
    __shared__ float st[CH], rk[CH];
    const int kp = w.kp, lds = kp + 8, h = blockIdx.y, grp = h / (g.heads / g.groups), r0 = blockIdx.x * CH;
    bf16* k = (bf16*) raw;
    float* A = (float*) (raw + CH * lds * 2);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, tq = lane & 3;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const bf16* src = w.qk + ((size_t) (g.groups + grp) * w.rows + r0) * kp;
    for (int i = threadIdx.x; i < CH * (kp / 8); i += 128)
        *reinterpret_cast<uint4*>(k + (i / (kp / 8)) * lds + (i % (kp / 8)) * 8) = *reinterpret_cast<const uint4*>(src + (size_t) i * 8);
    if (warp == 0) {
        const float2 ld = *reinterpret_cast<const float2*>(w.log_decay + (size_t) h * w.rows + r0 + 2 * lane);
        double s[2];
        decay_sums(ld.x, ld.y, lane, s);
        G[2 * lane] = s[0]; G[2 * lane + 1] = s[1];
    } else if (warp < 3) {
        const int i = threadIdx.x - 32;
        st[i] = w.step[(size_t) h * w.rows + r0 + i]; rk[i] = w.length[(size_t) (g.groups + grp) * w.rows + r0 + i];
    }
    __syncthreads();
    float c[8][4] = {};
    const uint32_t base = skd::smem_u32(k), a_at = base + ((warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * lds + (lane >> 4) * 8) * 2;
    const uint32_t b_at = base + (((lane & 7) + (lane >> 4) * 8) * lds + ((lane >> 3) & 1) * 8) * 2;
    for (int ks = 0; ks < kp / 16; ++ks) {
        uint32_t f[4], b[4];
        skd::ldsm4(f, a_at + ks * 32);
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
            if (n > 2 * warp) break;
            skd::ldsm4(b, b_at + (n * 8 * lds + ks * 16) * 2);
            skd::mma_bf16(c[n], f[0], f[1], f[2], f[3], b[0], b[1]);
            skd::mma_bf16(c[n + 1], f[0], f[1], f[2], f[3], b[2], b[3]);
        }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int t = warp * 16 + gr + (i >> 1) * 8, s = n * 8 + tq * 2 + (i & 1);
            A[t * INV_LD + s] = s < t ? st[t] * rk[t] * rk[s] * expf((float) (G[t] - G[s])) * c[n][i] : 0.0f;
        }
    __syncthreads();
    if (threadIdx.x >= CH) return;
    // column j of the inverse: x_i = [i = j] - sum_(m < i) A_im x_m
    float x[CH];
    const int j = threadIdx.x;
    bf16* out = w.inv + ((size_t) h * (w.rows / CH) + blockIdx.x) * 3 * CH * CH + j;
#pragma unroll
    for (int i = 0; i < CH; ++i) {
        float v = i == j ? 1.0f : 0.0f, v2 = 0.0f;
#pragma unroll
        for (int m = 0; m < i; m += 4) {
            const float4 q = *reinterpret_cast<const float4*>(A + i * INV_LD + m);
            v = fmaf(-q.x, x[m], v);
            if (m + 1 < i) v2 = fmaf(-q.y, x[m + 1], v2);
            if (m + 2 < i) v = fmaf(-q.z, x[m + 2], v);
            if (m + 3 < i) v2 = fmaf(-q.w, x[m + 3], v2);
        }
        x[i] = v + v2;
        float r = x[i];
#pragma unroll
        for (int t = 0; t < 3; ++t) {
            const bf16 b = __float2bfloat16_rn(r);
            out[(size_t) t * CH * CH + i * CH] = b;
            r -= __bfloat162float(b);
        }
    }
}

// KT: 16-row tiles of the state per warp (four warps hold it), so key sizes up to 64 * KT.
template <bool DELTA, int VT, int KT>
struct ScanShape {
    static constexpr int STAGES = KT <= 2 ? 2 : 1, LV = VT + 8, LT = CH + 8, V_TERM = CH * LV * 2;
    static constexpr int INV = DELTA ? 3 * CH * LT * 2 : 0;
    static __host__ __device__ int stage(int kp) { return 2 * CH * (kp + 8) * 2 + V_TERM + INV; }        // q | k | v | T
    static __host__ __device__ int smem(int kp) { return STAGES * stage(kp) + 3 * kp * LV * 2 + (DELTA ? 9 : 3) * V_TERM; }   // stages | S | U' | W | U
};

template <bool DELTA, int VT, int KT>
__global__ void __launch_bounds__(256, 1) recur_scan_kernel(const RecurArgs a, const Work w) {
    typedef ScanShape<DELTA, VT, KT> Z;
    constexpr int NT = VT / 8, LV = Z::LV;
    const RecurGeom& g = a.g;
    extern __shared__ __align__(16) uint8_t raw[];
    __shared__ double sG[2][CH];
    __shared__ float s_step[2][CH], s_rq[2][CH], s_rk[2][CH], s_e[2][CH], s_f[2][CH], s_col[2][CH];      // e^G, e^(G_end - G), the latter with |k|^-1 (and the step)
    const int kp = w.kp, lk = kp + 8, ksn = kp / 16, tiles = w.vp / VT, h = blockIdx.x / tiles, c0 = (blockIdx.x % tiles) * VT, grp = h / (g.heads / g.groups);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, tq = lane & 3, n_chunks = w.rows / CH;
    const uint32_t base = skd::smem_u32(raw), s_at = base + Z::STAGES * Z::stage(kp), up_at = s_at + 3 * kp * LV * 2, w_at = up_at + 3 * Z::V_TERM, u_at = w_at + 3 * Z::V_TERM;
    const int s_term = kp * LV * 2;
    float* state = a.state + (size_t) a.map.seq * g.state_size() + (size_t) h * g.kdim * g.vld();
    skd::pdl_launch_dependents();
    const int pos0 = a.map.pos[a.map.seq];
    const float skip = DELTA ? 0.0f : a.d[h];
    const bool holder = warp < 4;                                   // warps 0-3 hold the state, 4-7 the outputs
    const int mt = holder ? warp : 7 - warp;                        // the warp's 16 tokens; later tokens sum over more, so the two kinds run opposite ways

    // state rows 16 (mt + 4 i) + gr (+ 8), columns 8 n + 2 tq (+ 1); left by an earlier pass
    float S[KT][NT][4];
    if (holder)
#pragma unroll
        for (int i = 0; i < KT; ++i)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int r = 16 * (mt + 4 * i) + gr + 8 * e, c = c0 + n * 8 + tq * 2;
                    const float2 v = pos0 > 0 && r < g.kdim && c < g.vld() ? *reinterpret_cast<const float2*>(state + (size_t) r * g.vld() + c) : make_float2(0, 0);
                    S[i][n][2 * e] = v.x; S[i][n][2 * e + 1] = v.y;
                }
    skd::pdl_wait();

    auto load_chunk = [&](int c, int stage) {
        const uint32_t q = base + stage * Z::stage(kp), k = q + CH * lk * 2, v = k + CH * lk * 2, t = v + Z::V_TERM;
        const bf16 *gq = w.qk + ((size_t) grp * w.rows + c * CH) * kp, *gk = w.qk + ((size_t) (g.groups + grp) * w.rows + c * CH) * kp;
        const bf16* gv = w.v + ((size_t) h * w.rows + c * CH) * w.vp + c0;
        const int kc = kp / 8;
        for (int i = threadIdx.x; i < CH * kc; i += 256) {
            const uint32_t at = ((i / kc) * lk + (i % kc) * 8) * 2;
            skd::cp16(q + at, gq + (size_t) i * 8);
            skd::cp16(k + at, gk + (size_t) i * 8);
        }
        for (int i = threadIdx.x; i < CH * (VT / 8); i += 256) skd::cp16(v + ((i / (VT / 8)) * LV + (i % (VT / 8)) * 8) * 2, gv + (size_t) (i / (VT / 8)) * w.vp + (i % (VT / 8)) * 8);
        if (DELTA) {
            const bf16* gt = w.inv + ((size_t) h * n_chunks + c) * 3 * CH * CH;
            for (int i = threadIdx.x; i < 3 * CH * (CH / 8); i += 256) skd::cp16(t + ((i / (CH / 8)) * Z::LT + (i % (CH / 8)) * 8) * 2, gt + (size_t) i * 8);
        }
        skd::cp_commit();
    };
    // one warp turns a chunk's log decays into sums and factors
    struct Scal { float2 ld, st, rq, rk; };
    auto fetch_scal = [&](int c) {
        Scal s;
        const size_t at = (size_t) c * CH + 2 * lane;
        s.ld = *reinterpret_cast<const float2*>(w.log_decay + (size_t) h * w.rows + at); s.st = *reinterpret_cast<const float2*>(w.step + (size_t) h * w.rows + at);
        s.rq = *reinterpret_cast<const float2*>(w.length + (size_t) grp * w.rows + at); s.rk = *reinterpret_cast<const float2*>(w.length + (size_t) (g.groups + grp) * w.rows + at);
        return s;
    };
    auto store_scal = [&](const Scal& s, int b) {
        double d[2];
        decay_sums(s.ld.x, s.ld.y, lane, d);
        const double end = __shfl_sync(~0u, d[1], 31);
        const float st[2] = {s.st.x, s.st.y}, rq[2] = {s.rq.x, s.rq.y}, rk[2] = {s.rk.x, s.rk.y};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int t = 2 * lane + i;
            sG[b][t] = d[i]; s_step[b][t] = st[i]; s_rq[b][t] = rq[i]; s_rk[b][t] = rk[i];
            s_e[b][t] = expf((float) d[i]); s_f[b][t] = expf((float) (end - d[i]));
            s_col[b][t] = s_f[b][t] * rk[i] * (DELTA ? 1.0f : st[i]);
        }
    };
    // three bf16 terms of a value pair into the terms' tiles
    auto put3 = [&](uint32_t at, int term, float x, float y) {
        uint32_t t[3];
        skd::split3(x, y, t);
#pragma unroll
        for (int i = 0; i < 3; ++i) asm volatile("st.shared.u32 [%0], %1;" ::"r"(at + i * term), "r"(t[i]) : "memory");
    };
    auto put_state = [&]() {
#pragma unroll
        for (int i = 0; i < KT; ++i) {
            if (mt + 4 * i >= ksn) break;
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) put3(s_at + ((16 * (mt + 4 * i) + gr + 8 * e) * LV + n * 8 + tq * 2) * 2, s_term, S[i][n][2 * e], S[i][n][2 * e + 1]);
        }
    };
    const int lr = lane & 7, l8 = (lane >> 3) & 1, l16 = lane >> 4;
    const uint32_t bt_off = ((lr + l8 * 8) * LV + l16 * 8) * 2;     // B fragments of a [k][columns] tile, transposed on load

    load_chunk(0, 0);
    if (warp == 7) store_scal(fetch_scal(0), 0);
    if (holder) put_state();

    for (int c = 0; c < n_chunks; ++c) {
        const int b = c & 1, stage = Z::STAGES == 2 ? b : 0;
        const uint32_t q = base + stage * Z::stage(kp), k = q + CH * lk * 2, v = k + CH * lk * 2, t_at = v + Z::V_TERM;
        skd::cp_wait<0>();
        __syncthreads();
        if (Z::STAGES == 2 && c + 1 < n_chunks) load_chunk(c + 1, b ^ 1);
        Scal next = {};
        if (warp == 7 && c + 1 < n_chunks) next = fetch_scal(c + 1);
        const int t0 = mt * 16 + gr, t1 = t0 + 8;

        float acc[NT][4];
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) acc[n][i] = 0.0f;
        if (DELTA || !holder) {                                     // k S or q S, 16 tokens
            const uint32_t a_at = (holder ? k : q) + ((mt * 16 + lr + l8 * 8) * lk + l16 * 8) * 2;
            for (int ks = 0; ks < ksn; ++ks) {
                uint32_t f[4];
                skd::ldsm4(f, a_at + ks * 32);
#pragma unroll
                for (int n = 0; n < NT; n += 4) {                   // four sums in flight
                    uint32_t bb[3][2][4];
#pragma unroll
                    for (int j = 0; j < 3; ++j)
#pragma unroll
                        for (int e = 0; e < 2; ++e) skd::ldsm4_t(bb[j][e], s_at + j * s_term + bt_off + (ks * 16 * LV + (n + 2 * e) * 8) * 2);
#pragma unroll
                    for (int j = 2; j >= 0; --j)
#pragma unroll
                        for (int e = 0; e < 4; ++e) skd::mma_bf16(acc[n + e], f[0], f[1], f[2], f[3], bb[j][e >> 1][2 * (e & 1)], bb[j][e >> 1][2 * (e & 1) + 1]);
                }
            }
        }
        float p[8][4], row0 = 0.0f, row1 = 0.0f;
        if (holder) {
            const float e0 = DELTA ? s_e[b][t0] * s_rk[b][t0] : 0.0f, e1 = DELTA ? s_e[b][t1] * s_rk[b][t1] : 0.0f, b0 = s_step[b][t0], b1 = s_step[b][t1];
            const float f0 = s_f[b][t0] * s_rk[b][t0], f1 = s_f[b][t1] * s_rk[b][t1];
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                uint32_t x0, x1;
                const uint32_t at = (n * 8 + tq * 2) * 2;
                asm volatile("ld.shared.u32 %0, [%1];" : "=r"(x0) : "r"(v + t0 * LV * 2 + at));
                asm volatile("ld.shared.u32 %0, [%1];" : "=r"(x1) : "r"(v + t1 * LV * 2 + at));
                const float w0 = b0 * (skd::bf16_lo(x0) - e0 * acc[n][0]), w1 = b0 * (skd::bf16_hi(x0) - e0 * acc[n][1]);
                const float w2 = b1 * (skd::bf16_lo(x1) - e1 * acc[n][2]), w3 = b1 * (skd::bf16_hi(x1) - e1 * acc[n][3]);
                if (DELTA) { put3(w_at + t0 * LV * 2 + at, Z::V_TERM, w0, w1); put3(w_at + t1 * LV * 2 + at, Z::V_TERM, w2, w3); }
                else { put3(up_at + t0 * LV * 2 + at, Z::V_TERM, w0 * f0, w1 * f0); put3(up_at + t1 * LV * 2 + at, Z::V_TERM, w2 * f1, w3 * f1); }
            }
            if (DELTA) {
                asm volatile("bar.sync 1, 128;" ::: "memory");
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int i = 0; i < 4; ++i) acc[n][i] = 0.0f;
                for (int ks = 0; ks <= mt; ++ks) {                  // T is lower triangular
                    uint32_t f[3][4];
#pragma unroll
                    for (int i = 0; i < 3; ++i) skd::ldsm4(f[i], t_at + ((i * CH + mt * 16 + lr + l8 * 8) * Z::LT + ks * 16 + l16 * 8) * 2);
#pragma unroll
                    for (int n = 0; n < NT; n += 4)
#pragma unroll
                        for (int j = 2; j >= 0; --j) {
                            uint32_t bb[2][4];
#pragma unroll
                            for (int e = 0; e < 2; ++e) skd::ldsm4_t(bb[e], w_at + j * Z::V_TERM + bt_off + (ks * 16 * LV + (n + 2 * e) * 8) * 2);
#pragma unroll
                            for (int i = 2 - j; i >= 0; --i)
#pragma unroll
                                for (int e = 0; e < 4; ++e) skd::mma_bf16(acc[n + e], f[i][0], f[i][1], f[i][2], f[i][3], bb[e >> 1][2 * (e & 1)], bb[e >> 1][2 * (e & 1) + 1]);
                        }
                }
#pragma unroll
                for (int n = 0; n < NT; ++n) {
                    const uint32_t at = (n * 8 + tq * 2) * 2;
                    put3(u_at + t0 * LV * 2 + at, Z::V_TERM, acc[n][0], acc[n][1]); put3(u_at + t1 * LV * 2 + at, Z::V_TERM, acc[n][2], acc[n][3]);
                    put3(up_at + t0 * LV * 2 + at, Z::V_TERM, acc[n][0] * f0, acc[n][1] * f0); put3(up_at + t1 * LV * 2 + at, Z::V_TERM, acc[n][2] * f1, acc[n][3] * f1);
                }
            }
        } else {
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) p[n][i] = 0.0f;
            const uint32_t a_at = q + ((mt * 16 + lr + l8 * 8) * lk + l16 * 8) * 2, b_at = k + ((lr + l16 * 8) * lk + l8 * 8) * 2;
            for (int ks = 0; ks < ksn; ++ks) {
                uint32_t f[4];
                skd::ldsm4(f, a_at + ks * 32);
#pragma unroll
                for (int n = 0; n < 8; n += 2) {
                    if (n > 2 * mt) break;
                    uint32_t bb[4];
                    skd::ldsm4(bb, b_at + (n * 8 * lk + ks * 16) * 2);
                    skd::mma_bf16(p[n], f[0], f[1], f[2], f[3], bb[0], bb[1]);
                    skd::mma_bf16(p[n + 1], f[0], f[1], f[2], f[3], bb[2], bb[3]);
                }
            }
            const double G0 = sG[b][t0], G1 = sG[b][t1], end = sG[b][CH - 1];
            float e0, e1;                                           // factors of S^T q now, and of the outputs at the end
            row0 = s_rq[b][t0]; row1 = s_rq[b][t1];
            if (end > -MILD_DECAY) {
                // e^(G_t - G_s) = e^(G_t - G_end) e^(G_end - G_s): a factor per column here and one per row at the end, both in range
#pragma unroll
                for (int n = 0; n < 8; ++n) {
                    if (n > 2 * mt + 1) break;
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const int s = n * 8 + tq * 2 + i;
                        const float f = s_col[b][s];
                        p[n][i] *= s <= t0 ? f : 0.0f;
                        p[n][i + 2] *= s <= t1 ? f : 0.0f;
                    }
                }
                e0 = e1 = s_e[b][CH - 1];
                row0 *= expf((float) (G0 - end)); row1 *= expf((float) (G1 - end));
            } else {
#pragma unroll
                for (int n = 0; n < 8; ++n) {
                    if (n > 2 * mt + 1) break;
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int s = n * 8 + tq * 2 + (i & 1), t = i < 2 ? t0 : t1;
                        p[n][i] *= s <= t ? expf((float) ((i < 2 ? G0 : G1) - sG[b][s])) * s_rk[b][s] * (DELTA ? 1.0f : s_step[b][s]) : 0.0f;
                    }
                }
                e0 = s_e[b][t0]; e1 = s_e[b][t1];
            }
#pragma unroll
            for (int n = 0; n < NT; ++n) { acc[n][0] *= e0; acc[n][1] *= e0; acc[n][2] *= e1; acc[n][3] *= e1; }
        }
        __syncthreads();
        if (holder) {
            const float end = s_e[b][CH - 1];
#pragma unroll
            for (int i = 0; i < KT; ++i) {
                if (mt + 4 * i >= ksn) break;
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) S[i][n][e] *= end;
            }
#pragma unroll
            for (int ks = 0; ks < CH / 16; ++ks)
{
                uint32_t f[KT][4];                                  // k transposed: rows are key coordinates
#pragma unroll
                for (int i = 0; i < KT; ++i) if (mt + 4 * i < ksn) skd::ldsm4_t(f[i], k + ((ks * 16 + lr + l16 * 8) * lk + 16 * (mt + 4 * i) + l8 * 8) * 2);
#pragma unroll
                for (int n = 0; n < NT; n += 2) {
                    uint32_t bb[3][4];
#pragma unroll
                    for (int j = 0; j < 3; ++j) skd::ldsm4_t(bb[j], up_at + j * Z::V_TERM + bt_off + (ks * 16 * LV + n * 8) * 2);
#pragma unroll
                    for (int j = 2; j >= 0; --j)
#pragma unroll
                        for (int i = 0; i < KT; ++i) {
                            if (mt + 4 * i >= ksn) break;
                            skd::mma_bf16(S[i][n], f[i][0], f[i][1], f[i][2], f[i][3], bb[j][0], bb[j][1]);
                            skd::mma_bf16(S[i][n + 1], f[i][0], f[i][1], f[i][2], f[i][3], bb[j][2], bb[j][3]);
                        }
                }
            }
            put_state();
        } else {
#pragma unroll
            for (int ks = 0; ks < CH / 16; ++ks) {
                if (ks > mt) break;
                uint32_t f[4][3];
                skd::split3(p[2 * ks][0], p[2 * ks][1], f[0]); skd::split3(p[2 * ks][2], p[2 * ks][3], f[1]);
                skd::split3(p[2 * ks + 1][0], p[2 * ks + 1][1], f[2]); skd::split3(p[2 * ks + 1][2], p[2 * ks + 1][3], f[3]);
#pragma unroll
                for (int n = 0; n < NT; n += 4)
#pragma unroll
                    for (int j = DELTA ? 2 : 0; j >= 0; --j) {
                        uint32_t bb[2][4];
#pragma unroll
                        for (int e = 0; e < 2; ++e) skd::ldsm4_t(bb[e], (DELTA ? u_at + j * Z::V_TERM : v) + bt_off + (ks * 16 * LV + (n + 2 * e) * 8) * 2);
#pragma unroll
                        for (int i = 2 - j; i >= 0; --i)
#pragma unroll
                            for (int e = 0; e < 4; ++e) skd::mma_bf16(acc[n + e], f[0][i], f[1][i], f[2][i], f[3][i], bb[e >> 1][2 * (e & 1)], bb[e >> 1][2 * (e & 1) + 1]);
                    }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = e ? t1 : t0, row = c * CH + t;
                if (row >= a.rows) continue;
                float* out = a.out + (size_t) row * g.v_dim() + (size_t) h * g.vdim;
#pragma unroll
                for (int n = 0; n < NT; ++n) {
                    uint32_t x = 0;
                    if (!DELTA) asm volatile("ld.shared.u32 %0, [%1];" : "=r"(x) : "r"(v + (t * LV + n * 8 + tq * 2) * 2));
                    const int col = c0 + n * 8 + tq * 2;
                    const float f = e ? row1 : row0;
                    if (col < g.vdim) out[col] = fmaf(acc[n][2 * e], f, skip * skd::bf16_lo(x));
                    if (col + 1 < g.vdim) out[col + 1] = fmaf(acc[n][2 * e + 1], f, skip * skd::bf16_hi(x));
                }
            }
            if (warp == 7 && c + 1 < n_chunks) store_scal(next, b ^ 1);
        }
        if (Z::STAGES == 1 && c + 1 < n_chunks) { __syncthreads(); load_chunk(c + 1, 0); }
    }
    if (holder)
#pragma unroll
        for (int i = 0; i < KT; ++i)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int r = 16 * (mt + 4 * i) + gr + 8 * e, cc = c0 + n * 8 + tq * 2;
                    if (r < g.kdim && cc < g.vld()) *reinterpret_cast<float2*>(state + (size_t) r * g.vld() + cc) = make_float2(S[i][n][2 * e], S[i][n][2 * e + 1]);
                }
    // the convolution inputs the next pass needs; the kernel that reads the old ones is done
    const int keep = min(a.rows, g.taps), total = keep * g.conv_dim();
    for (int i = blockIdx.x * 256 + threadIdx.x; i < total; i += gridDim.x * 256) {
        const int row = a.rows - 1 - i / g.conv_dim(), ch = i % g.conv_dim();
        a.tail[(size_t) a.map.seq * g.tail_size() + (size_t) ((pos0 + row) % g.taps) * g.conv_dim() + ch] = a.proj[(size_t) row * a.proj_ld + a.conv_off + ch];
    }
}

template <bool DELTA, int VT, int KT>
int32_t run_scan(const RecurArgs& a, const Work& w, cudaStream_t s) {
    const int bytes = ScanShape<DELTA, VT, KT>::smem(w.kp);
    SK_TRY(ensure_dynamic_smem((const void*) recur_scan_kernel<DELTA, VT, KT>, bytes));
    SK_CUDA(launch_pdl(recur_scan_kernel<DELTA, VT, KT>, dim3(a.g.heads * (w.vp / VT)), dim3(256), bytes, s, a, w));
    return SKAINET_CUDA_OK;
}

}  // namespace

size_t recur_work_bytes(const RecurGeom& g, int rows) {
    if (g.kdim > 256 || g.vdim > 512 || g.taps > 32) return 0;
    return layout(g, rows, nullptr).bytes;
}

int32_t launch_recur_chunks(const RecurArgs& a, cudaStream_t s) {
    const RecurGeom& g = a.g;
    const Work w = layout(g, a.rows, a.work);
    const bool quads = (a.proj_ld | a.conv_off | a.q_off | a.k_off | a.v_off) % 4 == 0;
    if (g.taps == 4 && quads && g.kdim == w.kp && g.kdim <= 128 && g.vdim == w.vp) {
        const int v_blocks = (g.v_dim() + 127) / 128, units = 2 * g.groups + v_blocks + (g.heads + 31) / 32;
        SK_CUDA(launch_pdl(recur_conv4_kernel, dim3(w.rows / CONV_ROWS, (units + 7) / 8), dim3(256), 0, s, a, w, v_blocks));
    } else {
        const int conv_bytes = (CONV_ROWS + g.taps - 1) * std::max(g.kdim, g.vdim) * (int) sizeof(float);
        SK_TRY(ensure_dynamic_smem((const void*) recur_conv_kernel, conv_bytes));
        SK_CUDA(launch_pdl(recur_conv_kernel, dim3(w.rows / CONV_ROWS, 2 * g.groups + g.heads), dim3(256), conv_bytes, s, a, w));
    }
    if (!g.delta) {
        if (state_cols(g) == 64) return run_scan<false, 64, 2>(a, w, s);
        return w.kp <= 128 ? run_scan<false, 32, 2>(a, w, s) : run_scan<false, 32, 4>(a, w, s);
    }
    const int inv_bytes = CH * (w.kp + 8) * 2 + CH * INV_LD * 4;
    SK_TRY(ensure_dynamic_smem((const void*) recur_inverse_kernel, inv_bytes));
    SK_CUDA(launch_pdl(recur_inverse_kernel, dim3(w.rows / CH, g.heads), dim3(128), inv_bytes, s, a, w));
    return w.kp <= 128 ? run_scan<true, 32, 2>(a, w, s) : run_scan<true, 32, 4>(a, w, s);
}

}  // namespace sk
