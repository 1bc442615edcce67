// Latent attention kernels (contract: latent_attn.cuh).
//
// A step's chain for few rows (decode):  prep + fold of W_uk | attention over key splits | merge + W_uv + gate
// and for many rows (prefill):           prep | fold (grouped GEMM) | attention | [merge] | W_uv + gate (grouped GEMM)
//
// latent_attn_mma_kernel (bf16): the MMA rows are (activation row, head) pairs, which all read the same keys; one staged
// [key][latent | rotated part] tile is the B operand of the scores and, its latent columns transposed on load, of the mix.
// latent_attn_rows_kernel: the same in fp32 FMA, one CTA per (row, head); the 32-bit mode, and bf16 models whose latent does
// not fit the tile kernel's registers or shared memory.
#include "latent_attn.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr float NEG_BIG = -1e30f;            // running maximum of a row that has seen no key: finite, so differences stay defined
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float block_sum_256(float v, float* sh) {
    v = skd::warp_sum(v);
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
    for (int i = 0; i < (int) blockDim.x / 32; ++i) t += sh[i];
    __syncthreads();
    return t;
}

// (u, v) -> (u c - v s, v c + u s) with every product and sum rounded on its own
__device__ __forceinline__ float2 rotate(float u, float v, float c, float s) {
    return make_float2(__fsub_rn(__fmul_rn(u, c), __fmul_rn(v, s)), __fadd_rn(__fmul_rn(v, c), __fmul_rn(u, s)));
}

// The latent, the shared rotated key part and the gates of one row; run by a whole CTA of 256 threads.
template <typename T>
__device__ void prep_row(const LatentArgs& a, int row, float* sh) {
    const LatentGeom& g = a.g;
    const float* p = a.proj + (size_t) row * a.proj_ld;
    const int pos = a.map.pos_of(row), seq = a.map.seq_of(row), half = g.rot_dim >> 1;
    if (a.owner) {
        const float* kv = p + a.q_rows;
        T* dst = (T*) a.cache.rows + ((size_t) seq * a.cache.cap + pos % a.cache.cap) * g.key_ld();
        float ss = 0.0f;
        for (int i = threadIdx.x; i < g.kv_rank; i += blockDim.x) ss += kv[i] * kv[i];
        ss = block_sum_256(ss, sh);
        const float r = 1.0f / sqrtf(ss / (float) g.kv_rank + a.eps);
        for (int i = threadIdx.x; i < g.kv_rank; i += blockDim.x) skd::store_act(dst + i, kv[i] * r * a.norm[i]);
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            const float2 o = rotate(kv[g.kv_rank + i], kv[g.kv_rank + i + half], a.cos_t[(size_t) pos * half + i], a.sin_t[(size_t) pos * half + i]);
            skd::store_act(dst + g.rank_pad() + i, o.x); skd::store_act(dst + g.rank_pad() + i + half, o.y);
        }
    }
    const float* gt = p + a.q_rows + (a.owner ? g.kv_rank + g.rot_dim : 0);
    for (int i = threadIdx.x; i < g.heads; i += blockDim.x) a.gates[(size_t) row * g.heads + i] = skd::sigmoid(gt[i]);
}

template <typename T>
__device__ __forceinline__ void rotate_query(const LatentArgs& a, int row, int h, int i, int pos) {
    const LatentGeom& g = a.g;
    const int half = g.rot_dim >> 1;
    const float* q = a.proj + (size_t) row * a.proj_ld + (size_t) h * (g.dim + g.rot_dim) + g.dim;
    T* dst = (T*) a.qf + ((size_t) row * g.heads + h) * g.key_ld() + g.rank_pad();
    const float2 o = rotate(q[i], q[i + half], a.cos_t[(size_t) pos * half + i], a.sin_t[(size_t) pos * half + i]);
    skd::store_act(dst + i, o.x); skd::store_act(dst + i + half, o.y);
}

__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(skd::pack_bf16(v.x, v.y), skd::pack_bf16(v.z, v.w)); }

template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentArgs a) {
    __shared__ float sh[8];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const LatentGeom& g = a.g;
    const int row = blockIdx.x, half = g.rot_dim >> 1, hd = g.dim + g.rot_dim, pos = a.map.pos_of(row);
    const float* p = a.proj + (size_t) row * a.proj_ld;
    if (g.dim % 4 == 0 && hd % 4 == 0 && a.proj_ld % 4 == 0) {         // rows 16-byte aligned: four elements per thread
        const int q4 = g.dim >> 2;
        for (int i = threadIdx.x; i < g.heads * q4; i += 256) {
            const int h = i / q4, c = (i - h * q4) * 4;
            const float4 v = *reinterpret_cast<const float4*>(p + (size_t) h * hd + c);
            store4((T*) a.qn + ((size_t) row * g.heads + h) * g.dim_ld() + c, v);
        }
    } else
        for (int i = threadIdx.x; i < g.heads * g.dim; i += 256) {
            const int h = i / g.dim, c = i - h * g.dim;
            skd::store_act((T*) a.qn + ((size_t) row * g.heads + h) * g.dim_ld() + c, p[(size_t) h * hd + c]);
        }
    for (int i = threadIdx.x; i < g.heads * half; i += 256) { const int h = i / half; rotate_query<T>(a, row, h, i - h * half, pos); }
    prep_row<T>(a, row, sh);
}

// Eight weights of a bf16 row against eight fp32 values in shared memory.
__device__ __forceinline__ float dot8(uint4 w, const float* x) {
    return skd::bf16_lo(w.x) * x[0] + skd::bf16_hi(w.x) * x[1] + skd::bf16_lo(w.y) * x[2] + skd::bf16_hi(w.y) * x[3] +
           skd::bf16_lo(w.z) * x[4] + skd::bf16_hi(w.z) * x[5] + skd::bf16_lo(w.w) * x[6] + skd::bf16_hi(w.w) * x[7];
}

// y[o] = sum_k W[o][k] x[k] for output rows o0 <= o < o1 by a CTA of 256 threads: `lanes` (8, 16 or 32) threads per row. The
// first AHEAD loads of every thread are issued by the constructor, which needs no input from the preceding kernel.
constexpr int AHEAD = 8;
struct CtaMatvec {
    const bf16* w;
    int ld, lanes, l, r, per, o0, o1, nk, total;
    uint4 pre[AHEAD];
    __device__ __forceinline__ uint4 load(int i) const {
        const int o = o0 + (i / nk) * per + r, k = (i % nk) * lanes * 8 + l * 8;
        return i < total && o < o1 && k < ld ? skd::ld_ro(w + (size_t) o * ld + k) : make_uint4(0, 0, 0, 0);
    }
    __device__ __forceinline__ CtaMatvec(const bf16* w_, int ld_, int o0_, int o1_) : w(w_), ld(ld_), o0(o0_), o1(o1_) {
        lanes = ld >= 256 ? 32 : (ld >= 128 ? 16 : 8); per = 256 / lanes;
        l = threadIdx.x % lanes; r = threadIdx.x / lanes;
        nk = (ld + lanes * 8 - 1) / (lanes * 8);
        total = o1 > o0 ? (o1 - o0 + per - 1) / per * nk : 0;
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) pre[i] = load(i);
    }
    template <typename F>
    __device__ __forceinline__ void run(const float* x, F&& store) {
        float v = 0.0f;
        for (int i0 = 0; i0 < total; i0 += AHEAD) {
            if (i0 > 0) {
#pragma unroll
                for (int i = 0; i < AHEAD; ++i) pre[i] = load(i0 + i);
            }
#pragma unroll
            for (int i = 0; i < AHEAD; ++i) {
                if (i0 + i >= total) break;
                const int kb = (i0 + i) % nk, o = o0 + (i0 + i) / nk * per + r, k = kb * lanes * 8 + l * 8;
                if (k < ld) v += dot8(pre[i], x + k);
                if (kb == nk - 1) {
                    for (int m = lanes / 2; m > 0; m >>= 1) v += __shfl_xor_sync(~0u, v, m);
                    if (l == 0 && o < o1) store(o, v);
                    v = 0.0f;
                }
            }
        }
    }
};

// Few rows: grid (heads + 1, rows, parts). Head CTAs rotate their query and fold a part of W_uk into it; the last column
// prepares latent, key part and gates.
__global__ void __launch_bounds__(256) latent_prep_fold_kernel(const LatentArgs a) {
    extern __shared__ float sq[];
    __shared__ float sh[8];
    skd::pdl_launch_dependents();
    const LatentGeom& g = a.g;
    const int h = blockIdx.x, row = blockIdx.y;
    if (h == g.heads) {
        skd::pdl_wait();
        if (blockIdx.z == 0) prep_row<bf16>(a, row, sh);
        return;
    }
    const int ld = g.dim_ld(), per = (g.kv_rank + gridDim.z - 1) / gridDim.z, o0 = blockIdx.z * per;
    CtaMatvec mv(a.uk_t + (size_t) h * g.kv_rank * ld, ld, o0, min(g.kv_rank, o0 + per));
    skd::pdl_wait();
    const float* q = a.proj + (size_t) row * a.proj_ld + (size_t) h * (g.dim + g.rot_dim);
    for (int i = threadIdx.x; i < ld; i += 256) sq[i] = i < g.dim ? q[i] : 0.0f;
    if (blockIdx.z == 0) {
        const int pos = a.map.pos_of(row);
        for (int i = threadIdx.x; i < (g.rot_dim >> 1); i += 256) rotate_query<bf16>(a, row, h, i, pos);
    }
    __syncthreads();
    bf16* dst = (bf16*) a.qf + ((size_t) row * g.heads + h) * g.key_ld();
    mv.run(sq, [&](int o, float v) { dst[o] = __float2bfloat16_rn(v); });
}

// ---- attention over the cache ---------------------------------------------------------------------------------------
struct SplitArgs { int rows_per_block, heads_per_block, n_splits; };

__device__ __forceinline__ void cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(skd::smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(skd::smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(skd::smem_u32(p)) : "memory");
}

// MW warps over 16-row groups x NW warps over keys (scores, eight each) and over 16-column groups of the latent (mix, NT each).
// The scores and the mix are chains of dependent shared-memory loads and MMAs: with 64 rows, sixteen warps hide them better than
// eight that own twice the columns (304 -> 279 us for 1024 rows x 32 heads at a latent of 512).
template <int MW>
struct AttnShape {
    static constexpr int WARPS = MW == 4 ? 16 : 8, THREADS = WARPS * 32, NW = WARPS / MW, BK = NW * 8, ROWS = 16 * MW;
    static int smem(int key_ld, int stages) {
        return (ROWS + stages * BK) * (key_ld + 8) * 2 + ROWS * (BK + 8) * 2 + (2 * NW * ROWS + ROWS) * 4;
    }
};
constexpr int ATTN_MAX_SMEM = 225 * 1024;

template <int MW, int NT, int ST>
__global__ void __launch_bounds__(AttnShape<MW>::THREADS)
latent_attn_mma_kernel(const LatentArgs a, const SplitArgs sp) {
    typedef AttnShape<MW> S;
    constexpr int NW = S::NW, BK = S::BK, ROWS = S::ROWS;
    extern __shared__ __align__(16) uint8_t smem[];
    const LatentGeom& g = a.g;
    const int kld = g.key_ld(), sld = kld + 8, RP = g.rank_pad(), chunks = kld >> 3;
    bf16* sq = (bf16*) smem;                                  // [ROWS][sld]
    bf16* sk_ = sq + ROWS * sld;                              // [ST][BK][sld]
    bf16* spb = sk_ + ST * BK * sld;                          // [ROWS][BK + 8] weights of the current tile
    float* red_m = (float*) (spb + ROWS * (BK + 8));          // [NW][ROWS]
    float* red_l = red_m + NW * ROWS;
    int* qpos = (int*) (red_l + NW * ROWS);                   // position of each MMA row, -1: none
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, mw = warp % MW, nw = warp / MW;
    const int split = blockIdx.x, h0 = blockIdx.y * sp.heads_per_block, r0 = (gridDim.z - 1 - blockIdx.z) * sp.rows_per_block;   // the rows with the most keys first
    const int hb = sp.heads_per_block;
    skd::pdl_launch_dependents();
    skd::pdl_wait();

    const int r_last = min(r0 + sp.rows_per_block, a.rows) - 1;
    const int hi = a.map.pos_of(r_last), lo = max(0, a.map.pos_of(r0) - a.window + 1), seq = a.map.seq_of(r0);
    const int n_tiles = (hi - lo + BK) / BK, per = (n_tiles + sp.n_splits - 1) / sp.n_splits;
    const int t0 = split * per, t1 = min(n_tiles, t0 + per);
    const bf16* cache = (const bf16*) a.cache.rows + (size_t) seq * a.cache.cap * kld;

    auto fetch = [&](int t) {                                 // keys past hi repeat the newest one; their weights are masked
        if (t < t1) {
            bf16* dst = sk_ + (t % ST) * BK * sld;
            for (int j = warp; j < BK; j += S::WARPS) {
                const int p = min(lo + t * BK + j, hi);
                const bf16* src = cache + (size_t) (p % a.cache.cap) * kld;
                for (int c = lane; c < chunks; c += 32) cp16(dst + j * sld + c * 8, src + c * 8);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int i = 0; i < ST - 1; ++i) fetch(t0 + i);
    for (int m = warp; m < ROWS; m += S::WARPS) {             // query rows, zero where there is none
        const int r = r0 + m / hb, h = h0 + m % hb;
        const bool live = m < sp.rows_per_block * hb && r <= r_last && h < g.heads;
        if (lane == 0) qpos[m] = live ? a.map.pos_of(r) : -1;
        const uint4* src = (const uint4*) ((const bf16*) a.qf + ((size_t) (live ? r : 0) * g.heads + (live ? h : 0)) * kld);
        for (int c = lane; c < chunks; c += 32) *(uint4*) (sq + m * sld + c * 8) = live ? src[c] : make_uint4(0, 0, 0, 0);
    }

    float acc[NT][2][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[i][j][k] = 0.0f;
    float m_run[2] = {NEG_BIG, NEG_BIG}, l_run[2] = {0.0f, 0.0f};
    const int ra = mw * 16 + (lane >> 2), rb = ra + 8;        // MMA rows of this lane's accumulators
    const float sc = a.scale * LOG2E;
    const bf16* aq = sq + (mw * 16 + (lane & 15)) * sld + (lane >> 4) * 8;
    const bf16* ap = spb + (mw * 16 + (lane & 15)) * (BK + 8) + (lane >> 4) * 8;

    for (int t = t0; t < t1; ++t) {
        asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
        __syncthreads();                                      // tile t is staged; every warp is done with tile t - 1
        fetch(t + ST - 1);
        const bf16* kt = sk_ + (t % ST) * BK * sld;
        float s4[4] = {}, s1[4] = {}, s2[4] = {}, s3[4] = {};         // four independent accumulator chains
        {
            const bf16* bk = kt + (nw * 8 + (lane & 7)) * sld + (lane >> 3) * 8;
            int k = 0;
            for (; k + 64 <= kld; k += 64) {
                uint32_t fa[4], fb[4];
                ldsm4(fb, bk + k); ldsm4(fa, aq + k);
                skd::mma_bf16(s4, fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
                ldsm4(fa, aq + k + 16);
                skd::mma_bf16(s1, fa[0], fa[1], fa[2], fa[3], fb[2], fb[3]);
                ldsm4(fb, bk + k + 32); ldsm4(fa, aq + k + 32);
                skd::mma_bf16(s2, fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
                ldsm4(fa, aq + k + 48);
                skd::mma_bf16(s3, fa[0], fa[1], fa[2], fa[3], fb[2], fb[3]);
            }
            for (; k < kld; k += 16) {
                uint32_t fa[4], fb[2];
                ldsm4(fa, aq + k);
                asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(fb[0]), "=r"(fb[1])
                             : "r"(skd::smem_u32(kt + (nw * 8 + (lane & 7)) * sld + ((lane >> 3) & 1) * 8 + k)) : "memory");
                skd::mma_bf16(s4, fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) s4[j] += s1[j] + (s2[j] + s3[j]);
        }
        // scaled scores in powers of two, masked; row maxima over this warp's keys, then over the warps
        const int pa = qpos[ra], pb = qpos[rb];
        float mx[2] = {NEG_BIG, NEG_BIG};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int key = lo + t * BK + nw * 8 + 2 * (lane & 3) + (j & 1), p = j < 2 ? pa : pb;
            const float v = key <= p && p - key < a.window ? s4[j] * sc : -INFINITY;
            s4[j] = v;
            mx[j >> 1] = fmaxf(mx[j >> 1], v);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(~0u, mx[r], 1)); mx[r] = fmaxf(mx[r], __shfl_xor_sync(~0u, mx[r], 2));
        }
        if ((lane & 3) == 0) { red_m[nw * ROWS + ra] = mx[0]; red_m[nw * ROWS + rb] = mx[1]; }
        __syncthreads();
        float al[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float m = m_run[r];
#pragma unroll
            for (int w = 0; w < NW; ++w) m = fmaxf(m, red_m[w * ROWS + (r ? rb : ra)]);
            al[r] = exp2f(m_run[r] - m);
            m_run[r] = m; l_run[r] *= al[r];
        }
        {
            const float e0 = exp2f(s4[0] - m_run[0]), e1 = exp2f(s4[1] - m_run[0]), e2 = exp2f(s4[2] - m_run[1]), e3 = exp2f(s4[3] - m_run[1]);
            l_run[0] += e0 + e1; l_run[1] += e2 + e3;
            const int c = nw * 8 + 2 * (lane & 3);
            *(uint32_t*) (spb + ra * (BK + 8) + c) = skd::pack_bf16(e0, e1);
            *(uint32_t*) (spb + rb * (BK + 8) + c) = skd::pack_bf16(e2, e3);
        }
        __syncthreads();
        if (__any_sync(~0u, al[0] != 1.0f || al[1] != 1.0f))             // a running maximum moved
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) { acc[i][j][0] *= al[0]; acc[i][j][1] *= al[0]; acc[i][j][2] *= al[1]; acc[i][j][3] *= al[1]; }
#pragma unroll
        for (int k = 0; k < BK; k += 16) {
            uint32_t fp[4];
            ldsm4(fp, ap + k);
            const bf16* bv = kt + (k + (lane & 7) + ((lane >> 3) & 1) * 8) * sld + (lane >> 4) * 8;
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int c = (nw + NW * i) * 16;
                if (c < RP) {
                    uint32_t fb[4];
                    ldsm4_t(fb, bv + c);
                    skd::mma_bf16(acc[i][0], fp[0], fp[1], fp[2], fp[3], fb[0], fb[1]);
                    skd::mma_bf16(acc[i][1], fp[0], fp[1], fp[2], fp[3], fb[2], fb[3]);
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    // sums of the weights: within the quad, then over the warps that shared a row group
#pragma unroll
    for (int r = 0; r < 2; ++r) { l_run[r] += __shfl_xor_sync(~0u, l_run[r], 1); l_run[r] += __shfl_xor_sync(~0u, l_run[r], 2); }
    if ((lane & 3) == 0) { red_l[nw * ROWS + ra] = l_run[0]; red_l[nw * ROWS + rb] = l_run[1]; }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int m = r ? rb : ra;
        if (m >= sp.rows_per_block * hb || qpos[m] < 0) continue;
        float l = 0.0f;
#pragma unroll
        for (int w = 0; w < NW; ++w) l += red_l[w * ROWS + m];
        const size_t rh = (size_t) (r0 + m / hb) * g.heads + h0 + m % hb;
        if (a.part) {
            float* d = a.part + (rh * sp.n_splits + split) * (RP + 2);
            if (nw == 0 && (lane & 3) == 0) { d[RP] = m_run[r]; d[RP + 1] = l; }
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int c = (nw + NW * i) * 16;
                if (c < RP)
#pragma unroll
                    for (int j = 0; j < 2; ++j) *(float2*) (d + c + j * 8 + 2 * (lane & 3)) = make_float2(acc[i][j][2 * r], acc[i][j][2 * r + 1]);
            }
        } else {
            const float inv = 1.0f / l;
            bf16* d = (bf16*) a.mix + rh * g.rank_ld();
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int c = (nw + NW * i) * 16;
                if (c < RP)
#pragma unroll
                    for (int j = 0; j < 2; ++j) *(uint32_t*) (d + c + j * 8 + 2 * (lane & 3)) = skd::pack_bf16(acc[i][j][2 * r] * inv, acc[i][j][2 * r + 1] * inv);
            }
        }
    }
}

constexpr int ROWS_BK = 64;
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_rows_kernel(const LatentArgs a, int n_splits) {
    extern __shared__ float dyn[];
    __shared__ float ss[ROWS_BK];
    const LatentGeom& g = a.g;
    const int kld = g.key_ld(), RP = g.rank_pad(), split = blockIdx.x, h = blockIdx.y, row = blockIdx.z;
    float *sq = dyn, *so = dyn + kld;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int pos = a.map.pos_of(row), lo = max(0, pos - a.window + 1);
    const int n_tiles = (pos - lo + ROWS_BK) / ROWS_BK, per = (n_tiles + n_splits - 1) / n_splits;
    const T* cache = (const T*) a.cache.rows + (size_t) a.map.seq_of(row) * a.cache.cap * kld;
    const size_t rh = (size_t) row * g.heads + h;
    for (int i = threadIdx.x; i < kld; i += 128) sq[i] = skd::load_act((const T*) a.qf + rh * kld + i);
    for (int i = threadIdx.x; i < RP; i += 128) so[i] = 0.0f;
    __syncthreads();
    float m_run = NEG_BIG, l_run = 0.0f;
    for (int t = split * per; t < min(n_tiles, split * per + per); ++t) {
        const int k0 = lo + t * ROWS_BK, n = min(ROWS_BK, pos - k0 + 1);
        for (int j = threadIdx.x >> 5; j < n; j += 4) {
            const T* kr = cache + (size_t) ((k0 + j) % a.cache.cap) * kld;
            float v = 0.0f;
            for (int i = threadIdx.x & 31; i < kld; i += 32) v = fmaf(sq[i], skd::load_act(kr + i), v);
            v = skd::warp_sum(v);
            if ((threadIdx.x & 31) == 0) ss[j] = v * a.scale;
        }
        __syncthreads();
        float m = m_run;
        for (int j = 0; j < n; ++j) m = fmaxf(m, ss[j]);
        const float al = expf(m_run - m);
        float l = l_run * al;
        __syncthreads();
        if (threadIdx.x < n) ss[threadIdx.x] = expf(ss[threadIdx.x] - m);
        __syncthreads();
        for (int j = 0; j < n; ++j) l += ss[j];
        for (int c = threadIdx.x; c < RP; c += 128) {
            float o = so[c] * al;
            for (int j = 0; j < n; ++j) o = fmaf(ss[j], skd::load_act(cache + (size_t) ((k0 + j) % a.cache.cap) * kld + c), o);
            so[c] = o;
        }
        m_run = m; l_run = l;
        __syncthreads();
    }
    if (a.part) {
        float* d = a.part + (rh * n_splits + split) * (RP + 2);
        for (int c = threadIdx.x; c < RP; c += 128) d[c] = so[c];
        if (threadIdx.x == 0) { d[RP] = m_run * LOG2E; d[RP + 1] = l_run; }
    } else {
        for (int c = threadIdx.x; c < RP; c += 128) skd::store_act((T*) a.mix + rh * g.rank_ld() + c, so[c] / l_run);
    }
}

// ---- key splits -----------------------------------------------------------------------------------------------------
// The mixed latent of (row, head) from its split records by a CTA of 256 threads, handed to store(column, value). The factors
// of the splits are formed once; then groups of threads take every n-th split of four columns and meet in shared memory.
constexpr int MERGE_MAX_SPLITS = 256;
template <typename F>
__device__ __forceinline__ void merge_splits(const float* part, int n_splits, int RP, float* fac, float4* sums, F&& store) {
    const int rec = RP + 2;
    float m = NEG_BIG;
    for (int s = threadIdx.x & 31; s < n_splits; s += 32) if (part[(size_t) s * rec + RP + 1] > 0.0f) m = fmaxf(m, part[(size_t) s * rec + RP]);
    m = skd::warp_max(m);
    float l = 0.0f;
    for (int s = threadIdx.x & 31; s < n_splits; s += 32) {
        const float ls = part[(size_t) s * rec + RP + 1], f = ls > 0.0f ? exp2f(part[(size_t) s * rec + RP] - m) : 0.0f;
        l += ls * f;
        if (threadIdx.x < 32) fac[s] = f;
    }
    const float inv = 1.0f / skd::warp_sum(l);
    __syncthreads();
    const int q4 = RP / 4;                                  // column quads; RP is a multiple of 16
    for (int c0 = 0; c0 < q4; c0 += 256) {
        const int cols = min(256, q4 - c0), ways = 256 / cols, c = threadIdx.x % cols, w = threadIdx.x / cols;
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (w < ways) {
#pragma unroll 8
            for (int s = w; s < n_splits; s += ways) {
                const float f = fac[s];
                const float2* d = reinterpret_cast<const float2*>(part + (size_t) s * rec + 4 * (c0 + c));
                const float2 a = d[0], b = d[1];
                v.x = fmaf(a.x, f, v.x); v.y = fmaf(a.y, f, v.y); v.z = fmaf(b.x, f, v.z); v.w = fmaf(b.y, f, v.w);
            }
            sums[threadIdx.x] = v;
        }
        __syncthreads();
        if ((int) threadIdx.x < cols) {
            for (int k = 1; k < ways; ++k) { const float4 o = sums[k * cols + c]; v.x += o.x; v.y += o.y; v.z += o.z; v.w += o.w; }
            const int at = 4 * (c0 + c);
            store(at, v.x * inv); store(at + 1, v.y * inv); store(at + 2, v.z * inv); store(at + 3, v.w * inv);
        }
        __syncthreads();
    }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_merge_kernel(const LatentArgs a, int n_splits) {
    __shared__ float fac[MERGE_MAX_SPLITS];
    __shared__ float4 sums[256];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const LatentGeom& g = a.g;
    const size_t rh = (size_t) blockIdx.y * g.heads + blockIdx.x;
    T* d = (T*) a.mix + rh * g.rank_ld();
    merge_splits(a.part + rh * n_splits * (g.rank_pad() + 2), n_splits, g.rank_pad(), fac, sums, [&](int c, float v) { skd::store_act(d + c, v); });
}

// Few rows: grid (heads, rows, parts): merge, then a part of W_uv's rows, gated.
__global__ void __launch_bounds__(256) latent_merge_value_kernel(const LatentArgs a, int n_splits) {
    extern __shared__ float so[];
    __shared__ float fac[MERGE_MAX_SPLITS];
    __shared__ float4 sums[256];
    skd::pdl_launch_dependents();
    const LatentGeom& g = a.g;
    const int h = blockIdx.x, row = blockIdx.y, ld = g.rank_ld(), per = (g.vdim + gridDim.z - 1) / gridDim.z, o0 = blockIdx.z * per;
    CtaMatvec mv(a.uv + (size_t) h * g.vdim * ld, ld, o0, min(g.vdim, o0 + per));
    skd::pdl_wait();
    const size_t rh = (size_t) row * g.heads + h;
    for (int i = g.rank_pad() + threadIdx.x; i < ld; i += 256) so[i] = 0.0f;
    merge_splits(a.part + rh * n_splits * (g.rank_pad() + 2), n_splits, g.rank_pad(), fac, sums, [&](int c, float v) { so[c] = v; });
    const float gate = a.gates[rh];
    bf16* dst = (bf16*) a.out + (size_t) row * g.out_ld() + (size_t) h * g.vdim;
    mv.run(so, [&](int o, float v) { dst[o] = __float2bfloat16_rn(v * gate); });
}

__global__ void transpose_heads_kernel(const bf16* __restrict__ src, bf16* __restrict__ dst, int dim, int kv_rank, int src_ld, int dst_ld) {
    const int h = blockIdx.y;
    for (int64_t i = blockIdx.x * (int64_t) blockDim.x + threadIdx.x; i < (int64_t) kv_rank * dst_ld; i += (int64_t) gridDim.x * blockDim.x) {
        const int r = (int) (i / dst_ld), d = (int) (i % dst_ld);
        dst[(size_t) h * kv_rank * dst_ld + i] = d < dim ? src[((size_t) h * dim + d) * src_ld + r] : __float2bfloat16_rn(0.0f);
    }
}

template <int MW, int NT, int ST>
int32_t run_mma_st(const LatentArgs& a, const SplitArgs& sp, dim3 grid, cudaStream_t s) {
    const int bytes = AttnShape<MW>::smem(a.g.key_ld(), ST);
    SK_TRY(ensure_dynamic_smem((const void*) latent_attn_mma_kernel<MW, NT, ST>, bytes));
    SK_CUDA(launch_pdl(latent_attn_mma_kernel<MW, NT, ST>, grid, dim3(AttnShape<MW>::THREADS), bytes, s, a, sp));
    return SKAINET_CUDA_OK;
}
template <int MW, int NT>
int32_t run_mma(const LatentArgs& a, const SplitArgs& sp, dim3 grid, cudaStream_t s) {
    return AttnShape<MW>::smem(a.g.key_ld(), 3) <= ATTN_MAX_SMEM ? run_mma_st<MW, NT, 3>(a, sp, grid, s) : run_mma_st<MW, NT, 2>(a, sp, grid, s);
}

// 16-column groups of the latent per warp; 0: the tile kernel does not take this geometry.
template <int MW>
int mma_groups(const LatentGeom& g) {
    typedef AttnShape<MW> S;
    const int nt = (g.rank_pad() / 16 + S::NW - 1) / S::NW;
    return nt <= 8 && S::smem(g.key_ld(), 2) <= ATTN_MAX_SMEM ? nt : 0;
}
template <int MW>
int32_t launch_mma(const LatentArgs& a, const SplitArgs& sp, dim3 grid, cudaStream_t s) {
    const int nt = mma_groups<MW>(a.g);
    return nt <= 1 ? run_mma<MW, 1>(a, sp, grid, s) : nt <= 2 ? run_mma<MW, 2>(a, sp, grid, s) : nt <= 4 ? run_mma<MW, 4>(a, sp, grid, s) : run_mma<MW, 8>(a, sp, grid, s);
}

}  // namespace

int32_t launch_latent_attention(const LatentArgs& args, cudaStream_t s) {
    LatentArgs a = args;
    const LatentGeom& g = a.g;
    const bool few = !a.f32_act && a.rows <= LATENT_FUSED_ROWS && g.dim_ld() <= 4096 && g.rank_ld() <= 4096;
    SK_REQUIRE(g.heads <= 65535 && a.rows <= 65535, "latent attention: %d rows x %d heads", a.rows, g.heads);
    if (few) {
        const int parts = std::max(1, std::min(4, sm_count() / (g.heads * a.rows)));
        SK_CUDA(launch_pdl(latent_prep_fold_kernel, dim3(g.heads + 1, a.rows, parts), dim3(256), g.dim_ld() * sizeof(float), s, a));
    } else {
        if (a.f32_act) SK_CUDA(launch_pdl(latent_prep_kernel<float>, dim3(a.rows), dim3(256), 0, s, a));
        else SK_CUDA(launch_pdl(latent_prep_kernel<bf16>, dim3(a.rows), dim3(256), 0, s, a));
        LinearArgs l;
        l.w = a.uk_t; l.w_rows = g.kv_rank; l.ldw = g.dim_ld(); l.groups = g.heads; l.x = a.qn; l.ldx = g.heads * g.dim_ld(); l.x_group_stride = g.dim_ld();
        l.x_rows_alloc = a.rows_alloc; l.rows = a.rows; l.y = a.qf; l.ldy = g.heads * g.key_ld(); l.y_group_stride = g.key_ld(); l.f32_act = a.f32_act; l.out = LIN_OUT_ACT;
        SK_TRY(launch_linear_bf16(l, s));
    }
    // key splits: enough CTAs for the machine, no more than there are key tiles, records within the scratch
    const bool small = a.map.seq < 0 || a.rows <= LATENT_FUSED_ROWS;      // rows of different sequences share no keys
    const int mw = small ? 1 : 4;
    const bool mma = !a.f32_act && (mw == 4 ? mma_groups<4>(g) : mma_groups<1>(g)) > 0;
    SplitArgs sp = {1, 1, 1};
    dim3 grid;
    int bk = ROWS_BK;
    if (mma) {
        const int m_rows = 16 * mw, groups = (g.heads + m_rows - 1) / m_rows;
        sp.heads_per_block = (g.heads + groups - 1) / groups;
        sp.rows_per_block = small ? 1 : m_rows / sp.heads_per_block;
        grid = dim3(1, groups, (a.rows + sp.rows_per_block - 1) / sp.rows_per_block);
        bk = mw == 4 ? AttnShape<4>::BK : AttnShape<1>::BK;
    } else grid = dim3(1, g.heads, a.rows);
    const int64_t blocks = (int64_t) grid.y * grid.z, records = (int64_t) a.rows * g.heads;
    const int keys = std::min(a.kv_bound, a.window + sp.rows_per_block - 1), tiles = (keys + bk - 1) / bk;
    sp.n_splits = (int) std::max<int64_t>(1, std::min<int64_t>({(int64_t) sm_count() / std::max<int64_t>(1, blocks), (int64_t) (tiles + 1) / 2, MERGE_MAX_SPLITS, LATENT_PART_RECORDS / std::max<int64_t>(1, records)}));
    grid.x = sp.n_splits;
    if (!few && sp.n_splits == 1) a.part = nullptr;
    if (mma) SK_TRY(mw == 4 ? launch_mma<4>(a, sp, grid, s) : launch_mma<1>(a, sp, grid, s));
    else {
        const int bytes = (g.key_ld() + g.rank_pad()) * (int) sizeof(float);
        if (a.f32_act) {
            SK_TRY(ensure_dynamic_smem((const void*) latent_attn_rows_kernel<float>, bytes));
            SK_CUDA(launch_pdl(latent_attn_rows_kernel<float>, grid, dim3(128), bytes, s, a, sp.n_splits));
        } else {
            SK_TRY(ensure_dynamic_smem((const void*) latent_attn_rows_kernel<bf16>, bytes));
            SK_CUDA(launch_pdl(latent_attn_rows_kernel<bf16>, grid, dim3(128), bytes, s, a, sp.n_splits));
        }
    }
    if (few) {
        const int parts = std::max(1, std::min(4, sm_count() / (g.heads * a.rows)));
        SK_CUDA(launch_pdl(latent_merge_value_kernel, dim3(g.heads, a.rows, parts), dim3(256), g.rank_ld() * sizeof(float), s, a, sp.n_splits));
        return SKAINET_CUDA_OK;
    }
    if (a.part) {
        if (a.f32_act) SK_CUDA(launch_pdl(latent_merge_kernel<float>, dim3(g.heads, a.rows), dim3(256), 0, s, a, sp.n_splits));
        else SK_CUDA(launch_pdl(latent_merge_kernel<bf16>, dim3(g.heads, a.rows), dim3(256), 0, s, a, sp.n_splits));
    }
    LinearArgs l;
    l.w = a.uv; l.w_rows = g.vdim; l.ldw = g.rank_ld(); l.groups = g.heads; l.x = a.mix; l.ldx = g.heads * g.rank_ld(); l.x_group_stride = g.rank_ld();
    l.x_rows_alloc = a.rows_alloc; l.rows = a.rows; l.y = a.out; l.ldy = g.out_ld(); l.y_group_stride = g.vdim; l.scale = a.gates; l.scale_ld = g.heads;
    l.f32_act = a.f32_act; l.out = LIN_OUT_ACT;
    return launch_linear_bf16(l, s);
}

int32_t launch_transpose_heads(const bf16* src, bf16* dst, int heads, int dim, int kv_rank, cudaStream_t s) {
    const int n = kv_rank * bf16_ld(dim);
    transpose_heads_kernel<<<dim3(std::min((n + 255) / 256, 1024), heads), 256, 0, s>>>(src, dst, dim, kv_rank, bf16_ld(kv_rank), bf16_ld(dim));
    SK_CUDA(cudaGetLastError());
    return SKAINET_CUDA_OK;
}

}  // namespace sk
