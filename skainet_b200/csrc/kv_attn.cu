// Ring attention with a chunk mask and a sink (contract: kv_attn.cuh).
//
//   kv_prep_kernel       biases, unit-rms queries and keys, ring append.
//   kv_attn_rows_kernel  fp32 FMA, one CTA per (row, head), any size: the 32-bit mode, and bf16 models whose heads are too large
//                        for the tile kernel.
#include "kv_attn.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr float NEG_BIG = -1e30f;            // maximum over no key: finite, so differences stay defined

// First position that position i sees.
__device__ __forceinline__ int first_key(const KvAttnArgs& a, int i) { return a.chunk > 0 ? i / a.chunk * a.chunk : 0; }

// One warp prepares one vector of a row: u < heads a query, u < heads + kv_heads a key, else a value.
template <typename T>
__device__ void prep_vector(const KvAttnArgs& a, int row, int u, int lane) {
    const KvGeom& g = a.g;
    const bool is_q = u < g.heads, is_v = u >= g.heads + g.kv_heads;
    const int n = is_v ? g.vdim : g.dim, off = is_v ? (g.heads + g.kv_heads) * g.dim + (u - g.heads - g.kv_heads) * g.vdim : u * g.dim;
    const float *p = a.proj + (size_t) row * a.proj_ld + off, *b = a.bias ? a.bias + off : nullptr;
    float r = 1.0f;
    if (!is_v) {
        float ss = 0.0f;
        for (int i = lane; i < n; i += 32) { const float v = p[i] + (b ? b[i] : 0.0f); ss = fmaf(v, v, ss); }
        r = 1.0f / sqrtf(skd::warp_sum(ss) / (float) n + a.eps);
    }
    T* dst;
    if (is_q) dst = (T*) a.q + ((size_t) row * g.heads + u) * g.kld();
    else {
        const int slot = a.map.pos_of(row) % a.cache.cap, kh = u - g.heads - (is_v ? g.kv_heads : 0);
        const size_t at = ((size_t) a.map.seq_of(row) * g.kv_heads + kh) * a.cache.cap + slot;
        dst = is_v ? (T*) a.cache.v + at * g.vcld() : (T*) a.cache.k + at * g.kld();
    }
    for (int i = lane; i < n; i += 32) skd::store_act(dst + i, (p[i] + (b ? b[i] : 0.0f)) * r);
}

template <typename T>
__global__ void __launch_bounds__(256) kv_prep_kernel(const KvAttnArgs a) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int units = a.g.heads + 2 * a.g.kv_heads, u = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (u < units) prep_vector<T>(a, blockIdx.x, u, threadIdx.x & 31);
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

size_t kv_part_floats(const KvGeom& g) { (void) g; return 0; }

int32_t launch_kv_attention(const KvAttnArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return SKAINET_CUDA_OK;
    if (a.f32_act) { SK_TRY(run_prep<float>(a, s)); return run_rows<float>(a, s); }
    SK_TRY(run_prep<bf16>(a, s));
    return run_rows<bf16>(a, s);
}

}  // namespace sk
