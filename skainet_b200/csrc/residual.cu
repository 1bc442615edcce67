// Residual, norms and depth average (contract: residual.cuh). All HBM- or latency-bound: one pass over the row for
// the sum of squares, one that writes. With few rows a cluster of up to eight CTAs shares a row (the sum of squares through
// distributed shared memory), because a late layer's average reads every earlier state of the row.
#include "residual.cuh"
#include "tma.cuh"

#include <cooperative_groups.h>

#include <algorithm>

namespace sk {

namespace {

constexpr int RT = 256;

__device__ __forceinline__ float block_sum(float v, float* sh) {
    v = skd::warp_sum(v);
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.0f;
    for (int i = 0; i < RT / 32; ++i) t += sh[i];
    __syncthreads();
    return t;
}

// V = 4: cols and every stride are multiples of four; V = 1: any.
template <int V> struct Vec { float v[V]; };
template <int V> __device__ __forceinline__ Vec<V> ld(const float* p) {
    Vec<V> r;
    if (V == 4) { const float4 q = *reinterpret_cast<const float4*>(p); r.v[0] = q.x; r.v[V > 1 ? 1 : 0] = q.y; r.v[V > 2 ? 2 : 0] = q.z; r.v[V > 3 ? 3 : 0] = q.w; }
    else r.v[0] = *p;
    return r;
}
template <int V> __device__ __forceinline__ void st(float* p, const Vec<V>& r) {
    if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[V > 1 ? 1 : 0], r.v[V > 2 ? 2 : 0], r.v[V > 3 ? 3 : 0]);
    else *p = r.v[0];
}
template <int V> __device__ __forceinline__ void st_act(float* p, const Vec<V>& r) { st<V>(p, r); }
template <int V> __device__ __forceinline__ void st_act(bf16* p, const Vec<V>& r) {
    if (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(skd::pack_bf16(r.v[0], r.v[V > 1 ? 1 : 0]), skd::pack_bf16(r.v[V > 2 ? 2 : 0], r.v[V > 3 ? 3 : 0]));
    else *p = __float2bfloat16_rn(r.v[0]);
}

template <typename T, int V>
__global__ void __launch_bounds__(RT) sublayer_kernel(const SublayerArgs a) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) float sy[];                 // this CTA's part of the sublayer output
    __shared__ float sh[RT / 32], part;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    cg::cluster_group cl = cg::this_cluster();
    const int cs = (int) cl.num_blocks(), rank = (int) cl.block_rank(), row = blockIdx.x / cs;
    const int per = ((a.cols + cs - 1) / cs + 3) / 4 * 4, c0 = min(a.cols, rank * per), c1 = min(a.cols, c0 + per);
    float ss = 0.0f;
    for (int c = c0 + (int) threadIdx.x * V; c < c1; c += RT * V) {
        Vec<V> v;
        if (a.slot_pos) {
            v = ld<V>(a.y + (size_t) a.slot_pos[(size_t) row * a.top] * a.cols + c);
            for (int k = 1; k < a.top; ++k) {
                const Vec<V> u = ld<V>(a.y + (size_t) a.slot_pos[(size_t) row * a.top + k] * a.cols + c);
#pragma unroll
                for (int i = 0; i < V; ++i) v.v[i] += u.v[i];
            }
        } else v = ld<V>(a.y + (size_t) row * a.cols + c);
#pragma unroll
        for (int i = 0; i < V; ++i) ss += v.v[i] * v.v[i];
        st<V>(sy + c - c0, v);
    }
    ss = block_sum(ss, sh);
    if (cs > 1) {
        if (threadIdx.x == 0) part = ss;
        cl.sync();
        ss = 0.0f;
        for (int i = 0; i < cs; ++i) ss += *cl.map_shared_rank(&part, i);
    }
    const float r = 1.0f / sqrtf(ss / (float) a.cols + a.eps) * a.gain;
    const size_t at = (size_t) row * a.cols;
    for (int c = c0 + (int) threadIdx.x * V; c < c1; c += RT * V) {
        Vec<V> v = ld<V>(a.base + at + c);
        const Vec<V> y = ld<V>(sy + c - c0);
#pragma unroll
        for (int i = 0; i < V; ++i) v.v[i] += y.v[i] * r;
        st<V>(a.state + at + c, v);
        if (a.n_states > 0) {
            Vec<V> x;
            const float cl_ = a.coef[a.n_states - 1];
#pragma unroll
            for (int i = 0; i < V; ++i) x.v[i] = cl_ * v.v[i];
#pragma unroll 8
            for (int j = 0; j < a.n_states - 1; ++j) {
                const Vec<V> s = ld<V>(a.states + (size_t) j * a.state_stride + at + c);
                const float f = a.coef[j];
#pragma unroll
                for (int i = 0; i < V; ++i) x.v[i] = fmaf(f, s.v[i], x.v[i]);
            }
            st<V>(a.x + at + c, x);
            v = x;
        }
        st_act<V>((T*) a.act + (size_t) row * a.act_ld + c, v);
    }
    if (cs > 1) cl.sync();                                      // no CTA leaves while its partial sum may still be read
}

// Sum of v over the CTA, then over the cluster's CTAs through distributed shared memory. `part` is written once per call site.
__device__ __forceinline__ float cluster_sum(float v, float* sh, float* part, cooperative_groups::cluster_group& cl, int cs) {
    v = block_sum(v, sh);
    if (cs > 1) {
        if (threadIdx.x == 0) *part = v;
        cl.sync();
        v = 0.0f;
        for (int i = 0; i < cs; ++i) v += *cl.map_shared_rank(part, i);
    }
    return v;
}

// Columns of one row that a CTA of the cluster owns.
struct Span { int c0, c1; };
__device__ __forceinline__ Span cluster_span(int cols, int cs, int rank) {
    const int per = ((cols + cs - 1) / cs + 3) / 4 * 4, c0 = min(cols, rank * per);
    return {c0, min(cols, c0 + per)};
}

// The stream's row stays in shared memory between the residual sum and the next norm.
template <typename T, int V>
__global__ void __launch_bounds__(RT) sandwich_kernel(const SandwichArgs a) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) float sx[];
    __shared__ float sh[RT / 32], part[2];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    cg::cluster_group cl = cg::this_cluster();
    const int cs = (int) cl.num_blocks(), rank = (int) cl.block_rank(), row = blockIdx.x / cs;
    const Span sp = cluster_span(a.cols, cs, rank);
    const size_t at = (size_t) row * a.cols;
    float ss = 0.0f;
    for (int c = sp.c0 + (int) threadIdx.x * V; c < sp.c1; c += RT * V) {
        const Vec<V> y = ld<V>(a.y + at + c);
#pragma unroll
        for (int i = 0; i < V; ++i) ss += y.v[i] * y.v[i];
        st<V>(sx + c - sp.c0, y);
    }
    const float r = 1.0f / sqrtf(cluster_sum(ss, sh, part, cl, cs) / (float) a.cols + a.eps);
    ss = 0.0f;
    for (int c = sp.c0 + (int) threadIdx.x * V; c < sp.c1; c += RT * V) {
        Vec<V> x = ld<V>(a.x + at + c);
        const Vec<V> y = ld<V>(sx + c - sp.c0), g = ld<V>(a.post + c);
#pragma unroll
        for (int i = 0; i < V; ++i) x.v[i] += y.v[i] * r * g.v[i];
        if (a.add) {
            const Vec<V> e = ld<V>(a.add + at + c);
#pragma unroll
            for (int i = 0; i < V; ++i) x.v[i] += e.v[i];
        }
        st<V>(a.x + at + c, x);
        st<V>(sx + c - sp.c0, x);
#pragma unroll
        for (int i = 0; i < V; ++i) ss += x.v[i] * x.v[i];
    }
    if (a.pre) {
        const float q = 1.0f / sqrtf(cluster_sum(ss, sh, part + 1, cl, cs) / (float) a.cols + a.eps);
        for (int c = sp.c0 + (int) threadIdx.x * V; c < sp.c1; c += RT * V) {
            Vec<V> x = ld<V>(sx + c - sp.c0);
            const Vec<V> g = ld<V>(a.pre + c);
#pragma unroll
            for (int i = 0; i < V; ++i) x.v[i] = x.v[i] * q * g.v[i];
            st_act<V>((T*) a.act + (size_t) row * a.act_ld + c, x);
        }
    }
    if (cs > 1) cl.sync();                                      // no CTA leaves while its partial sums may still be read
}

// The angle is formed and reduced to one turn in double, so far positions lose nothing to its size.
__device__ __forceinline__ float2 sin_cos_turn(double angle) {
    angle -= rint(angle * 0.15915494309189535) * 6.283185307179586;
    float2 r;
    sincosf((float) angle, &r.x, &r.y);
    return r;
}
template <typename T>
__global__ void __launch_bounds__(RT) embed_pos_kernel(const EmbedPosArgs a) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) float sx[];
    __shared__ float sh[RT / 32], part;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    cg::cluster_group cl = cg::this_cluster();
    const int cs = (int) cl.num_blocks(), rank = (int) cl.block_rank(), row = blockIdx.x / cs;
    const Span sp = cluster_span(a.cols, cs, rank);                     // begins at an even column
    const int id = min(max(a.ids[row], 0), a.vocab - 1);
    const double pos = (double) a.map.pos_of(row);
    const size_t at = (size_t) row * a.cols;
    float ss = 0.0f;
    for (int c = sp.c0 + 2 * (int) threadIdx.x; c < sp.c1; c += 2 * RT) {
        const float2 sc = sin_cos_turn(pos * a.freq[c >> 1]);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            if (c + i >= sp.c1) break;
            const float v = __bfloat162float(a.table[(size_t) id * a.ld + c + i]) * a.scale + (i ? sc.y : sc.x);
            a.x[at + c + i] = v;
            if (a.x0) a.x0[at + c + i] = v;
            sx[c + i - sp.c0] = v;
            ss += v * v;
        }
    }
    const float q = 1.0f / sqrtf(cluster_sum(ss, sh, &part, cl, cs) / (float) a.cols + a.eps);
    for (int c = sp.c0 + (int) threadIdx.x; c < sp.c1; c += RT) skd::store_act((T*) a.act + (size_t) row * a.act_ld + c, sx[c - sp.c0] * q * a.pre[c]);
    if (cs > 1) cl.sync();
}

// A part of up to 512 columns per warp, its values in registers.
constexpr int GN_COLS = 512;
template <typename T, int V>
__global__ void __launch_bounds__(RT) gated_norm_warp_kernel(const GatedNormArgs a) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int parts = a.cols / a.part, lane = threadIdx.x & 31;
    const int64_t unit = (int64_t) blockIdx.x * (RT / 32) + (threadIdx.x >> 5);
    if (unit >= (int64_t) a.rows * parts) return;
    const int row = (int) (unit / parts), c0 = (int) (unit % parts) * a.part;
    const float *o = a.o + (size_t) row * a.cols + c0, *z = a.z + (size_t) row * a.z_ld + c0, *gain = a.gate_first ? a.gain + c0 : a.gain;
    Vec<V> v[GN_COLS / 32 / V];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < GN_COLS / 32 / V; ++k) {
        const int c = (k * 32 + lane) * V;
        if (c >= a.part) break;
        v[k] = ld<V>(o + c);
        const Vec<V> g = ld<V>(z + c);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            const float y = v[k].v[i] * skd::silu(g.v[i]);
            const float n = a.gate_first ? y : v[k].v[i];
            ss = fmaf(n, n, ss);
            v[k].v[i] = y;
        }
    }
    const float r = 1.0f / sqrtf(skd::warp_sum(ss) / (float) a.part + a.eps);
#pragma unroll
    for (int k = 0; k < GN_COLS / 32 / V; ++k) {
        const int c = (k * 32 + lane) * V;
        if (c >= a.part) break;
        const Vec<V> g = ld<V>(gain + c);
#pragma unroll
        for (int i = 0; i < V; ++i) v[k].v[i] *= r * g.v[i];
        st_act<V>((T*) a.act + (size_t) row * a.act_ld + c0 + c, v[k]);
    }
}
// A wider part per cluster.
template <typename T, int V>
__global__ void __launch_bounds__(RT) gated_norm_kernel(const GatedNormArgs a) {
    namespace cg = cooperative_groups;
    extern __shared__ __align__(16) float sx[];
    __shared__ float sh[RT / 32], part;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    cg::cluster_group cl = cg::this_cluster();
    const int cs = (int) cl.num_blocks(), rank = (int) cl.block_rank(), unit = blockIdx.x / cs, parts = a.cols / a.part, row = unit / parts, c0 = unit % parts * a.part;
    const Span sp = cluster_span(a.part, cs, rank);
    const float *o = a.o + (size_t) row * a.cols + c0, *z = a.z + (size_t) row * a.z_ld + c0, *gain = a.gate_first ? a.gain + c0 : a.gain;
    float ss = 0.0f;
#pragma unroll 4
    for (int c = sp.c0 + (int) threadIdx.x * V; c < sp.c1; c += RT * V) {
        Vec<V> v = ld<V>(o + c);
        const Vec<V> g = ld<V>(z + c);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            const float y = v.v[i] * skd::silu(g.v[i]);
            const float n = a.gate_first ? y : v.v[i];
            ss = fmaf(n, n, ss);
            v.v[i] = y;
        }
        st<V>(sx + c - sp.c0, v);
    }
    const float r = 1.0f / sqrtf(cluster_sum(ss, sh, &part, cl, cs) / (float) a.part + a.eps);
    for (int c = sp.c0 + (int) threadIdx.x * V; c < sp.c1; c += RT * V) {
        Vec<V> v = ld<V>(sx + c - sp.c0);
        const Vec<V> g = ld<V>(gain + c);
#pragma unroll
        for (int i = 0; i < V; ++i) v.v[i] *= r * g.v[i];
        st_act<V>((T*) a.act + (size_t) row * a.act_ld + c0 + c, v);
    }
    if (cs > 1) cl.sync();
}

template <typename T>
__global__ void __launch_bounds__(RT) embed_rows_kernel(const bf16* __restrict__ table, int ld_, const int32_t* __restrict__ ids, int cols, int vocab,
                                                        float* __restrict__ x, float* __restrict__ state0, T* __restrict__ act, int act_ld) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int row = blockIdx.x, id = min(max(ids[row], 0), vocab - 1);
    for (int c = threadIdx.x; c < cols; c += RT) {
        const float v = __bfloat162float(table[(size_t) id * ld_ + c]);
        x[(size_t) row * cols + c] = v; state0[(size_t) row * cols + c] = v;
        skd::store_act(act + (size_t) row * act_ld + c, v);
    }
}

template <typename T>
__global__ void __launch_bounds__(RT) row_norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ index, int cols, const float* __restrict__ gains, float gain, float eps,
                                                         T* __restrict__ act, int act_ld) {
    __shared__ float sh[RT / 32];
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const float* p = x + (size_t) (index ? index[blockIdx.x] : (int) blockIdx.x) * cols;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < cols; c += RT) ss += p[c] * p[c];
    ss = block_sum(ss, sh);
    const float r = 1.0f / sqrtf(ss / (float) cols + eps) * gain;
    for (int c = threadIdx.x; c < cols; c += RT) skd::store_act(act + (size_t) blockIdx.x * act_ld + c, gains ? p[c] * r * gains[c] : p[c] * r);
}

// One cluster per row (of `cols` columns, `rows` of them); a CTA keeps its columns of the row in dynamic shared memory.
template <typename A>
int32_t run_row_clusters(void (*kernel)(const A), const A& a, int rows, int cols, cudaStream_t s) {
    int cs = 1;                                                 // CTAs per row: while the machine has room and a CTA keeps 256 columns
    while (cs < 8 && rows * cs * 2 <= sm_count() && cols / (cs * 2) >= 256) cs *= 2;
    const int per = ((cols + cs - 1) / cs + 3) / 4 * 4;
    SK_TRY(ensure_dynamic_smem((const void*) kernel, per * (int) sizeof(float)));
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(rows * cs); cfg.blockDim = dim3(RT); cfg.dynamicSmemBytes = per * sizeof(float); cfg.stream = s;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization; at[0].val.programmaticStreamSerializationAllowed = 1;
    at[1].id = cudaLaunchAttributeClusterDimension; at[1].val.clusterDim.x = cs; at[1].val.clusterDim.y = 1; at[1].val.clusterDim.z = 1;
    cfg.attrs = at; cfg.numAttrs = 2;
    SK_CUDA(cudaLaunchKernelEx(&cfg, kernel, a));
    return SKAINET_CUDA_OK;
}

template <typename T>
int32_t run_gated_norm(const GatedNormArgs& a, cudaStream_t s) {
    const int64_t units = (int64_t) a.rows * (a.cols / a.part);
    SK_REQUIRE(units < (1 << 28), "gated_norm: too many parts");
    const bool vec = a.part % 4 == 0 && a.z_ld % 4 == 0 && ((uintptr_t) a.z & 15) == 0;
    if (a.part > GN_COLS) return run_row_clusters(vec ? gated_norm_kernel<T, 4> : gated_norm_kernel<T, 1>, a, (int) units, a.part, s);
    SK_CUDA(launch_pdl(vec ? gated_norm_warp_kernel<T, 4> : gated_norm_warp_kernel<T, 1>, dim3((unsigned) ((units + RT / 32 - 1) / (RT / 32))), dim3(RT), 0, s, a));
    return SKAINET_CUDA_OK;
}

}  // namespace

int32_t launch_sublayer(const SublayerArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return SKAINET_CUDA_OK;
    const bool vec = a.cols % 4 == 0 && a.act_ld % 4 == 0 && a.state_stride % 4 == 0;
    if (a.f32_act) return run_row_clusters(vec ? sublayer_kernel<float, 4> : sublayer_kernel<float, 1>, a, a.rows, a.cols, s);
    return run_row_clusters(vec ? sublayer_kernel<bf16, 4> : sublayer_kernel<bf16, 1>, a, a.rows, a.cols, s);
}

int32_t launch_sandwich(const SandwichArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return SKAINET_CUDA_OK;
    const bool vec = a.cols % 4 == 0 && a.act_ld % 4 == 0;
    if (a.f32_act) return run_row_clusters(vec ? sandwich_kernel<float, 4> : sandwich_kernel<float, 1>, a, a.rows, a.cols, s);
    return run_row_clusters(vec ? sandwich_kernel<bf16, 4> : sandwich_kernel<bf16, 1>, a, a.rows, a.cols, s);
}

int32_t launch_embed_pos(const EmbedPosArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return SKAINET_CUDA_OK;
    return a.f32_act ? run_row_clusters(embed_pos_kernel<float>, a, a.rows, a.cols, s) : run_row_clusters(embed_pos_kernel<bf16>, a, a.rows, a.cols, s);
}

int32_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return SKAINET_CUDA_OK;
    return a.f32_act ? run_gated_norm<float>(a, s) : run_gated_norm<bf16>(a, s);
}

int32_t launch_embed_rows(const bf16* table, int ld_, const int32_t* ids, int rows, int cols, int vocab, float* x, float* state0, void* act, int act_ld,
                          bool f32_act, cudaStream_t s) {
    if (rows <= 0) return SKAINET_CUDA_OK;
    if (f32_act) SK_CUDA(launch_pdl(embed_rows_kernel<float>, dim3(rows), dim3(RT), 0, s, table, ld_, ids, cols, vocab, x, state0, (float*) act, act_ld));
    else SK_CUDA(launch_pdl(embed_rows_kernel<bf16>, dim3(rows), dim3(RT), 0, s, table, ld_, ids, cols, vocab, x, state0, (bf16*) act, act_ld));
    return SKAINET_CUDA_OK;
}

int32_t launch_row_norm(const float* x, const int32_t* index, int rows, int cols, const float* gain, float eps, void* act, int act_ld, bool f32_act, cudaStream_t s) {
    if (rows <= 0) return SKAINET_CUDA_OK;
    if (f32_act) SK_CUDA(launch_pdl(row_norm_kernel<float>, dim3(rows), dim3(RT), 0, s, x, index, cols, gain, 1.0f, eps, (float*) act, act_ld));
    else SK_CUDA(launch_pdl(row_norm_kernel<bf16>, dim3(rows), dim3(RT), 0, s, x, index, cols, gain, 1.0f, eps, (bf16*) act, act_ld));
    return SKAINET_CUDA_OK;
}

int32_t launch_scalar_norm(const float* x, const int32_t* index, int rows, int cols, float gain, float eps, void* act, int act_ld, bool f32_act, cudaStream_t s) {
    if (rows <= 0) return SKAINET_CUDA_OK;
    if (f32_act) SK_CUDA(launch_pdl(row_norm_kernel<float>, dim3(rows), dim3(RT), 0, s, x, index, cols, (const float*) nullptr, gain, eps, (float*) act, act_ld));
    else SK_CUDA(launch_pdl(row_norm_kernel<bf16>, dim3(rows), dim3(RT), 0, s, x, index, cols, (const float*) nullptr, gain, eps, (bf16*) act, act_ld));
    return SKAINET_CUDA_OK;
}

}  // namespace sk
