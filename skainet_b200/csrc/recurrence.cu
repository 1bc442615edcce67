// Gated linear recurrences (contract: recurrence.cuh).
//
//   recur_step_kernel    one token of each sequence, or consecutive tokens of one: a CTA keeps 32 columns of a head's state in
//                        registers (columns of the state never meet), so a step reads and writes the state once.
//   recur_tail_kernel    the convolution inputs a prompt pass leaves for the next one.
//   recurrence_chunk.cu  prompts of bf16 models: chunks of 64 tokens on the tensor cores.
#include "recurrence.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr int ST = 256, SC = 32;                 // threads and state columns of a step CTA

using skd::conv_input;
using skd::softplus;

__device__ __forceinline__ float conv_silu(const RecurArgs& a, const float* tail, int row0, int pos0, int p, int c) {
    float v = a.conv_b ? a.conv_b[c] : 0.0f;
    for (int j = 0; j < a.g.taps; ++j) v = fmaf(a.conv_w[(size_t) c * a.g.taps + j], conv_input(a, tail, row0, pos0, p - (a.g.taps - 1) + j, c), v);
    return skd::silu(v);
}

// Thread (warp w, lane l) holds rows w * 4 + l / 8 + 32 i and columns 4 (l % 8) .. + 3 of the CTA's 32. With the unnormalised
// q and k one pass over the state gives S^T k, S^T q; with them k.q, |k|^2 and |q|^2,
//   o = g S^T q + (k.q) u.
template <bool DELTA, int NR>
__global__ void __launch_bounds__(ST)
recur_step_kernel(const RecurArgs a) {
    const RecurGeom& g = a.g;
    extern __shared__ float dyn[];                                  // two sets of q [kp] | k [kp] | v [32]
    __shared__ float red[2][ST / 32][2][SC];
    constexpr int kp = NR * 32;
    const int tiles = (g.vdim + SC - 1) / SC, h = blockIdx.x / tiles, c0 = (blockIdx.x % tiles) * SC, grp = h / (g.heads / g.groups);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c4 = (lane & 7) * 4, r0 = warp * 4 + (lane >> 3);
    const bool prompt = a.map.seq >= 0;
    const int seq = prompt ? a.map.seq : (int) blockIdx.y, row0 = prompt ? 0 : (int) blockIdx.y, n = prompt ? a.rows : 1;
    const bool col_ok = c0 + c4 < g.vld();
    float* state = a.state + (size_t) seq * g.state_size() + (size_t) h * g.kdim * g.vld() + c0 + c4;
    float* tail = a.tail + (size_t) seq * g.tail_size();
    skd::pdl_launch_dependents();
    // positions, state and tail were left by earlier steps, not by the predecessor kernel
    const int pos0 = a.map.pos[seq];
    float4 S[NR];
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int r = r0 + 32 * i;
        S[i] = pos0 > 0 && col_ok && r < g.kdim ? *reinterpret_cast<const float4*>(state + (size_t) r * g.vld()) : make_float4(0, 0, 0, 0);
    }
    const float neg_a = -expf(a.a_log[h]), dtb = a.dt_bias[h], skip = !DELTA ? a.d[h] : 0.0f;
    skd::pdl_wait();

    for (int t = 0; t < n; ++t) {
        const int row = row0 + t;
        float* sq = dyn + (t & 1) * (2 * kp + SC);
        float *sk_ = sq + kp, *sv = sk_ + kp;
        for (int i = threadIdx.x; i < 2 * kp + SC; i += ST) {
            int c = -1;
            if (i < kp) { if (i < g.kdim) c = a.q_off + grp * g.kdim + i; }
            else if (i < 2 * kp) { if (i - kp < g.kdim) c = a.k_off + grp * g.kdim + i - kp; }
            else if (c0 + i - 2 * kp < g.vdim) c = a.v_off + h * g.vdim + c0 + i - 2 * kp;
            sq[i] = c >= 0 ? conv_silu(a, tail, row0, pos0, pos0 + t, c) : 0.0f;
            // one token: its own slot of the tail is read by nobody in this launch
            if (!prompt && c >= 0 && (i >= 2 * kp || (blockIdx.x % tiles == 0 && h % (g.heads / g.groups) == 0)))
                tail[(size_t) (pos0 % g.taps) * g.conv_dim() + c] = a.proj[(size_t) row * a.proj_ld + a.conv_off + c];
        }
        const float dt = softplus(a.proj[(size_t) row * a.proj_ld + a.dt_off + h] + dtb), decay = expf(neg_a * dt);
        const float beta = DELTA ? skd::sigmoid(a.proj[(size_t) row * a.proj_ld + a.beta_off + h]) : 0.0f;
        __syncthreads();
        float4 ks = make_float4(0, 0, 0, 0), qs = ks;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const float k = DELTA ? sk_[r0 + 32 * i] : 0.0f, q = sq[r0 + 32 * i];
            if (DELTA) { ks.x = fmaf(k, S[i].x, ks.x); ks.y = fmaf(k, S[i].y, ks.y); ks.z = fmaf(k, S[i].z, ks.z); ks.w = fmaf(k, S[i].w, ks.w); }
            qs.x = fmaf(q, S[i].x, qs.x); qs.y = fmaf(q, S[i].y, qs.y); qs.z = fmaf(q, S[i].z, qs.z); qs.w = fmaf(q, S[i].w, qs.w);
        }
#pragma unroll
        for (int o = 8; o <= 16; o <<= 1) {
            if (DELTA) { ks.x += __shfl_xor_sync(~0u, ks.x, o); ks.y += __shfl_xor_sync(~0u, ks.y, o); ks.z += __shfl_xor_sync(~0u, ks.z, o); ks.w += __shfl_xor_sync(~0u, ks.w, o); }
            qs.x += __shfl_xor_sync(~0u, qs.x, o); qs.y += __shfl_xor_sync(~0u, qs.y, o); qs.z += __shfl_xor_sync(~0u, qs.z, o); qs.w += __shfl_xor_sync(~0u, qs.w, o);
        }
        float (*rd)[2][SC] = red[t & 1];
        if (lane < 8) { *reinterpret_cast<float4*>(&rd[warp][0][c4]) = ks; *reinterpret_cast<float4*>(&rd[warp][1][c4]) = qs; }
        float qq = 0.0f, kk = 0.0f, qk = 0.0f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const float q = sq[lane + 32 * i], k = sk_[lane + 32 * i];
            qq = fmaf(q, q, qq); kk = fmaf(k, k, kk); qk = fmaf(q, k, qk);
        }
        qk = skd::warp_sum(qk);
        float rq = 1.0f, rk = 1.0f;
        if (DELTA) { rq = 1.0f / sqrtf(skd::warp_sum(qq) + 1e-6f) * a.q_scale; rk = 1.0f / sqrtf(skd::warp_sum(kk) + 1e-6f); }
        __syncthreads();
        float4 kS = make_float4(0, 0, 0, 0), qS = kS;
#pragma unroll
        for (int w = 0; w < ST / 32; ++w) {
            if (DELTA) { const float4 v = *reinterpret_cast<const float4*>(&rd[w][0][c4]); kS.x += v.x; kS.y += v.y; kS.z += v.z; kS.w += v.w; }
            if (threadIdx.x < 8) { const float4 v = *reinterpret_cast<const float4*>(&rd[w][1][c4]); qS.x += v.x; qS.y += v.y; qS.z += v.z; qS.w += v.w; }
        }
        const float4 v = *reinterpret_cast<const float4*>(sv + c4);
        float4 u;
        if (DELTA) {
            const float f = decay * rk;
            u = make_float4(beta * (v.x - f * kS.x), beta * (v.y - f * kS.y), beta * (v.z - f * kS.z), beta * (v.w - f * kS.w));
        } else u = make_float4(dt * v.x, dt * v.y, dt * v.z, dt * v.w);
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const float k = sk_[r0 + 32 * i] * rk;
            S[i].x = fmaf(k, u.x, decay * S[i].x); S[i].y = fmaf(k, u.y, decay * S[i].y);
            S[i].z = fmaf(k, u.z, decay * S[i].z); S[i].w = fmaf(k, u.w, decay * S[i].w);
        }
        if (threadIdx.x < 8) {
            const float f = decay * rq, e = qk * rq * rk;
            const float o[4] = {fmaf(e, u.x, f * qS.x) + skip * v.x, fmaf(e, u.y, f * qS.y) + skip * v.y, fmaf(e, u.z, f * qS.z) + skip * v.z, fmaf(e, u.w, f * qS.w) + skip * v.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) if (c0 + c4 + j < g.vdim) a.out[(size_t) row * g.v_dim() + h * g.vdim + c0 + c4 + j] = o[j];
        }
    }
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int r = r0 + 32 * i;
        if (col_ok && r < g.kdim) *reinterpret_cast<float4*>(state + (size_t) r * g.vld()) = S[i];
    }
}

// The last inputs of a prompt pass into the tail of its sequence. grid.y: how far back
__global__ void __launch_bounds__(256) recur_tail_kernel(const RecurArgs a) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int c = blockIdx.x * 256 + threadIdx.x, row = a.rows - 1 - (int) blockIdx.y, p = a.map.pos[a.map.seq] + row;
    if (c >= a.g.conv_dim() || row < 0) return;
    a.tail[(size_t) a.map.seq * a.g.tail_size() + (size_t) (p % a.g.taps) * a.g.conv_dim() + c] = a.proj[(size_t) row * a.proj_ld + a.conv_off + c];
}

template <bool DELTA, int NR>
int32_t run_step(const RecurArgs& a, cudaStream_t s) {
    const int tiles = (a.g.vdim + SC - 1) / SC, bytes = 2 * (2 * NR * 32 + SC) * (int) sizeof(float);
    SK_CUDA(launch_pdl(recur_step_kernel<DELTA, NR>, dim3(a.g.heads * tiles, a.map.seq >= 0 ? 1 : a.rows), dim3(ST), bytes, s, a));
    return SKAINET_CUDA_OK;
}
template <bool DELTA>
int32_t run_step_rows(const RecurArgs& a, cudaStream_t s) {
    const int nr = (a.g.kdim + 31) / 32;
    if (nr <= 1) return run_step<DELTA, 1>(a, s);
    if (nr <= 2) return run_step<DELTA, 2>(a, s);
    if (nr <= 4) return run_step<DELTA, 4>(a, s);
    if (nr <= 8) return run_step<DELTA, 8>(a, s);
    return run_step<DELTA, 16>(a, s);
}

}  // namespace

int32_t launch_recurrence(const RecurArgs& a, cudaStream_t s) {
    if (a.rows <= 0) return SKAINET_CUDA_OK;
    SK_REQUIRE(a.g.kdim <= RECUR_MAX_KDIM, "recurrence: key size %d (at most %d)", a.g.kdim, RECUR_MAX_KDIM);
    if (a.map.seq >= 0 && !a.f32_act && a.work && a.rows >= RECUR_CHUNK_MIN_ROWS && recur_work_bytes(a.g, a.rows) > 0) return launch_recur_chunks(a, s);
    SK_TRY(a.g.delta ? run_step_rows<true>(a, s) : run_step_rows<false>(a, s));
    if (a.map.seq >= 0) SK_CUDA(launch_pdl(recur_tail_kernel, dim3((a.g.conv_dim() + 255) / 256, std::min(a.rows, a.g.taps)), dim3(256), 0, s, a));
    return SKAINET_CUDA_OK;
}

}  // namespace sk
