// Expert routing kernels (contract: moe.cuh). Few slots: one CTA picks, counts and sorts in one launch. Many: one warp per
// row picks, then one CTA per expert finds its offset from a histogram of all slots and compacts its own slots in order.
#include "moe.cuh"
#include "tma.cuh"

#include <algorithm>

namespace sk {

namespace {

constexpr int SMALL_SLOTS = 512;

// The `top` best scores of one row by a warp; each pass looks for the best score strictly after the previous one in
// (score descending, index ascending) order.
__device__ __forceinline__ void pick_row(const float* z, int experts, int top, int32_t* expert, float* weight) {
    const int lane = threadIdx.x & 31;
    float last = INFINITY; int last_i = -1;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY; int bi = 0x7fffffff;
        for (int e = lane; e < experts; e += 32) {
            const float s = skd::sigmoid(z[e]);
            if ((s < last || (s == last && e > last_i)) && (s > best || (s == best && e < bi))) { best = s; bi = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(~0u, best, o); const int oi = __shfl_xor_sync(~0u, bi, o);
            if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
        }
        if (bi == 0x7fffffff) { bi = k; best = 0.0f; }        // no ordered score left (not-a-number logits): a valid index, weight 0
        if (lane == 0) { expert[k] = bi; weight[k] = best; }
        last = best; last_i = bi;
    }
}

__global__ void __launch_bounds__(SMALL_SLOTS)
route_small_kernel(const float* __restrict__ z, int rows, int experts, int top, int seg_rows, const RouteBuffers b) {
    extern __shared__ int hist[];               // [experts] counts, then exclusive offsets; [experts] segment offsets
    __shared__ int se[SMALL_SLOTS];
    __shared__ float sw[SMALL_SLOTS];
    int* seg0 = hist + experts;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int slots = rows * top, warp = threadIdx.x >> 5;
    for (int e = threadIdx.x; e < experts; e += blockDim.x) hist[e] = 0;
    for (int r = warp; r < rows; r += (int) blockDim.x >> 5) pick_row(z + (size_t) r * experts, experts, top, se + r * top, sw + r * top);
    __syncthreads();
    const int me = threadIdx.x;
    int e = -1, rank = 0;
    if (me < slots) {
        e = se[me];
        for (int i = 0; i < me; ++i) rank += se[i] == e;
        atomicAdd(hist + e, 1);
    }
    __syncthreads();
    if (warp == 0) {                            // exclusive prefix sums over the experts, 32 at a time
        int base = 0, sbase = 0;
        for (int e0 = 0; e0 < experts; e0 += 32) {
            const int i = e0 + (int) (threadIdx.x & 31);
            const int n = i < experts ? hist[i] : 0, sg = (n + seg_rows - 1) / seg_rows;
            int pn = n, ps = sg;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int vn = __shfl_up_sync(~0u, pn, o), vs = __shfl_up_sync(~0u, ps, o);
                if ((int) (threadIdx.x & 31) >= o) { pn += vn; ps += vs; }
            }
            if (i < experts) {
                hist[i] = base + pn - n; seg0[i] = sbase + ps - sg;
                for (int k = 0; k < sg; ++k) b.segs[sbase + ps - sg + k] = {i, base + pn - n + k * seg_rows, min(seg_rows, n - k * seg_rows), 0};
            }
            base += __shfl_sync(~0u, pn, 31); sbase += __shfl_sync(~0u, ps, 31);
        }
        if (threadIdx.x == 0) *b.n_segs = sbase;
    }
    __syncthreads();
    if (me < slots) {
        const int p = hist[e] + rank;
        b.slot_pos[me] = p; b.sorted_row[p] = me / top; b.sorted_weight[p] = sw[me];
    }
}

__global__ void __launch_bounds__(256) route_pick_kernel(const float* __restrict__ z, int rows, int experts, int top, const RouteBuffers b) {
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    const int r = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (r < rows) pick_row(z + (size_t) r * experts, experts, top, b.slot_expert + (size_t) r * top, b.slot_weight + (size_t) r * top);
}

__global__ void __launch_bounds__(256) route_sort_kernel(int slots, int experts, int top, int seg_rows, const RouteBuffers b) {
    extern __shared__ int hist[];
    __shared__ int wsum[8], s_off, s_seg;
    const int me = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    skd::pdl_launch_dependents();
    skd::pdl_wait();
    for (int e = threadIdx.x; e < experts; e += 256) hist[e] = 0;
    if (threadIdx.x == 0) s_off = s_seg = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < slots; i += 256) atomicAdd(hist + b.slot_expert[i], 1);
    __syncthreads();
    int off = 0, seg = 0;
    for (int e = threadIdx.x; e < experts; e += 256) {
        const int sg = (hist[e] + seg_rows - 1) / seg_rows;
        if (e < me) { off += hist[e]; seg += sg; }
    }
    if (off | seg) { atomicAdd(&s_off, off); atomicAdd(&s_seg, seg); }
    __syncthreads();
    const int n = hist[me], start = s_off;
    for (int k = threadIdx.x; k * seg_rows < n; k += 256) b.segs[s_seg + k] = {me, start + k * seg_rows, min(seg_rows, n - k * seg_rows), 0};
    if (me == experts - 1 && threadIdx.x == 0) *b.n_segs = s_seg + (n + seg_rows - 1) / seg_rows;
    int done = 0;
    for (int i0 = 0; i0 < slots && done < n; i0 += 256) {      // slots of this expert, kept in order
        const int i = i0 + threadIdx.x;
        const bool mine = i < slots && b.slot_expert[i] == me;
        const unsigned mask = __ballot_sync(~0u, mine);
        if (lane == 0) wsum[warp] = __popc(mask);
        __syncthreads();
        int before = 0, total = 0;
        for (int w = 0; w < 8; ++w) { if (w < warp) before += wsum[w]; total += wsum[w]; }
        if (mine) {
            const int p = start + done + before + __popc(mask & ((1u << lane) - 1));
            b.slot_pos[i] = p; b.sorted_row[p] = i / top; b.sorted_weight[p] = b.slot_weight[i];
        }
        done += total;
        __syncthreads();
    }
}

}  // namespace

int32_t launch_route(const float* z, int rows, int experts, int top, int seg_rows, const RouteBuffers& b, cudaStream_t s) {
    if (rows <= 0) return SKAINET_CUDA_OK;
    SK_REQUIRE(experts >= 1 && experts <= ROUTE_MAX_EXPERTS && top >= 1 && top <= experts, "route: %d of %d experts", top, experts);
    const int slots = rows * top;
    if (slots <= SMALL_SLOTS) {
        SK_CUDA(launch_pdl(route_small_kernel, dim3(1), dim3(SMALL_SLOTS), 2 * experts * sizeof(int), s, z, rows, experts, top, seg_rows, b));
        return SKAINET_CUDA_OK;
    }
    SK_CUDA(launch_pdl(route_pick_kernel, dim3((rows + 7) / 8), dim3(256), 0, s, z, rows, experts, top, b));
    SK_CUDA(launch_pdl(route_sort_kernel, dim3(experts), dim3(256), experts * sizeof(int), s, slots, experts, top, seg_rows, b));
    return SKAINET_CUDA_OK;
}

}  // namespace sk
