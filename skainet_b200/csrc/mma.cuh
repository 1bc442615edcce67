// Warp-level matrix fragments and asynchronous 16-byte copies shared by the mma.sync kernels.
#pragma once
#include "linear_bf16.cuh"

#ifdef __CUDACC__
namespace skd {

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// x = sum of three bf16 terms of 8 bits each, exactly (while the last term does not underflow); two values per word.
__device__ __forceinline__ void split3(float a, float b, uint32_t (&t)[3]) {
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        const uint32_t x = __float_as_uint(a), y = __float_as_uint(b);
        t[i] = __byte_perm(x, y, 0x7632);
        a -= __uint_as_float(x & 0xffff0000u); b -= __uint_as_float(y & 0xffff0000u);
    }
}

}  // namespace skd
#endif
