// Tensor maps over row-major bf16 matrices [rows][ld] (ld a multiple of 64) for TMA loads in the 128-byte swizzle: a box row is
// 64 elements, its 16-byte chunks XORed with the row. Coordinates outside the matrix read as zero.
#pragma once
#include "linear_bf16.cuh"

#include <cuda.h>

namespace sk {

// boxes of box_rows x 64 k, coordinates (k, row)
int32_t tensor_map_rows(CUtensorMap* map, const bf16* base, int64_t rows, int ld, int box_rows);
// boxes of box_blocks blocks of 64 k, box_rows rows each, block-major; coordinates (0, row, block)
int32_t tensor_map_k_blocks(CUtensorMap* map, const bf16* base, int64_t rows, int ld, int box_rows, int box_blocks);

}  // namespace sk

#ifdef __CUDACC__
namespace skd {

__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* map, int x, int y, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];"
                 ::"r"((uint32_t) __cvta_generic_to_shared(dst)), "l"(map), "r"(x), "r"(y), "r"((uint32_t) __cvta_generic_to_shared(bar)) : "memory");
}
__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, int x, int y, int z, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];"
                 ::"r"((uint32_t) __cvta_generic_to_shared(dst)), "l"(map), "r"(x), "r"(y), "r"(z), "r"((uint32_t) __cvta_generic_to_shared(bar)) : "memory");
}

}  // namespace skd
#endif
