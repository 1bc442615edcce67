// Which sequence and position an activation row stands for: seq >= 0, consecutive tokens of that sequence from pos[seq];
// seq < 0, row b is the next token of sequence b.
#pragma once
#include <stdint.h>

namespace sk {

struct RowMap {
    const int32_t* pos; int seq;
#ifdef __CUDACC__
    __device__ __forceinline__ int seq_of(int row) const { return seq < 0 ? row : seq; }
    __device__ __forceinline__ int pos_of(int row) const { return seq < 0 ? pos[row] : pos[seq] + row; }
#endif
};

}  // namespace sk
