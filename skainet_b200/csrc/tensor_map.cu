// Tensor-map encoding (contract: tensor_map.cuh); the driver's encoder is looked up at run time.
#include "tensor_map.cuh"

namespace sk {

namespace {

typedef CUresult (*EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                             const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeFn encode_fn() {
    static EncodeFn fn = [] {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess) { cudaGetLastError(); p = nullptr; }
        return (EncodeFn) p;
    }();
    return fn;
}

int32_t encode(CUtensorMap* map, const bf16* base, int rank, const cuuint64_t* dims, const cuuint64_t* strides, const cuuint32_t* box) {
    EncodeFn fn = encode_fn();
    SK_REQUIRE(fn != nullptr, "tensor map: the driver has no encoder");
    const cuuint32_t es[3] = {1, 1, 1};
    const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<bf16*>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
                          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    SK_REQUIRE(r == CUDA_SUCCESS, "tensor map of %lld x %lld elements refused (%d)", (long long) dims[1], (long long) dims[0], (int) r);
    return SKAINET_CUDA_OK;
}

}  // namespace

int32_t tensor_map_rows(CUtensorMap* map, const bf16* base, int64_t rows, int ld, int box_rows) {
    const cuuint64_t dims[2] = {(cuuint64_t) ld, (cuuint64_t) rows}, strides[1] = {(cuuint64_t) ld * 2};
    const cuuint32_t box[2] = {64, (cuuint32_t) box_rows};
    return encode(map, base, 2, dims, strides, box);
}

int32_t tensor_map_k_blocks(CUtensorMap* map, const bf16* base, int64_t rows, int ld, int box_rows, int box_blocks) {
    const cuuint64_t dims[3] = {64, (cuuint64_t) rows, (cuuint64_t) ld / 64}, strides[2] = {(cuuint64_t) ld * 2, 128};
    const cuuint32_t box[3] = {64, (cuuint32_t) box_rows, (cuuint32_t) box_blocks};
    return encode(map, base, 3, dims, strides, box);
}

}  // namespace sk
