// Tensor maps for TMA copies: the driver's encoder, fetched at run time so that the library loads on a machine without a driver.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include "capi_common.cuh"

namespace qtb {

typedef CUresult (*TensorMapEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
                                      CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline int tensor_map_encoder(TensorMapEncodeFn* out) {
    static TensorMapEncodeFn fn = nullptr;
    if (fn == nullptr) {
        void* p = nullptr;
        cudaDriverEntryPointQueryResult q = cudaDriverEntryPointSymbolNotFound;
        const cudaError_t e = cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q);
        if (e != cudaSuccess || q != cudaDriverEntryPointSuccess || p == nullptr) return fail(QUINTRIT_ERR_DEVICE, "the CUDA driver does not provide cuTensorMapEncodeTiled");
        fn = reinterpret_cast<TensorMapEncodeFn>(p);
    }
    *out = fn;
    return QUINTRIT_OK;
}

// `count` row-major bf16 matrices of `rows` rows each, one after the other, rows `pitch` elements apart (a multiple of 8), read in boxes of
// box_cols x box_rows of one matrix with the 128-byte swizzle (box_cols at most 64); rows beyond a matrix read as zeros.
inline int tensor_map_bf16(CUtensorMap* map, void* base, size_t pitch, size_t rows, size_t count, int box_cols, int box_rows, int rank) {
    TensorMapEncodeFn encode = nullptr;
    const int rc = tensor_map_encoder(&encode);
    if (rc != QUINTRIT_OK) return rc;
    const cuuint64_t dims[3] = {pitch, rows, count}, strides[2] = {pitch * 2, pitch * rows * 2};
    const cuuint32_t box[3] = {static_cast<cuuint32_t>(box_cols), static_cast<cuuint32_t>(box_rows), 1}, elem[3] = {1, 1, 1};
    const CUresult cr = encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, static_cast<cuuint32_t>(rank), base, dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                               CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (cr != CUDA_SUCCESS) return fail(QUINTRIT_ERR_DEVICE, "cuTensorMapEncodeTiled failed with CUDA driver error %d", static_cast<int>(cr));
    return QUINTRIT_OK;
}
inline int tensor_map_2d_bf16(CUtensorMap* map, void* base, size_t pitch, size_t rows, int box_cols, int box_rows) { return tensor_map_bf16(map, base, pitch, rows, 1, box_cols, box_rows, 2); }
inline int tensor_map_3d_bf16(CUtensorMap* map, void* base, size_t pitch, size_t rows, size_t count, int box_cols, int box_rows) {
    return tensor_map_bf16(map, base, pitch, rows, count, box_cols, box_rows, 3);
}

}  // namespace qtb
