// Tensor maps for TMA loads of bf16 matrices in boxes of 64 columns (128 bytes, 128-byte swizzle).
#pragma once

#include <cuda.h>

#include "host_util.h"

namespace q38 {

using TensorMapEncodeFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                       const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                       CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline TensorMapEncodeFn tensor_map_encode_fn() {
  static TensorMapEncodeFn fn = [] {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess) p = nullptr;
    return reinterpret_cast<TensorMapEncodeFn>(p);
  }();
  return fn;
}

// [rows][cols] bf16 with rows `ld` elements apart, boxes of 64 columns x box_rows; what lies outside reads as zero
inline int encode_bf16_rows(CUtensorMap* map, const void* base, long long rows, int cols, int ld, int box_rows) {
  TensorMapEncodeFn enc = tensor_map_encode_fn();
  Q38_REQUIRE(enc != nullptr, "cuTensorMapEncodeTiled is not available from this driver");
  const cuuint64_t dims[2] = {cuuint64_t(cols), cuuint64_t(rows)};
  const cuuint64_t strides[1] = {cuuint64_t(ld) * 2};
  const cuuint32_t box[2] = {64, cuuint32_t(box_rows)};
  const cuuint32_t estr[2] = {1, 1};
  const CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
                         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
                         CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  Q38_REQUIRE(r == CUDA_SUCCESS, "tensor map of %lld x %d, rows %d apart: encode failed (%d)", rows, cols, ld, int(r));
  return Q38_OK;
}

}  // namespace q38
