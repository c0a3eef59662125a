// Tensor maps for TMA loads of bf16 tiles, 128-byte swizzle.
#pragma once
#include <cuda.h>
#include "common.cuh"

namespace mv {

// cuTensorMapEncodeTiled through the runtime's driver entry point (no link-time libcuda dependency).
typedef CUresult (*TmapEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                 const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                 CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline TmapEncodeFn tmap_encode_fn() {
  static TmapEncodeFn fn = [] {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) == cudaSuccess &&
        qres == cudaDriverEntryPointSuccess)
      return reinterpret_cast<TmapEncodeFn>(ptr);
    cudaGetLastError();
    return static_cast<TmapEncodeFn>(nullptr);
  }();
  return fn;
}

// bf16 tensor (d2, d1, d0), d0 innermost and dense, strides s1 and s2 in elements; box 64 x b1 x b2 (d0 x d1 x d2).
// Elements outside the tensor read as zero.
inline int make_tmap_bf16(CUtensorMap* m, const void* base, int64_t d0, int64_t d1, int64_t d2, int64_t s1, int64_t s2,
                          int b1, int b2, const char* what) {
  TmapEncodeFn fn = tmap_encode_fn();
  if (!fn) return fail(MV_ERR_CUDA, "%s: cuTensorMapEncodeTiled is not available", what);
  const cuuint64_t dims[3] = {static_cast<cuuint64_t>(d0), static_cast<cuuint64_t>(d1), static_cast<cuuint64_t>(d2)};
  const cuuint64_t strides[2] = {static_cast<cuuint64_t>(s1) * 2, static_cast<cuuint64_t>(s2) * 2};
  const cuuint32_t box[3] = {64, static_cast<cuuint32_t>(b1), static_cast<cuuint32_t>(b2)};
  const cuuint32_t estr[3] = {1, 1, 1};
  const CUresult r = fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return fail(MV_ERR_CUDA, "%s: cuTensorMapEncodeTiled failed with %d", what, static_cast<int>(r));
  return MV_OK;
}

}  // namespace mv
