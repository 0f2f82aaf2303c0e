// Host side of a TMA tile map over bf16 values: 64 of them (one 128-byte swizzled row of shared memory) innermost.
#pragma once
#include <cuda.h>

#include "common.cuh"

namespace fb {

using EncodeTiledFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                   const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

// the driver's encoder, asked for by name (the library does not link libcuda); null where there is no driver
inline EncodeTiledFn tma_encoder() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult res;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &res) == cudaSuccess && res == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeTiledFn>(p);
  }
  return fn;
}

// dims[0] innermost; strides in elements for dims 1.. (each a multiple of 8); what lies outside reads as zeros
inline int tma_map_bf16(CUtensorMap* map, const void* base, int rank, const int64_t* dims, const int64_t* strides, const int* box, const char* what) {
  cuuint64_t d[5], s[5];
  cuuint32_t b[5], e[5];
  for (int i = 0; i < rank; ++i) d[i] = (cuuint64_t)dims[i], b[i] = (cuuint32_t)box[i], e[i] = 1;
  for (int i = 0; i + 1 < rank; ++i) s[i] = (cuuint64_t)strides[i] * 2;
  const CUresult rc = tma_encoder()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), d, s, b, e, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                    CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (rc == CUDA_SUCCESS) return FB_OK;
  set_error("%s: cuTensorMapEncodeTiled failed (%d)", what, (int)rc);
  return FB_ERR_LAUNCH;
}

// SMs of the current device
inline int sm_count_of_device() {
  static int known[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
  if (!known[dev]) {
    int n = 0;
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n < 1) n = 1, cudaGetLastError();
    known[dev] = n;
  }
  return known[dev];
}

}  // namespace fb
