// A launch that may start while the kernel before it in the stream drains (programmatic dependent launch): for kernels that
// call griddep_wait() before they read or write anything.
#pragma once
#include "common.cuh"

namespace fb {

template <typename... Params, typename... Args>
int launch_after(void (*kernel)(Params...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, const char* what, const Args&... args) {
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = grid, cfg.blockDim = block, cfg.dynamicSmemBytes = smem, cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr, cfg.numAttrs = 1;
  cudaLaunchKernelEx(&cfg, kernel, Params(args)...);
  return launch_status(what);
}

}  // namespace fb
