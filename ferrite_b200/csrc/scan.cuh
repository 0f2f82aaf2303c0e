// Arguments of the scans with a decaying state (recurrent.cu, selective_prompt.cu) as their kernels see them.
#pragma once
#include "values.cuh"

namespace fb {

struct ScanArgs {
  const void* x;  // [tokens, ld]: of head h the query at q0 + h / rep * dim, the key at k0 + h / rep * dim, the value at v0 + h * vdim
  int64_t ld, q0, k0, v0;
  int rep, heads, dim, vdim;
  const float* decay;     // [heads] (a selective scan: none)
  const int32_t* places;  // a sequence whose first token is at place 0 starts from a zero state
  int dead;               // a sequence whose first token is at this place has no token (its state stays, its output is 0); -1: none
  int64_t tokens;         // per sequence, one sequence's after the other's
  float* state;           // [sequences, heads, dim, vdim], sequences state_stride apart
  int64_t state_stride;
  float* out;  // [tokens, ld_o]
  int64_t ld_o;
  const float* step;  // selective: [tokens, ld_step], head h's step size before its bias and softplus
  int64_t ld_step;
  const float *step_bias, *a_log, *skip;  // [heads]
};

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

// selective_prompt.cu: a selective scan over prompts on the 5th-generation tensor cores
bool selective_prompt_supports(const ScanArgs& a, int64_t sequences);
int selective_prompt(const ScanArgs& a, int64_t sequences, cudaStream_t s);

}  // namespace fb
