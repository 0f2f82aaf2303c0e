// Arguments of fb_heads_attention as its kernels see them.
#pragma once
#include "values.cuh"

namespace fb {

struct HeadsArgs {
  const void* q;  // [T, ld_q]: head h at h * dim
  int64_t T, ld_q;
  int heads, kv_heads, dim, vdim, rep;  // rep: query heads per key head
  const void* cache;  // [kv_heads, cache_rows, dim + vdim]
  int64_t cache_rows, head_stride;
  const int32_t *base, *last;  // token t sees cache rows base[t] + row0 + lo .. + last[t]; lo: where last[t]'s span begins
  int64_t row0;
  int chunk;  // the tokens are one sequence's, their places rising
  int span;   // 0: no spans
  int window; // 0: none; else a token sees the last `window` places only
  float scale, softcap;  // softcap > 0: a scaled score s becomes softcap tanh(s / softcap)
  const float* sink;  // [heads] or null
  const float* key_bias;  // [heads] or null; given: no softmax, a key's weight is sigmoid(score + key_bias[h])
  float out_scale;    // of the result
  int gate_dtype;
  const void* gate;  // [T, ld_g]: head h at h * vdim; the output times its sigmoid
  int64_t ld_g;
  void* out;  // [T, ld_o]: head h at h * vdim
  int64_t ld_o;
  int64_t seen;  // an upper bound of the keys a token sees
  int stages;  // tiles of keys in the ring
  int entries, pairs, tiles;  // entries of `pairs` pairs each (a token's, or the chunk's), cut into tiles
};

// the first place that a token at `place` sees
__device__ __forceinline__ int first_seen(const HeadsArgs& a, int place) {
  const int lo = a.span > 0 ? place - place % a.span : 0;
  return a.window > 0 ? max(lo, place - a.window + 1) : lo;
}

// an unscaled score s as the unscaled score that the cap leaves: (softcap / scale) tanh(s scale / softcap), tanh by one exponential
// (to about 2e-7 of 1)
struct SoftCap {
  float in, out;
};
__device__ __forceinline__ SoftCap soft_cap(const HeadsArgs& a) { return {a.softcap > 0.f ? 2.8853900817779268f * a.scale / a.softcap : 0.f, a.softcap > 0.f ? a.softcap / a.scale : 0.f}; }
__device__ __forceinline__ float capped(const SoftCap& c, float s) { return fmaf(-2.f * c.out, __fdividef(1.f, 1.f + exp2_of(fminf(s * c.in, 80.f))), c.out); }

// sigmoids of two numbers given times log2(e), by two exponentials and one reciprocal
__device__ __forceinline__ void sigmoid_pair(float x, float y, float& a, float& b) {
  const float u = 1.f + exp2_of(fminf(-x, 60.f)), v = 1.f + exp2_of(fminf(-y, 60.f)), r = __fdividef(1.f, u * v);
  a = r * v, b = r * u;
}

__device__ __forceinline__ float gate_value(const HeadsArgs& a, int64_t at) {
  return a.gate_dtype == FB_FP32 ? static_cast<const float*>(a.gate)[at] : bf16_bits_to_float(static_cast<const uint16_t*>(a.gate)[at]);
}
__device__ __forceinline__ float gate_of(const HeadsArgs& a, int64_t t, int64_t col) {
  return a.gate ? sigmoid_f(gate_value(a, t * a.ld_g + col)) : 1.f;
}

// heads_prompt.cu: a prompt's chunk on the 5th-generation tensor cores
bool heads_prompt_supports(const HeadsArgs& a);
int heads_prompt(const HeadsArgs& a, cudaStream_t s);

}  // namespace fb
