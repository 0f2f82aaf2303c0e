// bf16 / fp32 values behind one name, for the kernels that run in either: a pointer's type says how its values are stored,
// arithmetic is fp32 throughout.
#pragma once
#include "common.cuh"

namespace fb {

__device__ __forceinline__ float value_of(float x) { return x; }
__device__ __forceinline__ float value_of(uint16_t x) { return bf16_bits_to_float(x); }
__device__ __forceinline__ void store_value(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_value(uint16_t* p, float v) { *p = (uint16_t)float_to_bf16_bits(v); }

// four columns at a time
__device__ __forceinline__ float4 four(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 four(const uint16_t* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_bits_to_float(v.x & 0xffffu), bf16_bits_to_float(v.x >> 16), bf16_bits_to_float(v.y & 0xffffu), bf16_bits_to_float(v.y >> 16));
}
__device__ __forceinline__ void put_four(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put_four(uint16_t* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w)); }
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) { return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w)); }

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

// the same by the hardware's exponential and reciprocal (about 1e-6 of the result): beside bf16 values
__device__ __forceinline__ float sigmoid_near(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

// 2^x, the hardware's (x far below: 0)
__device__ __forceinline__ float exp2_of(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// tanh by one exponential, and by its power series where that would cancel: about 2e-7 of the result either way
__device__ __forceinline__ float tanh_of(float x) {
  const float y = x * x;
  const float near = x * fmaf(y, fmaf(y, fmaf(y, fmaf(y, 62.f / 2835.f, -17.f / 315.f), 2.f / 15.f), -1.f / 3.f), 1.f);
  const float far = 1.f - __fdividef(2.f, 1.f + __expf(2.f * fminf(fmaxf(x, -15.f), 15.f)));
  return y < 0.04f ? near : far;
}

// sum over a block of up to 1024 threads (whole warps); every thread gets it.  `red` is 32 floats of shared memory
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();  // (the words may still be read from a sum before)
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < (int)(blockDim.x + 31) / 32; ++w) total += red[w];
  return total;
}

// cos and sin of place * freq, times mag.  The angle is formed in double and brought into one turn there, so that a far
// place's angle is as exact as a near one's.
__device__ __forceinline__ void turn_of(int place, double freq, float mag, float& c, float& s) {
  const double turns = (double)place * freq * 0.15915494309189535;  // / (2 pi)
  float a = (float)((turns - rint(turns)) * 6.283185307179586);
  sincosf(a, &s, &c);
  c *= mag, s *= mag;
}

}  // namespace fb
