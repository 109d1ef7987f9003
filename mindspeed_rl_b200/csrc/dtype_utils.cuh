// Element access for kernels that are compiled for bf16 and for fp32 storage: everything is computed in
// fp32, `ld` / `st` convert at the memory boundary; the 4-wide forms move one 8- or 16-byte vector.
#pragma once
#include "common.cuh"

namespace msrl {

__device__ __forceinline__ float ldf(const float* p) { return *p; }
__device__ __forceinline__ float ldf(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stf(float* p, float v) { *p = v; }
__device__ __forceinline__ void stf(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ void ldf4(const float* p, float (&f)[4]) {
  const float4 t = *reinterpret_cast<const float4*>(p);
  f[0] = t.x; f[1] = t.y; f[2] = t.z; f[3] = t.w;
}
__device__ __forceinline__ void ldf4(const __nv_bfloat16* p, float (&f)[4]) {
  const uint2 t = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
__device__ __forceinline__ void stf4(float* p, const float (&f)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
__device__ __forceinline__ void stf4(__nv_bfloat16* p, const float (&f)[4]) {
  __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
  uint2 t;
  t.x = *reinterpret_cast<uint32_t*>(&a);
  t.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = t;
}

__device__ __forceinline__ void ldf2(const float* p, float (&f)[4]) {
  const float2 t = *reinterpret_cast<const float2*>(p);
  f[0] = t.x; f[1] = t.y;
}
__device__ __forceinline__ void ldf2(const __nv_bfloat16* p, float (&f)[4]) {
  const float2 t = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
  f[0] = t.x; f[1] = t.y;
}
__device__ __forceinline__ void stf2(float* p, const float (&f)[4]) { *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]); }
__device__ __forceinline__ void stf2(__nv_bfloat16* p, const float (&f)[4]) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(f[0], f[1]);
}

// V elements (1, 2 or 4) at once
template <int V, typename T>
__device__ __forceinline__ void ldv(const T* p, float (&f)[4]) {
  if constexpr (V == 4) ldf4(p, f);
  else if constexpr (V == 2) ldf2(p, f);
  else f[0] = ldf(p);
}
template <int V, typename T>
__device__ __forceinline__ void stv(T* p, const float (&f)[4]) {
  if constexpr (V == 4) stf4(p, f);
  else if constexpr (V == 2) stf2(p, f);
  else stf(p, f[0]);
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// for activations that are stored in T: bf16 results do not need the last bits of the exponential and the division
template <typename T>
__device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-x));
  else return sigmoid_f(x);
}
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

}  // namespace msrl
