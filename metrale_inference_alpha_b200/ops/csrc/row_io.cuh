// Row access of the elementwise kernels around a 32-bit residual stream: vectors of activations and fp32 values.
#pragma once
#include "common.cuh"

namespace {

using bf16 = __nv_bfloat16;

template <typename T>
__device__ __forceinline__ float ldv(const T* p) {
  if constexpr (sizeof(T) == 2) return __bfloat162float(*p);
  else return *p;
}
template <typename T>
__device__ __forceinline__ void stv(T* p, float v) {
  if constexpr (sizeof(T) == 2) *p = __float2bfloat16(v);
  else *p = v;
}
// VEC consecutive elements <-> floats (VEC is 1 or 4; 4 needs the natural vector alignment)
template <int VEC, typename T>
__device__ __forceinline__ void ldn(const T* p, float* o) {
  if constexpr (VEC == 1) {
    o[0] = ldv(p);
  } else if constexpr (sizeof(T) == 2) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y;
  } else {
    const float4 v = *reinterpret_cast<const float4*>(p);
    o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void stn(T* p, const float* o) {
  if constexpr (VEC == 1) {
    stv(p, o[0]);
  } else if constexpr (sizeof(T) == 2) {
    uint2 v;
    *reinterpret_cast<__nv_bfloat162*>(&v.x) = __floats2bfloat162_rn(o[0], o[1]);
    *reinterpret_cast<__nv_bfloat162*>(&v.y) = __floats2bfloat162_rn(o[2], o[3]);
    *reinterpret_cast<uint2*>(p) = v;
  } else {
    *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
  }
}

struct DytW {
  float alpha;
  const bf16* w;
  const bf16* b;
};

__device__ __forceinline__ float dyt(float x, float alpha, float w, float b) { return tanhf(alpha * x) * w + b; }

inline bool al(const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) % n) == 0; }
inline int row_threads(int W, int vec) {
  int n = 32;
  while (n < 256 && n * vec < W) n <<= 1;
  return n;
}

}  // namespace
