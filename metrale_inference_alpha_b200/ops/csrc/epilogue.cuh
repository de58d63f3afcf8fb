// GEMM epilogue numbering and the elementwise functions the two GEMM families share.
#pragma once
#include "common.cuh"

namespace mb {

enum { EPI_PLAIN = 0, EPI_SWIGLU = 1, EPI_CLAMP_GLU = 2, EPI_SILU_COLS = 3, EPI_NEG_EXP = 4, EPI_GEGLU = 5, EPI_BIAS = 6, EPI_LOG_SIGMOID = 7, EPI_RELU2 = 8, EPI_SIGMOID = 9 };

__device__ __forceinline__ float relu2(float z) { const float r = fmaxf(z, 0.f); return r * r; }
__device__ __forceinline__ float sigmoid_exact(float z) { return 1.f / (1.f + expf(-z)); }
// the same with the approximate exponential and divide (a few ulp)
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }
__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }

// g = min(gate, limit), u = clamp(up, -limit, limit): g sigmoid(alpha g) (u + 1)
__device__ __forceinline__ float clamp_glu(float gate, float up, float alpha, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g * sigmoid_exact(alpha * g) * (u + 1.f);
}
// the same with the approximate exponential and divide (a few ulp), for outputs that are rounded to bf16
__device__ __forceinline__ float clamp_glu_fast(float gate, float up, float alpha, float limit) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return __fdividef(g * (u + 1.f), 1.f + __expf(-alpha * g));
}


// gelu_tanh(gate) * up; 0.5 (1 + tanh(a)) = sigmoid(2 a), and 1.5957... = 2 sqrt(2 / pi)
__device__ __forceinline__ float gelu_tanh(float z) { return z * sigmoid_exact(1.5957691216057308f * (z + 0.044715f * z * z * z)); }
__device__ __forceinline__ float geglu_fast(float gate, float up) {
  return __fdividef(gate * up, 1.f + __expf(-1.5957691216057308f * (gate + 0.044715f * gate * gate * gate)));
}
// log(sigmoid(z)) = min(z, 0) - log(1 + u), u = exp(-|z|), without cancellation on either side: with s = u / (2 + u) <= 1/3,
// log(1 + u) = 2 atanh(s), its power series to s^15
__device__ __forceinline__ float log_sigmoid(float z) {
  const float u = __expf(-fabsf(z)), s = __fdividef(u, 2.f + u), q = s * s;
  float r = 1.f / 15.f;
  r = fmaf(r, q, 1.f / 13.f);
  r = fmaf(r, q, 1.f / 11.f);
  r = fmaf(r, q, 1.f / 9.f);
  r = fmaf(r, q, 1.f / 7.f);
  r = fmaf(r, q, 1.f / 5.f);
  r = fmaf(r, q, 1.f / 3.f);
  r = fmaf(r, q, 1.f);
  return fminf(z, 0.f) - 2.f * s * r;
}

}  // namespace mb
