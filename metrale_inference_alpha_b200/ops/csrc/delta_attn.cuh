// Inputs of the delta-rule kernels, and the gates made of them: shared by the token-by-token and the chunked kernels.
#pragma once
#include "common.cuh"
#include "epilogue.cuh"

namespace mb {

constexpr float kUnitEps = 1e-6f;      // added to a squared length before its root

template <typename T>
__device__ __forceinline__ float load1(const void* base, size_t i) {
  if constexpr (sizeof(T) == 2) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(base)[i]);
  else return reinterpret_cast<const float*>(base)[i];
}

// log(1 + exp(z))
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

struct DeltaInputs {
  const void* q;               // [T, HK DK]
  const void* k;
  const void* v;               // [T, H DV]
  long long q_ld, k_ld, v_ld;  // elements between tokens
  int H, HK, DK, DV, f32, general;
  // gated rule: logits [T, H] of the decay and the step size, and the decay's constants [H]
  const void* decay;
  const void* step;
  long long gate_ld;
  const float* A_log;
  const float* dt_bias;
  // general rule (HK = H): logits [T, H DK] of the removal rate, log decays [T, H DK]
  const void* removal;
  long long removal_ld;
  const float* log_w;

  template <typename T>
  __device__ __forceinline__ float query(size_t t, int h, int d) const { return load1<T>(q, t * q_ld + (size_t)(h / (H / HK)) * DK + d); }
  template <typename T>
  __device__ __forceinline__ float key(size_t t, int h, int d) const { return load1<T>(k, t * k_ld + (size_t)(h / (H / HK)) * DK + d); }
  template <typename T>
  __device__ __forceinline__ float value(size_t t, int h, int d) const { return load1<T>(v, t * v_ld + (size_t)h * DV + d); }
  template <typename T>
  __device__ __forceinline__ float log_gate(size_t t, int h) const { return -expf(A_log[h]) * softplus(load1<T>(decay, t * gate_ld + h) + dt_bias[h]); }
  template <typename T>
  __device__ __forceinline__ float step_size(size_t t, int h) const { return sigmoid_exact(load1<T>(step, t * gate_ld + h)); }
  template <typename T>
  __device__ __forceinline__ float rate(size_t t, int h, int d) const { return sigmoid_exact(load1<T>(removal, t * removal_ld + (size_t)h * DK + d)); }
};

inline bool delta_inputs_ok(const DeltaInputs& in, bool low_rank) {
  if (!in.q || !in.k || !in.v || in.H <= 0 || in.HK <= 0 || in.H % in.HK || in.DK <= 0 || in.DV <= 0) return false;
  if (in.general) return in.HK == in.H && in.removal && (low_rank || in.log_w);
  return in.decay && in.step && in.A_log && in.dt_bias;
}

}  // namespace mb
