// What the attention kernels share about masks and outputs beyond plain causal attention.
#pragma once
#include "common.cuh"

namespace mb {

// Cached tokens that any of a run of consecutive queries may see, as a dense list of whole 64-token tiles: the kept
// first tokens, then the window. Entry v stands for token v (v < keep64) or v + shift; without a window the list is
// the context itself. Queries still mask inside the first and last tiles.
struct VisibleTokens {
  int keep64;    // entries that stand for the kept first tokens, a multiple of 64
  int shift;     // token - entry behind them, a multiple of 64
  int len;       // entries

  // first: position of the run's first query; end: one past the last token that the last query sees
  __device__ __forceinline__ VisibleTokens(int first, int end, int window, int keep) {
    const int begin = window > 0 ? max(0, first + 1 - window) & ~63 : 0;
    keep64 = min((keep + 63) & ~63, begin);
    shift = begin - keep64;
    len = end - shift;
  }
  __device__ __forceinline__ int token(int v) const { return v < keep64 ? v : v + shift; }
};

// the query that sees the tokens below `limit`: does it see `tok`?
__device__ __forceinline__ bool sees(int tok, int limit, int window, int keep) {
  return tok < limit && (window <= 0 || tok >= limit - window || tok < keep);
}

// Scores squashed to (-cap, cap) before the softmax, cap tanh(s / cap), in the log2 domain of the kernels' scores and written
// with one exponential: cap - 2 cap / (1 + exp(2 s / cap)). `mul` takes a raw dot product into the exponent.
struct SoftCap {
  float mul, cap;    // cap 0: off
  static SoftCap make(float scale, float softcap) {
    constexpr float kLog2e = 1.44269504088896f;
    return softcap > 0.f ? SoftCap{2.f * scale * kLog2e / softcap, softcap * kLog2e} : SoftCap{0.f, 0.f};
  }
  __device__ __forceinline__ float operator()(float dot) const {
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(dot * mul));
    return cap - __fdividef(2.f * cap, 1.f + e);
  }
};

// An output row turned back by its own position (values that are cached turned by theirs): pair (m, m + dv / 2) by minus
// the angle in the tables' row of that position.
struct TurnBack {
  const float* cos_tab;   // [max_pos, dv / 2], or null: off
  const float* sin_tab;
  int half, max_pos;
  // N consecutive elements of the first half and their partners, element d on
  template <int N>
  __device__ __forceinline__ void operator()(int pos, int d, float* u, float* v) const {
    const size_t at = (size_t)(pos < max_pos ? pos : 0) * half + d;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const float c = __ldg(cos_tab + at + i), s = __ldg(sin_tab + at + i), a = u[i], b = v[i];
      u[i] = a * c + b * s;
      v[i] = b * c - a * s;
    }
  }
};

enum { GATE_NONE = 0, GATE_HEAD = 1, GATE_ELEMENT = 2 };

// Sigmoid gates on an attention output, read where the projection left their logits: one per head, or one per element
// (head h's at columns h * dv ...). Row m of the output has its logits gate_ld elements times m on.
template <typename T>
struct OutputGate {
  const T* logits;
  long long ld;
  int mode, dv;
  __device__ __forceinline__ float operator()(size_t row, int head, int d) const {
    if (mode == GATE_NONE) return 1.f;
    const T* z = logits + row * ld + (mode == GATE_HEAD ? head : head * dv + d);
    float v;
    if constexpr (sizeof(T) == 2) v = __bfloat162float(*z);
    else v = *z;
    return 1.f / (1.f + expf(-v));
  }
  // elements d .. d + 3 of a bf16 gate times v (d a multiple of 4; those past dv stay)
  __device__ __forceinline__ void scale4(size_t row, int head, int d, float* v) const {
    const T* z = logits + row * ld + (size_t)head * dv + d;
    if (d + 4 <= dv && (reinterpret_cast<uintptr_t>(z) & 7) == 0) {
      const uint2 w = __ldg(reinterpret_cast<const uint2*>(z));
      const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
      const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
      const float g[4] = {a.x, a.y, b.x, b.y};
#pragma unroll
      for (int i = 0; i < 4; ++i) v[i] *= __fdividef(1.f, 1.f + __expf(-g[i]));
      return;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (d + i < dv) v[i] *= (*this)(row, head, d + i);
  }
};

}  // namespace mb
