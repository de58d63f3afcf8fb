// Residual streams with static hyper-connections: a token keeps S copies x_1 .. x_S of its fp32 residual row.
//
//   mb_stream_hyper   everything between two sublayers in one pass. The pending sublayer's output Y joins all streams at
//                     once, x_t <- sum_s mix[s, t] x_s + out[t] Y, and the next sublayer's input is made from the new
//                     streams, u = sum_s in[s] x_s, through a Dynamic Tanh, or as it is (activation type or fp32).
//                     Y = y (times the sigmoid of one logit per token: a gated shared expert) + the weighted sum of the
//                     token's expert rows, gathered where the grouped GEMM left them.
//                     Before the first sublayer all streams are one row (x_one), which is stored once; nothing is
//                     pending there, and the streams are written out by the next call. With a row list only those
//                     tokens are produced (the rows whose logits are wanted) and the streams stay as they are.
//
// Nothing reduces over a row, so the grid splits rows into column ranges. S up to 4 is held in registers and may be
// updated in place; more streams are read again for every new one and need x_out elsewhere.
#include "common.cuh"
#include "row_io.cuh"

namespace {

enum { HYPER_NONE = 0, HYPER_DYT = 1, HYPER_RAW = 2, HYPER_F32 = 3 };

struct HyperParams {
  int W, S, x_one, out_mode, K;
  const float* x;            // [T, S, W], or [T, W] with x_one
  const void* y;             // [T, W] or null
  const float* y_gate;       // logits [T], y_gate_ld apart, or null
  long long y_gate_ld;
  const float* ye;           // expert rows, or null
  long long ye_ld;
  const int* pair_row;       // [T, K] rows of ye, -1 = none
  const float* pair_w;       // [T, K]
  const float* w_mix;        // [S (from), S (to)] of the pending sublayer, or null: nothing pending
  const float* w_out;        // [S]
  float* x_out;              // [T, S, W] or null
  const float* w_in;         // [S] of the next sublayer
  DytW norm;
  void* out;                 // [rows, W]
  const long long* rows;     // or null: all
  long long num_rows;        // of x, with `rows`
  uint32_t* status;
};

template <int kS, int VEC, typename T>
__global__ void __launch_bounds__(256) stream_hyper_kernel(const HyperParams p) {
  constexpr int kN = kS > 0 ? kS : 1;
  __shared__ int s_row[32];
  __shared__ float s_w[32];
  const int S = kS > 0 ? kS : p.S, W = p.W, tid = threadIdx.x;
  const int k = (blockIdx.y * blockDim.x + tid) * VEC;
  // the model's own numbers do not depend on the kernel before this one
  float wi[kN], wo[kN], wm[kN][kN];
  if constexpr (kS > 0) {
#pragma unroll
    for (int s = 0; s < kN; ++s) {
      wi[s] = p.w_in ? __ldg(p.w_in + s) : 0.f;
      wo[s] = p.w_mix ? __ldg(p.w_out + s) : 0.f;
#pragma unroll
      for (int t = 0; t < kN; ++t) wm[s][t] = p.w_mix ? __ldg(p.w_mix + s * kN + t) : 0.f;
    }
  }
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  long long t = blockIdx.x;
  if (p.rows) {
    t = p.rows[blockIdx.x];
    if (t < 0 || t >= p.num_rows) {
      if (tid == 0 && p.status) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
      return;
    }
  }
  if (p.ye) {
    if (tid < p.K) {
      s_row[tid] = p.pair_row[t * p.K + tid];
      s_w[tid] = p.pair_w[t * p.K + tid];
    }
    __syncthreads();
  }
  if (k >= W) return;
  const float* x = p.x + (size_t)t * (p.x_one ? 1 : S) * W + k;
  const size_t step = p.x_one ? 0 : W;
  float y[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) y[e] = 0.f;
  if (p.w_mix) {
    if (p.y) {
      ldn<VEC>(reinterpret_cast<const T*>(p.y) + (size_t)t * W + k, y);
      if (p.y_gate) {
        const float g = 1.f / (1.f + expf(-p.y_gate[t * p.y_gate_ld]));
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] *= g;
      }
    }
    if (p.ye) {
      float a[VEC];
      for (int j = 0; j < p.K; ++j) {
        if (s_row[j] < 0) continue;
        ldn<VEC>(p.ye + (size_t)s_row[j] * p.ye_ld + k, a);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = fmaf(s_w[j], a[e], y[e]);
      }
    }
  }
  float u[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) u[e] = 0.f;
  float* xo = p.x_out ? p.x_out + (size_t)t * S * W + k : nullptr;
  if constexpr (kS > 0) {
    float v[kN][VEC];
#pragma unroll
    for (int s = 0; s < kN; ++s) ldn<VEC>(x + s * step, v[s]);
#pragma unroll
    for (int to = 0; to < kN; ++to) {
      float n[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (p.w_mix) {
          n[e] = wo[to] * y[e];
#pragma unroll
          for (int s = 0; s < kN; ++s) n[e] = fmaf(wm[s][to], v[s][e], n[e]);
        } else {
          n[e] = v[to][e];
        }
        u[e] = fmaf(wi[to], n[e], u[e]);
      }
      if (xo) stn<VEC>(xo + (size_t)to * W, n);
    }
  } else {
    for (int to = 0; to < S; ++to) {
      float n[VEC], a[VEC];
      if (p.w_mix) {
        const float wo1 = p.w_out[to];
#pragma unroll
        for (int e = 0; e < VEC; ++e) n[e] = wo1 * y[e];
        for (int s = 0; s < S; ++s) {
          const float w = p.w_mix[s * S + to];
          ldn<VEC>(x + s * step, a);
#pragma unroll
          for (int e = 0; e < VEC; ++e) n[e] = fmaf(w, a[e], n[e]);
        }
      } else {
        ldn<VEC>(x + to * step, n);
      }
      const float wi1 = p.w_in ? p.w_in[to] : 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[e] = fmaf(wi1, n[e], u[e]);
      if (xo) stn<VEC>(xo + (size_t)to * W, n);
    }
  }
  if (p.out_mode == HYPER_NONE) return;
  const size_t o = (size_t)blockIdx.x * W + k;
  if (p.out_mode == HYPER_F32) {
    stn<VEC>(reinterpret_cast<float*>(p.out) + o, u);
    return;
  }
  if (p.out_mode == HYPER_DYT) {
    float w[VEC], b[VEC];
    ldn<VEC>(p.norm.w + k, w);
    ldn<VEC>(p.norm.b + k, b);
#pragma unroll
    for (int e = 0; e < VEC; ++e) u[e] = dyt(u[e], p.norm.alpha, w[e], b[e]);
  }
  stn<VEC>(reinterpret_cast<T*>(p.out) + o, u);
}

}  // namespace

struct MbStreamHyperArgs {
  int T, W, S, f32, x_one, out_mode, K;
  const float* x;
  const void* y;
  const float* y_gate;
  long long y_gate_ld;
  const float* ye;
  long long ye_ld;
  const int* pair_row;
  const float* pair_w;
  const float* w_mix;
  const float* w_out;
  float* x_out;
  const float* w_in;
  float alpha;
  const void* norm_w;
  const void* norm_b;
  void* out;
  const long long* rows;     // or null; T is their number then, num_rows that of x
  long long num_rows;
  uint32_t* status;
};

extern "C" int mb_stream_hyper(const MbStreamHyperArgs* a, cudaStream_t stream) {
  if (!a || a->T <= 0 || a->W <= 0 || a->S <= 0 || !a->x || a->out_mode < HYPER_NONE || a->out_mode > HYPER_F32) return MB_ERR_BAD_ARG;
  if (a->out_mode != HYPER_NONE && (!a->out || !a->w_in)) return MB_ERR_BAD_ARG;
  if (a->out_mode == HYPER_DYT && (!a->norm_w || !a->norm_b)) return MB_ERR_BAD_ARG;
  if (a->w_mix ? !a->w_out : (a->y || a->ye || a->x_out)) return MB_ERR_BAD_ARG;
  if (a->ye && (!a->pair_row || !a->pair_w || a->K <= 0 || a->K > 32 || a->ye_ld < a->W)) return MB_ERR_BAD_ARG;
  if (a->y_gate && !a->y) return MB_ERR_BAD_ARG;
  if (a->x_out && (a->rows || (a->x_out == a->x && (a->S > 4 || a->x_one)))) return MB_ERR_BAD_ARG;
  const HyperParams p{a->W, a->S, a->x_one, a->out_mode, a->K, a->x, a->y, a->y_gate, a->y_gate_ld, a->ye, a->ye_ld, a->pair_row, a->pair_w,
                      a->w_mix, a->w_out, a->x_out, a->w_in, DytW{a->alpha, (const bf16*)a->norm_w, (const bf16*)a->norm_b}, a->out, a->rows,
                      a->num_rows, a->status};
  const bool v4 = a->W % 4 == 0 && a->ye_ld % 4 == 0 && al(a->x, 16) && al(a->y, 16) && al(a->ye, 16) && al(a->x_out, 16) && al(a->out, 16) &&
                  al(a->norm_w, 8) && al(a->norm_b, 8);
  const int vec = v4 ? 4 : 1, nt = row_threads(a->W, vec);
  const dim3 g(a->T, (a->W + nt * vec - 1) / (nt * vec)), b(nt);
#define MB_HYPER(N, V)                                                                                  \
  return a->f32 ? (int)mb::launch_kernel(stream_hyper_kernel<N, V, float>, g, b, 0, stream, p)          \
                : (int)mb::launch_kernel(stream_hyper_kernel<N, V, bf16>, g, b, 0, stream, p)
#define MB_HYPER_S(N)      \
  if (v4) MB_HYPER(N, 4);  \
  MB_HYPER(N, 1)
  switch (a->S) {
    case 1: MB_HYPER_S(1);
    case 2: MB_HYPER_S(2);
    case 3: MB_HYPER_S(3);
    case 4: MB_HYPER_S(4);
    default: MB_HYPER_S(0);
  }
#undef MB_HYPER_S
#undef MB_HYPER
}
