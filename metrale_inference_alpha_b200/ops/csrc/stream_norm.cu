// Row kernels of models with a 32-bit residual stream and Dynamic-Tanh norms.
//
//   stream_norm   one pass over the stream between two sublayers: the previous sublayer's output y joins
//                 the fp32 stream x through its post-norm (Dynamic Tanh, or RMS with a plain weight), and
//                 the next sublayer's input is produced from the new value (Dynamic Tanh, or the value as
//                 it is). Dynamic Tanh needs no statistics, so both norms and the add are one elementwise
//                 pass; only the RMS add reduces a row. With `mu` set the consumer is a token-shift mixer:
//                 five mixes h + (h_prev - h) mu_s are written next to h, where h_prev is the previous
//                 token's h: recomputed from the previous row (elementwise), or read from the sequence's
//                 carried state on the first row of its portion (zero at position 0). The CTA of a
//                 sequence's first row also advances that state to its last row's h: it is the only
//                 reader of the old value, so no other CTA can see a half-updated state.
//   stream_rms    the same step for streams with RMS norms in front of their sublayers and none behind: x + y, plus
//                 (mixture of experts) the weighted sum of a token's expert rows, gathered where the grouped GEMM
//                 left them; then RMS norm, or the value as it is, into a row of a possibly wider matrix
//   shift_commit  state := h of the last accepted row (write-on-accept after speculative verification)
//   gated_norm    RMS over groups of channels x weight x act(gate) x scale, act = SiLU or sigmoid; the
//                 output may be a column range of a wider matrix
//   side_gate     gelu_tanh(z) * e, e gathered from a per-layer slice of a second embedding table
//   embed_scaled  fp32 embedding rows times a constant, optionally plus a learned position row, through a Dynamic
//                 Tanh, or with a copy in the activation type
//   rope_dims     per-head RMS norms (optional) and rotate-half positions (optional) on q and k with separate query/key
//                 and value head sizes, scattered into a paged cache whose rows are padded (with zeros) to the
//                 attention kernel's tile
// T is the activation type: bf16, or fp32 for models served in 32-bit.
#include "common.cuh"
#include "epilogue.cuh"
#include "row_io.cuh"

namespace {

enum { ADD_NONE = 0, ADD_DYT = 1, ADD_RMS = 2 };
enum { OUT_NONE = 0, OUT_DYT = 1, OUT_RAW = 2 };

struct StreamParams {
  int T, W;
  const float* x;
  const void* y;
  int add_mode, out_mode;
  DytW post, pre;            // ADD_RMS uses post.w and eps
  float eps;
  float* x_out;
  void* out;                 // [T, W]
  float* h32;                // optional fp32 copy of the produced rows
  const bf16* mu;            // [5, W] or null
  void* mixes;               // [5, T, W]
  float* state;              // [slots, W]
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_seqs, num_slots, write_state;
  uint32_t* status;
};

template <int VEC, typename T>
__global__ void __launch_bounds__(256) stream_norm_kernel(const StreamParams p) {
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, W = p.W;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const T* y = reinterpret_cast<const T*>(p.y);
  auto row_inv = [&](int row) -> float {
    if (p.add_mode != ADD_RMS) return 1.f;
    float ss = 0.f;
    for (int k = tid * VEC; k < W; k += nt * VEC) {
      float v[VEC];
      ldn<VEC>(y + (size_t)row * W + k, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
    }
    return rsqrtf(mb::block_sum(ss, red) / (float)W + p.eps);
  };
  // the stream after the pending add, elements k .. k + VEC - 1 of `row`
  auto value = [&](int row, int k, float inv, float* o) {
    ldn<VEC>(p.x + (size_t)row * W + k, o);
    if (p.add_mode == ADD_NONE) return;
    float v[VEC], w[VEC], b[VEC];
    ldn<VEC>(y + (size_t)row * W + k, v);
    ldn<VEC>(p.post.w + k, w);
    if (p.add_mode == ADD_DYT) {
      ldn<VEC>(p.post.b + k, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] += fmaf(tanhf(p.post.alpha * v[i]), w[i], b[i]);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] += v[i] * inv * w[i];
    }
  };
  auto normed = [&](int k, const float* x, float* o) {
    if (p.out_mode == OUT_RAW) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = x[i];
      return;
    }
    float w[VEC], b[VEC];
    ldn<VEC>(p.pre.w + k, w);
    ldn<VEC>(p.pre.b + k, b);
#pragma unroll
    for (int i = 0; i < VEC; ++i) o[i] = fmaf(tanhf(p.pre.alpha * x[i]), w[i], b[i]);
  };

  // token shift: which sequence this row belongs to, and where its previous token's h comes from
  int prev = -1, last = -1;          // rows; prev = -1: from the state, or zero
  const float* st = nullptr;
  float* st_out = nullptr;
  if (p.mu) {
    int lo = 0, hi = p.num_seqs - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.q_start[mid] <= t) lo = mid;
      else hi = mid - 1;
    }
    const int r0 = p.q_start[lo], n = p.q_len[lo];
    if (t < r0 || t >= r0 + n) return;
    if (t > r0) {
      prev = t - 1;
    } else {
      const int slot = p.slots[lo];
      if (slot < 0 || slot >= p.num_slots) {
        if (p.status && tid == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
      } else {
        if (p.positions[t] != 0) st = p.state + (size_t)slot * W;
        if (p.write_state) { st_out = p.state + (size_t)slot * W; last = r0 + n - 1; }
      }
    }
  }
  const float inv = row_inv(t);
  const float inv_prev = prev >= 0 ? row_inv(prev) : 1.f;
  const float inv_last = (st_out && last != t) ? row_inv(last) : inv;
  for (int k = tid * VEC; k < W; k += nt * VEC) {
    float x[VEC], h[VEC];
    value(t, k, inv, x);
    if (p.x_out) stn<VEC>(p.x_out + (size_t)t * W + k, x);
    if (p.out_mode == OUT_NONE) continue;
    normed(k, x, h);
    if (p.out) stn<VEC>(reinterpret_cast<T*>(p.out) + (size_t)t * W + k, h);
    if (p.h32) stn<VEC>(p.h32 + (size_t)t * W + k, h);
    if (!p.mu) continue;
    float hp[VEC];
    if (prev >= 0) {
      float xp[VEC];
      value(prev, k, inv_prev, xp);
      normed(k, xp, hp);
    } else if (st) {
      ldn<VEC>(st + k, hp);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) hp[i] = 0.f;
    }
#pragma unroll
    for (int s = 0; s < 5; ++s) {
      float m[VEC], o[VEC];
      ldn<VEC>(p.mu + (size_t)s * W + k, m);
#pragma unroll
      for (int i = 0; i < VEC; ++i) o[i] = fmaf(hp[i] - h[i], m[i], h[i]);
      stn<VEC>(reinterpret_cast<T*>(p.mixes) + ((size_t)s * p.T + t) * W + k, o);
    }
    if (st_out) {
      if (last != t) {
        float xl[VEC], hl[VEC];
        value(last, k, inv_last, xl);
        normed(k, xl, hl);
        stn<VEC>(st_out + k, hl);
      } else {
        stn<VEC>(st_out + k, h);
      }
    }
  }
}

// ------------------------------------------------------------------ add, gather experts, RMS norm
enum { RMS_NONE = 0, RMS_NORM = 1, RMS_RAW = 2 };

struct StreamRmsParams {
  int W;
  const float* x;
  const void* y;             // [T, W] or null
  const float* ye;           // expert rows, or null
  long long ye_ld;
  const int* pair_row;       // [T, K] rows of ye, -1 = none
  const float* pair_w;       // [T, K]
  int K, out_mode;
  const bf16* w;
  float eps;
  float* x_out;              // or null
  void* out;
  long long out_ld;
  float plus, scale;         // the norm's weight is (plus + w) scale
};

// a row is NIT vectors per thread, kept in registers between the sum of squares and the output
template <int VEC, int NIT, typename T>
__global__ void __launch_bounds__(256) stream_rms_kernel(const StreamRmsParams p) {
  __shared__ float red[32];
  __shared__ int s_row[32];
  __shared__ float s_w[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, W = p.W;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  if (p.ye) {
    if (tid < p.K) {
      s_row[tid] = p.pair_row[(size_t)t * p.K + tid];
      s_w[tid] = p.pair_w[(size_t)t * p.K + tid];
    }
    __syncthreads();
  }
  float v[NIT][VEC];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NIT; ++i) {
    const int k = (i * nt + tid) * VEC;
    if (k >= W) continue;
    ldn<VEC>(p.x + (size_t)t * W + k, v[i]);
    if (p.y) {
      float a[VEC];
      ldn<VEC>(reinterpret_cast<const T*>(p.y) + (size_t)t * W + k, a);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i][e] += a[e];
    }
    if (p.ye) {
      float s[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) s[e] = 0.f;
      for (int j = 0; j < p.K; ++j) {
        if (s_row[j] < 0) continue;
        float a[VEC];
        ldn<VEC>(p.ye + (size_t)s_row[j] * p.ye_ld + k, a);
#pragma unroll
        for (int e = 0; e < VEC; ++e) s[e] = fmaf(s_w[j], a[e], s[e]);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i][e] += s[e];
    }
    if (p.x_out) stn<VEC>(p.x_out + (size_t)t * W + k, v[i]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(v[i][e], v[i][e], ss);
  }
  if (p.out_mode == RMS_NONE) return;
  const float inv = p.out_mode == RMS_NORM ? rsqrtf(mb::block_sum(ss, red) / (float)W + p.eps) : 1.f;
#pragma unroll
  for (int i = 0; i < NIT; ++i) {
    const int k = (i * nt + tid) * VEC;
    if (k >= W) continue;
    if (p.out_mode == RMS_NORM) {
      float w[VEC];
      ldn<VEC>(p.w + k, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i][e] *= inv * (p.plus + w[e]) * p.scale;
    }
    stn<VEC>(reinterpret_cast<T*>(p.out) + (size_t)t * p.out_ld + k, v[i]);
  }
}

__global__ void __launch_bounds__(256) shift_commit_kernel(const float* h32, int W, float* state, const int* q_start, const int* q_len,
                                                           const int* slots, int num_slots, uint32_t* status) {
  const int s = blockIdx.x, n = q_len[s];
  if (n <= 0) return;
  const int slot = slots[s];
  if (slot < 0 || slot >= num_slots) {
    if (status && threadIdx.x == 0) atomicCAS(status, 0u, MB_ST_BOUNDS);
    return;
  }
  const float* src = h32 + (size_t)(q_start[s] + n - 1) * W;
  for (int k = threadIdx.x; k < W; k += blockDim.x) state[(size_t)slot * W + k] = src[k];
}

// ------------------------------------------------------------------ gated group RMS
struct GatedParams {
  int T, K, group;
  const float* x;
  const bf16* w;
  const void* gate;
  long long gate_ld;
  int sigmoid_gate;        // 0: SiLU
  float eps, scale;
  void* out;
  long long out_ld;
};

template <int VEC, typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedParams p) {
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const float* x = p.x + (size_t)t * p.K;
  const T* gate = reinterpret_cast<const T*>(p.gate) + (size_t)t * p.gate_ld;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.out_ld;
  auto emit = [&](int k, float inv) {
    float v[VEC], w[VEC], g[VEC], o[VEC];
    ldn<VEC>(x + k, v);
    ldn<VEC>(p.w + k, w);
    ldn<VEC>(gate + k, g);
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      const float a = p.sigmoid_gate ? mb::sigmoid_exact(g[i]) : mb::silu_exact(g[i]);
      o[i] = v[i] * inv * w[i] * a * p.scale;
    }
    stn<VEC>(out + k, o);
  };
  auto sumsq = [&](int k) {
    float v[VEC], ss = 0.f;
    ldn<VEC>(x + k, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
    return ss;
  };
  if (p.group >= p.K) {
    float ss = 0.f;
    for (int k = tid * VEC; k < p.K; k += nt * VEC) ss += sumsq(k);
    const float inv = rsqrtf(mb::block_sum(ss, red) / (float)p.K + p.eps);
    for (int k = tid * VEC; k < p.K; k += nt * VEC) emit(k, inv);
    return;
  }
  const int warp = tid >> 5, lane = tid & 31, nw = nt >> 5;
  for (int g0 = warp * p.group; g0 < p.K; g0 += nw * p.group) {
    float ss = 0.f;
    for (int k = lane * VEC; k < p.group; k += 32 * VEC) ss += sumsq(g0 + k);
    const float inv = rsqrtf(mb::warp_sum(ss) / (float)p.group + p.eps);
    for (int k = lane * VEC; k < p.group; k += 32 * VEC) emit(g0 + k, inv);
  }
}

// ------------------------------------------------------------------ token side input
template <int VEC, typename T>
__global__ void __launch_bounds__(256) side_gate_kernel(const float* z, const int* tokens, const bf16* table, long long table_ld, int off,
                                                        int dim, int rows, int num_rows, T* out, uint32_t* status) {
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const unsigned i = blockIdx.x * blockDim.x + threadIdx.x;            // one vector of one row
  const unsigned per = (unsigned)(dim / VEC), t = i / per, c = (i - t * per) * VEC;
  if (t >= (unsigned)rows) return;
  const int tok = tokens[t];
  float e[VEC], v[VEC], o[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) e[j] = 0.f;
  if (tok < 0 || tok >= num_rows) {
    if (status) atomicCAS(status, 0u, MB_ST_BOUNDS);
  } else {
    ldn<VEC>(table + (size_t)tok * table_ld + off + c, e);
  }
  ldn<VEC>(z + (size_t)t * dim + c, v);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const float x = v[j];
    o[j] = 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x))) * e[j];   // sqrt(2 / pi)
  }
  stn<VEC>(out + (size_t)t * dim + c, o);
}

// tanh(z) as two bf16 terms side by side: out[t] = [value (R) | remainder (R)], the operand of a GEMM against [W | W]
template <typename T>
__global__ void __launch_bounds__(256) tanh_split_kernel(const T* z, long long ld, bf16* out, long long total, int R) {
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const long long t = i / R, c = i - t * R;
  const float v = tanhf(ldv(z + t * ld + c));
  const bf16 h = __float2bfloat16(v);
  out[t * 2 * R + c] = h;
  out[t * 2 * R + R + c] = __float2bfloat16(v - __bfloat162float(h));
}

struct EmbedParams {
  const int* tokens;
  const bf16* table;
  float* out;
  int W, vocab;
  float scale;
  void* copy;                // [M, W] of the activation type, rows copy_ld apart, or null
  long long copy_ld;
  const int* positions;      // with pos
  const bf16* pos;           // [max_pos, W] added to the scaled row, or null
  int max_pos;
  DytW norm;                 // w null: none
  uint32_t* status;
};

template <int VEC, typename T>
__global__ void __launch_bounds__(256) embed_scaled_kernel(const EmbedParams p) {
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int t = blockIdx.x, tok = p.tokens[t], W = p.W;
  const int at = p.pos ? p.positions[t] : 0;
  const bool ok = tok >= 0 && tok < p.vocab, at_ok = p.pos && at >= 0 && at < p.max_pos;
  if ((!ok || (p.pos && !at_ok)) && p.status && threadIdx.x == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
  for (int k = threadIdx.x * VEC; k < W; k += blockDim.x * VEC) {
    float v[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    if (ok) ldn<VEC>(p.table + (size_t)tok * W + k, v);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] *= p.scale;
    if (at_ok) {
      float a[VEC];
      ldn<VEC>(p.pos + (size_t)at * W + k, a);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] += a[i];
    }
    if (p.norm.w) {
      float w[VEC], b[VEC];
      ldn<VEC>(p.norm.w + k, w);
      ldn<VEC>(p.norm.b + k, b);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = dyt(v[i], p.norm.alpha, w[i], b[i]);
    }
    stn<VEC>(p.out + (size_t)t * W + k, v);
    if (p.copy) stn<VEC>(reinterpret_cast<T*>(p.copy) + (size_t)t * p.copy_ld + k, v);
  }
}

// ------------------------------------------------------------------ rotary + cache write, separate head sizes
struct RopeDimsParams {
  int M, Hq, Hkv, dk, dv, rot, dkp, dvp;    // dkp / dvp: padded row lengths of q_out / K and of V
  const void* qkv;
  long long qkv_ld;
  const int* positions;
  const long long* slots;
  const float* cos_tab;
  const float* sin_tab;
  int max_pos;
  void* q_out;
  void* k_cache;
  void* v_cache;
  long long num_slots;
  uint32_t* status;
  const bf16* q_norm;        // [dk] per-head RMS norm weights, or null
  const bf16* k_norm;
  float eps;
};

// grid (tokens, y): the y CTAs of a token share its q | k | v output elements
template <int VEC, typename T>
__global__ void __launch_bounds__(256) rope_dims_kernel(const RopeDimsParams p) {
  const int m = blockIdx.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const T* src = reinterpret_cast<const T*>(p.qkv) + (size_t)m * p.qkv_ld;
  int pos = p.positions[m];
  if (pos < 0 || (p.rot > 0 && pos >= p.max_pos)) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    pos = 0;
  }
  long long slot = p.slots[m];
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    slot = -1;
  }
  const int half = p.rot / 2;
  const float* cs = p.cos_tab + (size_t)pos * half;
  const float* sn = p.sin_tab + (size_t)pos * half;
  const int nq = p.Hq * p.dkp, nk = p.Hkv * p.dkp, nv = p.Hkv * p.dvp;
  for (int e = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; e < nq + nk + nv; e += gridDim.y * blockDim.x * VEC) {
    float o[VEC];
    if (e < nq + nk) {
      const bool is_q = e < nq;
      const int i = is_q ? e : e - nq;
      const int h = i / p.dkp, d = i - h * p.dkp;
      const T* row = src + (is_q ? 0 : p.Hq * p.dk) + h * p.dk;
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = 0.f;
      if (d < p.dk) {
        ldn<VEC>(row + d, o);
        if (d < p.rot) {                       // VEC divides rot / 2: the whole vector is on one side
          float q[VEC];
          const bool first = d < half;
          ldn<VEC>(row + (first ? d + half : d - half), q);
          const int a = first ? d : d - half;
#pragma unroll
          for (int j = 0; j < VEC; ++j) {
            const float c = cs[a + j], s = sn[a + j];
            o[j] = first ? o[j] * c - q[j] * s : o[j] * c + q[j] * s;
          }
        }
      }
      if (is_q) stn<VEC>(reinterpret_cast<T*>(p.q_out) + (size_t)m * nq + i, o);
      else if (slot >= 0) stn<VEC>(reinterpret_cast<T*>(p.k_cache) + (size_t)slot * nk + i, o);
    } else if (slot >= 0) {
      const int i = e - nq - nk;
      const int h = i / p.dvp, d = i - h * p.dvp;
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = 0.f;
      if (d < p.dv) ldn<VEC>(src + (size_t)(p.Hq + p.Hkv) * p.dk + h * p.dv + d, o);
      stn<VEC>(reinterpret_cast<T*>(p.v_cache) + (size_t)slot * nv + i, o);
    }
  }
}

// The same with per-head RMS norms in front of the rotation: a warp per head (q, k or v). The sum of squares and the
// values run over the row twice; the second time it is in L1.
template <int VEC, typename T>
__global__ void __launch_bounds__(256) rope_heads_kernel(const RopeDimsParams p) {
  const int m = blockIdx.x, head = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (head >= p.Hq + 2 * p.Hkv) return;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const T* src = reinterpret_cast<const T*>(p.qkv) + (size_t)m * p.qkv_ld;
  long long slot = p.slots[m];
  int pos = p.positions[m];
  if (slot >= p.num_slots || pos < 0 || (p.rot > 0 && pos >= p.max_pos)) {
    if (lane == 0 && p.status) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    if (slot >= p.num_slots) slot = -1;
    pos = 0;
  }
  if (head >= p.Hq + p.Hkv) {                       // a value row
    if (slot < 0) return;
    const int h = head - p.Hq - p.Hkv;
    const T* row = src + (size_t)(p.Hq + p.Hkv) * p.dk + (size_t)h * p.dv;
    T* dst = reinterpret_cast<T*>(p.v_cache) + ((size_t)slot * p.Hkv + h) * p.dvp;
    for (int d = lane * VEC; d < p.dvp; d += 32 * VEC) {
      float o[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = 0.f;
      if (d < p.dv) ldn<VEC>(row + d, o);
      stn<VEC>(dst + d, o);
    }
    return;
  }
  const bool is_q = head < p.Hq;
  if (!is_q && slot < 0) return;
  const bf16* nw = is_q ? p.q_norm : p.k_norm;
  const T* row = src + (size_t)head * p.dk;         // k heads follow the q heads
  T* dst = is_q ? reinterpret_cast<T*>(p.q_out) + ((size_t)m * p.Hq + head) * p.dkp
                : reinterpret_cast<T*>(p.k_cache) + ((size_t)slot * p.Hkv + head - p.Hq) * p.dkp;
  float inv = 1.f;
  if (nw) {
    float ss = 0.f;
    for (int d = lane * VEC; d < p.dk; d += 32 * VEC) {
      float x[VEC];
      ldn<VEC>(row + d, x);
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(x[j], x[j], ss);
    }
    inv = 1.f / sqrtf(mb::warp_sum(ss) / (float)p.dk + p.eps);
  }
  const int half = p.rot / 2;
  const float* cs = p.cos_tab + (size_t)pos * half;
  const float* sn = p.sin_tab + (size_t)pos * half;
  auto load = [&](int d, float* o) {
    ldn<VEC>(row + d, o);
    if (nw) {
      float w[VEC];
      ldn<VEC>(nw + d, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] *= inv * w[j];
    }
  };
  for (int d = lane * VEC; d < p.dkp; d += 32 * VEC) {
    float o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    if (d < p.dk) {
      load(d, o);
      if (d < p.rot) {                              // VEC divides rot / 2: the whole vector is on one side
        float q[VEC];
        const bool first = d < half;
        load(first ? d + half : d - half, q);
        const int a = first ? d : d - half;
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          const float c = cs[a + j], s = sn[a + j];
          o[j] = first ? o[j] * c - q[j] * s : o[j] * c + q[j] * s;
        }
      }
    }
    stn<VEC>(dst + d, o);
  }
}

}  // namespace

struct MbStreamNormArgs {
  int T, W, f32, add_mode, out_mode;
  const float* x;
  const void* y;
  float post_alpha;
  const void* post_w;
  const void* post_b;
  float pre_alpha;
  const void* pre_w;
  const void* pre_b;
  float eps;
  float* x_out;
  void* out;
  float* h32;
  const void* mu;
  void* mixes;
  float* state;
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_seqs, num_slots, write_state;
  uint32_t* status;
};

struct MbStreamRmsArgs {
  int T, W, f32, out_mode;
  const float* x;
  const void* y;
  const float* ye;
  long long ye_ld;
  const int* pair_row;
  const float* pair_w;
  int K;
  const void* w;
  float eps;
  float* x_out;
  void* out;
  long long out_ld;
  int plus_one;              // the norm's weight is 1 + w
  float scale;               // factor on the normed output
};

struct MbGatedNormArgs {
  int T, K, group, f32;
  const float* x;
  const void* w;
  const void* gate;
  long long gate_ld;
  int sigmoid_gate;
  float eps, scale;
  void* out;
  long long out_ld;
};

struct MbEmbedArgs {
  int M, W, vocab, copy_f32;
  const int* tokens;
  const void* table;
  float* out;
  float scale;
  void* copy;                // or null: the same rows in the activation type, copy_ld elements apart
  long long copy_ld;
  const int* positions;
  const void* pos;           // [max_pos, W] or null
  int max_pos;
  float norm_alpha;
  const void* norm_w;        // or null
  const void* norm_b;
  uint32_t* status;
};

struct MbRopeDimsArgs {
  int M, Hq, Hkv, dk, dv, rot, dkp, dvp, f32;
  const void* qkv;
  long long qkv_ld;
  const int* positions;
  const long long* slots;
  const float* cos_tab;
  const float* sin_tab;
  int max_pos;
  void* q_out;
  void* k_cache;
  void* v_cache;
  long long num_slots;
  uint32_t* status;
  const void* q_norm;        // [dk] per-head RMS norm weights, or null
  const void* k_norm;
  float eps;
};

extern "C" {

int mb_stream_norm(const MbStreamNormArgs* a, cudaStream_t stream) {
  if (!a || a->T <= 0 || a->W <= 0 || !a->x) return MB_ERR_BAD_ARG;
  if (a->add_mode != ADD_NONE && (!a->y || !a->post_w || (a->add_mode == ADD_DYT && !a->post_b))) return MB_ERR_BAD_ARG;
  if (a->out_mode == OUT_DYT && (!a->pre_w || !a->pre_b)) return MB_ERR_BAD_ARG;
  if (a->mu && (!a->mixes || !a->state || !a->q_start || !a->q_len || !a->positions || !a->slots || a->num_seqs <= 0 || a->out_mode != OUT_DYT ||
                a->x_out == a->x))
    return MB_ERR_BAD_ARG;
  StreamParams p{};
  p.T = a->T; p.W = a->W; p.x = a->x; p.y = a->y; p.add_mode = a->add_mode; p.out_mode = a->out_mode;
  p.post = DytW{a->post_alpha, (const bf16*)a->post_w, (const bf16*)a->post_b};
  p.pre = DytW{a->pre_alpha, (const bf16*)a->pre_w, (const bf16*)a->pre_b};
  p.eps = a->eps; p.x_out = a->x_out; p.out = a->out; p.h32 = a->h32;
  p.mu = (const bf16*)a->mu; p.mixes = a->mixes; p.state = a->state;
  p.q_start = a->q_start; p.q_len = a->q_len; p.positions = a->positions; p.slots = a->slots;
  p.num_seqs = a->num_seqs; p.num_slots = a->num_slots; p.write_state = a->write_state; p.status = a->status;
  const bool v4 = a->W % 4 == 0 && al(a->x, 16) && al(a->y, 16) && al(a->x_out, 16) && al(a->out, 16) && al(a->h32, 16) && al(a->mixes, 16) &&
                  al(a->state, 16) && al(a->post_w, 8) && al(a->post_b, 8) && al(a->pre_w, 8) && al(a->pre_b, 8) && al(a->mu, 8);
  const dim3 g(a->T), b(row_threads(a->W, v4 ? 4 : 1));
  if (a->f32) return (int)(v4 ? mb::launch_kernel(stream_norm_kernel<4, float>, g, b, 0, stream, p) : mb::launch_kernel(stream_norm_kernel<1, float>, g, b, 0, stream, p));
  return (int)(v4 ? mb::launch_kernel(stream_norm_kernel<4, bf16>, g, b, 0, stream, p) : mb::launch_kernel(stream_norm_kernel<1, bf16>, g, b, 0, stream, p));
}

int mb_stream_rms(const MbStreamRmsArgs* a, cudaStream_t stream) {
  if (!a || a->T <= 0 || a->W <= 0 || !a->x || (a->out_mode != RMS_NONE && !a->out) || (a->out_mode == RMS_NORM && !a->w)) return MB_ERR_BAD_ARG;
  if (a->ye && (!a->pair_row || !a->pair_w || a->K <= 0 || a->K > 32 || a->ye_ld < a->W)) return MB_ERR_BAD_ARG;
  const StreamRmsParams p{a->W, a->x, a->y, a->ye, a->ye_ld, a->pair_row, a->pair_w, a->K, a->out_mode, (const bf16*)a->w, a->eps, a->x_out, a->out, a->out_ld,
                          a->plus_one ? 1.f : 0.f, a->scale};
  const bool v4 = a->W % 4 == 0 && a->out_ld % 4 == 0 && a->ye_ld % 4 == 0 && al(a->x, 16) && al(a->y, 16) && al(a->ye, 16) && al(a->x_out, 16) &&
                  al(a->out, a->f32 ? 16 : 8) && al(a->w, 8);
  const int vec = v4 ? 4 : 1, nt = max(row_threads(a->W, vec), 32), nit = (a->W + nt * vec - 1) / (nt * vec);
  const dim3 g(a->T), b(nt);
#define MB_RMS(V, N)                                                                                                   \
  return a->f32 ? (int)mb::launch_kernel(stream_rms_kernel<V, N, float>, g, b, 0, stream, p)                           \
                : (int)mb::launch_kernel(stream_rms_kernel<V, N, bf16>, g, b, 0, stream, p)
  if (v4) {
    if (nit <= 1) MB_RMS(4, 1);
    if (nit <= 3) MB_RMS(4, 3);
    if (nit <= 8) MB_RMS(4, 8);
    if (nit <= 16) MB_RMS(4, 16);
  } else {
    if (nit <= 4) MB_RMS(1, 4);
    if (nit <= 16) MB_RMS(1, 16);
    if (nit <= 64) MB_RMS(1, 64);
  }
#undef MB_RMS
  return MB_ERR_TOO_LARGE;
}

int mb_shift_commit(const float* h32, int W, float* state, const int* q_start, const int* q_len, const int* slots, int num_seqs, int num_slots,
                    uint32_t* status, cudaStream_t stream) {
  if (!h32 || !state || W <= 0 || num_seqs <= 0) return MB_ERR_BAD_ARG;
  return (int)mb::launch_kernel(shift_commit_kernel, dim3(num_seqs), dim3(256), 0, stream, h32, W, state, q_start, q_len, slots, num_slots, status);
}

int mb_gated_norm(const MbGatedNormArgs* a, cudaStream_t stream) {
  if (!a || a->T <= 0 || a->K <= 0 || a->group <= 0 || a->K % a->group || !a->x || !a->w || !a->gate || !a->out) return MB_ERR_BAD_ARG;
  GatedParams p{a->T, a->K, a->group, a->x, (const bf16*)a->w, a->gate, a->gate_ld, a->sigmoid_gate, a->eps, a->scale, a->out, a->out_ld};
  const size_t es = a->f32 ? 4 : 2;
  const bool v4 = a->group % 4 == 0 && a->gate_ld % 4 == 0 && a->out_ld % 4 == 0 && al(a->x, 16) && al(a->w, 8) && al(a->gate, 4 * es) && al(a->out, 4 * es);
  const dim3 g(a->T), b(row_threads(a->K, v4 ? 4 : 1));
  if (a->f32) return (int)(v4 ? mb::launch_kernel(gated_norm_kernel<4, float>, g, b, 0, stream, p) : mb::launch_kernel(gated_norm_kernel<1, float>, g, b, 0, stream, p));
  return (int)(v4 ? mb::launch_kernel(gated_norm_kernel<4, bf16>, g, b, 0, stream, p) : mb::launch_kernel(gated_norm_kernel<1, bf16>, g, b, 0, stream, p));
}

int mb_side_gate(const float* z, const int* tokens, const void* table, long long table_ld, int off, int dim, int rows, int num_rows, void* out,
                 int f32, uint32_t* status, cudaStream_t stream) {
  if (!z || !tokens || !table || !out || rows <= 0 || dim <= 0 || off < 0 || off + dim > table_ld) return MB_ERR_BAD_ARG;
  if ((long long)rows * dim > (1ll << 31)) return MB_ERR_TOO_LARGE;
  const bool v4 = dim % 4 == 0 && off % 4 == 0 && table_ld % 4 == 0 && al(table, 8) && al(z, 16) && al(out, 16);
  const long long n = (long long)rows * dim / (v4 ? 4 : 1);
  const dim3 g((unsigned)((n + 255) / 256)), b(256);
  const bf16* tb = (const bf16*)table;
  if (f32) return (int)(v4 ? mb::launch_kernel(side_gate_kernel<4, float>, g, b, 0, stream, z, tokens, tb, table_ld, off, dim, rows, num_rows, (float*)out, status)
                           : mb::launch_kernel(side_gate_kernel<1, float>, g, b, 0, stream, z, tokens, tb, table_ld, off, dim, rows, num_rows, (float*)out, status));
  return (int)(v4 ? mb::launch_kernel(side_gate_kernel<4, bf16>, g, b, 0, stream, z, tokens, tb, table_ld, off, dim, rows, num_rows, (bf16*)out, status)
                  : mb::launch_kernel(side_gate_kernel<1, bf16>, g, b, 0, stream, z, tokens, tb, table_ld, off, dim, rows, num_rows, (bf16*)out, status));
}

int mb_embed_scaled(const MbEmbedArgs* a, cudaStream_t stream) {
  if (!a || !a->tokens || !a->table || !a->out || a->M <= 0 || a->W <= 0 || (a->copy && a->copy_ld < a->W)) return MB_ERR_BAD_ARG;
  if ((a->pos && (!a->positions || a->max_pos <= 0)) || (a->norm_w && !a->norm_b)) return MB_ERR_BAD_ARG;
  const EmbedParams p{a->tokens, (const bf16*)a->table, a->out, a->W, a->vocab, a->scale, a->copy, a->copy_ld, a->positions, (const bf16*)a->pos,
                      a->max_pos, DytW{a->norm_alpha, (const bf16*)a->norm_w, (const bf16*)a->norm_b}, a->status};
  const bool v4 = a->W % 4 == 0 && al(a->table, 8) && al(a->out, 16) && a->copy_ld % 4 == 0 && al(a->copy, 16) && al(a->pos, 8) &&
                  al(a->norm_w, 8) && al(a->norm_b, 8);
  const dim3 g(a->M), b(row_threads(a->W, v4 ? 4 : 1));
  if (a->copy_f32) return (int)(v4 ? mb::launch_kernel(embed_scaled_kernel<4, float>, g, b, 0, stream, p) : mb::launch_kernel(embed_scaled_kernel<1, float>, g, b, 0, stream, p));
  return (int)(v4 ? mb::launch_kernel(embed_scaled_kernel<4, bf16>, g, b, 0, stream, p) : mb::launch_kernel(embed_scaled_kernel<1, bf16>, g, b, 0, stream, p));
}

// z [T, R] (fp32, or bf16), rows z_ld elements apart
int mb_tanh_split_cols(const void* z, long long z_ld, int z_bf16, void* out, int T, int R, cudaStream_t stream) {
  if (!z || !out || T <= 0 || R <= 0 || z_ld < R) return MB_ERR_BAD_ARG;
  const long long total = (long long)T * R;
  const dim3 g((unsigned)((total + 255) / 256)), b(256);
  return (int)(z_bf16 ? mb::launch_kernel(tanh_split_kernel<bf16>, g, b, 0, stream, (const bf16*)z, z_ld, (bf16*)out, total, R)
                      : mb::launch_kernel(tanh_split_kernel<float>, g, b, 0, stream, (const float*)z, z_ld, (bf16*)out, total, R));
}

int mb_tanh_split(const float* z, void* out, int T, int R, cudaStream_t stream) { return mb_tanh_split_cols(z, R, 0, out, T, R, stream); }

int mb_rope_dims(const MbRopeDimsArgs* a, cudaStream_t stream) {
  if (!a || a->M <= 0 || !a->qkv || !a->positions || !a->slots || !a->q_out || !a->k_cache || !a->v_cache) return MB_ERR_BAD_ARG;
  if (a->dk <= 0 || a->dv <= 0 || a->dk > a->dkp || a->dv > a->dvp || a->rot < 0 || a->rot > a->dk || a->rot % 2) return MB_ERR_UNSUPPORTED;
  if (a->rot > 0 && (!a->cos_tab || !a->sin_tab)) return MB_ERR_BAD_ARG;
  RopeDimsParams p{a->M, a->Hq, a->Hkv, a->dk, a->dv, a->rot, a->dkp, a->dvp, a->qkv, a->qkv_ld, a->positions, a->slots, a->cos_tab,
                   a->sin_tab, a->max_pos, a->q_out, a->k_cache, a->v_cache, a->num_slots, a->status, (const bf16*)a->q_norm, (const bf16*)a->k_norm, a->eps};
  const bool v4 = a->dk % 4 == 0 && a->dv % 4 == 0 && a->rot % 8 == 0 && a->dkp % 4 == 0 && a->dvp % 4 == 0 && a->qkv_ld % 4 == 0 &&
                  al(a->qkv, 16) && al(a->q_out, 16) && al(a->k_cache, 16) && al(a->v_cache, 16) && al(a->q_norm, 8) && al(a->k_norm, 8);
  if (a->q_norm || a->k_norm) {
    const dim3 g(a->M, (a->Hq + 2 * a->Hkv + 7) / 8), b(256);
    if (a->f32) return (int)(v4 ? mb::launch_kernel(rope_heads_kernel<4, float>, g, b, 0, stream, p) : mb::launch_kernel(rope_heads_kernel<1, float>, g, b, 0, stream, p));
    return (int)(v4 ? mb::launch_kernel(rope_heads_kernel<4, bf16>, g, b, 0, stream, p) : mb::launch_kernel(rope_heads_kernel<1, bf16>, g, b, 0, stream, p));
  }
  const int total = (a->Hq + a->Hkv) * a->dkp + a->Hkv * a->dvp;
  const int vec = v4 ? 4 : 1;
  const int want = (total + 256 * vec - 1) / (256 * vec);
  const dim3 g(a->M, a->M >= 2048 ? 1 : (want < 8 ? want : 8)), b(256);
  if (a->f32) return (int)(v4 ? mb::launch_kernel(rope_dims_kernel<4, float>, g, b, 0, stream, p) : mb::launch_kernel(rope_dims_kernel<1, float>, g, b, 0, stream, p));
  return (int)(v4 ? mb::launch_kernel(rope_dims_kernel<4, bf16>, g, b, 0, stream, p) : mb::launch_kernel(rope_dims_kernel<1, bf16>, g, b, 0, stream, p));
}

}  // extern "C"
