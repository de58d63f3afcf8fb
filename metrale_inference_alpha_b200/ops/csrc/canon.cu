// Short causal convolutions over time with a carried window, one filter per channel.
//
//   stream_canon   one pass between two sublayers of models that norm a sublayer's output and convolve its input: the
//                  pending output (a row, the weighted sum of a token's expert rows, or both) joins the fp32 stream
//                  through its RMS norm, x' = x + rms(y) w (or 1 + w), and the next sublayer's input is
//                  h_t = x'_t + sum_j f_j x'_(t - taps + 1 + j), zero in front of the sequence. Without a filter only x'.
//   canon_commit   state := the last taps - 1 rows of (state | x' of the accepted rows), after speculative verification
//   short_conv     the same convolution of a projection's columns, through SiLU instead of the residual
//
// A CTA of stream_canon owns up to kRun consecutive tokens of one sequence. It recomputes x' of the taps - 1 rows in front
// of them, so that no row waits for another CTA; rows in front of the portion come from the carried window. The CTA of a
// portion's first rows is the only reader of the window, and it alone writes the new one (recomputing the portion's last
// rows where they are not its own). All rows of a CTA live in shared memory: their sums of squares are taken by whole
// warps side by side, then every thread walks its own channels over the rows.
// Long portions take two launches instead, a join of whole rows and the convolution below over x'.
// short_conv follows the same rule with runs of tokens per thread. Windows are rows of a slot pool, win_ld floats from slot
// to slot, oldest row first.
#include "epilogue.cuh"
#include "row_io.cuh"

namespace {

constexpr int kRun = 8;            // tokens of a run, at most
constexpr int kMaxRows = 40;       // rows of a CTA: the run and the window
constexpr int kLongPortion = 96;   // portions this long take the join and the convolution as two launches

struct Window {
  float* base;                     // [slots, win_ld]: taps - 1 rows
  long long ld;
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_slots, write;
  uint32_t* status;
};

struct CanonParams {
  int T, W, taps, run;
  const float* x;
  const void* y;                   // [T, W] or null
  const float* ye;                 // expert rows, or null
  long long ye_ld;
  const int* pair_row;             // [T, K] rows of ye, -1 = none
  const float* pair_w;
  int K;
  const bf16* norm_w;              // null: nothing pending
  float plus, eps;                 // the norm's weight is plus + norm_w
  float* x_out;
  const bf16* filt;                // [taps, W], or null: only x_out
  void* out;
  Window win;
};

template <int VEC, typename T>
__global__ void __launch_bounds__(512) stream_canon_kernel(const CanonParams p) {
  extern __shared__ __align__(16) float rows[];          // [rows][W]
  __shared__ float red[kMaxRows][16];
  const int seq = blockIdx.y, tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, nw = nt >> 5, W = p.W;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.filt ? p.win.q_len[seq] : p.T;
  const int l0 = blockIdx.x * p.run;
  if (l0 >= n) return;
  const int q0 = p.filt ? p.win.q_start[seq] : 0;
  const int halo = p.filt ? p.taps - 1 : 0;
  float* win = nullptr;
  bool fresh = true;
  if (p.filt) {
    const int slot = p.win.slots[seq];
    fresh = p.win.positions[q0] == 0;
    if (slot < 0 || slot >= p.win.num_slots) {
      if (p.win.status && tid == 0) atomicCAS(p.win.status, 0u, MB_ST_BOUNDS);
      fresh = true;
    } else if (halo > 0) {
      win = p.win.base + (size_t)slot * p.win.ld;
    }
  }
  const T* y = reinterpret_cast<const T*>(p.y);
  // x' of the portion's rows first .. first + cnt - 1 into shared rows at, at + 1, ...; those from `own` on go to x_out
  auto join = [&](int first, int cnt, int at, int own) {
    const bool pend = p.norm_w != nullptr;
    const int wpr = cnt >= nw ? 1 : nw / cnt;            // warps side by side on a row
    if (pend) {
      for (int g = warp; g < cnt * wpr; g += nw) {
        const int r = g / wpr, part = g - r * wpr;
        const size_t t = (size_t)(q0 + first + r);
        float* dst = rows + (size_t)(at + r) * W;
        float ss = 0.f;
#pragma unroll 2
        for (int k = (part * 32 + lane) * VEC; k < W; k += wpr * 32 * VEC) {
          float v[VEC];
#pragma unroll
          for (int i = 0; i < VEC; ++i) v[i] = 0.f;
          if (y) ldn<VEC>(y + t * W + k, v);
          if (p.ye) {
            for (int j = 0; j < p.K; ++j) {
              const int row = p.pair_row[t * p.K + j];
              if (row < 0) continue;
              const float pw = p.pair_w[t * p.K + j];
              float a[VEC];
              ldn<VEC>(p.ye + (size_t)row * p.ye_ld + k, a);
#pragma unroll
              for (int i = 0; i < VEC; ++i) v[i] = fmaf(pw, a[i], v[i]);
            }
          }
#pragma unroll
          for (int i = 0; i < VEC; ++i) ss = fmaf(v[i], v[i], ss);
          stn<VEC>(dst + k, v);
        }
        ss = mb::warp_sum(ss);
        if (lane == 0) red[at + r][part] = ss;
      }
      __syncthreads();
    }
    for (int r = 0; r < cnt; ++r) {
      float inv = 0.f;
      if (pend) {
        for (int i = 0; i < wpr; ++i) inv += red[at + r][i];
        inv = 1.f / sqrtf(inv / (float)W + p.eps);
      }
      const size_t t = (size_t)(q0 + first + r);
      float* row = rows + (size_t)(at + r) * W;
      for (int k = tid * VEC; k < W; k += nt * VEC) {
        float x[VEC];
        ldn<VEC>(p.x + t * W + k, x);
        if (pend) {
          float v[VEC], w[VEC];
          ldn<VEC>(row + k, v);
          ldn<VEC>(p.norm_w + k, w);
#pragma unroll
          for (int i = 0; i < VEC; ++i) x[i] = fmaf(v[i] * inv, p.plus + w[i], x[i]);
          if (p.x_out && first + r >= own) stn<VEC>(p.x_out + t * W + k, x);
        }
        if (p.filt) stn<VEC>(row + k, x);
      }
    }
  };
  const int own = min(p.run, n - l0);
  const int from = max(0, l0 - halo), before = halo - (l0 - from);      // rows of the window that come from the state
  join(from, l0 - from + own, before, l0);
  if (!p.filt) return;
  // from here on every thread stays with its own channels
  for (int k = tid * VEC; k < W; k += nt * VEC) {
    for (int r = 0; r < before; ++r) {
      float v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      if (win && !fresh) ldn<VEC>(win + (size_t)(l0 + r) * W + k, v);    // l0 < halo here: row l0 + r of the window
      stn<VEC>(rows + (size_t)r * W + k, v);
    }
    for (int t = 0; t < own; ++t) {
      float h[VEC];
      ldn<VEC>(rows + (size_t)(halo + t) * W + k, h);
      for (int j = 0; j < p.taps; ++j) {
        float v[VEC], f[VEC];
        ldn<VEC>(rows + (size_t)(t + j) * W + k, v);
        ldn<VEC>(p.filt + (size_t)j * W + k, f);
#pragma unroll
        for (int i = 0; i < VEC; ++i) h[i] = fmaf(f[i], v[i], h[i]);
      }
      stn<VEC>(reinterpret_cast<T*>(p.out) + (size_t)(q0 + l0 + t) * W + k, h);
    }
  }
  if (blockIdx.x != 0 || !win || !p.win.write) return;
  int at = own;                                          // the portion's last `halo` rows end here: rows at .. at + halo - 1
  if (n > own) {
    __syncthreads();
    join(n - halo, halo, 0, n);
    at = 0;
  }
  for (int k = tid * VEC; k < W; k += nt * VEC)
    for (int r = 0; r < halo; ++r) {
      float v[VEC];
      ldn<VEC>(rows + (size_t)(at + r) * W + k, v);
      stn<VEC>(win + (size_t)r * W + k, v);
    }
}

// state := the last taps - 1 rows of (state | the sequence's rows of x)
template <int VEC>
__global__ void __launch_bounds__(256) canon_commit_kernel(const float* x, int W, int halo, const Window win) {
  const int seq = blockIdx.x, n = win.q_len[seq];
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  if (n <= 0) return;
  const int slot = win.slots[seq], q0 = win.q_start[seq];
  if (slot < 0 || slot >= win.num_slots) {
    if (win.status && threadIdx.x == 0) atomicCAS(win.status, 0u, MB_ST_BOUNDS);
    return;
  }
  float* st = win.base + (size_t)slot * win.ld;
  const bool fresh = win.positions[q0] == 0;
  for (int k = threadIdx.x * VEC; k < W; k += blockDim.x * VEC)
    for (int r = 0; r < halo; ++r) {                     // row r comes from row r + n of the old window: read before it is written
      const int l = n - halo + r;
      float v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      if (l >= 0) ldn<VEC>(x + (size_t)(q0 + l) * W + k, v);
      else if (!fresh) ldn<VEC>(st + (size_t)(halo + l) * W + k, v);
      stn<VEC>(st + (size_t)r * W + k, v);
    }
}

// Long portions: x' alone, a CTA per row with the row in registers; the convolution then reads x' from L2.
template <int VEC, int NIT, typename T>
__global__ void __launch_bounds__(256) stream_join_kernel(const CanonParams p) {
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
  float v[NIT][VEC], x[NIT][VEC], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NIT; ++i) {
    const int k = (i * nt + tid) * VEC;
    if (k >= W) continue;
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[i][e] = 0.f;
    if (p.y) ldn<VEC>(reinterpret_cast<const T*>(p.y) + (size_t)t * W + k, v[i]);
    ldn<VEC>(p.x + (size_t)t * W + k, x[i]);
    if (p.ye) {
      for (int j = 0; j < p.K; ++j) {
        if (s_row[j] < 0) continue;
        float a[VEC];
        ldn<VEC>(p.ye + (size_t)s_row[j] * p.ye_ld + k, a);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[i][e] = fmaf(s_w[j], a[e], v[i][e]);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(v[i][e], v[i][e], ss);
  }
  const float inv = 1.f / sqrtf(mb::block_sum(ss, red) / (float)W + p.eps);
#pragma unroll
  for (int i = 0; i < NIT; ++i) {
    const int k = (i * nt + tid) * VEC;
    if (k >= W) continue;
    float w[VEC];
    ldn<VEC>(p.norm_w + k, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[i][e] = fmaf(v[i][e] * inv, p.plus + w[e], x[i][e]);
    stn<VEC>(p.x_out + (size_t)t * W + k, x[i]);
  }
}

// ------------------------------------------------------------------ columns of a matrix
constexpr int kConvRun = 16;       // tokens of a thread

struct ShortConvParams {
  int C, taps, write_out;
  const void* x;
  long long x_ld;
  const void* filt;                // [taps, C]
  void* out;                       // [T, C]
  Window win;                      // rows of C floats
};

// TI, TF, TO: inputs, filter, output. TAPS > 0: that many, kept in registers; 0: any number, inputs read again. SILU: through
// SiLU, else the convolution is added to its input.
template <int VEC, int TAPS, bool SILU, typename TI, typename TF, typename TO>
__global__ void __launch_bounds__(128) short_conv_kernel(const ShortConvParams p) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * VEC, seq = blockIdx.z, l0 = blockIdx.y * kConvRun;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.win.q_len[seq];
  if (c >= p.C || l0 >= n) return;
  const int q0 = p.win.q_start[seq], slot = p.win.slots[seq], halo = p.taps - 1;
  if (slot < 0 || slot >= p.win.num_slots) {
    if (p.win.status) atomicCAS(p.win.status, 0u, MB_ST_BOUNDS);
    return;
  }
  float* st = p.win.base + (size_t)slot * p.win.ld + c;
  const bool fresh = p.win.positions[q0] == 0;
  const TI* x = reinterpret_cast<const TI*>(p.x) + (size_t)q0 * p.x_ld + c;
  const TF* filt = reinterpret_cast<const TF*>(p.filt) + c;
  auto input = [&](int l, float* v) {
    if (l >= 0) {
      ldn<VEC>(x + (size_t)l * p.x_ld, v);
    } else if (!fresh) {
      ldn<VEC>(st + (size_t)(halo + l) * p.C, v);
    } else {
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
    }
  };
  auto emit = [&](int l, const float* conv, const float* in) {
    float a[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) a[i] = !SILU ? conv[i] + in[i] : sizeof(TO) == 2 ? mb::silu(conv[i]) : mb::silu_exact(conv[i]);
    stn<VEC>(reinterpret_cast<TO*>(p.out) + (size_t)(q0 + l) * p.C + c, a);
  };
  if (p.write_out) {
    const int l1 = min(n, l0 + kConvRun);
    if constexpr (TAPS > 0) {
      float f[TAPS][VEC], w[TAPS][VEC];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        ldn<VEC>(filt + (size_t)j * p.C, f[j]);
        if (j + 1 < TAPS) input(l0 - TAPS + 1 + j, w[j]);
      }
      // four tokens' inputs are on their way at a time
      for (int lb = l0; lb < l1; lb += 4) {
        float nx[4][VEC];
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (lb + u < l1) ldn<VEC>(x + (size_t)(lb + u) * p.x_ld, nx[u]);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          if (lb + u >= l1) break;
          float a[VEC];
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            w[TAPS - 1][i] = nx[u][i];
            a[i] = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) a[i] = fmaf(f[j][i], w[j][i], a[i]);
#pragma unroll
            for (int j = 0; j + 1 < TAPS; ++j) w[j][i] = w[j + 1][i];
          }
          emit(lb + u, a, nx[u]);
        }
      }
    } else {
      for (int l = l0; l < l1; ++l) {
        float a[VEC], v[VEC], f[VEC];
#pragma unroll
        for (int i = 0; i < VEC; ++i) a[i] = 0.f;
        for (int j = 0; j < p.taps; ++j) {                 // ends with the token's own input in v
          input(l - halo + j, v);
          ldn<VEC>(filt + (size_t)j * p.C, f);
#pragma unroll
          for (int i = 0; i < VEC; ++i) a[i] = fmaf(f[i], v[i], a[i]);
        }
        emit(l, a, v);
      }
    }
  }
  if (l0 != 0 || !p.win.write) return;                   // the first run alone reads the window, and writes the new one
  for (int r = 0; r < halo; ++r) {
    float v[VEC];
    input(n - halo + r, v);
    stn<VEC>(st + (size_t)r * p.C, v);
  }
}

template <int VEC, bool SILU, typename TI, typename TF, typename TO>
int launch_conv(const ShortConvParams& p, int max_q_len, int num_seqs, cudaStream_t stream) {
  const int runs = p.write_out ? (max_q_len + kConvRun - 1) / kConvRun : 1;
  if (runs > 65535) return MB_ERR_TOO_LARGE;
  const dim3 g((p.C + 128 * VEC - 1) / (128 * VEC), runs, num_seqs), b(128);
  switch (p.taps) {
    case 2: return (int)mb::launch_kernel(short_conv_kernel<VEC, 2, SILU, TI, TF, TO>, g, b, 0, stream, p);
    case 3: return (int)mb::launch_kernel(short_conv_kernel<VEC, 3, SILU, TI, TF, TO>, g, b, 0, stream, p);
    case 4: return (int)mb::launch_kernel(short_conv_kernel<VEC, 4, SILU, TI, TF, TO>, g, b, 0, stream, p);
    default: return (int)mb::launch_kernel(short_conv_kernel<VEC, 0, SILU, TI, TF, TO>, g, b, 0, stream, p);
  }
}

}  // namespace

struct MbWindowArgs {
  void* base;                // [slots, ld] fp32, or null
  long long ld;
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_seqs, num_slots, max_q_len, write;
  uint32_t* status;
};

struct MbStreamCanonArgs {
  int T, W, taps, f32, K, plus_one;
  const float* x;
  const void* y;
  const float* ye;
  long long ye_ld;
  const int* pair_row;
  const float* pair_w;
  const void* norm_w;        // or null: nothing pending
  float eps;
  float* x_out;
  const void* filt;          // [taps, W] bf16, or null: only x_out
  void* out;
  MbWindowArgs win;
};

struct MbShortConvArgs {
  int C, taps, f32, write_out;
  const void* x;
  long long x_ld;
  const float* filt;
  void* out;
  MbWindowArgs win;
};

namespace {
Window window_of(const MbWindowArgs& w) {
  return Window{(float*)w.base, w.ld, w.q_start, w.q_len, w.positions, w.slots, w.num_slots, w.write, w.status};
}
bool window_ok(const MbWindowArgs& w, int taps, long long row) {
  return w.q_start && w.q_len && w.positions && w.slots && w.num_seqs > 0 && w.num_seqs <= 65535 && w.max_q_len > 0 && taps > 0 &&
         (taps == 1 || (w.base && w.ld >= (taps - 1) * row));
}

template <int VEC, typename T>
int launch_canon(const CanonParams& p, dim3 grid, int threads, size_t smem, cudaStream_t stream) {
  auto kern = stream_canon_kernel<VEC, T>;
  static size_t configured = 0;
  if (smem > configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return (int)mb::launch_kernel(kern, grid, dim3(threads), smem, stream, p);
}

template <typename T>
int join_rows(const CanonParams& p, bool v4, int nit, int threads, cudaStream_t stream) {
  const dim3 g(p.T), b(threads);
  if (p.K > 32) return MB_ERR_TOO_LARGE;
#define MB_JOIN(V, N) return (int)mb::launch_kernel(stream_join_kernel<V, N, T>, g, b, 0, stream, p)
  if (v4) {
    if (nit <= 1) MB_JOIN(4, 1);
    if (nit <= 3) MB_JOIN(4, 3);
    if (nit <= 8) MB_JOIN(4, 8);
    MB_JOIN(4, 16);
  }
  if (nit <= 4) MB_JOIN(1, 4);
  MB_JOIN(1, 16);
#undef MB_JOIN
}
}  // namespace

extern "C" {

int mb_stream_canon(const MbStreamCanonArgs* a, cudaStream_t stream) {
  if (!a || a->T <= 0 || a->W <= 0 || !a->x || (!a->filt && !a->x_out) || (a->filt && !a->out)) return MB_ERR_BAD_ARG;
  if (a->norm_w && ((!a->y && !a->ye) || !a->x_out || a->x_out == a->x)) return MB_ERR_BAD_ARG;   // neighbours are read again
  if (!a->norm_w && !a->filt) return MB_ERR_BAD_ARG;
  if (a->ye && (!a->pair_row || !a->pair_w || a->K <= 0 || a->ye_ld < a->W)) return MB_ERR_BAD_ARG;
  if (a->filt && !window_ok(a->win, a->taps, a->W)) return MB_ERR_BAD_ARG;
  const int halo = a->filt ? a->taps - 1 : 0, longest = a->filt ? a->win.max_q_len : a->T;
  if (halo > kMaxRows / 2) return MB_ERR_TOO_LARGE;
  // a run is no shorter than the window (so that the portion's first run alone needs the carried one) and its rows fit
  const size_t row = (size_t)a->W * sizeof(float);
  int run = kRun;
  while (run > 1 && (run + halo) * row > (size_t)104 * 1024) --run;
  if (run > longest) run = longest;
  if (run < halo && run < longest) run = halo < longest ? halo : longest;
  const size_t smem = (size_t)(run + halo) * row;
  if (smem > (size_t)220 * 1024) return MB_ERR_TOO_LARGE;
  const CanonParams p{a->T, a->W, a->taps, run, a->x, a->y, a->ye, a->ye_ld, a->pair_row, a->pair_w, a->K, (const bf16*)a->norm_w,
                      a->plus_one ? 1.f : 0.f, a->eps, a->x_out, (const bf16*)a->filt, a->out, window_of(a->win)};
  const bool v4 = a->W % 4 == 0 && a->ye_ld % 4 == 0 && a->win.ld % 4 == 0 && al(a->x, 16) && al(a->y, 16) && al(a->ye, 16) && al(a->norm_w, 8) &&
                  al(a->x_out, 16) && al(a->filt, 8) && al(a->out, 16) && al(a->win.base, 16);
  // long portions: the join by itself, then the convolution over x' (nothing is recomputed, and rows need no shared memory)
  if (a->filt && halo <= kConvRun && longest >= kLongPortion) {
    const int vec = v4 ? 4 : 1, nt = row_threads(a->W, vec), nit = (a->W + nt * vec - 1) / (nt * vec);
    if (nit <= 16) {
      if (a->norm_w) {
        const int rc = a->f32 ? join_rows<float>(p, v4, nit, nt, stream) : join_rows<bf16>(p, v4, nit, nt, stream);
        if (rc != 0) return rc;
      }
      const ShortConvParams c{a->W, a->taps, 1, a->norm_w ? a->x_out : a->x, a->W, a->filt, a->out, p.win};
      const int S = a->win.num_seqs;
      if (a->f32) return v4 ? launch_conv<4, false, float, bf16, float>(c, longest, S, stream) : launch_conv<1, false, float, bf16, float>(c, longest, S, stream);
      return v4 ? launch_conv<4, false, float, bf16, bf16>(c, longest, S, stream) : launch_conv<1, false, float, bf16, bf16>(c, longest, S, stream);
    }
  }
  const int threads = a->W >= 1024 ? 512 : 256;
  const dim3 grid((longest + run - 1) / run, a->filt ? a->win.num_seqs : 1);
  if (a->f32) return v4 ? launch_canon<4, float>(p, grid, threads, smem, stream) : launch_canon<1, float>(p, grid, threads, smem, stream);
  return v4 ? launch_canon<4, bf16>(p, grid, threads, smem, stream) : launch_canon<1, bf16>(p, grid, threads, smem, stream);
}

int mb_canon_commit(const float* x, int W, int taps, const MbWindowArgs* w, cudaStream_t stream) {
  if (!x || !w || W <= 0 || taps < 2 || !window_ok(*w, taps, W)) return MB_ERR_BAD_ARG;
  const bool v4 = W % 4 == 0 && w->ld % 4 == 0 && al(x, 16) && al(w->base, 16);
  const dim3 g(w->num_seqs), b(256);
  return (int)(v4 ? mb::launch_kernel(canon_commit_kernel<4>, g, b, 0, stream, x, W, taps - 1, window_of(*w))
                  : mb::launch_kernel(canon_commit_kernel<1>, g, b, 0, stream, x, W, taps - 1, window_of(*w)));
}

int mb_short_conv(const MbShortConvArgs* a, cudaStream_t stream) {
  if (!a || a->C <= 0 || !a->x || !a->filt || (a->write_out && !a->out) || !window_ok(a->win, a->taps, a->C)) return MB_ERR_BAD_ARG;
  if (a->taps - 1 > kConvRun) return MB_ERR_TOO_LARGE;
  const ShortConvParams p{a->C, a->taps, a->write_out, a->x, a->x_ld, a->filt, a->out, window_of(a->win)};
  const size_t es = a->f32 ? 16 : 8;
  const bool v4 = a->C % 4 == 0 && a->x_ld % 4 == 0 && a->win.ld % 4 == 0 && al(a->x, es) && al(a->filt, 16) && al(a->out, es) && al(a->win.base, 16);
  const int mq = a->win.max_q_len, S = a->win.num_seqs;
  if (a->f32) return v4 ? launch_conv<4, true, float, float, float>(p, mq, S, stream) : launch_conv<1, true, float, float, float>(p, mq, S, stream);
  return v4 ? launch_conv<4, true, bf16, float, bf16>(p, mq, S, stream) : launch_conv<1, true, bf16, float, bf16>(p, mq, S, stream);
}

}  // extern "C"
