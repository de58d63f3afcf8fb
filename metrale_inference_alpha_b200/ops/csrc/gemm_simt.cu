// GEMM on the CUDA cores, fp32 accumulation with plain FMAs: out[m, n] = sum_k a(X[m, k]) W[n, k].
//
// Two kinds of caller need it next to the tensor-core GEMM:
//   * models served in true 32-bit (fp32 activations and weights; no tensor-core mode keeps 24 bits);
//   * products whose operands stay 32-bit in an otherwise bf16 model (low-rank decay projections of a
//     recurrence), and bf16 layers whose row length is not a multiple of 16 bytes, which no tensor map
//     can describe.
// X is fp32 or bf16, W fp32 or bf16, out fp32 or bf16, any M, N, K and row strides.
// Operand function a(): identity or tanh. Epilogues (shared numbering with the tensor-core GEMM):
//   plain; SwiGLU, tanh-GELU GLU and clamped GLU on interleaved (gate, up) rows; SiLU on the first epi_n columns;
//   y + bias; -exp(y + bias), the logarithm of a decay exp(-exp(.)); epi_a log(sigmoid(y + bias)), that of a
//   decay sigmoid(.)^epi_a; epi_a sigmoid(y + bias), that of a decay bounded below; relu(y)^2.
// Grouped mode: a work list of (expert, first row, rows) tiles over rows sorted by expert, weights stacked
// [experts * n_per_expert, K]; the rows may be read through an index (row r = X[row_index[r] / row_div]).
// A CTA owns 64 x 64 outputs (64 x 16 when M <= 16), 256 threads, k steps of 16 through shared memory,
// the next step's operands fetched into registers while the current one is consumed.
#include "common.cuh"
#include "epilogue.cuh"

namespace {

struct SimtParams {
  int M, N, K;
  const void* X;
  long long ldx;
  const void* W;
  long long ldw;
  void* out;
  long long ldo;
  int a_op, epilogue;
  const float* bias;
  float epi_a, epi_b;
  int epi_n;
  const int* tile_expert;      // grouped mode, else null
  const int* tile_row0;
  const int* tile_nrows;
  const int* row_index;        // or null: rows as they are
  int row_div;
};

template <typename T>
__device__ __forceinline__ float ld1(const T* p) {
  if constexpr (sizeof(T) == 2) return __bfloat162float(*p);
  else return *p;
}
template <typename T>
__device__ __forceinline__ void st1(T* p, float v) {
  if constexpr (sizeof(T) == 2) *p = __float2bfloat16(v);
  else *p = v;
}

constexpr int kBN = 64, kBK = 16;

// kBM x 64 tile; thread (ty, tx) of a 16 x 16 grid owns kBM / 16 rows and 4 consecutive columns
template <int kBM, typename TX, typename TW, typename TO>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const SimtParams p) {
  constexpr int kRM = kBM / 16;
  __shared__ float sX[kBK][kBM + 4];
  __shared__ float sW[kBK][kBN + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int n0 = blockIdx.x * kBN;
  int m0 = blockIdx.y * kBM, m_end = p.M;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const TX* X = reinterpret_cast<const TX*>(p.X);
  const TW* W = reinterpret_cast<const TW*>(p.W);
  if (p.tile_expert) {
    const int e = p.tile_expert[blockIdx.y];
    if (e < 0) return;
    W += (size_t)e * p.N * p.ldw;                  // N is one expert's rows
    m0 = p.tile_row0[blockIdx.y];
    m_end = min(p.M, m0 + p.tile_nrows[blockIdx.y]);
  }
  __shared__ long long s_row[kBM];                 // source row of every tile row, -1 past the end
  for (int i = tid; i < kBM; i += 256) {
    const int m = m0 + i;
    s_row[i] = m < m_end ? (p.row_index ? p.row_index[m] / p.row_div : m) : -1;
  }
  __syncthreads();
  constexpr int kLX = kBM * kBK / 256, kLW = kBN * kBK / 256;
  float rx[kLX], rw[kLW];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int i = 0; i < kLX; ++i) {
      const int e = tid + i * 256, r = e / kBK, k = k0 + e % kBK;
      float v = 0.f;
      if (s_row[r] >= 0 && k < p.K) v = ld1(X + (size_t)s_row[r] * p.ldx + k);
      rx[i] = p.a_op == 1 ? tanhf(v) : v;
    }
#pragma unroll
    for (int i = 0; i < kLW; ++i) {
      const int e = tid + i * 256, r = e / kBK, k = k0 + e % kBK;
      rw[i] = (n0 + r < p.N && k < p.K) ? ld1(W + (size_t)(n0 + r) * p.ldw + k) : 0.f;
    }
  };
  float acc[kRM][4];
#pragma unroll
  for (int i = 0; i < kRM; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  fetch(0);
  for (int k0 = 0; k0 < p.K; k0 += kBK) {
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kLX; ++i) { const int e = tid + i * 256; sX[e % kBK][e / kBK] = rx[i]; }
#pragma unroll
    for (int i = 0; i < kLW; ++i) { const int e = tid + i * 256; sW[e % kBK][e / kBK] = rw[i]; }
    __syncthreads();
    if (k0 + kBK < p.K) fetch(k0 + kBK);
    // every step's 16 products are summed by themselves: rounding grows with 16 + K / 16, not with K
    float part[kRM][4];
#pragma unroll
    for (int i = 0; i < kRM; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) part[i][j] = 0.f;
#pragma unroll
    for (int k = 0; k < kBK; ++k) {
      const float4 w = *reinterpret_cast<const float4*>(&sW[k][tx * 4]);
#pragma unroll
      for (int i = 0; i < kRM; ++i) {
        const float x = sX[k][ty * kRM + i];
        part[i][0] = fmaf(x, w.x, part[i][0]);
        part[i][1] = fmaf(x, w.y, part[i][1]);
        part[i][2] = fmaf(x, w.z, part[i][2]);
        part[i][3] = fmaf(x, w.w, part[i][3]);
      }
    }
#pragma unroll
    for (int i = 0; i < kRM; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
  }
#pragma unroll
  for (int i = 0; i < kRM; ++i) {
    const int m = m0 + ty * kRM + i;
    if (m >= m_end) continue;
    TO* row = reinterpret_cast<TO*>(p.out) + (size_t)m * p.ldo;
    const int n = n0 + tx * 4;
    if (p.epilogue == mb::EPI_CLAMP_GLU || p.epilogue == mb::EPI_SWIGLU || p.epilogue == mb::EPI_GEGLU) {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        if (n + 2 * j + 1 >= p.N) continue;
        const float g = acc[i][2 * j], u = acc[i][2 * j + 1];
        st1(row + (n >> 1) + j, p.epilogue == mb::EPI_CLAMP_GLU ? mb::clamp_glu(g, u, p.epi_a, p.epi_b)
                                : p.epilogue == mb::EPI_SWIGLU  ? mb::silu_exact(g) * u
                                                                : mb::gelu_tanh(g) * u);
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (n + j >= p.N) continue;
      float y = acc[i][j];
      if (p.epilogue == mb::EPI_SILU_COLS) {
        if (n + j < p.epi_n) y = mb::silu_exact(y);
      } else if (p.epilogue == mb::EPI_NEG_EXP) {
        y = -expf(y + (p.bias ? p.bias[n + j] : 0.f));
      } else if (p.epilogue == mb::EPI_BIAS) {
        y += p.bias[n + j];
      } else if (p.epilogue == mb::EPI_LOG_SIGMOID) {
        y = p.epi_a * mb::log_sigmoid(y + p.bias[n + j]);
      } else if (p.epilogue == mb::EPI_SIGMOID) {
        y = p.epi_a * mb::sigmoid_exact(y + p.bias[n + j]);
      } else if (p.epilogue == mb::EPI_RELU2) {
        y = mb::relu2(y);
      }
      st1(row + n + j, y);
    }
  }
}

template <int kBM, typename TX, typename TW, typename TO>
int launch_t(const SimtParams& p, int max_tiles, cudaStream_t stream) {
  const dim3 grid((p.N + kBN - 1) / kBN, max_tiles > 0 ? max_tiles : (p.M + kBM - 1) / kBM);
  if (grid.y > 65535) return MB_ERR_TOO_LARGE;
  return (int)mb::launch_kernel(gemm_simt_kernel<kBM, TX, TW, TO>, grid, dim3(256), 0, stream, p);
}
template <typename TX, typename TW, typename TO>
int launch_m(const SimtParams& p, int max_tiles, int tile_rows, cudaStream_t stream) {
  const bool small = max_tiles > 0 ? tile_rows == 16 : p.M <= 16;
  return small ? launch_t<16, TX, TW, TO>(p, max_tiles, stream) : launch_t<64, TX, TW, TO>(p, max_tiles, stream);
}

}  // namespace

struct MbSimtGemmArgs {
  int M, N, K;
  int x_bf16, w_bf16, out_bf16;
  const void* X;
  long long ldx;
  const void* W;
  long long ldw;
  void* out;
  long long ldo;
  int a_op, epilogue;
  const float* bias;
  float epi_a, epi_b;
  int epi_n;
  // grouped mode (tile_expert set): N is one expert's rows, a tile has at most tile_rows (16 or 64) rows
  const int* tile_expert;
  const int* tile_row0;
  const int* tile_nrows;
  int max_tiles, tile_rows;
  const int* row_index;
  int row_div;
};

extern "C" int mb_gemm_simt(const MbSimtGemmArgs* a, cudaStream_t stream) {
  if (!a || !a->X || !a->W || !a->out || a->M <= 0 || a->N <= 0 || a->K <= 0) return MB_ERR_BAD_ARG;
  const bool glu = a->epilogue == mb::EPI_SWIGLU || a->epilogue == mb::EPI_CLAMP_GLU || a->epilogue == mb::EPI_GEGLU;
  if (glu && (a->N & 1)) return MB_ERR_BAD_ARG;
  if ((a->epilogue == mb::EPI_BIAS || a->epilogue == mb::EPI_LOG_SIGMOID || a->epilogue == mb::EPI_SIGMOID) && !a->bias) return MB_ERR_BAD_ARG;
  const bool grouped = a->tile_expert != nullptr;
  if (grouped && (!a->tile_row0 || !a->tile_nrows || a->max_tiles <= 0 || (a->tile_rows != 16 && a->tile_rows != 64))) return MB_ERR_BAD_ARG;
  if (a->row_index && a->row_div <= 0) return MB_ERR_BAD_ARG;
  SimtParams p{a->M, a->N, a->K, a->X, a->ldx, a->W, a->ldw, a->out, a->ldo, a->a_op, a->epilogue, a->bias, a->epi_a, a->epi_b, a->epi_n,
               a->tile_expert, a->tile_row0, a->tile_nrows, a->row_index, a->row_div};
  const int mt = grouped ? a->max_tiles : 0, tr = a->tile_rows;
  using B = __nv_bfloat16;
  const int key = (a->x_bf16 ? 4 : 0) | (a->w_bf16 ? 2 : 0) | (a->out_bf16 ? 1 : 0);
  switch (key) {
    case 0: return launch_m<float, float, float>(p, mt, tr, stream);
    case 2: return launch_m<float, B, float>(p, mt, tr, stream);
    case 3: return launch_m<float, B, B>(p, mt, tr, stream);
    case 6: return launch_m<B, B, float>(p, mt, tr, stream);
    case 7: return launch_m<B, B, B>(p, mt, tr, stream);
    default: return MB_ERR_UNSUPPORTED;
  }
}
