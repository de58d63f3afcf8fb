// GEMM on the CUDA cores, fp32 accumulation with plain FMAs: out[m, n] = sum_k a(X[m, k]) W[n, k].
//
// Two kinds of caller need it next to the tensor-core GEMM:
//   * models served in true 32-bit (fp32 activations and weights; no tensor-core mode keeps 24 bits);
//   * products whose operands stay 32-bit in an otherwise bf16 model (low-rank decay projections of a
//     recurrence), and bf16 layers whose row length is not a multiple of 16 bytes, which no tensor map
//     can describe.
// X is fp32 or bf16, W fp32 or bf16, out fp32 or bf16, any M, N, K and row strides.
// Operand function a(): identity or tanh. Epilogues (shared numbering with the tensor-core GEMM):
//   plain; clamped GLU on interleaved (gate, up) rows; SiLU on the first epi_n columns;
//   -exp(y + bias), the logarithm of a decay exp(-exp(.)).
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
  const int n0 = blockIdx.x * kBN, m0 = blockIdx.y * kBM;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const TX* X = reinterpret_cast<const TX*>(p.X);
  const TW* W = reinterpret_cast<const TW*>(p.W);
  constexpr int kLX = kBM * kBK / 256, kLW = kBN * kBK / 256;
  float rx[kLX], rw[kLW];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int i = 0; i < kLX; ++i) {
      const int e = tid + i * 256, r = e / kBK, k = k0 + e % kBK;
      float v = 0.f;
      if (m0 + r < p.M && k < p.K) v = ld1(X + (size_t)(m0 + r) * p.ldx + k);
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
#pragma unroll
    for (int k = 0; k < kBK; ++k) {
      const float4 w = *reinterpret_cast<const float4*>(&sW[k][tx * 4]);
#pragma unroll
      for (int i = 0; i < kRM; ++i) {
        const float x = sX[k][ty * kRM + i];
        acc[i][0] = fmaf(x, w.x, acc[i][0]);
        acc[i][1] = fmaf(x, w.y, acc[i][1]);
        acc[i][2] = fmaf(x, w.z, acc[i][2]);
        acc[i][3] = fmaf(x, w.w, acc[i][3]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < kRM; ++i) {
    const int m = m0 + ty * kRM + i;
    if (m >= p.M) continue;
    TO* row = reinterpret_cast<TO*>(p.out) + (size_t)m * p.ldo;
    const int n = n0 + tx * 4;
    if (p.epilogue == mb::EPI_CLAMP_GLU) {
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (n + 2 * j + 1 < p.N) st1(row + (n >> 1) + j, mb::clamp_glu(acc[i][2 * j], acc[i][2 * j + 1], p.epi_a, p.epi_b));
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
      }
      st1(row + n + j, y);
    }
  }
}

template <int kBM, typename TX, typename TW, typename TO>
int launch_t(const SimtParams& p, cudaStream_t stream) {
  const dim3 grid((p.N + kBN - 1) / kBN, (p.M + kBM - 1) / kBM);
  if (grid.y > 65535) return MB_ERR_TOO_LARGE;
  return (int)mb::launch_kernel(gemm_simt_kernel<kBM, TX, TW, TO>, grid, dim3(256), 0, stream, p);
}
template <typename TX, typename TW, typename TO>
int launch_m(const SimtParams& p, cudaStream_t stream) {
  return p.M <= 16 ? launch_t<16, TX, TW, TO>(p, stream) : launch_t<64, TX, TW, TO>(p, stream);
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
};

extern "C" int mb_gemm_simt(const MbSimtGemmArgs* a, cudaStream_t stream) {
  if (!a || !a->X || !a->W || !a->out || a->M <= 0 || a->N <= 0 || a->K <= 0) return MB_ERR_BAD_ARG;
  if (a->epilogue == mb::EPI_SWIGLU || (a->epilogue == mb::EPI_CLAMP_GLU && (a->N & 1))) return MB_ERR_BAD_ARG;
  SimtParams p{a->M, a->N, a->K, a->X, a->ldx, a->W, a->ldw, a->out, a->ldo, a->a_op, a->epilogue, a->bias, a->epi_a, a->epi_b, a->epi_n};
  using B = __nv_bfloat16;
  const int key = (a->x_bf16 ? 4 : 0) | (a->w_bf16 ? 2 : 0) | (a->out_bf16 ? 1 : 0);
  switch (key) {
    case 0: return launch_m<float, float, float>(p, stream);
    case 2: return launch_m<float, B, float>(p, stream);
    case 3: return launch_m<float, B, B>(p, stream);
    case 6: return launch_m<B, B, float>(p, stream);
    case 7: return launch_m<B, B, B>(p, stream);
    default: return MB_ERR_UNSUPPORTED;
  }
}
