// Row kernels of latent attention with per-layer sizes (queries through a normed latent, keys and values linear in
// a cached latent, one rotated key part for all heads).
//
//   latent_norm    one CTA per token over the input projection's row [query latent | latent | key part | ...]:
//                  RMS norm of the query latent (the next GEMM's operand), RMS norm of the key-value latent and
//                  rotation of the key part, both written as one cache row at the token's slot
//   latent_query   completes absorbed query rows [T, H, row]: the latent columns come from a batched product with
//                  the heads' key matrices, the rotated part and the zero padding are written here
// A cache row is [latent (L) | zeros | rotated key (R) at rope_at | zeros]. Rotation pairs dimension i with i + R / 2.
// The projection's rows are fp32 or of the activation type T (bf16, or fp32 for models served in 32-bit).
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

struct NormParams {
  int q_rank, L, R, row, rope_at;
  const void* x;
  long long x_ld;
  const bf16* q_w;
  const bf16* kv_w;
  float eps;
  const float* cos_tab;
  const float* sin_tab;
  int max_pos;
  const int* positions;
  const long long* slots;
  long long num_slots;
  void* cache;
  void* cq;
  uint32_t* status;
};

template <typename TX, typename T>
__global__ void __launch_bounds__(256) latent_norm_kernel(const NormParams p) {
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const TX* x = reinterpret_cast<const TX*>(p.x) + (size_t)t * p.x_ld;
  const TX* kv = x + p.q_rank;
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < p.q_rank; i += 256) { const float v = ldv(x + i); sq = fmaf(v, v, sq); }
  for (int i = tid; i < p.L; i += 256) { const float v = ldv(kv + i); sk = fmaf(v, v, sk); }
  const float iq = rsqrtf(mb::block_sum(sq, red) / (float)p.q_rank + p.eps);
  const float ik = rsqrtf(mb::block_sum(sk, red) / (float)p.L + p.eps);
  T* cq = reinterpret_cast<T*>(p.cq) + (size_t)t * p.q_rank;
  for (int i = tid; i < p.q_rank; i += 256) stv(cq + i, ldv(x + i) * iq * __bfloat162float(p.q_w[i]));
  const long long slot = p.slots[t];
  if (slot >= p.num_slots) {
    if (p.status && tid == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    return;
  }
  if (slot < 0) return;
  int pos = p.positions[t];
  if (pos < 0 || (p.R > 0 && pos >= p.max_pos)) {
    if (p.status && tid == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    pos = 0;
  }
  T* dst = reinterpret_cast<T*>(p.cache) + (size_t)slot * p.row;
  const int half = p.R / 2;
  for (int i = tid; i < p.row; i += 256) {
    float v = 0.f;
    const int r = i - p.rope_at;
    if (i < p.L) {
      v = ldv(kv + i) * ik * __bfloat162float(p.kv_w[i]);
    } else if (r >= 0 && r < p.R) {
      const int a = r < half ? r : r - half;
      const float c = p.cos_tab[(size_t)pos * half + a], s = p.sin_tab[(size_t)pos * half + a];
      const float u = ldv(kv + p.L + a), w = ldv(kv + p.L + half + a);
      v = r < half ? u * c - w * s : w * c + u * s;
    }
    stv(dst + i, v);
  }
}

struct QueryParams {
  int T, H, dim, R, L, row, rope_at;
  const void* q;
  const float* cos_tab;
  const float* sin_tab;
  int max_pos;
  const int* positions;
  void* qq;
  uint32_t* status;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_query_kernel(const QueryParams p) {
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int t = blockIdx.x;
  int pos = p.positions[t];
  if (pos < 0 || (p.R > 0 && pos >= p.max_pos)) {
    if (p.status && threadIdx.x == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    pos = 0;
  }
  const int half = p.R / 2, rest = p.row - p.L;
  const float* cs = p.cos_tab + (size_t)pos * half;
  const float* sn = p.sin_tab + (size_t)pos * half;
  for (int e = blockIdx.y * 256 + threadIdx.x; e < p.H * rest; e += gridDim.y * 256) {
    const int h = e / rest, i = p.L + e - h * rest, r = i - p.rope_at;
    float v = 0.f;
    if (r >= 0 && r < p.R) {
      const T* src = reinterpret_cast<const T*>(p.q) + ((size_t)t * p.H + h) * (p.dim + p.R) + p.dim;
      const int a = r < half ? r : r - half;
      const float u = ldv(src + a), w = ldv(src + half + a);
      v = r < half ? u * cs[a] - w * sn[a] : w * cs[a] + u * sn[a];
    }
    stv(reinterpret_cast<T*>(p.qq) + ((size_t)t * p.H + h) * p.row + i, v);
  }
}

}  // namespace

struct MbLatentNormArgs {
  int T, in_f32, f32, q_rank, L, R, row, rope_at;
  const void* x;
  long long x_ld;
  const void* q_w;
  const void* kv_w;
  float eps;
  const float* cos_tab;
  const float* sin_tab;
  int max_pos;
  const int* positions;
  const long long* slots;
  long long num_slots;
  void* cache;
  void* cq;
  uint32_t* status;
};

struct MbLatentQueryArgs {
  int T, H, f32, dim, R, L, row, rope_at;
  const void* q;
  const float* cos_tab;
  const float* sin_tab;
  int max_pos;
  const int* positions;
  void* qq;
  uint32_t* status;
};

extern "C" int mb_latent_norm(const MbLatentNormArgs* a, cudaStream_t stream) {
  if (!a || !a->x || !a->q_w || !a->kv_w || !a->cache || !a->cq || !a->positions || !a->slots || a->T <= 0) return MB_ERR_BAD_ARG;
  if (a->q_rank <= 0 || a->L <= 0 || a->R < 0 || (a->R & 1) || a->rope_at < a->L || a->rope_at + a->R > a->row) return MB_ERR_BAD_ARG;
  if (a->R > 0 && (!a->cos_tab || !a->sin_tab || a->max_pos <= 0)) return MB_ERR_BAD_ARG;
  if (a->x_ld < (long long)a->q_rank + a->L + a->R) return MB_ERR_BAD_ARG;
  const NormParams p{a->q_rank, a->L, a->R, a->row, a->rope_at, a->x, a->x_ld, (const bf16*)a->q_w, (const bf16*)a->kv_w, a->eps, a->cos_tab,
                     a->sin_tab, a->max_pos, a->positions, a->slots, a->num_slots, a->cache, a->cq, a->status};
  const dim3 grid(a->T), block(256);
  if (a->f32) return a->in_f32 ? (int)mb::launch_kernel(latent_norm_kernel<float, float>, grid, block, 0, stream, p) : MB_ERR_UNSUPPORTED;
  if (a->in_f32) return (int)mb::launch_kernel(latent_norm_kernel<float, bf16>, grid, block, 0, stream, p);
  return (int)mb::launch_kernel(latent_norm_kernel<bf16, bf16>, grid, block, 0, stream, p);
}

extern "C" int mb_latent_query(const MbLatentQueryArgs* a, cudaStream_t stream) {
  if (!a || !a->q || !a->qq || !a->positions || a->T <= 0 || a->H <= 0) return MB_ERR_BAD_ARG;
  if (a->dim <= 0 || a->R < 0 || (a->R & 1) || a->rope_at < a->L || a->rope_at + a->R > a->row) return MB_ERR_BAD_ARG;
  if (a->R > 0 && (!a->cos_tab || !a->sin_tab || a->max_pos <= 0)) return MB_ERR_BAD_ARG;
  const QueryParams p{a->T, a->H, a->dim, a->R, a->L, a->row, a->rope_at, a->q, a->cos_tab, a->sin_tab, a->max_pos, a->positions, a->qq, a->status};
  const int per = (a->H * (a->row - a->L) + 255) / 256;
  const dim3 grid(a->T, a->T >= 1024 ? 1 : (per < 8 ? (per < 1 ? 1 : per) : 8));
  if (a->f32) return (int)mb::launch_kernel(latent_query_kernel<float>, grid, dim3(256), 0, stream, p);
  return (int)mb::launch_kernel(latent_query_kernel<bf16>, grid, dim3(256), 0, stream, p);
}
