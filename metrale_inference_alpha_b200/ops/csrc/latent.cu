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

template <int VEC, typename TX, typename T>
__global__ void __launch_bounds__(256) latent_norm_kernel(const NormParams p) {
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const TX* x = reinterpret_cast<const TX*>(p.x) + (size_t)t * p.x_ld;
  const TX* kv = x + p.q_rank;
  float sq = 0.f, sk = 0.f;
#pragma unroll 2
  for (int i = tid * VEC; i < p.q_rank + p.L; i += 256 * VEC) {        // a vector lies on one side
    float v[VEC], s = 0.f;
    ldn<VEC>(x + i, v);
#pragma unroll
    for (int e = 0; e < VEC; ++e) s = fmaf(v[e], v[e], s);
    if (i < p.q_rank) sq += s;
    else sk += s;
  }
  const float iq = rsqrtf(mb::block_sum(sq, red) / (float)p.q_rank + p.eps);
  const float ik = rsqrtf(mb::block_sum(sk, red) / (float)p.L + p.eps);
  T* cq = reinterpret_cast<T*>(p.cq) + (size_t)t * p.q_rank;
  for (int i = tid * VEC; i < p.q_rank; i += 256 * VEC) {
    float v[VEC], w[VEC];
    ldn<VEC>(x + i, v);
    ldn<VEC>(p.q_w + i, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= iq * w[e];
    stn<VEC>(cq + i, v);
  }
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
  for (int i = tid * VEC; i < p.L; i += 256 * VEC) {
    float v[VEC], w[VEC];
    ldn<VEC>(kv + i, v);
    ldn<VEC>(p.kv_w + i, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] *= ik * w[e];
    stn<VEC>(dst + i, v);
  }
  for (int i = p.L + tid; i < p.row; i += 256) {
    const int r = i - p.rope_at;
    float v = 0.f;
    if (r >= 0 && r < p.R) {
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
  const auto al = [](const void* q, int n) { return reinterpret_cast<uintptr_t>(q) % n == 0; };
  const bool v4 = a->q_rank % 4 == 0 && a->L % 4 == 0 && a->row % 4 == 0 && a->x_ld % 4 == 0 && al(a->x, 16) && al(a->cq, 16) && al(a->cache, 16) &&
                  al(a->q_w, 8) && al(a->kv_w, 8);
  const dim3 grid(a->T), block(256);
#define MB_LATENT(TX, T)                                                                                         \
  return (int)(v4 ? mb::launch_kernel(latent_norm_kernel<4, TX, T>, grid, block, 0, stream, p)                   \
                  : mb::launch_kernel(latent_norm_kernel<1, TX, T>, grid, block, 0, stream, p))
  if (a->f32 && !a->in_f32) return MB_ERR_UNSUPPORTED;
  if (a->f32) MB_LATENT(float, float);
  if (a->in_f32) MB_LATENT(float, bf16);
  MB_LATENT(bf16, bf16);
#undef MB_LATENT
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
