// Rows of an attention layer whose queries and keys are normed over the whole projection (all heads at once).
//
//   attention_rows  queries, keys and values are column ranges of one projection; the value range may be the key range
//                   itself (keys as projected, before norm and rotation, serve as values). RMS norms with plain weights,
//                   rotate-half positions on the leading `rot` dimensions, optionally a rotation of the values by their
//                   own position over all of dv; queries to a padded buffer, keys and values to the paged cache. A CTA
//                   per token: the sums of squares first, then one elementwise pass.
//   turn_rows       an attention output turned by minus its own position, in place: what undoes rotated values
#include "row_io.cuh"

namespace {

struct AttnRowsParams {
  int Hq, Hkv, dk, dv, rot, dkp, dvp;
  const void* y;
  long long ld;
  int q_at, k_at, v_at;
  const int* positions;
  const long long* slots;
  const float* cos_tab;        // [max_pos, rot / 2]
  const float* sin_tab;
  const float* v_cos;          // [max_pos, dv / 2], or null: values as they are
  const float* v_sin;
  int max_pos;
  const bf16* q_norm;          // [Hq dk], or null
  const bf16* k_norm;          // [Hkv dk], or null
  float eps;
  void* q_out;
  void* k_cache;
  void* v_cache;
  long long num_slots;
  uint32_t* status;
};

template <int VEC, typename T>
__global__ void __launch_bounds__(256) attention_rows_kernel(const AttnRowsParams p) {
  __shared__ float red[2][8];
  const int m = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const T* src = reinterpret_cast<const T*>(p.y) + (size_t)m * p.ld;
  int pos = p.positions[m];
  long long slot = p.slots[m];
  if (slot >= p.num_slots || pos < 0 || pos >= p.max_pos) {
    if (tid == 0 && p.status) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    if (slot >= p.num_slots) slot = -1;
    if (pos < 0 || pos >= p.max_pos) pos = 0;
  }
  float inv_q = 1.f, inv_k = 1.f;
  if (p.q_norm || p.k_norm) {
    auto sumsq = [&](const T* r, int n) {
      float ss = 0.f;
      for (int d = tid * VEC; d < n; d += blockDim.x * VEC) {
        float x[VEC];
        ldn<VEC>(r + d, x);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(x[i], x[i], ss);
      }
      return mb::warp_sum(ss);
    };
    const float a = sumsq(src + p.q_at, p.Hq * p.dk), b = sumsq(src + p.k_at, p.Hkv * p.dk);
    if (lane == 0) {
      red[0][warp] = a;
      red[1][warp] = b;
    }
    __syncthreads();
    float ta = 0.f, tb = 0.f;
    for (int w = 0; w < nw; ++w) {
      ta += red[0][w];
      tb += red[1][w];
    }
    if (p.q_norm) inv_q = 1.f / sqrtf(ta / (float)(p.Hq * p.dk) + p.eps);
    if (p.k_norm) inv_k = 1.f / sqrtf(tb / (float)(p.Hkv * p.dk) + p.eps);
  }
  const int half = p.rot / 2, vhalf = p.dv / 2;
  const float* cs = p.cos_tab + (size_t)pos * half;
  const float* sn = p.sin_tab + (size_t)pos * half;
  // elements d .. d + VEC - 1 of a head's row turned with their partners; VEC divides `half`: they are on one side
  auto turned = [&](float* o, const float* q, bool first, const float* c, const float* s) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = first ? o[j] * c[j] - q[j] * s[j] : o[j] * c[j] + q[j] * s[j];
  };
  const int nq = p.Hq * p.dkp, nk = p.Hkv * p.dkp, nv = p.Hkv * p.dvp;
  for (int e = tid * VEC; e < nq + nk + nv; e += blockDim.x * VEC) {
    float o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = 0.f;
    if (e < nq + nk) {
      const bool is_q = e < nq;
      if (!is_q && slot < 0) continue;
      const int i = is_q ? e : e - nq, h = i / p.dkp, d = i - h * p.dkp;
      const T* row = src + (is_q ? p.q_at : p.k_at) + h * p.dk;
      const bf16* nw_ = is_q ? p.q_norm : p.k_norm;
      const float inv = is_q ? inv_q : inv_k;
      auto load = [&](int at, float* v) {
        ldn<VEC>(row + at, v);
        if (nw_) {
          float w[VEC];
          ldn<VEC>(nw_ + h * p.dk + at, w);
#pragma unroll
          for (int j = 0; j < VEC; ++j) v[j] *= inv * w[j];
        }
      };
      if (d < p.dk) {
        load(d, o);
        if (d < p.rot) {
          float q[VEC];
          const bool first = d < half;
          load(first ? d + half : d - half, q);
          turned(o, q, first, cs + (first ? d : d - half), sn + (first ? d : d - half));
        }
      }
      if (is_q) stn<VEC>(reinterpret_cast<T*>(p.q_out) + (size_t)m * nq + i, o);
      else stn<VEC>(reinterpret_cast<T*>(p.k_cache) + (size_t)slot * nk + i, o);
    } else if (slot >= 0) {
      const int i = e - nq - nk, h = i / p.dvp, d = i - h * p.dvp;
      const T* row = src + p.v_at + h * p.dv;
      if (d < p.dv) {
        ldn<VEC>(row + d, o);
        if (p.v_cos) {
          float q[VEC];
          const bool first = d < vhalf;
          const int a = first ? d : d - vhalf;
          ldn<VEC>(row + (first ? d + vhalf : a), q);
          turned(o, q, first, p.v_cos + (size_t)pos * vhalf + a, p.v_sin + (size_t)pos * vhalf + a);
        }
      }
      stn<VEC>(reinterpret_cast<T*>(p.v_cache) + (size_t)slot * nv + i, o);
    }
  }
}

template <int VEC, typename T>
__global__ void __launch_bounds__(256) turn_rows_kernel(T* x, long long ld, int M, int H, int dv, const int* positions, const float* cos_tab,
                                                        const float* sin_tab, int max_pos, uint32_t* status) {
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int half = dv / 2, per = H * half / VEC;           // vectors of a token's first halves
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int m = (int)(i / per), r = (int)(i - (long long)m * per) * VEC;
  if (m >= M) return;
  int pos = positions[m];
  if (pos < 0 || pos >= max_pos) {
    if (status) atomicCAS(status, 0u, MB_ST_BOUNDS);
    pos = 0;
  }
  const int h = r / half, d = r - h * half;
  T* row = x + (size_t)m * ld + (size_t)h * dv + d;
  float u[VEC], v[VEC], c[VEC], s[VEC], a[VEC], b[VEC];
  ldn<VEC>(row, u);
  ldn<VEC>(row + half, v);
  ldn<VEC>(cos_tab + (size_t)pos * half + d, c);
  ldn<VEC>(sin_tab + (size_t)pos * half + d, s);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    a[j] = u[j] * c[j] + v[j] * s[j];
    b[j] = v[j] * c[j] - u[j] * s[j];
  }
  stn<VEC>(row, a);
  stn<VEC>(row + half, b);
}

}  // namespace

struct MbAttnRowsArgs {
  int M, Hq, Hkv, dk, dv, rot, dkp, dvp, f32;
  const void* y;
  long long ld;
  int q_at, k_at, v_at;
  const int* positions;
  const long long* slots;
  const float* cos_tab;
  const float* sin_tab;
  const float* v_cos;
  const float* v_sin;
  int max_pos;
  const void* q_norm;
  const void* k_norm;
  float eps;
  void* q_out;
  void* k_cache;
  void* v_cache;
  long long num_slots;
  uint32_t* status;
};

extern "C" {

int mb_attention_rows(const MbAttnRowsArgs* a, cudaStream_t stream) {
  if (!a || a->M <= 0 || !a->y || !a->positions || !a->slots || !a->q_out || !a->k_cache || !a->v_cache || a->max_pos <= 0) return MB_ERR_BAD_ARG;
  if (a->dk <= 0 || a->dv <= 0 || a->dk > a->dkp || a->dv > a->dvp || a->rot < 0 || a->rot > a->dk || a->rot % 2) return MB_ERR_UNSUPPORTED;
  if (a->q_at < 0 || a->k_at < 0 || a->v_at < 0 || a->q_at + a->Hq * a->dk > a->ld || a->k_at + a->Hkv * a->dk > a->ld || a->v_at + a->Hkv * a->dv > a->ld)
    return MB_ERR_BAD_ARG;
  if ((a->rot > 0 && (!a->cos_tab || !a->sin_tab)) || (a->v_cos && (!a->v_sin || a->dv % 2))) return MB_ERR_BAD_ARG;
  const AttnRowsParams p{a->Hq, a->Hkv, a->dk, a->dv, a->rot, a->dkp, a->dvp, a->y, a->ld, a->q_at, a->k_at, a->v_at, a->positions, a->slots,
                         a->cos_tab, a->sin_tab, a->v_cos, a->v_sin, a->max_pos, (const bf16*)a->q_norm, (const bf16*)a->k_norm, a->eps, a->q_out,
                         a->k_cache, a->v_cache, a->num_slots, a->status};
  const size_t es = a->f32 ? 16 : 8;
  const bool v4 = a->dk % 4 == 0 && a->dv % 4 == 0 && a->rot % 8 == 0 && (!a->v_cos || a->dv % 8 == 0) && a->dkp % 4 == 0 && a->dvp % 4 == 0 &&
                  a->ld % 4 == 0 && a->q_at % 4 == 0 && a->k_at % 4 == 0 && a->v_at % 4 == 0 && al(a->y, es) && al(a->q_out, es) &&
                  al(a->k_cache, es) && al(a->v_cache, es) && al(a->q_norm, 8) && al(a->k_norm, 8);
  const dim3 g(a->M), b(256);
  if (a->f32) return (int)(v4 ? mb::launch_kernel(attention_rows_kernel<4, float>, g, b, 0, stream, p) : mb::launch_kernel(attention_rows_kernel<1, float>, g, b, 0, stream, p));
  return (int)(v4 ? mb::launch_kernel(attention_rows_kernel<4, bf16>, g, b, 0, stream, p) : mb::launch_kernel(attention_rows_kernel<1, bf16>, g, b, 0, stream, p));
}

int mb_turn_rows(void* x, long long ld, int M, int H, int dv, int f32, const int* positions, const float* cos_tab, const float* sin_tab, int max_pos,
                 uint32_t* status, cudaStream_t stream) {
  if (!x || M <= 0 || H <= 0 || dv <= 0 || dv % 2 || !positions || !cos_tab || !sin_tab || max_pos <= 0 || ld < (long long)H * dv) return MB_ERR_BAD_ARG;
  const size_t es = f32 ? 16 : 8;
  const bool v4 = dv % 8 == 0 && ld % 4 == 0 && al(x, es) && al(cos_tab, 16) && al(sin_tab, 16);
  const long long n = (long long)M * (H * (dv / 2) / (v4 ? 4 : 1));
  if (n > (1ll << 38)) return MB_ERR_TOO_LARGE;
  const dim3 g((unsigned)((n + 255) / 256)), b(256);
  if (f32) return (int)(v4 ? mb::launch_kernel(turn_rows_kernel<4, float>, g, b, 0, stream, (float*)x, ld, M, H, dv, positions, cos_tab, sin_tab, max_pos, status)
                           : mb::launch_kernel(turn_rows_kernel<1, float>, g, b, 0, stream, (float*)x, ld, M, H, dv, positions, cos_tab, sin_tab, max_pos, status));
  return (int)(v4 ? mb::launch_kernel(turn_rows_kernel<4, bf16>, g, b, 0, stream, (bf16*)x, ld, M, H, dv, positions, cos_tab, sin_tab, max_pos, status)
                  : mb::launch_kernel(turn_rows_kernel<1, bf16>, g, b, 0, stream, (bf16*)x, ld, M, H, dv, positions, cos_tab, sin_tab, max_pos, status));
}

}  // extern "C"
