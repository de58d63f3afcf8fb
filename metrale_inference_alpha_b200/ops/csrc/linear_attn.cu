// Decaying linear attention, token by token, for a ragged batch: per head a [DK, DV] fp32 state with
//     S_t = diag(w_t) S_(t-1) + k_t v_t^T
// and one of two readouts
//     after the update        o_t = S_t^T q_t
//     before it, with a bonus o_t = (S_(t-1) + diag(u) k_t v_t^T)^T q_t
// w_t is a constant of the head, or exp(log_w) of a per-token, per-channel fp32 tensor. q, k, v are bf16 or
// fp32, DK <= 256, any DV; everything inside is fp32. The state is carried in a slot pool; a sequence whose
// first row is at position 0 starts from zero. Serves decode, speculative verification and its commit pass
// (write_out = 0), prefill of head sizes the chunked kernels do not take, and models served in 32-bit.
//
// A CTA owns one (sequence, head, block of value columns). Its compute warps hold the state in registers,
// 8 key rows x 4 value columns per thread; KG lanes share a column and meet in a shuffle reduction. Two
// key rows sit in one 64-bit register pair, so the update runs on the packed fp32 FMA. Producer warps load
// and convert the next 16 tokens into the other half of a double buffer meanwhile (and compute each token's
// bonus coefficient sum_i q_i u_i k_i), so the recurrence never waits on global memory.
//
// Steps of one token per sequence take linear_decode_kernel instead: one CTA per (sequence, head) streams the
// state once, 16 rows of 16-byte vectors in flight per thread, and can finish the head's output itself (RMS over
// the head, weight, gate, scale), so decode needs no separate norm launch; decays given as a low-rank projection are
// computed there too, one channel per thread.
#include "common.cuh"
#include "epilogue.cuh"

namespace {

using bf16 = __nv_bfloat16;

// log decays c log(sigmoid(a2 a1 + bias)): a1 [T, rank] of the activation type, a2 [H * DK, rank], bias [H * DK]
struct LowRank {
  const void* a1;                  // null: not used
  long long a1_ld;
  const bf16* a2;
  const float* bias;
  int rank;
  float c;
};

struct LinParams {
  const void* q;
  const void* k;
  const void* v;
  long long q_ld, k_ld, v_ld;      // elements between tokens
  int H, DK, DV;
  const float* log_w;              // [T, H * DK] or null
  const float* decay;              // [H] when log_w is null
  LowRank lr;                      // decode: the decays from their low-rank projection instead of log_w
  const float* u;                  // [H, DK]: bonus readout before the update; null: readout after it
  float* state;                    // [slots, H, DK, DV]
  float* out;                      // [T, H * DV]
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_slots, write_state, write_out;
  uint32_t* status;
};

constexpr int kTB = 16;            // tokens per buffer
constexpr int kNW = 4;             // compute warps
constexpr int kPW = 4;             // producer warps

template <typename T>
__device__ __forceinline__ float ldx(const void* base, size_t i) {
  if constexpr (sizeof(T) == 2) return __bfloat162float(reinterpret_cast<const bf16*>(base)[i]);
  else return reinterpret_cast<const float*>(base)[i];
}

using f2 = unsigned long long;     // two packed fp32
__device__ __forceinline__ f2 pk(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void upk(f2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

template <int KG>
constexpr int cols_per_cta() { return kNW * (32 / KG) * 4; }
template <int KG, bool CH>
constexpr size_t lin_smem() { return (size_t)2 * kTB * ((CH ? 3 : 2) * 8 * KG + cols_per_cta<KG>() + 4) * sizeof(float); }

// KG lanes per value column, 8 key rows each (DK <= 8 KG); CH: per-channel decays; BONUS: readout before the update
template <typename T, int KG, bool CH, bool BONUS>
__global__ void __launch_bounds__(32 * (kNW + kPW)) linear_attn_kernel(const LinParams p) {
  constexpr int DKP = 8 * KG, VB = cols_per_cta<KG>();
  extern __shared__ __align__(16) float sm[];
  float* sQ = sm;                                  // [2][kTB][DKP]
  float* sK = sQ + 2 * kTB * DKP;
  float* sV = sK + 2 * kTB * DKP;                  // [2][kTB][VB]
  float* sB = sV + 2 * kTB * VB;                   // [2][kTB][4]: bonus coefficients
  float* sW = sB + 2 * kTB * 4;                    // [2][kTB][DKP], CH only
  const int vb = blockIdx.x, hd = blockIdx.y, seq = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (n <= 0) return;
  const int t0 = p.q_start[seq];
  const int slot = p.slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (p.status && tid == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    return;
  }
  const int DK = p.DK, DV = p.DV, col0 = vb * VB;

  auto produce = [&](int tile, int pw) {
    const int buf = tile & 1;
    const int cnt = min(kTB, n - tile * kTB);
#pragma unroll 2
    for (int tt = pw; tt < cnt; tt += kPW) {
      const size_t t = (size_t)(t0 + tile * kTB + tt);
      float* q = sQ + (buf * kTB + tt) * DKP;
      float* k = sK + (buf * kTB + tt) * DKP;
      float bonus = 0.f;
#pragma unroll
      for (int j = 0; j < (DKP + 31) / 32; ++j) {
        const int d = lane + 32 * j;
        if (d < DKP) {
          float qv = 0.f, kv = 0.f, wv = 0.f;
          if (d < DK) {
            qv = ldx<T>(p.q, t * p.q_ld + (size_t)hd * DK + d);
            kv = ldx<T>(p.k, t * p.k_ld + (size_t)hd * DK + d);
            if constexpr (CH) wv = expf(p.log_w[(t * p.H + hd) * DK + d]);
            if constexpr (BONUS) bonus += qv * p.u[hd * DK + d] * kv;
          }
          q[d] = qv;
          k[d] = kv;
          if constexpr (CH) sW[(buf * kTB + tt) * DKP + d] = wv;
        }
      }
      if constexpr (BONUS) {
        bonus = mb::warp_sum(bonus);
        if (lane == 0) sB[(buf * kTB + tt) * 4] = bonus;
      }
      for (int c = lane; c < VB; c += 32)
        sV[(buf * kTB + tt) * VB + c] = col0 + c < DV ? ldx<T>(p.v, t * p.v_ld + (size_t)hd * DV + col0 + c) : 0.f;
    }
  };

  const int tiles = (n + kTB - 1) / kTB;
  const bool compute = warp < kNW;
  const int kg = lane % KG, vg = lane / KG;
  const int lc = (warp * (32 / KG) + vg) * 4;      // first of this thread's four columns inside the block
  const int col = col0 + lc;
  // s[pair][c]: key rows row(pair), row(pair) + 1 of column c; pair 0, 1 = rows 4 kg .. 4 kg + 3, pair 2, 3 = 4 KG further
  f2 s[4][4];
  float* st = p.state + ((size_t)slot * p.H + hd) * DK * DV;
  auto row_of = [&](int pair) { return (pair >> 1) * 4 * KG + kg * 4 + (pair & 1) * 2; };
  const bool vec = DV % 4 == 0;
  if (compute) {
    const bool fresh = p.positions[t0] == 0;
#pragma unroll
    for (int pr = 0; pr < 4; ++pr) {
      float a[2][4];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = row_of(pr) + e;
        const float* src = st + (size_t)r * DV + col;
        if (!fresh && r < DK && vec && col < DV) {
          const float4 v = *reinterpret_cast<const float4*>(src);
          a[e][0] = v.x; a[e][1] = v.y; a[e][2] = v.z; a[e][3] = v.w;
        } else {
#pragma unroll
          for (int c = 0; c < 4; ++c) a[e][c] = (!fresh && r < DK && col + c < DV) ? src[c] : 0.f;
        }
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) s[pr][c] = pk(a[0][c], a[1][c]);
    }
  } else {
    produce(0, warp - kNW);
  }
  const float wconst = CH ? 0.f : p.decay[hd];
  const f2 w2c = pk(wconst, wconst);
  __syncthreads();
  for (int tile = 0; tile < tiles; ++tile) {
    if (!compute) {
      if (tile + 1 < tiles) produce(tile + 1, warp - kNW);
    } else {
      const int buf = tile & 1;
      const int cnt = min(kTB, n - tile * kTB);
      for (int tt = 0; tt < cnt; ++tt) {
        const float4 v = *reinterpret_cast<const float4*>(sV + (buf * kTB + tt) * VB + lc);
        const f2 vv[4] = {pk(v.x, v.x), pk(v.y, v.y), pk(v.z, v.z), pk(v.w, v.w)};
        f2 o[4] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          const int off = (buf * kTB + tt) * DKP + g * 4 * KG + kg * 4;
          const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(sQ + off);
          const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(sK + off);
          ulonglong2 w4;
          if constexpr (CH) w4 = *reinterpret_cast<const ulonglong2*>(sW + off);
          else w4.x = w4.y = w2c;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const f2 q2 = e ? q4.y : q4.x, k2 = e ? k4.y : k4.x, w2 = e ? w4.y : w4.x;
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              f2& sr = s[g * 2 + e][c];
              if constexpr (BONUS) o[c] = fma2(q2, sr, o[c]);
              sr = fma2(w2, sr, mul2(k2, vv[c]));
              if constexpr (!BONUS) o[c] = fma2(q2, sr, o[c]);
            }
          }
        }
        if (p.write_out) {
          float r[4];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            float a, b;
            upk(o[c], a, b);
            r[c] = a + b;
          }
          // reduce over the KG lanes of a column group; with KG >= 4 every lane ends up with one column
          float y;
          int cc;
          if constexpr (KG >= 4) {
            const bool b0 = kg & 1, b1 = kg & 2;
            const float s0 = b0 ? r[0] : r[2], s1 = b0 ? r[1] : r[3];         // what the neighbour keeps
            float k0 = b0 ? r[2] : r[0], k1 = b0 ? r[3] : r[1];
            k0 += __shfl_xor_sync(0xffffffffu, s0, 1);
            k1 += __shfl_xor_sync(0xffffffffu, s1, 1);
            const float s2 = b1 ? k0 : k1;
            y = (b1 ? k1 : k0) + __shfl_xor_sync(0xffffffffu, s2, 2);
#pragma unroll
            for (int o2 = 4; o2 < KG; o2 <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o2);
            cc = (b0 ? 2 : 0) + (b1 ? 1 : 0);
          } else {
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
              for (int o2 = 1; o2 < KG; o2 <<= 1) r[c] += __shfl_xor_sync(0xffffffffu, r[c], o2);
            y = 0.f;
            cc = 0;
          }
          const float bonus = BONUS ? sB[(buf * kTB + tt) * 4] : 0.f;
          const size_t t = (size_t)(t0 + tile * kTB + tt);
          float* dst = p.out + (t * p.H + hd) * DV;
          if constexpr (KG >= 4) {
            if (kg < 4 && col + cc < DV) {
              if constexpr (BONUS) y = fmaf(bonus, sV[(buf * kTB + tt) * VB + lc + cc], y);
              dst[col + cc] = y;
            }
          } else {
            if (kg == 0) {
#pragma unroll
              for (int c = 0; c < 4; ++c)
                if (col + c < DV) dst[col + c] = BONUS ? fmaf(bonus, sV[(buf * kTB + tt) * VB + lc + c], r[c]) : r[c];
            }
          }
        }
      }
    }
    __syncthreads();
  }
  if (compute && p.write_state) {
#pragma unroll
    for (int pr = 0; pr < 4; ++pr) {
      float a[2][4];
#pragma unroll
      for (int c = 0; c < 4; ++c) upk(s[pr][c], a[0][c], a[1][c]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = row_of(pr) + e;
        float* dst = st + (size_t)r * DV + col;
        if (r < DK && vec && col < DV) {
          *reinterpret_cast<float4*>(dst) = make_float4(a[e][0], a[e][1], a[e][2], a[e][3]);
        } else {
#pragma unroll
          for (int c = 0; c < 4; ++c)
            if (r < DK && col + c < DV) dst[c] = a[e][c];
        }
      }
    }
  }
}

// ------------------------------------------------------------------ one token per sequence
struct DecodeNorm {
  const bf16* w;                   // [H * DV] or null: no norm, fp32 output
  const void* gate;
  long long gate_ld;
  int sigmoid_gate;
  float eps, scale;
  void* out;                       // row stride out_ld
  long long out_ld;
};

constexpr int kDecRows = 16;       // state rows in flight per thread

// QV threads cover the DV / 4 column vectors of a row; 256 / QV rows are in work side by side
template <typename T, int QV, bool CH, bool BONUS>
__global__ void __launch_bounds__(256, 2) linear_decode_kernel(const LinParams p, const DecodeNorm nm) {
  constexpr int RG = 256 / QV;
  __shared__ float sq[256], sk[256], sw[CH ? 256 : 1], so[RG * QV * 4], red[32];
  const int hd = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  if (p.q_len[seq] <= 0) return;
  const size_t t = (size_t)p.q_start[seq];
  const int slot = p.slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (p.status && tid == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    return;
  }
  const bool fresh = p.positions[t] == 0;
  const int DK = p.DK, DV = p.DV, c4 = (tid % QV) * 4, rg = tid / QV;
  const bool col_ok = c4 < DV;
  float* st = p.state + ((size_t)slot * p.H + hd) * DK * DV + c4;
  float4 s[kDecRows];
  auto load = [&](int r0) {
#pragma unroll
    for (int i = 0; i < kDecRows; ++i) {
      const int r = r0 + rg + i * RG;
      s[i] = (!fresh && col_ok && r < DK) ? *reinterpret_cast<const float4*>(st + (size_t)r * DV) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(0);
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (col_ok) {
    const size_t b = t * p.v_ld + (size_t)hd * DV + c4;
    v = make_float4(ldx<T>(p.v, b), ldx<T>(p.v, b + 1), ldx<T>(p.v, b + 2), ldx<T>(p.v, b + 3));
  }
  float bonus = 0.f;
  if (tid < DK) {
    const float qv = ldx<T>(p.q, t * p.q_ld + (size_t)hd * DK + tid), kv = ldx<T>(p.k, t * p.k_ld + (size_t)hd * DK + tid);
    sq[tid] = qv;
    sk[tid] = kv;
    if constexpr (CH) {
      if (p.lr.a1) {
        const size_t n = (size_t)hd * DK + tid;
        const bf16* a2 = p.lr.a2 + n * p.lr.rank;
        float z = p.lr.bias[n];
        for (int r = 0; r < p.lr.rank; ++r) z = fmaf(ldx<T>(p.lr.a1, t * p.lr.a1_ld + r), __bfloat162float(a2[r]), z);
        sw[tid] = expf(p.lr.c * mb::log_sigmoid(z));
      } else {
        sw[tid] = expf(p.log_w[(t * p.H + hd) * DK + tid]);
      }
    }
    if constexpr (BONUS) bonus = qv * p.u[hd * DK + tid] * kv;
  }
  if constexpr (BONUS) bonus = mb::block_sum(bonus, red);
  __syncthreads();
  const float wc = CH ? 0.f : p.decay[hd];
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int r0 = 0; r0 < DK; r0 += kDecRows * RG) {
    if (r0 > 0) load(r0);
#pragma unroll
    for (int i = 0; i < kDecRows; ++i) {
      const int r = r0 + rg + i * RG;
      if (r < DK) {
        const float q = sq[r], k = sk[r], w = CH ? sw[r] : wc;
        float4 x = s[i];
        if constexpr (BONUS) { o.x = fmaf(q, x.x, o.x); o.y = fmaf(q, x.y, o.y); o.z = fmaf(q, x.z, o.z); o.w = fmaf(q, x.w, o.w); }
        x.x = fmaf(w, x.x, k * v.x); x.y = fmaf(w, x.y, k * v.y); x.z = fmaf(w, x.z, k * v.z); x.w = fmaf(w, x.w, k * v.w);
        if constexpr (!BONUS) { o.x = fmaf(q, x.x, o.x); o.y = fmaf(q, x.y, o.y); o.z = fmaf(q, x.z, o.z); o.w = fmaf(q, x.w, o.w); }
        if (p.write_state && col_ok) *reinterpret_cast<float4*>(st + (size_t)r * DV) = x;
      }
    }
  }
  if (!p.write_out) return;
  *reinterpret_cast<float4*>(so + (rg * QV) * 4 + c4) = o;
  __syncthreads();
  float y = 0.f;
  if (tid < DV) {
#pragma unroll
    for (int g = 0; g < RG; ++g) y += so[g * QV * 4 + tid];
    if constexpr (BONUS) y = fmaf(bonus, ldx<T>(p.v, t * p.v_ld + (size_t)hd * DV + tid), y);
  }
  if (!nm.w) {
    if (tid < DV) p.out[(t * p.H + hd) * DV + tid] = y;
    return;
  }
  const float inv = rsqrtf(mb::block_sum(y * y, red) / (float)DV + nm.eps);
  if (tid < DV) {
    const int col = hd * DV + tid;
    const float z = ldx<T>(nm.gate, t * nm.gate_ld + col);
    const float a = nm.sigmoid_gate ? mb::sigmoid_exact(z) : mb::silu_exact(z);
    const float r = y * inv * __bfloat162float(nm.w[col]) * a * nm.scale;
    if constexpr (sizeof(T) == 2) reinterpret_cast<bf16*>(nm.out)[t * nm.out_ld + col] = __float2bfloat16(r);
    else reinterpret_cast<float*>(nm.out)[t * nm.out_ld + col] = r;
  }
}

template <typename T, bool CH, bool BONUS>
int launch_decode(const LinParams& p, const DecodeNorm& nm, int num_seqs, cudaStream_t stream) {
  const dim3 grid(p.H, num_seqs), block(256);
  const int quads = p.DV / 4;
  if (quads <= 8) return (int)mb::launch_kernel(linear_decode_kernel<T, 8, CH, BONUS>, grid, block, 0, stream, p, nm);
  if (quads <= 16) return (int)mb::launch_kernel(linear_decode_kernel<T, 16, CH, BONUS>, grid, block, 0, stream, p, nm);
  if (quads <= 32) return (int)mb::launch_kernel(linear_decode_kernel<T, 32, CH, BONUS>, grid, block, 0, stream, p, nm);
  return (int)mb::launch_kernel(linear_decode_kernel<T, 64, CH, BONUS>, grid, block, 0, stream, p, nm);
}
template <typename T>
int decode_mode(const LinParams& p, const DecodeNorm& nm, int num_seqs, cudaStream_t stream) {
  if (p.log_w || p.lr.a1) return p.u ? launch_decode<T, true, true>(p, nm, num_seqs, stream) : launch_decode<T, true, false>(p, nm, num_seqs, stream);
  return p.u ? launch_decode<T, false, true>(p, nm, num_seqs, stream) : launch_decode<T, false, false>(p, nm, num_seqs, stream);
}

template <typename T, int KG, bool CH, bool BONUS>
int launch_k(const LinParams& p, int num_seqs, cudaStream_t stream) {
  constexpr size_t smem = lin_smem<KG, CH>();
  auto kern = linear_attn_kernel<T, KG, CH, BONUS>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int VB = cols_per_cta<KG>();
  return (int)mb::launch_kernel(kern, dim3((p.DV + VB - 1) / VB, p.H, num_seqs), dim3(32 * (kNW + kPW)), smem, stream, p);
}
template <typename T, bool CH, bool BONUS>
int launch_kg(const LinParams& p, int num_seqs, cudaStream_t stream) {
  if (p.DK <= 16) return launch_k<T, 2, CH, BONUS>(p, num_seqs, stream);
  if (p.DK <= 32) return launch_k<T, 4, CH, BONUS>(p, num_seqs, stream);
  if (p.DK <= 64) return launch_k<T, 8, CH, BONUS>(p, num_seqs, stream);
  if (p.DK <= 128) return launch_k<T, 16, CH, BONUS>(p, num_seqs, stream);
  if (p.DK <= 256) return launch_k<T, 32, CH, BONUS>(p, num_seqs, stream);
  return MB_ERR_UNSUPPORTED;
}
template <typename T>
int launch_mode(const LinParams& p, int num_seqs, cudaStream_t stream) {
  if (p.log_w) return p.u ? launch_kg<T, true, true>(p, num_seqs, stream) : launch_kg<T, true, false>(p, num_seqs, stream);
  return p.u ? launch_kg<T, false, true>(p, num_seqs, stream) : launch_kg<T, false, false>(p, num_seqs, stream);
}

}  // namespace

struct MbLinearAttnArgs {
  const void* q;
  const void* k;
  const void* v;
  long long q_ld, k_ld, v_ld;
  int H, DK, DV, f32;
  const float* log_w;
  const float* decay;
  const float* u;
  float* state;
  float* out;
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_seqs, num_slots, write_state, write_out;
  uint32_t* status;
  int decode;                // every sequence has at most one row: the streaming kernel (DV % 4 == 0, DK and DV <= 256)
  const void* norm_w;        // decode: finish the head's output (RMS, weight, gate, scale) into norm_out
  const void* gate;
  long long gate_ld;
  int sigmoid_gate;
  float eps, scale;
  void* norm_out;
  long long norm_out_ld;
  const void* lr_a1;         // decode: low-rank decays (log_w and decay null)
  long long lr_a1_ld;
  const void* lr_a2;
  const float* lr_bias;
  int lr_rank;
  float lr_c;
};

extern "C" int mb_linear_attn(const MbLinearAttnArgs* a, cudaStream_t stream) {
  if (!a || !a->q || !a->k || !a->v || !a->state || (a->write_out && !a->out && !a->norm_w) || (!a->log_w && !a->decay && !a->lr_a1)) return MB_ERR_BAD_ARG;
  if (a->H <= 0 || a->DK <= 0 || a->DV <= 0 || a->num_seqs <= 0 || a->num_seqs > 65535 || a->H > 65535) return MB_ERR_BAD_ARG;
  if (reinterpret_cast<uintptr_t>(a->state) % 16) return MB_ERR_BAD_ARG;
  LinParams p{a->q, a->k, a->v, a->q_ld, a->k_ld, a->v_ld, a->H, a->DK, a->DV, a->log_w, a->decay,
              LowRank{a->lr_a1, a->lr_a1_ld, (const bf16*)a->lr_a2, a->lr_bias, a->lr_rank, a->lr_c}, a->u, a->state, a->out, a->q_start, a->q_len, a->positions, a->slots, a->num_slots, a->write_state, a->write_out, a->status};
  if (a->lr_a1 && (!a->lr_a2 || !a->lr_bias || a->lr_rank <= 0)) return MB_ERR_BAD_ARG;
  if (a->decode) {
    if (a->DV % 4 || a->DV > 256 || a->DK > 256) return MB_ERR_UNSUPPORTED;
    if (a->norm_w && (!a->gate || !a->norm_out)) return MB_ERR_BAD_ARG;
    const DecodeNorm nm{(const bf16*)a->norm_w, a->gate, a->gate_ld, a->sigmoid_gate, a->eps, a->scale, a->norm_out, a->norm_out_ld};
    return a->f32 ? decode_mode<float>(p, nm, a->num_seqs, stream) : decode_mode<bf16>(p, nm, a->num_seqs, stream);
  }
  if (a->norm_w || a->lr_a1) return MB_ERR_UNSUPPORTED;
  return a->f32 ? launch_mode<float>(p, a->num_seqs, stream) : launch_mode<bf16>(p, a->num_seqs, stream);
}
