// Chunked prefill of decaying linear attention (the recurrences of linear_attn.cu), 64 tokens per chunk, all
// large products on the tensor cores (mma.sync m16n8k16, fp32 accumulation).
//
// With L_t the running sum of log2 decays inside a chunk (per key channel, or a multiple of the head's own):
//     end state   S' = 2^L_last S + sum_j (k_j 2^(L_last - L_j)) v_j^T
//     readout     o_i = (q_i 2^L_(i-1 | i)) S + sum_j A_ij v_j
// Three launches for the whole ragged batch:
//   chunk_state  per (chunk, head, sequence): the chunk's own contribution to the state
//   chunk_scan   per element of a head's state: the short recurrence over chunks; leaves every chunk's start
//                state as two bf16 planes (value and remainder), the final state in the pool
//   chunk_out    per (chunk, head, sequence): scores, readout of the start state, and A V
// bf16 inputs are exact tensor-core operands. 32-bit operands (decayed keys and queries, states, scores) enter
// as value + remainder, two bf16 terms with 16 mantissa bits, so a product costs two or three passes instead of
// one and keeps 32-bit quantities 32-bit to a few 1e-6.
//
// Per-channel decays make a plain factorisation q_i 2^L_i . k_j 2^-L_j overflow. The scores are built in 16 x 16
// blocks: off the diagonal both factors are taken relative to the end of the block before the query's, so both
// exponents are <= 0; on the diagonal the decay between j and i is multiplied up step by step, without a logarithm
// or an exponential. Modes: per-head decay read after the update, per-channel decay read after it or, with a bonus,
// before it.
// Head sizes 64 and 128. Sequence s keeps its chunks from index q_start[s] / 64 + s on, which never overlaps.
#include "common.cuh"

namespace {

using bf16 = __nv_bfloat16;
constexpr int kC = 64;

struct ChunkParams {
  const bf16* q;
  const bf16* k;
  const bf16* v;
  long long q_ld, k_ld, v_ld;
  int H;
  const float* log_w;          // [T, H * DK] or null
  const float* decay;          // [H] when log_w is null
  const float* u;              // [H, DK]: bonus readout (with log_w)
  float* state;                // [slots, H, DK, DV]
  float* out;                  // [T, H * DV]
  float* ws_c;                 // [chunks, H, DK * DV] contributions
  bf16* ws_hi;                 // [chunks, H, DK * DV] start states, value ...
  bf16* ws_lo;                 // ... and remainder
  float* ws_d;                 // [chunks, H, DK] decay of a whole chunk
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_slots, write_state;
  uint32_t* status;
};

constexpr float kLog2e = 1.4426950408889634f;
// A step's log2 decay counts as at least this in running sums: 2^-40 is nothing next to the step's own key, and
// the sums stay small enough for their differences to be exact.
constexpr float kMinLog = -40.f;
__device__ __forceinline__ float head_log(float decay) { return fmaxf(log2f(decay), -140.f); }

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mb::smem_u32(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mb::smem_u32(p)));
}
__device__ __forceinline__ void cp16(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mb::smem_u32(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
// (a, b) -> packed bf16 pair, and the packed pair of what rounding took off
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 bf2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

// rows [0, 64) of one head's D columns into padded shared rows (zero past `valid`)
template <int D>
__device__ __forceinline__ void stage_rows(bf16 (*dst)[D + 8], const bf16* src, long long ld, int valid) {
  for (int i = threadIdx.x; i < kC * (D / 8); i += 256) {
    const int r = i / (D / 8), c = i - r * (D / 8);
    const bool ok = r < valid;
    cp16(&dst[r][c * 8], src + (ok ? (size_t)r * ld + c * 8 : 0), ok);
  }
}
// running sums of log2 decays over the chunk's tokens; rows past `valid` repeat the last. All 256 threads: 256 / D
// groups of rows side by side, joined through each group's last row. Ends with a barrier.
template <int D>
__device__ __forceinline__ void running_logs(float (*sL)[D + 4], const float* lw, size_t ld, int valid) {
  constexpr int kR = kC * D / 256;
  const int d = threadIdx.x % D, grp = threadIdx.x / D, r0 = grp * kR;
  float v[kR];
#pragma unroll
  for (int i = 0; i < kR; ++i) v[i] = r0 + i < valid ? fmaxf(lw[(size_t)(r0 + i) * ld + d] * kLog2e, kMinLog) : 0.f;
#pragma unroll
  for (int i = 1; i < kR; ++i) v[i] += v[i - 1];
  sL[r0 + kR - 1][d] = v[kR - 1];
  __syncthreads();
  float before = 0.f;
  for (int g = 0; g < grp; ++g) before += sL[g * kR + kR - 1][d];
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kR; ++i) sL[r0 + i][d] = before + v[i];
  __syncthreads();
}

// ------------------------------------------------------------------ a chunk's contribution to the state
template <int DK, int DV>
struct StateSmem {
  bf16 kh[kC][DK + 8], kl[kC][DK + 8], v[kC][DV + 8];
  float L[kC][DK + 4];
};

template <int DK, int DV, bool CH>
__global__ void __launch_bounds__(256) chunk_state_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) uint8_t raw[];
  auto& s = *reinterpret_cast<StateSmem<DK, DV>*>(raw);
  const int c = blockIdx.x, hd = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (c * kC >= n) return;
  const int t0 = p.q_start[seq] + c * kC, valid = min(kC, n - c * kC);
  const size_t ci = ((size_t)(p.q_start[seq] / kC + seq + c)) * p.H + hd;
  stage_rows<DK>(s.kh, p.k + (size_t)t0 * p.k_ld + (size_t)hd * DK, p.k_ld, valid);
  stage_rows<DV>(s.v, p.v + (size_t)t0 * p.v_ld + (size_t)hd * DV, p.v_ld, valid);
  asm volatile("cp.async.commit_group;" ::: "memory");
  float ld2 = 0.f;
  if constexpr (CH) running_logs<DK>(s.L, p.log_w + ((size_t)t0 * p.H + hd) * DK, (size_t)p.H * DK, valid);
  else ld2 = head_log(p.decay[hd]);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  // keys decayed to the end of the chunk, value and remainder
  for (int i = tid; i < kC * (DK / 2); i += 256) {
    const int r = i / (DK / 2), d = (i - r * (DK / 2)) * 2;
    const float2 kv = bf2(&s.kh[r][d]);
    float fa, fb;
    if constexpr (CH) {
      fa = ex2(s.L[kC - 1][d] - s.L[r][d]);
      fb = ex2(s.L[kC - 1][d + 1] - s.L[r][d + 1]);
    } else {
      fa = fb = exp2f((float)(valid - 1 - r) * ld2);     // rows past valid hold zero keys
    }
    uint32_t hi, lo;
    split2(r < valid ? kv.x * fa : 0.f, r < valid ? kv.y * fb : 0.f, hi, lo);
    *reinterpret_cast<uint32_t*>(&s.kh[r][d]) = hi;
    *reinterpret_cast<uint32_t*>(&s.kl[r][d]) = lo;
  }
  if (tid < DK) p.ws_d[ci * DK + tid] = CH ? ex2(s.L[kC - 1][tid]) : exp2f((float)valid * ld2);
  __syncthreads();
  constexpr int kMB = DK / 16, kCW = 8 / kMB, kN = DV / 8 / kCW;      // m blocks, column groups of warps, n8 tiles per warp
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int m0 = (warp % kMB) * 16, n0 = (warp / kMB) * kN * 8;
  float acc[kN][4];
#pragma unroll
  for (int i = 0; i < kN; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
  for (int k0 = 0; k0 < kC; k0 += 16) {
    uint32_t ah[4], al[4];
    const int ar = k0 + (lane >> 4) * 8 + (lane & 7), ac = m0 + ((lane >> 3) & 1) * 8;
    ldsm4t(ah, &s.kh[ar][ac]);
    ldsm4t(al, &s.kl[ar][ac]);
#pragma unroll
    for (int i = 0; i < kN; i += 2) {
      uint32_t b[4];
      ldsm4t(b, &s.v[k0 + (lane & 15)][n0 + i * 8 + (lane >> 4) * 8]);
      mma(acc[i], ah, b[0], b[1]);
      mma(acc[i], al, b[0], b[1]);
      mma(acc[i + 1], ah, b[2], b[3]);
      mma(acc[i + 1], al, b[2], b[3]);
    }
  }
  float* dst = p.ws_c + ci * (DK * DV);
#pragma unroll
  for (int i = 0; i < kN; ++i) {
    *reinterpret_cast<float2*>(dst + (m0 + g) * DV + n0 + i * 8 + 2 * t) = make_float2(acc[i][0], acc[i][1]);
    *reinterpret_cast<float2*>(dst + (m0 + g + 8) * DV + n0 + i * 8 + 2 * t) = make_float2(acc[i][2], acc[i][3]);
  }
}

// ------------------------------------------------------------------ recurrence over chunks
template <int DK, int DV>
__global__ void __launch_bounds__(256) chunk_scan_kernel(const ChunkParams p) {
  const int hd = blockIdx.y, seq = blockIdx.z;
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;          // four consecutive value columns of one key row
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (n <= 0) return;
  const int slot = p.slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (p.status && threadIdx.x == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    return;
  }
  const int row = e / DV;
  float4* st = reinterpret_cast<float4*>(p.state + ((size_t)slot * p.H + hd) * (DK * DV) + e);
  float4 h = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.positions[p.q_start[seq]] != 0) h = *st;
  const int chunks = (n + kC - 1) / kC;
  const size_t c0 = (size_t)(p.q_start[seq] / kC + seq);
#pragma unroll 4
  for (int c = 0; c < chunks; ++c) {
    const size_t ci = (c0 + c) * p.H + hd;
    const float4 w = *reinterpret_cast<const float4*>(p.ws_c + ci * (DK * DV) + e);
    const float d = p.ws_d[ci * DK + row];
    uint2 hi, lo;
    split2(h.x, h.y, hi.x, lo.x);
    split2(h.z, h.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(p.ws_hi + ci * (DK * DV) + e) = hi;
    *reinterpret_cast<uint2*>(p.ws_lo + ci * (DK * DV) + e) = lo;
    h.x = fmaf(d, h.x, w.x); h.y = fmaf(d, h.y, w.y); h.z = fmaf(d, h.z, w.z); h.w = fmaf(d, h.w, w.w);
  }
  if (p.write_state) *st = h;
}

// ------------------------------------------------------------------ outputs of a chunk
// The scores are built first, from q, k and the logs. Then the decayed queries replace q and k (value and remainder)
// and the logs' space takes the start state, 64 key rows at a time: 105 KB at 128 x 128, two CTAs per SM, so that one
// CTA's loads run under the other's products.
template <int DK, int DV>
struct OutSmem {
  bf16 q[kC][DK + 8], k[kC][DK + 8], v[kC][DV + 8];
  bf16 ah[kC][kC + 8], al[kC][kC + 8];              // scores, value and remainder
  union {
    float L[kC][DK + 4];                            // per-channel mode: decays of each step, then their running logs
    struct { bf16 h[64][DV + 8], l[64][DV + 8]; } st;
  };
};

// sum over the 32 lanes of each of 16 values; lane l returns value l & 15
__device__ __forceinline__ float reduce16(float (&v)[16], int lane) {
#pragma unroll
  for (int o = 8; o >= 1; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < o) {
        const float send = up ? v[i] : v[i + o];
        const float keep = up ? v[i + o] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
  }
  return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 16);
}

template <int DK, int DV, bool CH, bool BONUS>
__global__ void __launch_bounds__(256, 2) chunk_out_kernel(const ChunkParams p) {
  extern __shared__ __align__(16) uint8_t raw[];
  auto& s = *reinterpret_cast<OutSmem<DK, DV>*>(raw);
  const int c = blockIdx.x, hd = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (c * kC >= n) return;
  const int t0 = p.q_start[seq] + c * kC, valid = min(kC, n - c * kC);
  const size_t ci = ((size_t)(p.q_start[seq] / kC + seq + c)) * p.H + hd;
  stage_rows<DK>(s.q, p.q + (size_t)t0 * p.q_ld + (size_t)hd * DK, p.q_ld, valid);
  stage_rows<DK>(s.k, p.k + (size_t)t0 * p.k_ld + (size_t)hd * DK, p.k_ld, valid);
  asm volatile("cp.async.commit_group;" ::: "memory");
  stage_rows<DV>(s.v, p.v + (size_t)t0 * p.v_ld + (size_t)hd * DV, p.v_ld, valid);
  asm volatile("cp.async.commit_group;" ::: "memory");
  const bf16 *gh = p.ws_hi + ci * (DK * DV), *gl = p.ws_lo + ci * (DK * DV);
  auto stage_state = [&](int row0) {
    for (int i = tid; i < 64 * (DV / 8); i += 256) {
      const int r = i / (DV / 8), cc = (i - r * (DV / 8)) * 8;
      cp16(&s.st.h[r][cc], gh + (row0 + r) * DV + cc, true);
      cp16(&s.st.l[r][cc], gl + (row0 + r) * DV + cc, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if constexpr (!CH) stage_state(0);                                  // nothing else needs that space
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int rb = warp & 3, half = warp >> 2, i0 = rb * 16;            // this warp's 16 tokens and column half
  const float ld2 = CH ? 0.f : head_log(p.decay[hd]);
  const float* lw = CH ? p.log_w + ((size_t)t0 * p.H + hd) * DK : nullptr;

  if constexpr (CH) {
    for (int i = tid; i < kC * DK; i += 256) {
      const int r = i / DK, d = i - r * DK;
      s.L[r][d] = r < valid ? ex2(lw[(size_t)r * p.H * DK + d] * kLog2e) : 1.f;
    }
  }
  asm volatile("cp.async.wait_group %0;" ::"n"(CH ? 1 : 2) : "memory");
  __syncthreads();
  if constexpr (CH) {
    // ---- diagonal blocks: key j times the decays of the steps between j and i, multiplied up step by step
    constexpr int kCh = DK / 32;
    float uu[kCh];
#pragma unroll
    for (int e = 0; e < kCh; ++e) uu[e] = BONUS ? p.u[hd * DK + e * 32 + lane] : 1.f;
    for (int j = half; j < 16; j += 2) {
      float kk[kCh], val[16];
#pragma unroll
      for (int e = 0; e < kCh; ++e) kk[e] = __bfloat162float(s.k[i0 + j][e * 32 + lane]);
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        val[i] = 0.f;
        if (i >= j) {
#pragma unroll
          for (int e = 0; e < kCh; ++e) {
            const float qv = __bfloat162float(s.q[i0 + i][e * 32 + lane]);
            if (i == j) {
              val[i] = fmaf(qv * uu[e], kk[e], val[i]);              // the bonus stands in for the token itself
            } else if constexpr (!BONUS) {
              kk[e] *= s.L[i0 + i][e * 32 + lane];                   // read after step i's decay
              val[i] = fmaf(qv, kk[e], val[i]);
            } else {
              val[i] = fmaf(qv, kk[e], val[i]);
              kk[e] *= s.L[i0 + i][e * 32 + lane];
            }
          }
        }
      }
      const float a = reduce16(val, lane);
      if (lane < 16) {
        const bf16 h = __float2bfloat16(a);
        s.ah[i0 + lane][i0 + j] = h;
        s.al[i0 + lane][i0 + j] = __float2bfloat16(a - __bfloat162float(h));
      }
    }
    __syncthreads();
    running_logs<DK>(s.L, lw, (size_t)p.H * DK, valid);
  }
  // query fragments of this warp's rows decayed from the reference on: q_i 2^(L_(i-1) - ref), or L_i when read after
  // the update; value and remainder
  constexpr int kBefore = BONUS ? 1 : 0;
  auto q_frag = [&](int k0, const float* refL, uint32_t* hi, uint32_t* lo) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = i0 + g + (e & 1) * 8, d = k0 + 2 * t + (e >> 1) * 8;
      const float2 qv = bf2(&s.q[i][d]);
      float la = 0.f, lb = 0.f;
      if (i >= kBefore) {
        la = s.L[i - kBefore][d];
        lb = s.L[i - kBefore][d + 1];
      }
      la -= refL[d];
      lb -= refL[d + 1];
      split2(qv.x * ex2(la), qv.y * ex2(lb), hi[e], lo[e]);
    }
  };
  auto put = [&](int i, int j, float a, float b) {
    uint32_t hi, lo;
    split2(a, b, hi, lo);
    *reinterpret_cast<uint32_t*>(&s.ah[i][j]) = hi;
    *reinterpret_cast<uint32_t*>(&s.al[i][j]) = lo;
  };
  // ---- scores of this warp's rows; its half takes 8 of the 16 columns of every block
  if constexpr (CH) {
    if (rb > 0) {
      const float* refL = s.L[i0 - 1];
      float acc[3][4];
#pragma unroll
      for (int J = 0; J < 3; ++J)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[J][e] = 0.f;
      for (int k0 = 0; k0 < DK; k0 += 16) {
        uint32_t hi[4], lo[4];
        q_frag(k0, refL, hi, lo);
#pragma unroll
        for (int J = 0; J < 3; ++J) {
          if (J < rb) {
            const int j = J * 16 + half * 8 + g;
            uint32_t bh[2], bl[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int d = k0 + 2 * t + e * 8;
              const float2 kv = bf2(&s.k[j][d]);
              split2(kv.x * ex2(refL[d] - s.L[j][d]), kv.y * ex2(refL[d + 1] - s.L[j][d + 1]), bh[e], bl[e]);
            }
            mma(acc[J], hi, bh[0], bh[1]);
            mma(acc[J], hi, bl[0], bl[1]);
            mma(acc[J], lo, bh[0], bh[1]);
          }
        }
      }
#pragma unroll
      for (int J = 0; J < 3; ++J)
        if (J < rb) {
          const int j = J * 16 + half * 8 + 2 * t;
          put(i0 + g, j, acc[J][0], acc[J][1]);
          put(i0 + g + 8, j, acc[J][2], acc[J][3]);
        }
    }
  } else {
    float acc[4][4];
#pragma unroll
    for (int J = 0; J < 4; ++J)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[J][e] = 0.f;
    for (int k0 = 0; k0 < DK; k0 += 16) {
      uint32_t a[4];
      ldsm4(a, &s.q[i0 + (lane & 15)][k0 + (lane >> 4) * 8]);
#pragma unroll
      for (int J = 0; J < 4; ++J)
        if (J <= rb) {
          const bf16* kr = &s.k[J * 16 + half * 8 + g][k0 + 2 * t];
          mma(acc[J], a, *reinterpret_cast<const uint32_t*>(kr), *reinterpret_cast<const uint32_t*>(kr + 8));
        }
    }
#pragma unroll
    for (int J = 0; J < 4; ++J)
      if (J <= rb) {
        const int j = J * 16 + half * 8 + 2 * t;
#pragma unroll
        for (int hr = 0; hr < 2; ++hr) {
          const int i = i0 + g + hr * 8;
          put(i, j, j <= i ? acc[J][hr * 2] * exp2f((float)(i - j) * ld2) : 0.f,
              j + 1 <= i ? acc[J][hr * 2 + 1] * exp2f((float)(i - j - 1) * ld2) : 0.f);
        }
      }
  }
  // ---- per-channel mode: q and k become the queries decayed from the chunk's start, value and remainder
  if constexpr (CH) {
    __syncthreads();
    for (int i = tid; i < kC * (DK / 2); i += 256) {
      const int r = i / (DK / 2), d = (i - r * (DK / 2)) * 2;
      const float2 qv = bf2(&s.q[r][d]);
      float la = 0.f, lb = 0.f;
      if (r >= kBefore) {
        la = s.L[r - kBefore][d];
        lb = s.L[r - kBefore][d + 1];
      }
      split2(qv.x * ex2(la), qv.y * ex2(lb), *reinterpret_cast<uint32_t*>(&s.q[r][d]), *reinterpret_cast<uint32_t*>(&s.k[r][d]));
    }
    __syncthreads();
    stage_state(0);
  }
  // ---- o = (decayed q) S + A V for 16 rows and DV / 2 columns
  constexpr int kN = DV / 16;
  const int n0 = half * (DV / 2);
  float o[kN][4];
#pragma unroll
  for (int i = 0; i < kN; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  for (int row0 = 0; row0 < DK; row0 += 64) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 64; kk += 16) {
      uint32_t hi[4], lo[4];
      ldsm4(hi, &s.q[i0 + (lane & 15)][row0 + kk + (lane >> 4) * 8]);
      if constexpr (CH) ldsm4(lo, &s.k[i0 + (lane & 15)][row0 + kk + (lane >> 4) * 8]);
#pragma unroll
      for (int i = 0; i < kN; i += 2) {
        uint32_t bh[4], bl[4];
        const int r = kk + (lane & 15), cc = n0 + i * 8 + (lane >> 4) * 8;
        ldsm4t(bh, &s.st.h[r][cc]);
        ldsm4t(bl, &s.st.l[r][cc]);
        mma(o[i], hi, bh[0], bh[1]);
        mma(o[i + 1], hi, bh[2], bh[3]);
        mma(o[i], hi, bl[0], bl[1]);
        mma(o[i + 1], hi, bl[2], bl[3]);
        if constexpr (CH) {
          mma(o[i], lo, bh[0], bh[1]);
          mma(o[i + 1], lo, bh[2], bh[3]);
        }
      }
    }
    if (row0 + 64 < DK) {
      __syncthreads();
      stage_state(row0 + 64);
    }
  }
  if constexpr (!CH) {
    const float f0 = exp2f((float)(i0 + g + 1) * ld2), f1 = exp2f((float)(i0 + g + 9) * ld2);
#pragma unroll
    for (int i = 0; i < kN; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
  }
  for (int k0 = 0; k0 <= i0; k0 += 16) {
    uint32_t ah[4], al[4];
    ldsm4(ah, &s.ah[i0 + (lane & 15)][k0 + (lane >> 4) * 8]);
    ldsm4(al, &s.al[i0 + (lane & 15)][k0 + (lane >> 4) * 8]);
#pragma unroll
    for (int i = 0; i < kN; i += 2) {
      uint32_t b[4];
      ldsm4t(b, &s.v[k0 + (lane & 15)][n0 + i * 8 + (lane >> 4) * 8]);
      mma(o[i], ah, b[0], b[1]);
      mma(o[i], al, b[0], b[1]);
      mma(o[i + 1], ah, b[2], b[3]);
      mma(o[i + 1], al, b[2], b[3]);
    }
  }
#pragma unroll
  for (int hr = 0; hr < 2; ++hr) {
    const int i = i0 + g + hr * 8;
    if (i >= valid) continue;
    float* dst = p.out + ((size_t)(t0 + i) * p.H + hd) * DV + n0 + 2 * t;
#pragma unroll
    for (int e = 0; e < kN; ++e) *reinterpret_cast<float2*>(dst + e * 8) = make_float2(o[e][hr * 2], o[e][hr * 2 + 1]);
  }
}

template <int DK, int DV, bool CH, bool BONUS>
int launch_chunks(const ChunkParams& p, int num_seqs, int max_q_len, cudaStream_t stream) {
  using SS = StateSmem<DK, DV>;
  using SO = OutSmem<DK, DV>;
  const size_t ss = CH ? sizeof(SS) : offsetof(SS, L), so = sizeof(SO);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(chunk_state_kernel<DK, DV, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ss);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(chunk_out_kernel<DK, DV, CH, BONUS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)so);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((max_q_len + kC - 1) / kC, p.H, num_seqs);
  cudaError_t e = mb::launch_kernel(chunk_state_kernel<DK, DV, CH>, grid, dim3(256), ss, stream, p);
  if (e == cudaSuccess) e = mb::launch_kernel(chunk_scan_kernel<DK, DV>, dim3(DK * DV / 1024, p.H, num_seqs), dim3(256), 0, stream, p);
  if (e == cudaSuccess) e = mb::launch_kernel(chunk_out_kernel<DK, DV, CH, BONUS>, grid, dim3(256), so, stream, p);
  return (int)e;
}
template <bool CH, bool BONUS>
int dispatch_dims(const ChunkParams& p, int DK, int DV, int num_seqs, int max_q_len, cudaStream_t stream) {
  if (DK == 64 && DV == 64) return launch_chunks<64, 64, CH, BONUS>(p, num_seqs, max_q_len, stream);
  if (DK == 64 && DV == 128) return launch_chunks<64, 128, CH, BONUS>(p, num_seqs, max_q_len, stream);
  if (DK == 128 && DV == 64) return launch_chunks<128, 64, CH, BONUS>(p, num_seqs, max_q_len, stream);
  if (DK == 128 && DV == 128) return launch_chunks<128, 128, CH, BONUS>(p, num_seqs, max_q_len, stream);
  return MB_ERR_UNSUPPORTED;
}

}  // namespace

struct MbLinearChunkedArgs {
  const void* q;
  const void* k;
  const void* v;
  long long q_ld, k_ld, v_ld;
  int H, DK, DV, total_rows;
  const float* log_w;
  const float* decay;
  const float* u;
  float* state;
  float* out;
  void* ws;
  size_t ws_bytes;
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_seqs, num_slots, max_q_len, write_state;
  uint32_t* status;
};

extern "C" size_t mb_linear_chunked_ws_bytes(int total_rows, int num_seqs, int H, int DK, int DV) {
  return ((size_t)total_rows / kC + num_seqs) * H * ((size_t)DK * DV * 8 + DK * 4) + 1024;
}

extern "C" int mb_linear_chunked(const MbLinearChunkedArgs* a, cudaStream_t stream) {
  if (!a || !a->q || !a->k || !a->v || !a->state || !a->out || !a->ws) return MB_ERR_BAD_ARG;
  if (a->num_seqs <= 0 || a->num_seqs > 65535 || a->H <= 0 || a->H > 65535 || a->max_q_len <= 0 || a->total_rows <= 0) return MB_ERR_BAD_ARG;
  if ((a->u && !a->log_w) || (!a->log_w && !a->decay)) return MB_ERR_UNSUPPORTED;
  const uintptr_t al = reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->k) | reinterpret_cast<uintptr_t>(a->v) |
                       reinterpret_cast<uintptr_t>(a->state) | reinterpret_cast<uintptr_t>(a->out) | reinterpret_cast<uintptr_t>(a->ws);
  if ((al & 15) || (a->q_ld | a->k_ld | a->v_ld) % 8) return MB_ERR_UNSUPPORTED;      // 16-byte copies
  if (a->ws_bytes < mb_linear_chunked_ws_bytes(a->total_rows, a->num_seqs, a->H, a->DK, a->DV)) return MB_ERR_TOO_LARGE;
  ChunkParams p{};
  p.q = (const bf16*)a->q; p.k = (const bf16*)a->k; p.v = (const bf16*)a->v;
  p.q_ld = a->q_ld; p.k_ld = a->k_ld; p.v_ld = a->v_ld; p.H = a->H;
  p.log_w = a->log_w; p.decay = a->decay; p.u = a->u; p.state = a->state; p.out = a->out;
  const size_t chunks = ((size_t)a->total_rows / kC + a->num_seqs) * a->H, per = (size_t)a->DK * a->DV;
  p.ws_c = reinterpret_cast<float*>(a->ws);
  p.ws_hi = reinterpret_cast<bf16*>(p.ws_c + chunks * per);
  p.ws_lo = p.ws_hi + chunks * per;
  p.ws_d = reinterpret_cast<float*>(p.ws_lo + chunks * per);
  p.q_start = a->q_start; p.q_len = a->q_len; p.positions = a->positions; p.slots = a->slots;
  p.num_slots = a->num_slots; p.write_state = a->write_state; p.status = a->status;
  if (a->u) return dispatch_dims<true, true>(p, a->DK, a->DV, a->num_seqs, a->max_q_len, stream);
  return a->log_w ? dispatch_dims<true, false>(p, a->DK, a->DV, a->num_seqs, a->max_q_len, stream)
                  : dispatch_dims<false, false>(p, a->DK, a->DV, a->num_seqs, a->max_q_len, stream);
}
