// Chunked prefill of the delta rules of delta_attn.cu, 64 tokens per chunk, all large products on the tensor cores
// (mma.sync m16n8k16, fp32 accumulation).
//
// Over a chunk with start state S0, the rows X_j that the rule adds to the state (besides k v^T in the general rule) solve
// a unit lower-triangular system, so with M = (I + A)^-1
//     X = Xw S0 + Xu        o = R' S0 + O'        S' = diag(d) S0 + T S0 + E
// and everything but S0 is known without the state:
//   general  (L the running sums of log2 decays per key channel, L_-1 = 0; d = 2^L_last)
//     U_i = u_i 2^L_(i-1)   R_i = r_i 2^L_i   B_j = a_j u_j 2^-L_j   K_j = k_j 2^-L_j
//     A = tril(U B^T, -1)   Xw = -M U   Xu = -M tril(U K^T, -1) V
//     Q = tril(R B^T)       R' = R + Q Xw   O' = tril(R K^T) V + Q Xu
//     T = diag(d) B^T Xw    E = diag(d) (K^T V + B^T Xu)
//     The decays are bounded below (at most 100 octaves in a chunk), so no factor overflows.
//   gated    (G the running sums of one log2 decay per token; d = 2^G_last)
//     A_ij = beta_i 2^(G_i - G_j) k_i.k_j (j < i)   Xw = -M diag(beta 2^G) K   Xu = M diag(beta) V
//     Q_ij = 2^(G_i - G_j) q_i.k_j (j <= i)         R' = diag(2^G) q + Q Xw    O' = Q Xu
//     T = k^T diag(2^(G_last - G)) Xw               E = k^T diag(2^(G_last - G)) Xu
//     Every exponent is <= 0 however strong the decay.
// Three launches for the whole ragged batch:
//   delta_prep  per (chunk, head, sequence): all of the above into a workspace
//   delta_scan  per (16 or 32 value columns, head, sequence): the recurrence over chunks, S in registers; leaves every chunk's
//               start state as two bf16 planes (value and remainder), the final state in the pool
//   delta_out   per (chunk, head, sequence): o, optionally finished by the head's gated RMS norm
// Values are exact bf16 operands, and so are the gated rule's queries and keys (their lengths enter as factors, above
// written into k and q); every other one is 32-bit and enters as value + remainder (16 mantissa bits), so a product
// costs two or three passes and keeps 32-bit quantities 32-bit to a few 1e-6. The triangular inverse is fp32, by 16 x 16
// blocks. Head sizes 64 and 128. Sequence s keeps its chunks from index q_start[s] / 64 + s on, which never overlaps.
#include "common.cuh"
#include "delta_attn.cuh"
#include "epilogue.cuh"

namespace {

using bf16 = __nv_bfloat16;
using mb::DeltaInputs;
constexpr int kC = 64;
constexpr float kLog2e = 1.4426950408889634f;

struct ChunkParams {
  DeltaInputs in;
  float* state;                // [slots, H, DK, DV]
  float* out;                  // [T, H DV], or null with a norm
  // T, R', E and O' are kept as the tensor cores' fragments, a warp's accumulators one vector per lane: see put_frag, put_c
  uint4* ws_t;                 // [chunks, H] of DK x DK, two planes
  float4* ws_e;                // [chunks, H] of DK x DV
  bf16* ws_s;                  // [chunks, H, 2 planes, DK, DV] start states
  uint4* ws_r;                 // [chunks, H] of 64 x DK, two planes
  float4* ws_o;                // [chunks, H] of 64 x DV
  float* ws_d;                 // [chunks, H, DK]
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_slots, write_state;
  uint32_t* status;
  const bf16* norm_w;          // [H DV] or null
  const bf16* gate;
  long long gate_ld;
  int sigmoid_gate;
  float eps, scale;
  bf16* norm_out;
  long long norm_out_ld;
};

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
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mb::smem_u32(p)) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(mb::smem_u32(p)) : "memory");
}
__device__ __forceinline__ void cp16(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(mb::smem_u32(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
// (a, b) -> packed bf16 pair, and the packed pair of what rounding took off
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
// two planes of a matrix in shared or global memory, ld elements per row
struct Planes {
  bf16* hi;
  bf16* lo;
  int ld;
  __device__ __forceinline__ void put(int r, int c, float a, float b) const {
    uint32_t h, l;
    split2(a, b, h, l);
    *reinterpret_cast<uint32_t*>(hi + (size_t)r * ld + c) = h;
    *reinterpret_cast<uint32_t*>(lo + (size_t)r * ld + c) = l;
  }
  __device__ __forceinline__ float2 get(int r, int c) const {
    const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(hi + (size_t)r * ld + c));
    const float2 l = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(lo + (size_t)r * ld + c));
    return make_float2(h.x + l.x, h.y + l.y);
  }
};

// acc (16 rows m0 .., 8 N8 columns n0 ..) += A B over k in [k0, k1): A is [row][k], or [k][row] with AT; B is [k][column];
// exact (one plane) without AL, BL
template <int N8, bool AT, bool BL, bool AL = true>
__device__ __forceinline__ void mm(float (*acc)[4], const Planes& A, int m0, const Planes& B, int n0, int k0, int k1) {
  const int lane = threadIdx.x & 31;
#pragma unroll 2
  for (int k = k0; k < k1; k += 16) {
    uint32_t ah[4], al[4];
    if constexpr (AT) {
      const size_t o = (size_t)(k + (lane >> 4) * 8 + (lane & 7)) * A.ld + m0 + ((lane >> 3) & 1) * 8;
      ldsm4t(ah, A.hi + o);
      if constexpr (AL) ldsm4t(al, A.lo + o);
    } else {
      const size_t o = (size_t)(m0 + (lane & 15)) * A.ld + k + (lane >> 4) * 8;
      ldsm4(ah, A.hi + o);
      if constexpr (AL) ldsm4(al, A.lo + o);
    }
#pragma unroll
    for (int i = 0; i < N8; i += 2) {
      uint32_t b[4];
      const size_t o = (size_t)(k + (lane & 15)) * B.ld + n0 + i * 8 + (lane >> 4) * 8;
      ldsm4t(b, B.hi + o);
      mma(acc[i], ah, b[0], b[1]);
      mma(acc[i + 1], ah, b[2], b[3]);
      if constexpr (AL) {
        mma(acc[i], al, b[0], b[1]);
        mma(acc[i + 1], al, b[2], b[3]);
      }
      if constexpr (BL) {
        ldsm4t(b, B.lo + o);
        mma(acc[i], ah, b[0], b[1]);
        mma(acc[i + 1], ah, b[2], b[3]);
      }
    }
  }
}
template <int N8>
__device__ __forceinline__ void zero(float (*acc)[4]) {
#pragma unroll
  for (int i = 0; i < N8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
}
// the accumulators (times f) into planes
template <int N8>
__device__ __forceinline__ void put_acc(const Planes& P, int m0, int n0, const float (*acc)[4], float f) {
  const int lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int i = 0; i < N8; ++i) {
    P.put(m0 + g, n0 + i * 8 + 2 * t, acc[i][0] * f, acc[i][1] * f);
    P.put(m0 + g + 8, n0 + i * 8 + 2 * t, acc[i][2] * f, acc[i][3] * f);
  }
}

// Fragments: a 16 x 16 block of an A operand is four registers per lane, which are the accumulators of two neighbouring
// 8-column tiles. Block (row block, column block) of a matrix of `blocks` column blocks: value plane, then remainder, a
// 16-byte vector per lane.
template <int N8>
__device__ __forceinline__ void put_frag(uint4* dst, int blocks, int m0, int n0, const float (*acc)[4]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int i = 0; i < N8; i += 2) {
    uint4 h, l;
    split2(acc[i][0], acc[i][1], h.x, l.x);
    split2(acc[i][2], acc[i][3], h.y, l.y);
    split2(acc[i + 1][0], acc[i + 1][1], h.z, l.z);
    split2(acc[i + 1][2], acc[i + 1][3], h.w, l.w);
    uint4* d = dst + ((size_t)((m0 >> 4) * blocks + (n0 >> 4) + (i >> 1)) * 2) * 32 + lane;
    d[0] = h;
    d[32] = l;
  }
}
// acc += A B with A's blocks as above, `frag` at this warp's row of blocks
template <int N8>
__device__ __forceinline__ void mm_frag(float (*acc)[4], const uint4* frag, const Planes& B, int n0, int blocks) {
  const int lane = threadIdx.x & 31;
#pragma unroll 2
  for (int kb = 0; kb < blocks; ++kb) {
    const uint4 h = frag[kb * 64 + lane], l = frag[kb * 64 + 32 + lane];
    const uint32_t ah[4] = {h.x, h.y, h.z, h.w}, al[4] = {l.x, l.y, l.z, l.w};
#pragma unroll
    for (int i = 0; i < N8; i += 2) {
      uint32_t b[4];
      const size_t o = (size_t)(kb * 16 + (lane & 15)) * B.ld + n0 + i * 8 + (lane >> 4) * 8;
      ldsm4t(b, B.hi + o);
      mma(acc[i], ah, b[0], b[1]);
      mma(acc[i + 1], ah, b[2], b[3]);
      mma(acc[i], al, b[0], b[1]);
      mma(acc[i + 1], al, b[2], b[3]);
      ldsm4t(b, B.lo + o);
      mma(acc[i], ah, b[0], b[1]);
      mma(acc[i + 1], ah, b[2], b[3]);
    }
  }
}
// accumulators of 8-column tiles, tile (row block, column tile) of a matrix of `tiles` column tiles a vector per lane
template <int N8>
__device__ __forceinline__ void put_c(float4* dst, int tiles, int m0, int n0, const float (*acc)[4]) {
#pragma unroll
  for (int i = 0; i < N8; ++i)
    dst[(size_t)((m0 >> 4) * tiles + (n0 >> 3) + i) * 32 + (threadIdx.x & 31)] = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
}
template <int N8>
__device__ __forceinline__ void get_c(const float4* src, int tiles, int m0, int n0, float (*acc)[4]) {
#pragma unroll
  for (int i = 0; i < N8; ++i) {
    const float4 v = src[(size_t)((m0 >> 4) * tiles + (n0 >> 3) + i) * 32 + (threadIdx.x & 31)];
    acc[i][0] = v.x; acc[i][1] = v.y; acc[i][2] = v.z; acc[i][3] = v.w;
  }
}

// ------------------------------------------------------------------ per-chunk preparation
constexpr int kPrep = 512;         // threads
constexpr int kLdF = kC + 4;       // fp32 rows of the inverse
constexpr int kLdC = kC + 8;       // bf16 rows of 64 x 64 matrices

template <int DK, int DV>
struct PrepLayout {
  static constexpr int ldk = DK + 8, ldv = DV + 8, ldx = (DK > DV ? DK : DV) + 8;
  static constexpr size_t plane_k = (size_t)kC * ldk * 2, plane_x = (size_t)kC * ldx * 2;
  static constexpr size_t u = 0, r = 2 * plane_k, b = 4 * plane_k, k = 6 * plane_k, v = k + 2 * plane_x, z0 = v + (size_t)kC * ldv * 2;
  static constexpr size_t zsize = 2 * (size_t)kC * kLdC * 2;                   // two planes of a 64 x 64 matrix, or one in fp32
  static constexpr size_t z1 = z0 + zsize, tmp = z1 + zsize, vec = tmp + 3 * 16 * 17 * 4, bytes = vec + (DK + 5 * kC) * 4;
  static_assert(2 * zsize >= (size_t)kC * (DK + 4) * 4, "the running logs live where the 64 x 64 matrices come later");
  static_assert(zsize >= (size_t)kC * kLdF * 4, "");
};

template <int DK, int DV, bool GEN>
__global__ void __launch_bounds__(kPrep, 1) delta_prep_kernel(const ChunkParams p) {
  using Lay = PrepLayout<DK, DV>;
  extern __shared__ __align__(16) uint8_t sm[];
  const DeltaInputs& in = p.in;
  const int c = blockIdx.x, hd = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (c * kC >= n) return;
  const int t0 = p.q_start[seq] + c * kC, valid = min(kC, n - c * kC), H = in.H;
  const size_t ci = ((size_t)(p.q_start[seq] / kC + seq + c)) * H + hd;
  auto planes = [&](size_t at, int ld) { return Planes{reinterpret_cast<bf16*>(sm + at), reinterpret_cast<bf16*>(sm + at) + kC * ld, ld}; };
  const Planes U = planes(Lay::u, Lay::ldk), R = planes(Lay::r, Lay::ldk), B = planes(Lay::b, Lay::ldk), K = planes(Lay::k, Lay::ldx);
  const Planes V{reinterpret_cast<bf16*>(sm + Lay::v), nullptr, Lay::ldv};
  const Planes Z0 = planes(Lay::z0, kLdC), Z1 = planes(Lay::z1, kLdC);
  float* sA = reinterpret_cast<float*>(sm + Lay::z0);                         // [64][kLdF]
  float* sM = reinterpret_cast<float*>(sm + Lay::z1);
  float* sT = reinterpret_cast<float*>(sm + Lay::tmp);
  float* sD = reinterpret_cast<float*>(sm + Lay::vec);                         // decay of the whole chunk, [DK]
  // gated: running log2 decays (sums of strong decays grow; their differences must not lose the mild ones), step sizes
  double* sG = reinterpret_cast<double*>(sD + DK);
  float* sBeta = reinterpret_cast<float*>(sG + kC);
  float* sNk = sBeta + kC;                                                     // gated: one over the lengths of keys and queries
  float* sNq = sNk + kC;
  float* sL = sA;                                                              // general: running logs [64][DK + 4]
  constexpr int ldl = DK + 4;

  // everything the chunk reads, at once: values and the raw rows of keys, queries and removal logits (a row's owner makes
  // its operands of them in place), log decays
  auto rows_in = [&](const void* base, long long ld, int head, int D, bf16* dst, int dst_ld) {
    for (int i = tid; i < kC * (D / 8); i += kPrep) {
      const int r = i / (D / 8), cc = (i - r * (D / 8)) * 8;
      const bool ok = r < valid;
      cp16(dst + r * dst_ld + cc, reinterpret_cast<const bf16*>(base) + (ok ? (size_t)(t0 + r) * ld + (size_t)head * D + cc : 0), ok);
    }
  };
  const int hk = hd / (H / in.HK);
  rows_in(in.k, in.k_ld, hk, DK, U.hi, Lay::ldk);
  rows_in(in.q, in.q_ld, hk, DK, R.hi, Lay::ldk);
  rows_in(in.v, in.v_ld, hd, DV, V.hi, Lay::ldv);
  if constexpr (GEN) {
    rows_in(in.removal, in.removal_ld, hd, DK, B.hi, Lay::ldk);
    for (int i = tid; i < kC * (DK / 4); i += kPrep) {
      const int r = i / (DK / 4), cc = (i - r * (DK / 4)) * 4;
      const bool ok = r < valid;
      cp16(sL + r * ldl + cc, in.log_w + (ok ? ((size_t)(t0 + r) * H + hd) * DK + cc : 0), ok);
    }
  }
  cp_commit();
  if constexpr (GEN) {
    // running sums of log2 decays; rows past `valid` repeat the last
    constexpr int kR = kC * DK / kPrep;
    const int d = tid % DK, grp = tid / DK, r0 = grp * kR;
    cp_wait<0>();
    __syncthreads();
    float v[kR];
#pragma unroll
    for (int i = 0; i < kR; ++i) v[i] = sL[(r0 + i) * ldl + d] * kLog2e;
#pragma unroll
    for (int i = 1; i < kR; ++i) v[i] += v[i - 1];
    sL[(r0 + kR - 1) * ldl + d] = v[kR - 1];
    __syncthreads();
    float before = 0.f;
    for (int i = 0; i < grp; ++i) before += sL[(i * kR + kR - 1) * ldl + d];
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kR; ++i) sL[(r0 + i) * ldl + d] = before + v[i];
    __syncthreads();
    if (tid < DK) {
      sD[tid] = ex2(sL[(kC - 1) * ldl + tid]);
      p.ws_d[ci * DK + tid] = sD[tid];
    }
  } else {
    if (tid < kC) {
      double lg = 0.0;
      float beta = 0.f;
      if (tid < valid) {
        lg = (double)in.log_gate<bf16>(t0 + tid, hd) * 1.4426950408889634;
        beta = in.step_size<bf16>(t0 + tid, hd);
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, lg, o);
        if (lane >= o) lg += up;
      }
      sG[tid] = lg;
      sBeta[tid] = beta;
    }
    __syncthreads();
    if (tid >= 32 && tid < kC) sG[tid] += sG[31];
    __syncthreads();
    if (tid < DK) p.ws_d[ci * DK + tid] = ex2((float)sG[kC - 1]);
    cp_wait<0>();
    __syncthreads();
  }
  // ---- operands, a warp per row
  {
    constexpr int E = DK / 32;
    const int d0 = lane * E;
    auto load = [&](const bf16* src, float* o) {
      if constexpr (E == 4) {
        const uint2 w = *reinterpret_cast<const uint2*>(src);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w.y));
        o[0] = a.x; o[1] = a.y; o[2] = b.x; o[3] = b.y;
      } else {
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src));
        o[0] = a.x; o[1] = a.y;
      }
    };
#pragma unroll 2
    for (int i = warp; i < kC; i += kPrep / 32) {
      float q[E], k[E], a[E];
      load(R.hi + i * Lay::ldk + d0, q);
      load(U.hi + i * Lay::ldk + d0, k);
      if constexpr (GEN) load(B.hi + i * Lay::ldk + d0, a);
      float sq = 0.f, sk = 0.f;
#pragma unroll
      for (int e = 0; e < E; ++e) {
        sq = fmaf(q[e], q[e], sq);
        sk = fmaf(k[e], k[e], sk);
      }
      const float nk = rsqrtf(mb::warp_sum(sk) + mb::kUnitEps);
      if constexpr (GEN) {
        float u[E], rr[E], bb[E], kk[E];
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const float l = sL[i * ldl + d0 + e], l1 = i > 0 ? sL[(i - 1) * ldl + d0 + e] : 0.f, up = ex2(-l), un = k[e] * nk;
          u[e] = un * ex2(l1);
          rr[e] = q[e] * ex2(l);
          bb[e] = mb::sigmoid_fast(a[e]) * un * up;
          kk[e] = k[e] * up;
        }
#pragma unroll
        for (int e = 0; e < E; e += 2) {
          U.put(i, d0 + e, u[e], u[e + 1]);
          R.put(i, d0 + e, rr[e], rr[e + 1]);
          B.put(i, d0 + e, bb[e], bb[e + 1]);
          K.put(i, d0 + e, kk[e], kk[e + 1]);
        }
      } else {
        const float nq = rsqrtf(mb::warp_sum(sq) + mb::kUnitEps) * rsqrtf((float)DK);
        if (lane == 0) {                                  // the rows stay as they are, exact; their lengths enter the scores
          sNk[i] = nk;
          sNq[i] = nq;
        }
      }
    }
  }
  __syncthreads();
  // ---- scores of this warp's 16 rows and 16 columns, blocks up to the diagonal: rows U and R against columns B (and K)
  // (warps w, w + 4 ... share a scheduler: a long row block of a triangle goes with a short one)
  const int quarter = warp >> 2, rb = quarter & 1 ? 3 - (warp & 3) : warp & 3, i0 = rb * 16, j0 = quarter * 16;
  float sa[2][4], sb[GEN ? 2 : 1][4], sp[GEN ? 2 : 1][4], sq[2][4];
  zero<2>(sa);
  zero<2>(sq);
  if constexpr (GEN) {
    zero<2>(sb);
    zero<2>(sp);
  }
  const Planes& CB = GEN ? B : U;
  if (j0 <= i0) {
#pragma unroll 1
    for (int k0 = 0; k0 < DK; k0 += 16) {
      uint32_t uh[4], ul[4], rh[4], rl[4];
      const size_t o = (size_t)(i0 + (lane & 15)) * Lay::ldk + k0 + (lane >> 4) * 8;
      ldsm4(uh, U.hi + o);
      ldsm4(rh, R.hi + o);
      if constexpr (GEN) {
        ldsm4(ul, U.lo + o);
        ldsm4(rl, R.lo + o);
      }
      {
        const int row = j0 + (lane & 7) + ((lane >> 4) << 3), col = k0 + ((lane >> 3) & 1) * 8;
        uint32_t bh[4], bl[4];
        ldsm4(bh, CB.hi + (size_t)row * CB.ld + col);
        if constexpr (GEN) ldsm4(bl, CB.lo + (size_t)row * CB.ld + col);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma(sa[e], uh, bh[2 * e], bh[2 * e + 1]);
          mma(sq[e], rh, bh[2 * e], bh[2 * e + 1]);
          if constexpr (GEN) {
            mma(sa[e], uh, bl[2 * e], bl[2 * e + 1]);
            mma(sq[e], rh, bl[2 * e], bl[2 * e + 1]);
            mma(sa[e], ul, bh[2 * e], bh[2 * e + 1]);
            mma(sq[e], rl, bh[2 * e], bh[2 * e + 1]);
          }
        }
        if constexpr (GEN) {
          ldsm4(bh, K.hi + (size_t)row * K.ld + col);
          ldsm4(bl, K.lo + (size_t)row * K.ld + col);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            mma(sb[e], uh, bh[2 * e], bh[2 * e + 1]);
            mma(sp[e], rh, bh[2 * e], bh[2 * e + 1]);
            mma(sb[e], uh, bl[2 * e], bl[2 * e + 1]);
            mma(sp[e], rh, bl[2 * e], bl[2 * e + 1]);
            mma(sb[e], ul, bh[2 * e], bh[2 * e + 1]);
            mma(sp[e], rl, bh[2 * e], bh[2 * e + 1]);
          }
        }
      }
    }
  }
  __syncthreads();                                        // the logs are consumed: their space takes A
#pragma unroll
  for (int e = 0; e < 2; ++e)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int i = i0 + g + (x >> 1) * 8, j = j0 + e * 8 + 2 * t + (x & 1);
      float fa = 1.f, fq = 1.f;
      if constexpr (!GEN) {
        const float dec = j <= i ? ex2((float)(sG[i] - sG[j])) * sNk[j] : 0.f;
        fa = dec * sBeta[i] * sNk[i];
        fq = dec * sNq[i];
      }
      sa[e][x] = j < i ? sa[e][x] * fa : 0.f;
      sq[e][x] = j <= i ? sq[e][x] * fq : 0.f;
      if constexpr (GEN) {
        sb[e][x] = j < i ? sb[e][x] : 0.f;
        sp[e][x] = j <= i ? sp[e][x] : 0.f;
      }
      sA[i * kLdF + j] = sa[e][x];
    }
  __syncthreads();
  // ---- M = (I + A)^-1: 16 x 16 diagonal blocks by substitution, a column per thread, then block by block below
  for (int e = tid; e < kC * kC; e += kPrep) {
    const int i = e >> 6, j = e & 63;
    if ((j >> 4) > (i >> 4)) sM[i * kLdF + j] = 0.f;
  }
  if (tid < kC) {
    const int b0 = tid & ~15, cc = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s = i == cc ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < 16; ++j)
        if (j < i) s = fmaf(-sA[(b0 + i) * kLdF + b0 + j], x[j], s);
      x[i] = s;
      sM[(b0 + i) * kLdF + b0 + cc] = s;
    }
  }
  __syncthreads();
  {
    const int r = (tid >> 4) & 15, cc = tid & 15, side = tid >> 8;
    for (int lev = 1; lev < 4; ++lev) {
      for (int jb = side; jb + lev < 4; jb += kPrep / 256) {
        const int ib = jb + lev;
        float s = 0.f;
        for (int k = jb * 16; k < ib * 16; ++k) s = fmaf(sA[(ib * 16 + r) * kLdF + k], sM[k * kLdF + jb * 16 + cc], s);
        sT[(jb * 16 + r) * 17 + cc] = s;
      }
      __syncthreads();
      for (int jb = side; jb + lev < 4; jb += kPrep / 256) {
        const int ib = jb + lev;
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < 16; ++k) s = fmaf(sM[(ib * 16 + r) * kLdF + ib * 16 + k], sT[(jb * 16 + k) * 17 + cc], s);
        sM[(ib * 16 + r) * kLdF + jb * 16 + cc] = -s;
      }
      __syncthreads();
    }
  }
  // M as planes; gated: times diag(beta 2^G / |k|) for Xw, diag(beta) for Xu
  auto put_m = [&](bool decayed) {
    for (int e = tid; e < kC * kC / 2; e += kPrep) {
      const int i = e >> 5, j = (e & 31) * 2;
      float a = sM[i * kLdF + j], b = sM[i * kLdF + j + 1];
      if constexpr (!GEN) {
        a *= sBeta[j] * (decayed ? ex2((float)sG[j]) * sNk[j] : 1.f);
        b *= sBeta[j + 1] * (decayed ? ex2((float)sG[j + 1]) * sNk[j + 1] : 1.f);
      }
      Z0.put(i, j, a, b);
    }
  };
  put_m(true);
  __syncthreads();
  // ---- Xw = -M U and Xu; this warp's 16 rows and a quarter of the columns
  constexpr int NK = DK / 32, NV = DV / 32;
  const int nk0 = quarter * (DK / 4), nv0 = quarter * (DV / 4), kend = i0 + 16;
  float xw[NK][4], xu[NV][4];
  zero<NK>(xw);
  zero<NV>(xu);
  mm<NK, false, GEN>(xw, Z0, i0, U, nk0, 0, kend);
  const Planes& XW = GEN ? U : B;
  float po[NV][4];                                        // O'
  zero<NV>(po);
  if constexpr (GEN) {
    put_acc<2>(Z1, i0, j0, sb, 1.f);
    __syncthreads();
    float mbv[2][4];
    zero<2>(mbv);
    mm<2, false, true>(mbv, Z0, i0, Z1, j0, 0, kend);
    __syncthreads();
    put_acc<2>(Z0, i0, j0, mbv, -1.f);
    put_acc<2>(Z1, i0, j0, sp, 1.f);
    put_acc<NK>(XW, i0, nk0, xw, -1.f);
    __syncthreads();
    mm<NV, false, false>(xu, Z0, i0, V, nv0, 0, kend);
    mm<NV, false, false>(po, Z1, i0, V, nv0, 0, kend);
    __syncthreads();
    put_acc<2>(Z0, i0, j0, sq, 1.f);
  } else {
    __syncthreads();
    put_m(false);
    put_acc<NK>(XW, i0, nk0, xw, -1.f);
    __syncthreads();
    mm<NV, false, false>(xu, Z0, i0, V, nv0, 0, kend);
    __syncthreads();
    put_acc<2>(Z0, i0, j0, sq, 1.f);
    put_acc<NV>(K, i0, nv0, xu, 1.f);
  }
  __syncthreads();
  // ---- R' = R (gated: decayed) + Q Xw
  {
    float acc[NK][4];
#pragma unroll
    for (int i = 0; i < NK; ++i)
#pragma unroll
      for (int h2 = 0; h2 < 2; ++h2) {
        const int row = i0 + g + 8 * h2;
        float2 r;
        float f = 1.f;
        if constexpr (GEN) {
          r = R.get(row, nk0 + i * 8 + 2 * t);
        } else {
          r = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(R.hi + row * Lay::ldk + nk0 + i * 8 + 2 * t));
          f = ex2((float)sG[row]) * sNq[row];
        }
        acc[i][2 * h2] = r.x * f;
        acc[i][2 * h2 + 1] = r.y * f;
      }
    mm<NK, false, true>(acc, Z0, i0, XW, nk0, 0, kend);
    put_frag<NK>(p.ws_r + ci * (kC * DK / 4), DK / 16, i0, nk0, acc);
  }
  // ---- the state's side: 16 key rows and a part of the columns per warp
  constexpr int kMB = DK / 16, kCW = kPrep / 32 / kMB, NE = DV / 8 / kCW, NT = DK / 8 / kCW;
  const int m0 = (warp % kMB) * 16, e0 = (warp / kMB) * NE * 8, x0 = (warp / kMB) * NT * 8;
  float acc_e[NE][4];
  zero<NE>(acc_e);
  if constexpr (GEN) {
    mm<NE, true, false>(acc_e, K, m0, V, e0, 0, kC);
    __syncthreads();                                      // K is consumed: its space takes Xu
    put_acc<NV>(K, i0, nv0, xu, 1.f);
    __syncthreads();
  }
  mm<NV, false, true>(po, Z0, i0, K, nv0, 0, kend);        // O' += Q Xu
  put_c<NV>(p.ws_o + ci * (kC * DV / 4), DV / 8, i0, nv0, po);
  if constexpr (!GEN) {                                   // rows of X decayed to the chunk's end and over the keys' lengths, in place
    __syncthreads();
    const double gl = sG[kC - 1];
    for (int e = tid; e < kC * (DK + DV) / 2; e += kPrep) {
      const int i = e / ((DK + DV) / 2), d = (e - i * ((DK + DV) / 2)) * 2;
      const float f = i < valid ? ex2((float)(gl - sG[i])) * sNk[i] : 0.f;
      const Planes& X = d < DK ? XW : K;
      const int cc = d < DK ? d : d - DK;
      const float2 x = X.get(i, cc);
      X.put(i, cc, x.x * f, x.y * f);
    }
    __syncthreads();
  }
  mm<NE, true, true, GEN>(acc_e, GEN ? B : U, m0, K, e0, 0, kC);
  const float d0 = GEN ? sD[m0 + g] : 1.f, d1 = GEN ? sD[m0 + g + 8] : 1.f;
#pragma unroll
  for (int i = 0; i < NE; ++i) {
    acc_e[i][0] *= d0; acc_e[i][1] *= d0; acc_e[i][2] *= d1; acc_e[i][3] *= d1;
  }
  put_c<NE>(p.ws_e + ci * (DK * DV / 4), DV / 8, m0, e0, acc_e);
  float acc_t[NT][4];
  zero<NT>(acc_t);
  mm<NT, true, true, GEN>(acc_t, GEN ? B : U, m0, XW, x0, 0, kC);
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    acc_t[i][0] *= d0; acc_t[i][1] *= d0; acc_t[i][2] *= d1; acc_t[i][3] *= d1;
  }
  put_frag<NT>(p.ws_t + ci * (DK * DK / 4), DK / 16, m0, x0, acc_t);
}

// ------------------------------------------------------------------ recurrence over chunks
// SLICE value columns per CTA: 32, or 16 where those CTAs, too, have an SM each
template <int DK, int SLICE>
struct ScanLayout {
  static constexpr int lds = SLICE + 8;
  static constexpr size_t t_stage = (size_t)DK * DK * 4, s = 2 * t_stage, bytes = s + 2 * (size_t)DK * lds * 2;
};

template <int DK, int SLICE>
constexpr int scan_threads() { return SLICE == 32 || DK == 128 ? 256 : 128; }

template <int DK, int DV, int SLICE>
__global__ void __launch_bounds__(scan_threads<DK, SLICE>(), 1) delta_scan_kernel(const ChunkParams p) {
  using Lay = ScanLayout<DK, SLICE>;
  extern __shared__ __align__(16) uint8_t sm[];
  const int slice = blockIdx.x, hd = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (n <= 0) return;
  const int slot = p.slots[seq], H = p.in.H;
  if (slot < 0 || slot >= p.num_slots) {
    if (p.status && tid == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    return;
  }
  const int chunks = (n + kC - 1) / kC, c0 = slice * SLICE;
  const size_t first = (size_t)(p.q_start[seq] / kC + seq);
  constexpr int kMB = DK / 16, kThreads = scan_threads<DK, SLICE>(), kCW = kThreads / 32 / kMB, N8 = SLICE / 8 / kCW;
  const int m0 = (warp % kMB) * 16, n0 = (warp / kMB) * N8 * 8;
  const Planes S{reinterpret_cast<bf16*>(sm + Lay::s), reinterpret_cast<bf16*>(sm + Lay::s) + DK * Lay::lds, Lay::lds};
  auto issue = [&](int c) {
    if (c < chunks) {
      const uint4* src = p.ws_t + ((first + c) * H + hd) * (DK * DK / 4);
      uint4* dst = reinterpret_cast<uint4*>(sm + (c & 1) * Lay::t_stage);
      for (int i = tid; i < DK * DK / 4; i += kThreads) cp16(dst + i, src + i, true);
    }
    cp_commit();
  };
  float* st = p.state + ((size_t)slot * H + hd) * DK * DV + c0;
  const bool fresh = p.positions[p.q_start[seq]] == 0;
  float s[N8][4];
#pragma unroll
  for (int i = 0; i < N8; ++i)
#pragma unroll
    for (int h2 = 0; h2 < 2; ++h2) {
      float2 v = make_float2(0.f, 0.f);
      if (!fresh) v = *reinterpret_cast<const float2*>(st + (size_t)(m0 + g + 8 * h2) * DV + n0 + i * 8 + 2 * t);
      s[i][2 * h2] = v.x;
      s[i][2 * h2 + 1] = v.y;
    }
  issue(0);
  for (int c = 0; c < chunks; ++c) {
    const size_t ci = (first + c) * H + hd;
    issue(c + 1);
    // this chunk's additions, on their way while the start state is laid out
    float e[N8][4];
    const float d0 = p.ws_d[ci * DK + m0 + g], d1 = p.ws_d[ci * DK + m0 + g + 8];
    get_c<N8>(p.ws_e + ci * (DK * DV / 4), DV / 8, m0, c0 + n0, e);
    put_acc<N8>(S, m0, n0, s, 1.f);
    bf16* gs = p.ws_s + ci * 2 * DK * DV + c0;
    put_acc<N8>(Planes{gs, gs + DK * DV, DV}, m0, n0, s, 1.f);
    cp_wait<1>();
    __syncthreads();
#pragma unroll
    for (int i = 0; i < N8; ++i) {
      s[i][0] = fmaf(d0, s[i][0], e[i][0]); s[i][1] = fmaf(d0, s[i][1], e[i][1]);
      s[i][2] = fmaf(d1, s[i][2], e[i][2]); s[i][3] = fmaf(d1, s[i][3], e[i][3]);
    }
    mm_frag<N8>(s, reinterpret_cast<const uint4*>(sm + (c & 1) * Lay::t_stage) + (m0 >> 4) * (DK / 16) * 64, S, n0, DK / 16);
    __syncthreads();                                      // S and this stage are consumed
  }
  cp_wait<0>();
  if (p.write_state) {
#pragma unroll
    for (int i = 0; i < N8; ++i)
#pragma unroll
      for (int h2 = 0; h2 < 2; ++h2)
        *reinterpret_cast<float2*>(st + (size_t)(m0 + g + 8 * h2) * DV + n0 + i * 8 + 2 * t) = make_float2(s[i][2 * h2], s[i][2 * h2 + 1]);
  }
}

// ------------------------------------------------------------------ outputs of a chunk
template <int DK, int DV>
struct OutLayout {
  static constexpr int lds = DV + 8;
  static constexpr size_t r = 0, s = (size_t)kC * DK * 4, bytes = s + 2 * (size_t)DK * lds * 2;
};

template <int DK, int DV>
__global__ void __launch_bounds__(256, 2) delta_out_kernel(const ChunkParams p) {
  using Lay = OutLayout<DK, DV>;
  extern __shared__ __align__(16) uint8_t sm[];
  __shared__ float s_ss[kC][2];
  const int c = blockIdx.x, hd = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (c * kC >= n) return;
  const int t0 = p.q_start[seq] + c * kC, valid = min(kC, n - c * kC), H = p.in.H;
  const size_t ci = ((size_t)(p.q_start[seq] / kC + seq + c)) * H + hd;
  const Planes S{reinterpret_cast<bf16*>(sm + Lay::s), reinterpret_cast<bf16*>(sm + Lay::s) + DK * Lay::lds, Lay::lds};
  const uint4* gr = p.ws_r + ci * (kC * DK / 4);
  const bf16* gs = p.ws_s + ci * 2 * DK * DV;
  for (int i = tid; i < kC * DK / 4; i += 256) cp16(sm + Lay::r + (size_t)i * 16, gr + i, true);
  for (int i = tid; i < 2 * DK * (DV / 8); i += 256) {
    const int pl = i / (DK * (DV / 8)), e = i - pl * (DK * (DV / 8)), r = e / (DV / 8), cc = (e - r * (DV / 8)) * 8;
    cp16((pl ? S.lo : S.hi) + r * Lay::lds + cc, gs + (size_t)i * 8, true);
  }
  cp_commit();
  constexpr int NV = DV / 16;
  const int i0 = (warp & 3) * 16, half = warp >> 2, nv0 = half * (DV / 2);
  float o[NV][4];
  get_c<NV>(p.ws_o + ci * (kC * DV / 4), DV / 8, i0, nv0, o);
  cp_wait<0>();
  __syncthreads();
  mm_frag<NV>(o, reinterpret_cast<const uint4*>(sm + Lay::r) + (i0 >> 4) * (DK / 16) * 64, S, nv0, DK / 16);
  if (!p.norm_w) {
#pragma unroll
    for (int h2 = 0; h2 < 2; ++h2) {
      const int row = i0 + g + 8 * h2;
      if (row >= valid) continue;
      float* dst = p.out + ((size_t)(t0 + row) * H + hd) * DV + nv0 + 2 * t;
#pragma unroll
      for (int i = 0; i < NV; ++i) *reinterpret_cast<float2*>(dst + i * 8) = make_float2(o[i][2 * h2], o[i][2 * h2 + 1]);
    }
    return;
  }
#pragma unroll
  for (int h2 = 0; h2 < 2; ++h2) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss = fmaf(o[i][2 * h2], o[i][2 * h2], fmaf(o[i][2 * h2 + 1], o[i][2 * h2 + 1], ss));
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if (t == 0) s_ss[i0 + g + 8 * h2][half] = ss;
  }
  __syncthreads();
#pragma unroll
  for (int h2 = 0; h2 < 2; ++h2) {
    const int row = i0 + g + 8 * h2;
    if (row >= valid) continue;
    const float inv = rsqrtf((s_ss[row][0] + s_ss[row][1]) / (float)DV + p.eps) * p.scale;
    const int col = hd * DV + nv0 + 2 * t;
    const bf16* gz = p.gate + (size_t)(t0 + row) * p.gate_ld + col;
    bf16* dst = p.norm_out + (size_t)(t0 + row) * p.norm_out_ld + col;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gz + i * 8));
      const float2 w = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p.norm_w + col + i * 8));
      const float a = p.sigmoid_gate ? mb::sigmoid_fast(z.x) : mb::silu(z.x), b = p.sigmoid_gate ? mb::sigmoid_fast(z.y) : mb::silu(z.y);
      *reinterpret_cast<__nv_bfloat162*>(dst + i * 8) = __floats2bfloat162_rn(o[i][2 * h2] * inv * w.x * a, o[i][2 * h2 + 1] * inv * w.y * b);
    }
  }
}

template <int DK, int DV, bool GEN>
int launch_chunks(const ChunkParams& p, int num_seqs, int max_q_len, cudaStream_t stream) {
  constexpr size_t sp = PrepLayout<DK, DV>::bytes, so = OutLayout<DK, DV>::bytes;
  static bool configured = false;
  static int sms = 0;
  if (!configured) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) sms = 148;
    cudaError_t e = cudaFuncSetAttribute(delta_prep_kernel<DK, DV, GEN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sp);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_scan_kernel<DK, DV, 32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ScanLayout<DK, 32>::bytes);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_scan_kernel<DK, DV, 16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ScanLayout<DK, 16>::bytes);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_out_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)so);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((max_q_len + kC - 1) / kC, p.in.H, num_seqs);
  cudaError_t e = mb::launch_kernel(delta_prep_kernel<DK, DV, GEN>, grid, dim3(kPrep), sp, stream, p);
  if (e == cudaSuccess) {
    if ((long long)DV / 16 * p.in.H * num_seqs <= sms)
      e = mb::launch_kernel(delta_scan_kernel<DK, DV, 16>, dim3(DV / 16, p.in.H, num_seqs), dim3(scan_threads<DK, 16>()), ScanLayout<DK, 16>::bytes, stream, p);
    else
      e = mb::launch_kernel(delta_scan_kernel<DK, DV, 32>, dim3(DV / 32, p.in.H, num_seqs), dim3(scan_threads<DK, 32>()), ScanLayout<DK, 32>::bytes, stream, p);
  }
  if (e == cudaSuccess) e = mb::launch_kernel(delta_out_kernel<DK, DV>, grid, dim3(256), so, stream, p);
  return (int)e;
}
template <int DK, int DV>
int launch_rule(const ChunkParams& p, int num_seqs, int max_q_len, cudaStream_t stream) {
  return p.in.general ? launch_chunks<DK, DV, true>(p, num_seqs, max_q_len, stream) : launch_chunks<DK, DV, false>(p, num_seqs, max_q_len, stream);
}

size_t per_chunk(int DK, int DV) { return (size_t)DK * DK * 4 + (size_t)DK * DV * 8 + (size_t)kC * DK * 4 + (size_t)kC * DV * 4 + (size_t)DK * 4; }

}  // namespace

struct MbDeltaChunkedArgs {
  mb::DeltaInputs in;
  float* state;
  float* out;
  void* ws;
  size_t ws_bytes;
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int total_rows, num_seqs, num_slots, max_q_len, write_state;
  uint32_t* status;
  const void* norm_w;        // or null: fp32 rows to `out`
  const void* gate;
  long long gate_ld;
  int sigmoid_gate;
  float eps, scale;
  void* norm_out;
  long long norm_out_ld;
};

extern "C" size_t mb_delta_chunked_ws_bytes(int total_rows, int num_seqs, int H, int DK, int DV) {
  return ((size_t)total_rows / kC + num_seqs) * H * per_chunk(DK, DV) + 1024;
}

extern "C" int mb_delta_chunked(const MbDeltaChunkedArgs* a, cudaStream_t stream) {
  if (!a || !mb::delta_inputs_ok(a->in, false) || !a->state || (!a->out && !a->norm_w) || !a->ws || a->in.f32) return MB_ERR_BAD_ARG;
  if (a->num_seqs <= 0 || a->num_seqs > 65535 || a->in.H > 65535 || a->max_q_len <= 0 || a->total_rows <= 0) return MB_ERR_BAD_ARG;
  const DeltaInputs& in = a->in;
  const auto bad = [](const void* ptr, long long ld) { return (reinterpret_cast<uintptr_t>(ptr) & 15) || ld % 8; };
  if (bad(in.q, in.q_ld) || bad(in.k, in.k_ld) || bad(in.v, in.v_ld) || (in.general && (bad(in.removal, in.removal_ld) || bad(in.log_w, 0))) || bad(a->state, 0) ||
      bad(a->out, 0) || bad(a->ws, 0))
    return MB_ERR_UNSUPPORTED;                             // 16-byte copies
  if (a->norm_w && (!a->gate || !a->norm_out || a->gate_ld % 2 || a->norm_out_ld % 2 || (reinterpret_cast<uintptr_t>(a->gate) & 3) ||
                    (reinterpret_cast<uintptr_t>(a->norm_out) & 3) || (reinterpret_cast<uintptr_t>(a->norm_w) & 3)))
    return MB_ERR_UNSUPPORTED;
  if (a->ws_bytes < mb_delta_chunked_ws_bytes(a->total_rows, a->num_seqs, in.H, in.DK, in.DV)) return MB_ERR_TOO_LARGE;
  ChunkParams p{};
  p.in = in; p.state = a->state; p.out = a->out;
  const size_t chunks = ((size_t)a->total_rows / kC + a->num_seqs) * in.H, kk = (size_t)in.DK * in.DK, kv = (size_t)in.DK * in.DV;
  p.ws_t = reinterpret_cast<uint4*>(a->ws);
  p.ws_e = reinterpret_cast<float4*>(p.ws_t + chunks * (kk / 4));
  p.ws_s = reinterpret_cast<bf16*>(p.ws_e + chunks * (kv / 4));
  p.ws_r = reinterpret_cast<uint4*>(p.ws_s + chunks * 2 * kv);
  p.ws_o = reinterpret_cast<float4*>(p.ws_r + chunks * (kC * in.DK / 4));
  p.ws_d = reinterpret_cast<float*>(p.ws_o + chunks * (kC * in.DV / 4));
  p.q_start = a->q_start; p.q_len = a->q_len; p.positions = a->positions; p.slots = a->slots;
  p.num_slots = a->num_slots; p.write_state = a->write_state; p.status = a->status;
  p.norm_w = (const bf16*)a->norm_w; p.gate = (const bf16*)a->gate; p.gate_ld = a->gate_ld; p.sigmoid_gate = a->sigmoid_gate;
  p.eps = a->eps; p.scale = a->scale; p.norm_out = (bf16*)a->norm_out; p.norm_out_ld = a->norm_out_ld;
  if (in.DK == 64 && in.DV == 64) return launch_rule<64, 64>(p, a->num_seqs, a->max_q_len, stream);
  if (in.DK == 64 && in.DV == 128) return launch_rule<64, 128>(p, a->num_seqs, a->max_q_len, stream);
  if (in.DK == 128 && in.DV == 64) return launch_rule<128, 64>(p, a->num_seqs, a->max_q_len, stream);
  if (in.DK == 128 && in.DV == 128) return launch_rule<128, 128>(p, a->num_seqs, a->max_q_len, stream);
  return MB_ERR_UNSUPPORTED;
}
