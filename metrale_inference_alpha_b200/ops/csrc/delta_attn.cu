// Delta-rule linear attention over a ragged batch, token by token: per head a [DK, DV] fp32 state S and one of two rules,
// both read after the update, o_t = S_t^T q_t:
//
//   gated     S <- g_t S; S <- S + k_t (beta_t (v_t - S^T k_t))^T with unit keys, unit queries times DK^-1/2, one decay
//             g = exp(-exp(A_log) softplus(a + dt_bias)) and one step size beta = sigmoid(b) per head; several heads may
//             share a query/key head
//   general   S <- diag(w_t) S - (a_t u_t) (u_t^T S)^T + k_t v_t^T where both terms read the old state, u is the unit key and
//             k the key itself, w = exp(log_w) and the removal rate a = sigmoid(.) per key channel
//
// q, k, v and the logits are bf16 or fp32 column ranges, everything inside is fp32, DK <= 256, any DV. The state is carried
// in a slot pool; a sequence whose first row is at position 0 starts from zero. Serves decode, speculative verification and
// its commit pass (write_out = 0), prompts whose head sizes the chunked kernels do not take, and models served in 32-bit.
//
// delta_attn_kernel: a CTA owns one (sequence, head, block of value columns). Compute warps hold the state in registers,
// 16 key rows x 2 value columns per thread on packed fp32 FMAs; KG lanes share a column. A token costs one reduction over
// those lanes on the critical path (S^T k); the read-out's reduction of the token before rides along with it. Producer
// warps load the next 16 tokens meanwhile and make unit vectors, decays and rates of them.
//
// delta_decode_kernel: steps of one token per sequence. A CTA per (sequence, head) holds the whole head in registers
// (16 rows of 16-byte vectors per thread), reads and writes the state once, and can finish the head's output itself
// (RMS over the head, weight, gate, scale); log decays may come as a low-rank projection, computed there too.
#include "common.cuh"
#include "delta_attn.cuh"
#include "epilogue.cuh"

namespace {

using bf16 = __nv_bfloat16;
using mb::DeltaInputs;

struct DeltaParams {
  DeltaInputs in;
  // general rule, decode: log decays lr_c sigmoid(lr_w2 tanh(lr_z) + lr_bias) instead of log_w
  const void* lr_z;                // [T, rank]
  long long lr_ld;
  const bf16* lr_w2;               // [H DK, rank]
  const float* lr_bias;            // [H DK]
  int lr_rank;
  float lr_c;
  float* state;                    // [slots, H, DK, DV]
  float* out;                      // [T, H DV]
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_slots, write_state, write_out;
  uint32_t* status;
};

constexpr int kTB = 16;            // tokens per buffer
constexpr int kNW = 4;             // compute warps
constexpr int kPW = 8;             // producer warps

using f2 = unsigned long long;     // two packed fp32
__device__ __forceinline__ f2 pk(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float sum2(f2 v) {
  float a, b;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
  return a + b;
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
constexpr int cols_per_cta() { return kNW * (32 / KG) * 2; }
template <int KG, bool GENERAL>
constexpr size_t delta_smem() { return (size_t)2 * kTB * ((GENERAL ? 4 : 2) * 16 * KG + cols_per_cta<KG>() + 4) * sizeof(float); }

// KG lanes per value column, 16 key rows each (DK <= 16 KG)
template <typename T, int KG, bool GENERAL>
__global__ void __launch_bounds__(32 * (kNW + kPW)) delta_attn_kernel(const DeltaParams p) {
  constexpr int DKP = 16 * KG, VB = cols_per_cta<KG>();
  extern __shared__ __align__(16) float sm[];
  float* sQ = sm;                                  // [2][kTB][DKP]
  float* sK = sQ + 2 * kTB * DKP;
  float* sV = sK + 2 * kTB * DKP;                  // [2][kTB][VB]
  float* sS = sV + 2 * kTB * VB;                   // [2][kTB][4]: gated g, beta; general 1 / |k|^2
  float* sW = sS + 2 * kTB * 4;                    // general: decays, and minus rate times key
  float* sA = sW + 2 * kTB * DKP;
  const int hd = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  const int n = p.q_len[seq];
  if (n <= 0) return;
  const int t0 = p.q_start[seq], slot = p.slots[seq];
  if (slot < 0 || slot >= p.num_slots) {
    if (p.status && tid == 0) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
    return;
  }
  const DeltaInputs& in = p.in;
  const int DK = in.DK, DV = in.DV, col0 = blockIdx.x * VB;

  // two tokens per producer warp and tile; everything they read is on its way before the first reduction
  const float neg_a = GENERAL ? 0.f : -expf(in.A_log[hd]), dtb = GENERAL ? 0.f : in.dt_bias[hd];
  auto produce = [&](int tile, int pw) {
    constexpr int kE = (DKP + 31) / 32, kV = (VB + 31) / 32, kN = kTB / kPW;
    const int buf = tile & 1, cnt = min(kTB, n - tile * kTB);
    float q[kN][kE], k[kN][kE], w[kN][kE], a[kN][kE], v[kN][kV], ga[kN], gb[kN];
#pragma unroll
    for (int i = 0; i < kN; ++i) {
      const int tt = pw + i * kPW;
      const bool ok = tt < cnt;
      const size_t t = (size_t)(t0 + tile * kTB + (ok ? tt : 0));
#pragma unroll
      for (int j = 0; j < kE; ++j) {
        const int d = lane + 32 * j;
        const bool in_row = ok && d < DK;
        q[i][j] = in_row ? in.query<T>(t, hd, d) : 0.f;
        k[i][j] = in_row ? in.key<T>(t, hd, d) : 0.f;
        if constexpr (GENERAL) {
          w[i][j] = in_row ? in.log_w[(t * in.H + hd) * DK + d] : 0.f;
          a[i][j] = in_row ? mb::load1<T>(in.removal, t * in.removal_ld + (size_t)hd * DK + d) : 0.f;
        }
      }
#pragma unroll
      for (int j = 0; j < kV; ++j) {
        const int c = lane + 32 * j;
        v[i][j] = ok && c < VB && col0 + c < DV ? in.value<T>(t, hd, col0 + c) : 0.f;
      }
      if constexpr (!GENERAL) {
        ga[i] = mb::load1<T>(in.decay, t * in.gate_ld + hd);
        gb[i] = mb::load1<T>(in.step, t * in.gate_ld + hd);
      }
    }
#pragma unroll
    for (int i = 0; i < kN; ++i) {
      const int tt = pw + i * kPW;
      if (tt >= cnt) break;
      const int at = (buf * kTB + tt) * DKP;
      float sq = 0.f, sk = 0.f;
#pragma unroll
      for (int j = 0; j < kE; ++j) {
        sq = fmaf(q[i][j], q[i][j], sq);
        sk = fmaf(k[i][j], k[i][j], sk);
      }
      sk = mb::warp_sum(sk);
      float nq = 1.f, nk = 1.f;
      if constexpr (!GENERAL) {
        nq = rsqrtf(mb::warp_sum(sq) + mb::kUnitEps) * rsqrtf((float)DK);
        nk = rsqrtf(sk + mb::kUnitEps);
      }
#pragma unroll
      for (int j = 0; j < kE; ++j) {
        const int d = lane + 32 * j;
        if (d >= DKP) continue;
        sQ[at + d] = q[i][j] * nq;
        sK[at + d] = k[i][j] * nk;
        if constexpr (GENERAL) {
          sW[at + d] = expf(w[i][j]);
          sA[at + d] = -mb::sigmoid_exact(a[i][j]) * k[i][j];
        }
      }
      if (lane == 0) {
        if constexpr (GENERAL) {
          sS[(buf * kTB + tt) * 4] = 1.f / (sk + mb::kUnitEps);
        } else {
          sS[(buf * kTB + tt) * 4] = expf(neg_a * mb::softplus(ga[i] + dtb));
          sS[(buf * kTB + tt) * 4 + 1] = mb::sigmoid_exact(gb[i]);
        }
      }
#pragma unroll
      for (int j = 0; j < kV; ++j)
        if (lane + 32 * j < VB) sV[(buf * kTB + tt) * VB + lane + 32 * j] = v[i][j];
    }
  };

  const int tiles = (n + kTB - 1) / kTB;
  const bool compute = warp < kNW;
  const int kg = lane % KG, lc = (warp * (32 / KG) + lane / KG) * 2, col = col0 + lc;
  f2 s[8][2];                                      // pair p: key rows row_of(p), row_of(p) + 1; two value columns
  float* st = p.state + ((size_t)slot * in.H + hd) * DK * DV;
  auto row_of = [&](int pair) { return (pair >> 1) * 4 * KG + kg * 4 + (pair & 1) * 2; };
  if (compute) {
    const bool fresh = p.positions[t0] == 0;
#pragma unroll
    for (int pr = 0; pr < 8; ++pr) {
      float a[2][2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = row_of(pr) + e;
#pragma unroll
        for (int c = 0; c < 2; ++c) a[e][c] = (!fresh && r < DK && col + c < DV) ? st[(size_t)r * DV + col + c] : 0.f;
      }
#pragma unroll
      for (int c = 0; c < 2; ++c) s[pr][c] = pk(a[0][c], a[1][c]);
    }
  } else {
    produce(0, warp - kNW);
  }
  __syncthreads();
  float po[2] = {0.f, 0.f};                        // this lane's share of the last token's read-out, not reduced yet
  auto store = [&](int t, float y) {               // after the exchange over bit 0: lane kg < 2 holds column kg
    if (kg < 2 && col + kg < DV) p.out[((size_t)(t0 + t) * in.H + hd) * DV + col + kg] = y;
  };
  for (int tile = 0; tile < tiles; ++tile) {
    if (!compute) {
      if (tile + 1 < tiles) produce(tile + 1, warp - kNW);
    } else {
      const int buf = tile & 1, cnt = min(kTB, n - tile * kTB);
      for (int tt = 0; tt < cnt; ++tt) {
        const int at = (buf * kTB + tt) * DKP + kg * 4;
        const float2 v = *reinterpret_cast<const float2*>(sV + (buf * kTB + tt) * VB + lc);
        const float2 sc = *reinterpret_cast<const float2*>(sS + (buf * kTB + tt) * 4);
        ulonglong2 k4[4];
        f2 acc[2][2] = {{0ull, 0ull}, {0ull, 0ull}};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          k4[j] = *reinterpret_cast<const ulonglong2*>(sK + at + j * 4 * KG);
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            acc[0][c] = fma2(k4[j].x, s[2 * j][c], acc[0][c]);
            acc[1][c] = fma2(k4[j].y, s[2 * j + 1][c], acc[1][c]);
          }
        }
        float d0 = sum2(acc[0][0]) + sum2(acc[1][0]), d1 = sum2(acc[0][1]) + sum2(acc[1][1]);
        // S^T k of this token and the read-out of the last one, reduced over the KG lanes together
        float y = (kg & 1 ? po[1] : po[0]) + __shfl_xor_sync(0xffffffffu, kg & 1 ? po[0] : po[1], 1);
        d0 += __shfl_xor_sync(0xffffffffu, d0, 1);
        d1 += __shfl_xor_sync(0xffffffffu, d1, 1);
#pragma unroll
        for (int o = 2; o < KG; o <<= 1) {
          d0 += __shfl_xor_sync(0xffffffffu, d0, o);
          d1 += __shfl_xor_sync(0xffffffffu, d1, o);
          y += __shfl_xor_sync(0xffffffffu, y, o);
        }
        f2 ro[2][2] = {{0ull, 0ull}, {0ull, 0ull}};
        if constexpr (GENERAL) {
          const f2 e0 = pk(d0 * sc.x, d0 * sc.x), e1 = pk(d1 * sc.x, d1 * sc.x), v0 = pk(v.x, v.x), v1 = pk(v.y, v.y);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(sQ + at + j * 4 * KG);
            const ulonglong2 w4 = *reinterpret_cast<const ulonglong2*>(sW + at + j * 4 * KG);
            const ulonglong2 a4 = *reinterpret_cast<const ulonglong2*>(sA + at + j * 4 * KG);
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              const f2 q2 = h ? q4.y : q4.x, k2 = h ? k4[j].y : k4[j].x, w2 = h ? w4.y : w4.x, a2 = h ? a4.y : a4.x;
              f2 &x = s[2 * j + h][0], &z = s[2 * j + h][1];
              x = fma2(a2, e0, fma2(k2, v0, mul2(w2, x)));
              z = fma2(a2, e1, fma2(k2, v1, mul2(w2, z)));
              ro[h][0] = fma2(q2, x, ro[h][0]);
              ro[h][1] = fma2(q2, z, ro[h][1]);
            }
          }
        } else {
          const float u0 = sc.y * (v.x - sc.x * d0), u1 = sc.y * (v.y - sc.x * d1);
          const f2 g2 = pk(sc.x, sc.x), e0 = pk(u0, u0), e1 = pk(u1, u1);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(sQ + at + j * 4 * KG);
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              const f2 q2 = h ? q4.y : q4.x, k2 = h ? k4[j].y : k4[j].x;
              f2 &x = s[2 * j + h][0], &z = s[2 * j + h][1];
              x = fma2(k2, e0, mul2(g2, x));
              z = fma2(k2, e1, mul2(g2, z));
              ro[h][0] = fma2(q2, x, ro[h][0]);
              ro[h][1] = fma2(q2, z, ro[h][1]);
            }
          }
        }
        const int t = tile * kTB + tt;
        if (p.write_out && t > 0) store(t - 1, y);
        po[0] = sum2(ro[0][0]) + sum2(ro[1][0]);
        po[1] = sum2(ro[0][1]) + sum2(ro[1][1]);
      }
    }
    __syncthreads();
  }
  if (!compute) return;
  if (p.write_out) {
    float y = (kg & 1 ? po[1] : po[0]) + __shfl_xor_sync(0xffffffffu, kg & 1 ? po[0] : po[1], 1);
#pragma unroll
    for (int o = 2; o < KG; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    store(n - 1, y);
  }
  if (p.write_state) {
#pragma unroll
    for (int pr = 0; pr < 8; ++pr)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float a, b;
        upk(s[pr][c], a, b);
        const int r = row_of(pr);
        if (col + c < DV) {
          if (r < DK) st[(size_t)r * DV + col + c] = a;
          if (r + 1 < DK) st[(size_t)(r + 1) * DV + col + c] = b;
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
constexpr int kMaxRank = 256;

// QV threads cover the DV / 4 column vectors of a row; 256 / QV rows are in work side by side
template <typename T, int QV, bool GENERAL>
__global__ void __launch_bounds__(256, 2) delta_decode_kernel(const DeltaParams p, const DecodeNorm nm) {
  constexpr int RG = 256 / QV, kBlock = kDecRows * RG;
  __shared__ __align__(16) float so[RG * QV * 4];
  __shared__ float sq[256], sk[256], sw[GENERAL ? 256 : 1], sa[GENERAL ? 256 : 1], sz[GENERAL ? kMaxRank : 1], red[32];
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
  const DeltaInputs& in = p.in;
  const bool fresh = p.positions[t] == 0;
  const int DK = in.DK, DV = in.DV, c4 = (tid % QV) * 4, rg = tid / QV;
  const bool col_ok = c4 < DV;
  float* st = p.state + ((size_t)slot * in.H + hd) * DK * DV + c4;
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
  if (col_ok) v = make_float4(in.value<T>(t, hd, c4), in.value<T>(t, hd, c4 + 1), in.value<T>(t, hd, c4 + 2), in.value<T>(t, hd, c4 + 3));
  const float q = tid < DK ? in.query<T>(t, hd, tid) : 0.f, k = tid < DK ? in.key<T>(t, hd, tid) : 0.f;
  float g = 0.f, beta = 0.f, inv2 = 0.f;
  if constexpr (GENERAL) {
    if (p.lr_z) {
      if (tid < p.lr_rank) sz[tid] = tanhf(mb::load1<T>(p.lr_z, t * p.lr_ld + tid));
    }
    inv2 = 1.f / (mb::block_sum(k * k, red) + mb::kUnitEps);       // its barriers publish sz
    if (tid < DK) {
      sq[tid] = q;
      sk[tid] = k;
      sa[tid] = -in.rate<T>(t, hd, tid) * k;
      const size_t ch = (size_t)hd * DK + tid;
      float lw;
      if (p.lr_z) {
        const bf16* w2 = p.lr_w2 + ch * p.lr_rank;
        float z = p.lr_bias[ch];
        int r = 0;
        if ((p.lr_rank & 7) == 0 && (reinterpret_cast<uintptr_t>(p.lr_w2) & 15) == 0) {      // rows of whole 16-byte vectors
#pragma unroll 8
          for (; r < p.lr_rank; r += 8) {
            const uint4 w8 = __ldg(reinterpret_cast<const uint4*>(w2 + r));
            const __nv_bfloat162* wb = reinterpret_cast<const __nv_bfloat162*>(&w8);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const float2 f = __bfloat1622float2(wb[i]);
              z = fmaf(sz[r + 2 * i], f.x, fmaf(sz[r + 2 * i + 1], f.y, z));
            }
          }
        }
        for (; r < p.lr_rank; ++r) z = fmaf(sz[r], __bfloat162float(w2[r]), z);
        lw = p.lr_c * mb::sigmoid_exact(z);
      } else {
        lw = in.log_w[t * in.H * DK + ch];
      }
      sw[tid] = expf(lw);
    }
  } else {
    const float nk = rsqrtf(mb::block_sum(k * k, red) + mb::kUnitEps);
    const float nq = rsqrtf(mb::block_sum(q * q, red) + mb::kUnitEps) * rsqrtf((float)DK);
    sq[tid] = q * nq;
    sk[tid] = k * nk;
    g = expf(in.log_gate<T>(t, hd));
    beta = in.step_size<T>(t, hd);
  }
  __syncthreads();
  // ---- S^T k over all rows
  float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int r0 = 0; r0 < DK; r0 += kBlock) {
    if (r0 > 0) load(r0);
#pragma unroll
    for (int i = 0; i < kDecRows; ++i) {
      const int r = r0 + rg + i * RG;
      if (r < DK) {
        const float kr = sk[r];
        d.x = fmaf(kr, s[i].x, d.x); d.y = fmaf(kr, s[i].y, d.y); d.z = fmaf(kr, s[i].z, d.z); d.w = fmaf(kr, s[i].w, d.w);
      }
    }
  }
  *reinterpret_cast<float4*>(so + (rg * QV) * 4 + c4) = d;
  __syncthreads();
  d = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < RG; ++i) {
    const float4 a = *reinterpret_cast<const float4*>(so + (i * QV) * 4 + c4);
    d.x += a.x; d.y += a.y; d.z += a.z; d.w += a.w;
  }
  __syncthreads();
  // what the rows take: gated k u, general k v + (-a k) e
  float4 u;
  if constexpr (GENERAL) {
    u = make_float4(inv2 * d.x, inv2 * d.y, inv2 * d.z, inv2 * d.w);
  } else {
    u = make_float4(beta * (v.x - g * d.x), beta * (v.y - g * d.y), beta * (v.z - g * d.z), beta * (v.w - g * d.w));
  }
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  const bool one = DK <= kBlock;
  for (int r0 = 0; r0 < DK; r0 += kBlock) {
    if (!one) load(r0);
#pragma unroll
    for (int i = 0; i < kDecRows; ++i) {
      const int r = r0 + rg + i * RG;
      if (r < DK) {
        const float qr = sq[r], kr = sk[r];
        float4 x = s[i];
        if constexpr (GENERAL) {
          const float w = sw[r], a = sa[r];
          x.x = fmaf(a, u.x, fmaf(kr, v.x, w * x.x)); x.y = fmaf(a, u.y, fmaf(kr, v.y, w * x.y));
          x.z = fmaf(a, u.z, fmaf(kr, v.z, w * x.z)); x.w = fmaf(a, u.w, fmaf(kr, v.w, w * x.w));
        } else {
          x.x = fmaf(kr, u.x, g * x.x); x.y = fmaf(kr, u.y, g * x.y); x.z = fmaf(kr, u.z, g * x.z); x.w = fmaf(kr, u.w, g * x.w);
        }
        o.x = fmaf(qr, x.x, o.x); o.y = fmaf(qr, x.y, o.y); o.z = fmaf(qr, x.z, o.z); o.w = fmaf(qr, x.w, o.w);
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
    for (int i = 0; i < RG; ++i) y += so[i * QV * 4 + tid];
  }
  if (!nm.w) {
    if (tid < DV) p.out[(t * in.H + hd) * DV + tid] = y;
    return;
  }
  const float inv = 1.f / sqrtf(mb::block_sum(y * y, red) / (float)DV + nm.eps);
  if (tid < DV) {
    const int col = hd * DV + tid;
    const float z = mb::load1<T>(nm.gate, t * nm.gate_ld + col);
    const float a = nm.sigmoid_gate ? mb::sigmoid_exact(z) : mb::silu_exact(z);
    const float r = y * inv * __bfloat162float(nm.w[col]) * a * nm.scale;
    if constexpr (sizeof(T) == 2) reinterpret_cast<bf16*>(nm.out)[t * nm.out_ld + col] = __float2bfloat16(r);
    else reinterpret_cast<float*>(nm.out)[t * nm.out_ld + col] = r;
  }
}

template <typename T, bool GENERAL>
int launch_decode(const DeltaParams& p, const DecodeNorm& nm, int num_seqs, cudaStream_t stream) {
  const dim3 grid(p.in.H, num_seqs), block(256);
  const int quads = p.in.DV / 4;
  if (quads <= 8) return (int)mb::launch_kernel(delta_decode_kernel<T, 8, GENERAL>, grid, block, 0, stream, p, nm);
  if (quads <= 16) return (int)mb::launch_kernel(delta_decode_kernel<T, 16, GENERAL>, grid, block, 0, stream, p, nm);
  if (quads <= 32) return (int)mb::launch_kernel(delta_decode_kernel<T, 32, GENERAL>, grid, block, 0, stream, p, nm);
  return (int)mb::launch_kernel(delta_decode_kernel<T, 64, GENERAL>, grid, block, 0, stream, p, nm);
}

template <typename T, int KG, bool GENERAL>
int launch_seq(const DeltaParams& p, int num_seqs, cudaStream_t stream) {
  constexpr size_t smem = delta_smem<KG, GENERAL>();
  auto kern = delta_attn_kernel<T, KG, GENERAL>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int VB = cols_per_cta<KG>();
  return (int)mb::launch_kernel(kern, dim3((p.in.DV + VB - 1) / VB, p.in.H, num_seqs), dim3(32 * (kNW + kPW)), smem, stream, p);
}
template <typename T, bool GENERAL>
int launch_kg(const DeltaParams& p, int num_seqs, cudaStream_t stream) {
  if (p.in.DK <= 32) return launch_seq<T, 2, GENERAL>(p, num_seqs, stream);
  if (p.in.DK <= 64) return launch_seq<T, 4, GENERAL>(p, num_seqs, stream);
  if (p.in.DK <= 128) return launch_seq<T, 8, GENERAL>(p, num_seqs, stream);
  if (p.in.DK <= 256) return launch_seq<T, 16, GENERAL>(p, num_seqs, stream);
  return MB_ERR_UNSUPPORTED;
}
template <typename T, bool GENERAL>
int run_delta(const DeltaParams& p, const DecodeNorm& nm, int decode, int num_seqs, cudaStream_t stream) {
  return decode ? launch_decode<T, GENERAL>(p, nm, num_seqs, stream) : launch_kg<T, GENERAL>(p, num_seqs, stream);
}

}  // namespace

struct MbDeltaAttnArgs {
  mb::DeltaInputs in;
  const void* lr_z;
  long long lr_ld;
  const void* lr_w2;
  const float* lr_bias;
  int lr_rank;
  float lr_c;
  float* state;
  float* out;
  const int* q_start;
  const int* q_len;
  const int* positions;
  const int* slots;
  int num_seqs, num_slots, write_state, write_out;
  uint32_t* status;
  int decode;                // every sequence has at most one row: the streaming kernel (DV % 4 == 0, DV <= 256)
  const void* norm_w;        // decode: finish the head's output (RMS, weight, gate, scale) into norm_out
  const void* gate;
  long long gate_ld;
  int sigmoid_gate;
  float eps, scale;
  void* norm_out;
  long long norm_out_ld;
};

extern "C" int mb_delta_attn(const MbDeltaAttnArgs* a, cudaStream_t stream) {
  if (!a || !mb::delta_inputs_ok(a->in, a->lr_z != nullptr) || !a->state || (a->write_out && !a->out && !a->norm_w)) return MB_ERR_BAD_ARG;
  if (a->num_seqs <= 0 || a->num_seqs > 65535 || a->in.H > 65535 || a->in.DK > 256) return MB_ERR_BAD_ARG;
  if (reinterpret_cast<uintptr_t>(a->state) % 16) return MB_ERR_BAD_ARG;
  if (a->lr_z && (!a->decode || !a->in.general || !a->lr_w2 || !a->lr_bias || a->lr_rank <= 0 || a->lr_rank > kMaxRank)) return MB_ERR_UNSUPPORTED;
  if (a->decode && (a->in.DV % 4 || a->in.DV > 256)) return MB_ERR_UNSUPPORTED;
  if (a->norm_w && (!a->decode || !a->gate || !a->norm_out)) return MB_ERR_BAD_ARG;
  const DeltaParams p{a->in, a->lr_z, a->lr_ld, (const bf16*)a->lr_w2, a->lr_bias, a->lr_rank, a->lr_c, a->state, a->out, a->q_start, a->q_len,
                      a->positions, a->slots, a->num_slots, a->write_state, a->write_out, a->status};
  const DecodeNorm nm{(const bf16*)a->norm_w, a->gate, a->gate_ld, a->sigmoid_gate, a->eps, a->scale, a->norm_out, a->norm_out_ld};
  if (a->in.general) return a->in.f32 ? run_delta<float, true>(p, nm, a->decode, a->num_seqs, stream) : run_delta<bf16, true>(p, nm, a->decode, a->num_seqs, stream);
  return a->in.f32 ? run_delta<float, false>(p, nm, a->decode, a->num_seqs, stream) : run_delta<bf16, false>(p, nm, a->decode, a->num_seqs, stream);
}
