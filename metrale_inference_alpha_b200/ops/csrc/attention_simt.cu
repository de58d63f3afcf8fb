// Paged causal attention on the CUDA cores in fp32 arithmetic: any query/key and value head size (up to
// 2048 / 1024), bf16 or fp32 cache, optional sink (a key without a value: score 0, or one per head), window with kept
// first tokens, sigmoid gates on the output. It serves models that run in true 32-bit, and head sizes beyond the
// tensor-core kernels' tiles.
//
// One CTA per (query head, query row), 128 threads. Per tile of 128 cached tokens: thread j scores token j
// (dot product over the query held in shared memory), the block agrees on the running maximum and sum, and
// thread d accumulates value columns d, d + 128, ... over the tile. Cache rows are [slot, kv head, dkp] and
// [slot, kv head, dvp]; the padding columns are never read.
#include "common.cuh"
#include "visible.cuh"

namespace {

struct SimtAttnParams {
  const void* q;             // [T, Hq, dkp]
  const void* k_cache;
  const void* v_cache;
  const int* block_table;
  int max_blocks;
  const int* q_start;
  const int* q_len;
  const int* ctx_len;
  int num_seqs, Hq, Hkv, dk, dv, dkp, dvp, block_size;
  long long num_blocks;
  float scale, out_scale;
  int sink;
  const float* sink_w;       // [Hq] or null
  int window, keep;
  const void* gate;
  long long gate_ld;
  int gate_mode;
  float softcap;             // 0: off
  void* out;                 // row stride out_ld, head stride dv
  long long out_ld;
  uint32_t* status;
};

template <typename T>
__device__ __forceinline__ float lda(const T* p) {
  if constexpr (sizeof(T) == 2) return __bfloat162float(*p);
  else return *p;
}

constexpr int kMaxDv = 1024;

template <typename T>
__global__ void __launch_bounds__(128) attn_simt_kernel(const SimtAttnParams p) {
  extern __shared__ float sq[];            // [dk]
  __shared__ float sp[128];
  __shared__ long long sslot[128];
  __shared__ float red[32];
  const int head = blockIdx.x, t = blockIdx.y, tid = threadIdx.x;
  mb::pdl_wait();
  mb::pdl_launch_dependents();
  int lo = 0, hi = p.num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.q_start[mid] <= t) lo = mid;
    else hi = mid - 1;
  }
  const int r0 = p.q_start[lo], n = p.q_len[lo], ctx = p.ctx_len[lo];
  if (t < r0 || t >= r0 + n) return;
  const int limit = ctx - n + (t - r0) + 1;
  const int kvh = head / (p.Hq / p.Hkv);
  const int* bt = p.block_table + (size_t)lo * p.max_blocks;
  for (int d = tid; d < p.dk; d += 128) sq[d] = lda(reinterpret_cast<const T*>(p.q) + ((size_t)t * p.Hq + head) * p.dkp + d);
  float acc[kMaxDv / 128];
#pragma unroll
  for (int i = 0; i < kMaxDv / 128; ++i) acc[i] = 0.f;
  // the sink is a key of score 0 without a value: it starts the running maximum and sum
  float m = p.sink ? (p.sink_w ? p.sink_w[head] : 0.f) : -INFINITY, l = p.sink ? 1.f : 0.f;
  // one query: the visible tokens are the kept first ones and the window behind them, exactly
  const int begin = p.window > 0 ? max(0, limit - p.window) : 0;
  const int kept = min(p.keep, begin), shift = begin - kept, len = limit - shift;
  for (int j0 = 0; j0 < len; j0 += 128) {
    __syncthreads();                       // sq ready / the previous tile's sp and sslot consumed
    const int j = j0 + tid;
    float s = -INFINITY;
    long long slot = 0;
    if (j < len) {
      const int tok = j < kept ? j : j + shift;
      long long blk = bt[tok / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) {
        if (p.status) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
        blk = 0;
      }
      slot = blk * p.block_size + tok % p.block_size;
      const T* k = reinterpret_cast<const T*>(p.k_cache) + ((size_t)slot * p.Hkv + kvh) * p.dkp;
      float a = 0.f;
      for (int d = 0; d < p.dk; ++d) a = fmaf(sq[d], lda(k + d), a);
      s = a * p.scale;
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    }
    const float m_new = fmaxf(m, mb::block_max(s, red));
    const float e = j < len ? expf(s - m_new) : 0.f;
    sp[tid] = e;
    sslot[tid] = slot;
    const float sum = mb::block_sum(e, red);       // its barriers also publish sp and sslot
    const float alpha = expf(m - m_new);
    l = l * alpha + sum;
    m = m_new;
    const int cnt = min(128, len - j0);
#pragma unroll
    for (int i = 0; i < kMaxDv / 128; ++i) {
      const int d = tid + i * 128;
      if (d < p.dv) {
        float a = acc[i] * alpha;
        for (int jj = 0; jj < cnt; ++jj)
          a = fmaf(sp[jj], lda(reinterpret_cast<const T*>(p.v_cache) + ((size_t)sslot[jj] * p.Hkv + kvh) * p.dvp + d), a);
        acc[i] = a;
      }
    }
  }
  const float inv = p.out_scale / l;
  const mb::OutputGate<T> gate{reinterpret_cast<const T*>(p.gate), p.gate_ld, p.gate_mode, p.dv};
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.out_ld + (size_t)head * p.dv;
#pragma unroll
  for (int i = 0; i < kMaxDv / 128; ++i) {
    const int d = tid + i * 128;
    if (d < p.dv) {
      const float v = acc[i] * inv * gate((size_t)t, head, d);
      if constexpr (sizeof(T) == 2) out[d] = __float2bfloat16(v);
      else out[d] = v;
    }
  }
}

}  // namespace

struct MbSimtAttnArgs {
  const void* q;
  const void* k_cache;
  const void* v_cache;
  const int* block_table;
  int max_blocks;
  const int* q_start;
  const int* q_len;
  const int* ctx_len;
  int total_rows, num_seqs, Hq, Hkv, dk, dv, dkp, dvp, block_size;
  long long num_blocks;
  float scale, out_scale;
  int sink, f32;
  void* out;
  long long out_ld;
  uint32_t* status;
  const float* sink_w;
  int window, keep;
  const void* gate;
  long long gate_ld;
  int gate_mode;
  float softcap;
};

extern "C" int mb_attn_simt(const MbSimtAttnArgs* a, cudaStream_t stream) {
  if (!a || !a->q || !a->k_cache || !a->v_cache || !a->block_table || !a->out || a->total_rows <= 0 || a->num_seqs <= 0) return MB_ERR_BAD_ARG;
  if (a->Hkv <= 0 || a->Hq % a->Hkv || a->dk <= 0 || a->dv <= 0 || a->dv > kMaxDv || a->dk > 2048 || a->dk > a->dkp || a->dv > a->dvp) return MB_ERR_UNSUPPORTED;
  if (a->total_rows > 65535) return MB_ERR_TOO_LARGE;
  SimtAttnParams p{a->q, a->k_cache, a->v_cache, a->block_table, a->max_blocks, a->q_start, a->q_len, a->ctx_len, a->num_seqs, a->Hq, a->Hkv,
                   a->dk, a->dv, a->dkp, a->dvp, a->block_size, a->num_blocks, a->scale, a->out_scale, a->sink, a->sink_w, a->window, a->window > 0 ? a->keep : 0,
                   a->gate, a->gate_ld, a->gate ? a->gate_mode : mb::GATE_NONE, a->softcap, a->out, a->out_ld, a->status};
  if (p.keep < 0 || p.gate_mode < 0 || p.gate_mode > mb::GATE_ELEMENT) return MB_ERR_BAD_ARG;
  const dim3 grid(a->Hq, a->total_rows);
  const size_t smem = (size_t)a->dk * sizeof(float);
  if (a->f32) return (int)mb::launch_kernel(attn_simt_kernel<float>, grid, dim3(128), smem, stream, p);
  return (int)mb::launch_kernel(attn_simt_kernel<__nv_bfloat16>, grid, dim3(128), smem, stream, p);
}
