// Paged causal attention on the CUDA cores in fp32 arithmetic: any query/key and value head size (up to
// 2048 / 1024), bf16 or fp32 cache, optional sink (one added to the softmax denominator). It serves models that
// run in true 32-bit, and head sizes beyond the tensor-core kernels' tiles.
//
// One CTA per (query head, query row), 128 threads. Per tile of 128 cached tokens: thread j scores token j
// (dot product over the query held in shared memory), the block agrees on the running maximum and sum, and
// thread d accumulates value columns d, d + 128, ... over the tile. Cache rows are [slot, kv head, dkp] and
// [slot, kv head, dvp]; the padding columns are never read.
#include "common.cuh"

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
  float m = p.sink ? 0.f : -INFINITY, l = p.sink ? 1.f : 0.f;
  for (int j0 = 0; j0 < limit; j0 += 128) {
    __syncthreads();                       // sq ready / the previous tile's sp and sslot consumed
    const int j = j0 + tid;
    float s = -INFINITY;
    long long slot = 0;
    if (j < limit) {
      long long blk = bt[j / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) {
        if (p.status) atomicCAS(p.status, 0u, MB_ST_BOUNDS);
        blk = 0;
      }
      slot = blk * p.block_size + j % p.block_size;
      const T* k = reinterpret_cast<const T*>(p.k_cache) + ((size_t)slot * p.Hkv + kvh) * p.dkp;
      float a = 0.f;
      for (int d = 0; d < p.dk; ++d) a = fmaf(sq[d], lda(k + d), a);
      s = a * p.scale;
    }
    const float m_new = fmaxf(m, mb::block_max(s, red));
    const float e = j < limit ? expf(s - m_new) : 0.f;
    sp[tid] = e;
    sslot[tid] = slot;
    const float sum = mb::block_sum(e, red);       // its barriers also publish sp and sslot
    const float alpha = expf(m - m_new);
    l = l * alpha + sum;
    m = m_new;
    const int cnt = min(128, limit - j0);
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
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.out_ld + (size_t)head * p.dv;
#pragma unroll
  for (int i = 0; i < kMaxDv / 128; ++i) {
    const int d = tid + i * 128;
    if (d < p.dv) {
      if constexpr (sizeof(T) == 2) out[d] = __float2bfloat16(acc[i] * inv);
      else out[d] = acc[i] * inv;
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
};

extern "C" int mb_attn_simt(const MbSimtAttnArgs* a, cudaStream_t stream) {
  if (!a || !a->q || !a->k_cache || !a->v_cache || !a->block_table || !a->out || a->total_rows <= 0 || a->num_seqs <= 0) return MB_ERR_BAD_ARG;
  if (a->Hkv <= 0 || a->Hq % a->Hkv || a->dk <= 0 || a->dv <= 0 || a->dv > kMaxDv || a->dk > 2048 || a->dk > a->dkp || a->dv > a->dvp) return MB_ERR_UNSUPPORTED;
  if (a->total_rows > 65535) return MB_ERR_TOO_LARGE;
  SimtAttnParams p{a->q, a->k_cache, a->v_cache, a->block_table, a->max_blocks, a->q_start, a->q_len, a->ctx_len, a->num_seqs, a->Hq, a->Hkv,
                   a->dk, a->dv, a->dkp, a->dvp, a->block_size, a->num_blocks, a->scale, a->out_scale, a->sink, a->out, a->out_ld, a->status};
  const dim3 grid(a->Hq, a->total_rows);
  const size_t smem = (size_t)a->dk * sizeof(float);
  if (a->f32) return (int)mb::launch_kernel(attn_simt_kernel<float>, grid, dim3(128), smem, stream, p);
  return (int)mb::launch_kernel(attn_simt_kernel<__nv_bfloat16>, grid, dim3(128), smem, stream, p);
}
