// Pooled blocks of a paged KV cache: block b of a sequence is the mean of its cached keys (and values) at positions b P .. b P + P - 1.  A query at position i
// sees it when b P + P - 1 <= i - window, so a step over positions [s, e) forms the blocks that become visible there -- their tokens lie in the cache by
// then, the step's own included -- and a block's row lives in a pool page beside the cache page of the block's last token: block b at page g = (b P + P - 1)
// / bs, row b - g bs / P.
//
// Long queries run on the tensor-core prefill kernel, whose tiles are dense: for them every visible block is also laid out in dense pages [sequence][page]
// [kv head][128] (older ones copied from the pool pages, rows behind the last one zeroed up to a whole page, so that a weight of zero meets a finite value).
// Steps of one token per sequence form their block inside the head epilogue (elementwise.cu).
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

struct PoolParams {
  const void* k_cache;         // [blocks][n_kv][bs][dk]
  const void* v_cache;
  void* pk;                    // [blocks][n_kv][rows][dk]
  void* pv;
  void* dense_k;               // [B * dense_pages][n_kv][128][dk], or null
  void* dense_v;
  const int* block_table;      // [B][max_blocks]
  const int* seq_lens;
  const int* cu_q;
  int n_kv, bs, dk, dv, pool, rows, window, max_blocks, dense_pages;
};
constexpr int POOL_WARPS = 4;

// four columns per lane and pass; T bf16 or fp32
template <typename T>
__device__ __forceinline__ void pool_row_mean(const PoolParams& p, const T* cache, T* out, T* dense, int b, int seq, int kvh, int width, int lane) {
  const int* table = p.block_table + (size_t)seq * p.max_blocks;
  for (int c = lane * 4; c < width; c += 128) {
    float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
    for (int j = 0; j < p.pool; ++j) {
      const int at = b * p.pool + j;
      float v[4];
      loadv<4>(cache + (((size_t)table[at / p.bs] * p.n_kv + kvh) * p.bs + at % p.bs) * width + c, v);
#pragma unroll
      for (int e = 0; e < 4; ++e) a[e] += v[e];
    }
    const float n = (float)p.pool;
#pragma unroll
    for (int e = 0; e < 4; ++e) a[e] /= n;
    storev<4>(out + c, a);
    if (dense) storev<4>(dense + c, a);
  }
}

// blockIdx: (four blocks, sequence, kv head), a warp per block
template <typename T>
__global__ void __launch_bounds__(POOL_WARPS * 32) pool_blocks_kernel(const PoolParams p) {
  pdl_prologue();
  const int seq = blockIdx.y, kvh = blockIdx.z, lane = threadIdx.x & 31;
  const int n = p.cu_q[seq + 1] - p.cu_q[seq];
  if (n <= 0) return;
  const int end = p.seq_lens[seq], start = end - n;
  const int seen = end > p.window ? (end - p.window) / p.pool : 0;                // blocks that the last query sees
  const int first = start > p.window ? (start - p.window) / p.pool : 0;           // ... that earlier steps saw
  int b = blockIdx.x * POOL_WARPS + (threadIdx.x >> 5);
  if (!p.dense_k) b += first;
  T *dk = nullptr, *dv = nullptr;
  if (p.dense_k) {
    if (b >= (seen + 127) / 128 * 128) return;
    const size_t row = (((size_t)seq * p.dense_pages + b / 128) * p.n_kv + kvh) * 128 + b % 128;
    dk = reinterpret_cast<T*>(p.dense_k) + row * p.dk;
    dv = reinterpret_cast<T*>(p.dense_v) + row * p.dv;
    if (b >= seen) {
      const float zero[4] = {0.f, 0.f, 0.f, 0.f};
      for (int c = lane * 4; c < p.dk; c += 128) storev<4>(dk + c, zero);
      for (int c = lane * 4; c < p.dv; c += 128) storev<4>(dv + c, zero);
      return;
    }
  } else if (b >= seen) {
    return;
  }
  const int page = (b * p.pool + p.pool - 1) / p.bs;
  const size_t at = ((size_t)p.block_table[(size_t)seq * p.max_blocks + page] * p.n_kv + kvh) * p.rows + (b - page * p.bs / p.pool);
  T* pk = reinterpret_cast<T*>(p.pk) + at * p.dk;
  T* pv = reinterpret_cast<T*>(p.pv) + at * p.dv;
  if (b >= first) {
    pool_row_mean(p, reinterpret_cast<const T*>(p.k_cache), pk, dk, b, seq, kvh, p.dk, lane);
    pool_row_mean(p, reinterpret_cast<const T*>(p.v_cache), pv, dv, b, seq, kvh, p.dv, lane);
  } else {                                                                        // (dense only)
    float v[4];
    for (int c = lane * 4; c < p.dk; c += 128) { loadv<4>(pk + c, v); storev<4>(dk + c, v); }
    for (int c = lane * 4; c < p.dv; c += 128) { loadv<4>(pv + c, v); storev<4>(dv + c, v); }
  }
}

}  // namespace mx

using namespace mx;

// See the head of this file.  max_blocks_seen: at least the blocks that any sequence's last query sees (dense), or that a step sees first (dense_k null).
// dense_pages * 128 >= max_blocks_seen.  Widths are multiples of 8.
MX_HOST_API int mx_pool_blocks(const void* k_cache, const void* v_cache, void* pk, void* pv, void* dense_k, void* dense_v, const int* block_table,
                               const int* seq_lens, const int* cu_q, int B, int n_kv, int bs, int dk, int dv, int pool, int rows, int window, int max_blocks,
                               int dense_pages, int max_blocks_seen, int elem_f32, cudaStream_t st) {
  if (B <= 0 || max_blocks_seen <= 0) return 0;
  if (pool < 1 || window < 1 || dk % 8 || dv % 8 || rows < (bs + pool - 1) / pool || (dense_k && (!dense_v || dense_pages * 128 < max_blocks_seen))) return -116;
  PoolParams p{k_cache, v_cache, pk, pv, dense_k, dense_v, block_table, seq_lens, cu_q, n_kv, bs, dk, dv, pool, rows, window, max_blocks, dense_pages};
  const int units = dense_k ? dense_pages * 128 : max_blocks_seen;
  const dim3 grid((unsigned)((units + POOL_WARPS - 1) / POOL_WARPS), B, n_kv), block(POOL_WARPS * 32);
  if (elem_f32) launch_pdl(pool_blocks_kernel<float>, grid, block, 0, st, p);
  else launch_pdl(pool_blocks_kernel<__nv_bfloat16>, grid, block, 0, st, p);
  return (int)cudaGetLastError();
}
