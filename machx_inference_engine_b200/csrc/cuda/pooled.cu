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

// A warp forms the mean of `pool` rows: groups of lanes take rows in turn, 16 bytes per lane.
template <typename T>
__device__ __forceinline__ void pool_row_mean(const PoolParams& p, const T* cache, T* out, T* dense, int b, int seq, int kvh, int width, int lane) {
  const int* table = p.block_table + (size_t)seq * p.max_blocks;
  constexpr int VE = 16 / sizeof(T);
  for (int p0 = 0; p0 < width / VE; p0 += 32) {
    const int per = min(32, width / VE - p0), groups = 32 / per, g = lane / per, c = (p0 + lane % per) * VE;
    float a[VE];
#pragma unroll
    for (int e = 0; e < VE; ++e) a[e] = 0.f;
    if (g < groups) {
#pragma unroll 8
      for (int j = g; j < p.pool; j += groups) {
        const int at = b * p.pool + j;
        const T* row = cache + (((size_t)table[at / p.bs] * p.n_kv + kvh) * p.bs + at % p.bs) * width + c;
#pragma unroll
        for (int i = 0; i < VE; i += 4) {
          float v[4];
          loadv<4>(row + i, v);
#pragma unroll
          for (int e = 0; e < 4; ++e) a[i + e] += v[e];
        }
      }
    }
    const float n = (float)p.pool;
#pragma unroll
    for (int e = 0; e < VE; ++e) {
      const float mine = a[e];
      for (int k = 1; k < groups; ++k) a[e] += __shfl_sync(0xffffffffu, mine, (lane + k * per) & 31);
      a[e] /= n;
    }
    if (g == 0) {
#pragma unroll
      for (int i = 0; i < VE; i += 4) {
        const float v[4] = {a[i], a[i + 1], a[i + 2], a[i + 3]};
        storev<4>(out + c + i, v);
        if (dense) storev<4>(dense + c + i, v);
      }
    }
  }
}

// blockIdx: (two blocks, sequence, kv head), a warp per block for its key and one for its value
template <typename T>
__global__ void __launch_bounds__(POOL_WARPS * 32) pool_blocks_kernel(const PoolParams p) {
  pdl_prologue();
  const int seq = blockIdx.y, kvh = blockIdx.z, lane = threadIdx.x & 31;
  const int n = p.cu_q[seq + 1] - p.cu_q[seq];
  if (n <= 0) return;
  const int end = p.seq_lens[seq], start = end - n;
  const int seen = end > p.window ? (end - p.window) / p.pool : 0;                // blocks that the last query sees
  const int first = start > p.window ? (start - p.window) / p.pool : 0;           // ... that earlier steps saw
  const bool vals = threadIdx.x & 32;
  const int width = vals ? p.dv : p.dk;
  int b = blockIdx.x * (POOL_WARPS / 2) + (threadIdx.x >> 6);
  if (!p.dense_k) b += first;
  T* dense = nullptr;
  if (p.dense_k) {
    if (b >= (seen + 127) / 128 * 128) return;
    const size_t row = (((size_t)seq * p.dense_pages + b / 128) * p.n_kv + kvh) * 128 + b % 128;
    dense = reinterpret_cast<T*>(vals ? p.dense_v : p.dense_k) + row * width;
    if (b >= seen) {
      const float zero[4] = {0.f, 0.f, 0.f, 0.f};
      for (int c = lane * 4; c < width; c += 128) storev<4>(dense + c, zero);
      return;
    }
  } else if (b >= seen) {
    return;
  }
  const int page = (b * p.pool + p.pool - 1) / p.bs;
  const size_t at = ((size_t)p.block_table[(size_t)seq * p.max_blocks + page] * p.n_kv + kvh) * p.rows + (b - page * p.bs / p.pool);
  T* out = reinterpret_cast<T*>(vals ? p.pv : p.pk) + at * width;
  if (b >= first) {
    pool_row_mean(p, reinterpret_cast<const T*>(vals ? p.v_cache : p.k_cache), out, dense, b, seq, kvh, width, lane);
  } else {                                                                        // (dense only)
    float v[4];
    for (int c = lane * 4; c < width; c += 128) { loadv<4>(out + c, v); storev<4>(dense + c, v); }
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
  const dim3 grid((unsigned)((units + POOL_WARPS / 2 - 1) / (POOL_WARPS / 2)), B, n_kv), block(POOL_WARPS * 32);
  if (elem_f32) launch_pdl(pool_blocks_kernel<float>, grid, block, 0, st, p);
  else launch_pdl(pool_blocks_kernel<__nv_bfloat16>, grid, block, 0, st, p);
  return (int)cudaGetLastError();
}
