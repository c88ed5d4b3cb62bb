// Paged attention on CUDA cores: split-KV flash-decode, small-T verify, and the general
// varlen causal kernel (sliding window, attention sinks, GQA sharing, logit soft-cap).
//
// One CTA owns (query tile, kv head, kv split).  Each 64-key K/V tile is staged in shared
// memory once and shared by every (query token, query head) pair of the group; a warp runs
// the online softmax for its pairs with one key per lane, so there is no per-key reduction.
// Every split writes an un-normalised partial (acc, m, l); the CTA of a (query tile, kv head)
// group that finishes last (an atomic ticket per group, reset by its last taker) merges the
// splits and folds the per-head sink into the denominator exactly once, so that decode is one
// launch.  Splits that would get no key tile exit at once and are not counted.  The separate
// combine kernel remains for batches with more groups than there are tickets.
//
// Keys and values may have different widths (multiples of 8, at most 512), the score scale may depend on the query's position
// (a table over positions: query temperature) and the output may be multiplied by the sigmoid of a gate.  Shapes with equal widths of
// 64 / 128 / 256 / 512 run on instances whose widths are compile-time constants; all other shapes, and caches in fp32, run on
// instances that take the widths at run time and only round the value width up to 64 / 128 / 256 / 512 (accumulator registers).
//
// Pooled blocks: with a window, means of whole runs of `pool` tokens before it are keys and values too; they lie in pool pages beside the cache pages (row
// layout: pool_row below) and are walked as tiles of their own in front of the window's.  The output may be turned back by the query's position (a rotation
// of neighbouring pairs, before the gate), which undoes a rotation of the cached values.
//
// A latent cache has no value pages: the values are the first dv elements of the key rows (v_cache null), which are staged once.
//
// KV cache layout: [block][kv_head][block_size][head_dim] bf16 (or fp32), block_size a multiple of 64.  An int8 cache has the
// same layout with one byte per element plus an fp32 scale per (block, kv head, token) row (value = q * scale); the
// staging loop widens it to bf16, so the math below is shared.  kv_dequant_pages_kernel expands the pages of a prefill
// batch into a bf16 scratch cache for the tensor-core prefill kernel.
//
// Reference parity: src/ops/attention.cpp:229-454 (naive / gpt-oss window + sink),
// :685-1036 (split-K flash decode, sink folded in combine), :2456-2714 (wide tile prefill with
// causal + window masks and whole-tile skipping).
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"
#include "mx_noalloc.h"

#include <cstdio>

namespace mx {

constexpr int ATT_WARPS = 8;
constexpr int ATT_TILE = 64;

struct AttnParams {
  const void* q;               // [Tq] rows of [n_q][dk], q_ld elements apart
  const void* k_cache;
  const void* v_cache;
  const float* k_scale;        // non-null: the caches hold int8 and these are the per-row scales [block][kv_head][block_size]
  const float* v_scale;
  const int* block_table;      // [B][max_blocks]
  const int* seq_lens;         // [B] kv length including this step's tokens
  const int* cu_q;             // [B+1]
  const float* q_scale;        // [q_scale_n] factor on the scores of a query at that position, or null
  const void* gate;            // out is multiplied by sigmoid(gate): [Tq] rows of [n_q][dv], gate_ld elements apart, or null
  int q_scale_n, q_ld, gate_ld, dk, dv;
  int gate_heads;              // the gate has one number per head: rows of [n_q]
  int keep_first;              // with a window: the first keys of the sequence that stay visible
  float* o_part;               // [splits][Tq][n_q][dv]
  float* ml_part;              // [splits][Tq][n_q][2]
  int* tickets;                // non-null: one counter per (batch entry, query tile, kv head) group; the last split merges
  const float* sinks;          // [n_q] or null (used by the merging CTA)
  void* out;                   // [Tq][n_q][dv] (written by the merging CTA)
  int B, n_q, n_kv, max_blocks, block_size;
  int q_tile;                  // query tokens per CTA
  int max_q_tiles;             // per sequence
  int n_splits;
  int Tq;
  int window;                  // 0 = full causal
  float scale, softcap;
};
// what only the extended instances take: pooled blocks and the turned output
struct AttnExtParams : AttnParams {
  const void* pk;              // pool pages [block][kv_head][pool_rows][dk], or null
  const void* pv;
  int pool, pool_rows;
  const float* out_cos;        // [out_n][out_half] or null: the output is turned by minus its position
  const float* out_sin;
  int out_n, out_half;
};
template <bool EXT> struct AttnArgs { using T = AttnParams; };
template <> struct AttnArgs<true> { using T = AttnExtParams; };

// blocks of `pool` tokens that a query at `pos` sees: those whose last token lies `window` or more before it
__device__ __forceinline__ int pool_visible(int pos, int window, int pool) { return pos >= window ? (pos - window + 1) / pool : 0; }
// row of a pool page that holds block b; the page is that of the block's last token
__device__ __forceinline__ int pool_row(int b, int pool, int page, int block_size) { return b - page * block_size / pool; }

// element d of the pair (2m, 2m + 1) turned by minus the angle; other: its neighbour
__device__ __forceinline__ float turn_back(float own, float other, int d, float c, float s) { return d & 1 ? own * c - other * s : own * c + other * s; }

// bytes `first`, `first + 1` of w as signed 8-bit integers, times scale, packed as two bf16
__device__ __forceinline__ uint32_t s8x2_to_bf16x2(uint32_t w, int first, float scale) {
  const float a = (float)(int8_t)(w >> (8 * first)) * scale, b = (float)(int8_t)(w >> (8 * first + 8)) * scale;
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&h);
}

// Pages of an int8 cache expanded to bf16: dst page (b * nb + j) = page block_table[b][j] of the source, for every page
// that holds keys of sequence b.  One CTA per (j, b, kv head).
__global__ void __launch_bounds__(256) kv_dequant_pages_kernel(const int8_t* __restrict__ k8, const int8_t* __restrict__ v8,
                                                               const float* __restrict__ ks, const float* __restrict__ vs,
                                                               const int* __restrict__ block_table, const int* __restrict__ seq_lens,
                                                               __nv_bfloat16* __restrict__ dk, __nv_bfloat16* __restrict__ dv, int n_kv,
                                                               int block_size, int hd, int max_blocks, int nb) {
  pdl_prologue();
  const int j = blockIdx.x, b = blockIdx.y, kvh = blockIdx.z;
  if ((long long)j * block_size >= seq_lens[b]) return;
  const int blk = block_table[(size_t)b * max_blocks + j];
  const size_t src = ((size_t)blk * n_kv + kvh) * block_size, dst = (((size_t)b * nb + j) * n_kv + kvh) * block_size;
  const int per_row = hd / 8;
  for (int i = threadIdx.x; i < block_size * per_row; i += blockDim.x) {
    const int r = i / per_row, c = (i % per_row) * 8;
    const uint2 kq = *reinterpret_cast<const uint2*>(k8 + (src + r) * hd + c);
    const uint2 vq = *reinterpret_cast<const uint2*>(v8 + (src + r) * hd + c);
    const float sk_ = ks[src + r], sv_ = vs[src + r];
    uint4 ko, vo;
    ko.x = s8x2_to_bf16x2(kq.x, 0, sk_); ko.y = s8x2_to_bf16x2(kq.x, 2, sk_); ko.z = s8x2_to_bf16x2(kq.y, 0, sk_); ko.w = s8x2_to_bf16x2(kq.y, 2, sk_);
    vo.x = s8x2_to_bf16x2(vq.x, 0, sv_); vo.y = s8x2_to_bf16x2(vq.x, 2, sv_); vo.z = s8x2_to_bf16x2(vq.y, 0, sv_); vo.w = s8x2_to_bf16x2(vq.y, 2, sv_);
    *reinterpret_cast<uint4*>(dk + (dst + r) * hd + c) = ko;
    *reinterpret_cast<uint4*>(dv + (dst + r) * hd + c) = vo;
  }
}

// elements by which a K row is padded in shared memory: an odd number of words apart, conflict-free one-key-per-lane reads
template <typename T> __host__ __device__ constexpr int att_kpad() { return sizeof(T) == 2 ? 2 : 1; }
// two consecutive K elements of a padded row (an fp32 row may start on an odd word)
__device__ __forceinline__ float2 k_pair(const __nv_bfloat16* r, int c) { return load2(r + 2 * c); }
__device__ __forceinline__ float2 k_pair(const float* r, int c) { return make_float2(r[2 * c], r[2 * c + 1]); }
template <bool PRECISE> __device__ __forceinline__ float att_exp(float x) { return PRECISE ? expf(x) : __expf(x); }

// EXACT: keys and values are both HD wide; otherwise the widths come from the parameters (dv <= HD).  EXT: pooled blocks, turned output.
template <typename T, int HD, int PPW, bool EXACT, bool EXT>
__global__ void __launch_bounds__(ATT_WARPS * 32, HD == 512 ? 2 : PPW == 1 ? 4 : (PPW == 2 || HD <= 128) ? 3 : 2) attn_partial_kernel(const typename AttnArgs<EXT>::T p) {
  pdl_prologue();
  constexpr int PAIRS = ATT_WARPS * PPW;
  constexpr bool PRECISE = sizeof(T) == 4;
  constexpr int VE = 16 / sizeof(T);                                               // elements per 16-byte access
  const int DK = EXACT ? HD : p.dk, DV = EXACT ? HD : p.dv;
  const int KSTR = DK + att_kpad<T>();
  const bool v_in_k = !EXACT && p.v_cache == nullptr;
  const int VSTR = v_in_k ? KSTR : DV;
  extern __shared__ uint8_t smem_raw[];
  float* sq = reinterpret_cast<float*>(smem_raw);                                  // [PAIRS][DK]
  T* sv = reinterpret_cast<T*>(sq + PAIRS * DK);                                   // [64][DV]
  T* sk = v_in_k ? sv : sv + ATT_TILE * DV;                                        // [64][KSTR] (v_in_k: the values are its first columns)
  const T* kc = reinterpret_cast<const T*>(p.k_cache);
  const T* vc = reinterpret_cast<const T*>(p.v_cache);

  const int b = blockIdx.x / p.max_q_tiles, qt = blockIdx.x % p.max_q_tiles;
  const int kvh = blockIdx.y, split = blockIdx.z;
  const int q_begin = p.cu_q[b], q_len = p.cu_q[b + 1] - q_begin;
  const int t0 = qt * p.q_tile;
  if (t0 >= q_len) return;
  const int nt = min(p.q_tile, q_len - t0);
  const int seq_len = p.seq_lens[b];
  const int pos0 = seq_len - q_len + t0;          // absolute position of the tile's first query
  const int gqa = p.n_q / p.n_kv;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  // kv range needed by this query tile, in whole 64-key tiles, then this split's share
  const int kv_hi = min(seq_len, pos0 + nt);
  const int kv_lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;
  const int tile_lo = kv_lo / ATT_TILE, tile_hi = (kv_hi + ATT_TILE - 1) / ATT_TILE;
  const int n_keep = min((p.keep_first + ATT_TILE - 1) / ATT_TILE, tile_lo);       // kept tiles before the window's
  int n_pooled = 0;
  if constexpr (EXT) {
    if (p.pk) n_pooled = pool_visible(pos0 + nt - 1, p.window, p.pool);
  }
  const int n_pool = (n_pooled + ATT_TILE - 1) / ATT_TILE;                         // tiles of pooled blocks, the first ones
  const int n_tiles = n_pool + n_keep + tile_hi - tile_lo;
  const int per = (n_tiles + p.n_splits - 1) / p.n_splits;
  const int my_lo = split * per, my_hi = min(n_tiles, my_lo + per);
  // splits that own at least one key tile (n_tiles >= 1: a query always sees its own position's tile)
  const int eff = p.tickets ? (n_tiles + per - 1) / per : p.n_splits;
  if (split >= eff) return;

  __shared__ long long s_prow[EXT ? ATT_TILE : 1];
  const int total_pairs = nt * gqa;
  for (int round0 = 0; round0 < total_pairs; round0 += PAIRS) {
    __syncthreads();
    // stage the queries of this round as fp32, pre-scaled
    for (int i = threadIdx.x; i < PAIRS * DK; i += blockDim.x) {
      const int pr = round0 + i / DK, d = i % DK;
      float v = 0.f;
      if (pr < total_pairs) {
        const int tq = pr / gqa, hq = kvh * gqa + pr % gqa;
        float sc = p.scale;
        if (p.q_scale) sc *= p.q_scale[min(pos0 + tq, p.q_scale_n - 1)];
        v = to_f32(reinterpret_cast<const T*>(p.q)[(size_t)(q_begin + t0 + tq) * p.q_ld + (size_t)hq * DK + d]) * sc;
      }
      sq[i] = v;
    }
    float m[PPW], l[PPW], acc[PPW][HD / 32];
#pragma unroll
    for (int i = 0; i < PPW; ++i) {
      m[i] = -1e30f; l[i] = 0.f;
#pragma unroll
      for (int j = 0; j < HD / 32; ++j) acc[i][j] = 0.f;
    }
    for (int tile = my_lo; tile < my_hi; ++tile) {
      __syncthreads();
      const bool pooled = EXT && tile < n_pool;
      const int tl = tile - n_pool;
      const int key0 = (pooled ? tile : tl < n_keep ? tl : tile_lo + tl - n_keep) * ATT_TILE;           // (of a pooled tile: its first block)
      const int blk = pooled ? 0 : p.block_table[(size_t)b * p.max_blocks + key0 / p.block_size];
      const size_t row0 = ((size_t)blk * p.n_kv + kvh) * p.block_size + key0 % p.block_size;
      if constexpr (EXT) if (pooled) {
        if (threadIdx.x < ATT_TILE) {
          const int pb = key0 + threadIdx.x;
          long long at = -1;
          if (pb < n_pooled) {
            const int page = (pb * p.pool + p.pool - 1) / p.block_size;
            at = ((long long)p.block_table[(size_t)b * p.max_blocks + page] * p.n_kv + kvh) * p.pool_rows + pool_row(pb, p.pool, page, p.block_size);
          }
          s_prow[threadIdx.x] = at;
        }
        __syncthreads();
        const int pk = DK / VE, pv = DV / VE;
        const uint4 zero = make_uint4(0, 0, 0, 0);
        for (int i = threadIdx.x; i < ATT_TILE * pk; i += blockDim.x) {
          const int r = i / pk, c = (i % pk) * VE;
          const long long at = s_prow[r];
          const uint4 kv4 = at >= 0 ? *reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(p.pk) + at * DK + c) : zero;
          uint32_t* kd = reinterpret_cast<uint32_t*>(sk + r * KSTR + c);
          kd[0] = kv4.x; kd[1] = kv4.y; kd[2] = kv4.z; kd[3] = kv4.w;
        }
        for (int i = threadIdx.x; i < ATT_TILE * pv; i += blockDim.x) {
          const int r = i / pv, c = (i % pv) * VE;
          const long long at = s_prow[r];
          *reinterpret_cast<uint4*>(sv + r * DV + c) = at >= 0 ? *reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(p.pv) + at * DV + c) : zero;
        }
      }
      if (pooled) {
      } else if (EXACT && sizeof(T) == 2 && p.k_scale) {
        const size_t base = row0 * HD;
        const int8_t* k8 = reinterpret_cast<const int8_t*>(p.k_cache);
        const int8_t* v8 = reinterpret_cast<const int8_t*>(p.v_cache);
        const size_t srow = row0;
        for (int i = threadIdx.x; i < ATT_TILE * HD / 8; i += blockDim.x) {
          const int r = i / (HD / 8), c = (i % (HD / 8)) * 8;
          const uint2 kq = *reinterpret_cast<const uint2*>(k8 + base + (size_t)r * HD + c);
          const uint2 vq = *reinterpret_cast<const uint2*>(v8 + base + (size_t)r * HD + c);
          const float ks = p.k_scale[srow + r], vs = p.v_scale[srow + r];
          uint32_t* kd = reinterpret_cast<uint32_t*>(sk + r * KSTR + c);
          kd[0] = s8x2_to_bf16x2(kq.x, 0, ks); kd[1] = s8x2_to_bf16x2(kq.x, 2, ks);
          kd[2] = s8x2_to_bf16x2(kq.y, 0, ks); kd[3] = s8x2_to_bf16x2(kq.y, 2, ks);
          uint4 vv;
          vv.x = s8x2_to_bf16x2(vq.x, 0, vs); vv.y = s8x2_to_bf16x2(vq.x, 2, vs);
          vv.z = s8x2_to_bf16x2(vq.y, 0, vs); vv.w = s8x2_to_bf16x2(vq.y, 2, vs);
          *reinterpret_cast<uint4*>(sv + r * HD + c) = vv;
        }
      } else {
        const int pk = DK / VE, pv = DV / VE;
        const T* kp = kc + row0 * DK;
        const T* vp = vc + row0 * DV;
        if constexpr (EXACT) {
          for (int i = threadIdx.x; i < ATT_TILE * pk; i += blockDim.x) {
            const int r = i / pk, c = (i % pk) * VE;
            const uint4 kv4 = *reinterpret_cast<const uint4*>(kp + (size_t)r * DK + c);
            uint32_t* kd = reinterpret_cast<uint32_t*>(sk + r * KSTR + c);
            kd[0] = kv4.x; kd[1] = kv4.y; kd[2] = kv4.z; kd[3] = kv4.w;
            *reinterpret_cast<uint4*>(sv + r * DV + c) = *reinterpret_cast<const uint4*>(vp + (size_t)r * DV + c);
          }
        } else {
          for (int i = threadIdx.x; i < ATT_TILE * pk; i += blockDim.x) {
            const int r = i / pk, c = (i % pk) * VE;
            const uint4 kv4 = *reinterpret_cast<const uint4*>(kp + (size_t)r * DK + c);
            uint32_t* kd = reinterpret_cast<uint32_t*>(sk + r * KSTR + c);
            kd[0] = kv4.x; kd[1] = kv4.y; kd[2] = kv4.z; kd[3] = kv4.w;
          }
          for (int i = threadIdx.x; i < (v_in_k ? 0 : ATT_TILE * pv); i += blockDim.x)            // the tile's rows are one dense run
            reinterpret_cast<uint4*>(sv)[i] = reinterpret_cast<const uint4*>(vp)[i];
        }
      }
      __syncthreads();
      // Scores of the warp's PPW pairs against the tile's 64 keys (a lane owns keys lane and lane + 32).  One pass over the key
      // row serves all pairs: a key element is read from shared memory once and multiplied into PPW dot products.
      if (round0 + warp * PPW >= total_pairs) continue;          // this warp has no live pair (barriers sit at the loop top)
      float p0[PPW], p1[PPW];
      {
        float sc[PPW][2];
        {
          // both keys of the lane in one pass: a query element read from shared memory feeds two dot products
          const T* kr0 = sk + lane * KSTR;
          const T* kr1 = sk + (lane + 32) * KSTR;
          const float* qv = sq + warp * PPW * DK;
          float d0[PPW], d1[PPW];
#pragma unroll
          for (int pi = 0; pi < PPW; ++pi) d0[pi] = d1[pi] = 0.f;
#pragma unroll 8
          for (int c = 0; c < DK / 2; ++c) {
            const float2 ka = k_pair(kr0, c), kb = k_pair(kr1, c);
            const float a0 = ka.x, a1 = ka.y, b0 = kb.x, b1 = kb.y;
#pragma unroll
            for (int pi = 0; pi < PPW; ++pi) {
              const float2 qq = *reinterpret_cast<const float2*>(qv + pi * DK + 2 * c);
              d0[pi] = fmaf(qq.x, a0, d0[pi]); d0[pi] = fmaf(qq.y, a1, d0[pi]);
              d1[pi] = fmaf(qq.x, b0, d1[pi]); d1[pi] = fmaf(qq.y, b1, d1[pi]);
            }
          }
#pragma unroll
          for (int pi = 0; pi < PPW; ++pi) {
            const int pr = round0 + warp * PPW + pi;
            const int qpos = pos0 + pr / gqa;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
              const int kpos = key0 + lane + 32 * half;
              float dd = half ? d1[pi] : d0[pi];
              if (p.softcap > 0.f) dd = p.softcap * tanhf(dd / p.softcap);
              bool ok = pr < total_pairs;
              if constexpr (EXT) {
                if (pooled) ok = ok && kpos < pool_visible(qpos, p.window, p.pool);
              }
              if (!pooled) ok = ok && kpos < seq_len && kpos <= qpos && (p.window <= 0 || kpos > qpos - p.window || kpos < p.keep_first);
              sc[pi][half] = ok ? dd : -INFINITY;
            }
          }
        }
#pragma unroll
        for (int pi = 0; pi < PPW; ++pi) {
          const float tmax = warp_max(fmaxf(sc[pi][0], sc[pi][1]));
          const float m_new = fmaxf(m[pi], tmax);
          const float corr = att_exp<PRECISE>(m[pi] - m_new);
          p0[pi] = att_exp<PRECISE>(sc[pi][0] - m_new);
          p1[pi] = att_exp<PRECISE>(sc[pi][1] - m_new);
          l[pi] = l[pi] * corr + warp_sum(p0[pi] + p1[pi]);
          m[pi] = m_new;
#pragma unroll
          for (int c = 0; c < HD / 32; ++c) acc[pi][c] *= corr;
        }
      }
      // P V: a value element is read once per key and feeds all PPW pairs
#pragma unroll 2
      for (int j = 0; j < ATT_TILE; ++j) {
        const T* vr = sv + j * VSTR;
        float vv[HD / 32];
#pragma unroll
        for (int c = 0; c < HD / 32; ++c) vv[c] = (EXACT || lane + 32 * c < DV) ? to_f32(vr[lane + 32 * c]) : 0.f;
#pragma unroll
        for (int pi = 0; pi < PPW; ++pi) {
          const float pj = __shfl_sync(0xffffffffu, j < 32 ? p0[pi] : p1[pi], j & 31);
#pragma unroll
          for (int c = 0; c < HD / 32; ++c) acc[pi][c] = fmaf(pj, vv[c], acc[pi][c]);
        }
      }
    }
    // write partials
#pragma unroll
    for (int pi = 0; pi < PPW; ++pi) {
      const int pr = round0 + warp * PPW + pi;
      if (pr >= total_pairs) continue;
      const int tq = pr / gqa, hq = kvh * gqa + pr % gqa;
      const size_t row = ((size_t)split * p.Tq + (q_begin + t0 + tq)) * p.n_q + hq;
#pragma unroll
      for (int c = 0; c < HD / 32; ++c)
        if (EXACT || lane + 32 * c < DV) p.o_part[row * DV + lane + 32 * c] = acc[pi][c];
      if (lane == 0) { p.ml_part[row * 2] = m[pi]; p.ml_part[row * 2 + 1] = l[pi]; }
    }
  }
  if (!p.tickets) return;
  // ---- the group's last CTA merges the splits
  __shared__ int s_last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    int* tk = p.tickets + (size_t)blockIdx.x * p.n_kv + kvh;
    const int prev = atomicAdd(tk, 1);
    s_last = prev == eff - 1;
    if (s_last) *tk = 0;                 // every counted split has arrived: the counter is ready for the next launch
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  const size_t sstride = (size_t)p.Tq * p.n_q;
  for (int pr = warp; pr < total_pairs; pr += ATT_WARPS) {
    const int tq = pr / gqa, hq = kvh * gqa + pr % gqa;
    const size_t r = (size_t)(q_begin + t0 + tq) * p.n_q + hq;
    float M = p.sinks ? p.sinks[hq] : -1e30f;
    for (int s = lane; s < eff; s += 32) M = fmaxf(M, __ldcg(p.ml_part + (s * sstride + r) * 2));
    M = warp_max(M);
    float L = 0.f;
    for (int s = lane; s < eff; s += 32) {
      const float2 ml = __ldcg(reinterpret_cast<const float2*>(p.ml_part + (s * sstride + r) * 2));
      L += ml.y * att_exp<PRECISE>(ml.x - M);
    }
    L = warp_sum(L) + (p.sinks ? att_exp<PRECISE>(p.sinks[hq] - M) : 0.f);
    const float inv = L > 0.f ? 1.f / L : 0.f;
    float acc[HD / 32];
#pragma unroll
    for (int c = 0; c < HD / 32; ++c) acc[c] = 0.f;
    for (int s0 = 0; s0 < eff; s0 += 32) {
      const float sc_l = s0 + lane < eff ? att_exp<PRECISE>(__ldcg(p.ml_part + ((s0 + lane) * sstride + r) * 2) - M) : 0.f;
      const int cnt = min(32, eff - s0);
#pragma unroll 4
      for (int j = 0; j < cnt; ++j) {
        const float sc = __shfl_sync(0xffffffffu, sc_l, j);
        const float* op = p.o_part + ((s0 + j) * sstride + r) * DV;
#pragma unroll
        for (int c = 0; c < HD / 32; ++c)
          if (EXACT || lane + 32 * c < DV) acc[c] = fmaf(__ldcg(op + lane + 32 * c), sc, acc[c]);
      }
    }
#pragma unroll
    for (int c = 0; c < HD / 32; ++c) {
      const int d = lane + 32 * c;
      float o = acc[c] * inv;
      if constexpr (EXT) if (p.out_cos) {
        const float other = __shfl_xor_sync(0xffffffffu, o, 1);
        if ((d >> 1) < p.out_half) {
          const size_t at = (size_t)min(pos0 + tq, p.out_n - 1) * p.out_half + (d >> 1);
          o = turn_back(o, other, d, __ldg(p.out_cos + at), __ldg(p.out_sin + at));
        }
      }
      if (!EXACT && d >= DV) continue;
      if (p.gate) o *= sigmoid_f<PRECISE>(to_f32(reinterpret_cast<const T*>(p.gate)[(size_t)(q_begin + t0 + tq) * p.gate_ld + (p.gate_heads ? hq : (size_t)hq * DV + d)]));
      reinterpret_cast<T*>(p.out)[r * DV + d] = from_f32<T>(o);
    }
  }
}

// out[t][h][:] = sum_s acc_s e^{m_s - M} / (sum_s l_s e^{m_s - M} + e^{sink_h - M}) [* sigmoid(gate)].  blockIdx: (row, run of 256 columns);
// every warp forms the weights of the splits, a lane per split, and a thread sums two columns over them.
constexpr int CMB_COLS = 256;
struct AttnTurn {              // out_cos .. of AttnParams and what gives a row its position
  const float* cos;
  const float* sin;
  const int* seq_lens;
  const int* cu_q;
  int n, half, B;
};
template <typename T>
__global__ void __launch_bounds__(CMB_COLS / 2) attn_combine_kernel(const float* __restrict__ o_part, const float* __restrict__ ml_part,
                                                                    const float* __restrict__ sinks, const T* __restrict__ gate, int gate_ld, int gate_heads,
                                                                    T* __restrict__ out, int Tq, int n_q, int hd, int n_splits, const AttnTurn turn) {
  constexpr bool PRECISE = sizeof(T) == 4;
  pdl_prologue();
  const int r = blockIdx.x, lane = threadIdx.x & 31, h = r % n_q;
  const int d = blockIdx.y * CMB_COLS + threadIdx.x * 2;
  const size_t rows = (size_t)Tq * n_q;
  const float2* ml = reinterpret_cast<const float2*>(ml_part);
  float M = sinks ? sinks[h] : -1e30f;
  for (int s = lane; s < n_splits; s += 32) M = fmaxf(M, ml[s * rows + r].x);
  M = warp_max(M);
  float L = 0.f;
  float a0 = 0.f, a1 = 0.f;
  for (int s0 = 0; s0 < n_splits; s0 += 32) {
    float w = 0.f;
    if (s0 + lane < n_splits) {
      const float2 v = ml[(s0 + lane) * rows + r];
      w = att_exp<PRECISE>(v.x - M);
      L = fmaf(v.y, w, L);
    }
    const int cnt = min(32, n_splits - s0);
    const float* op = o_part + ((size_t)s0 * rows + r) * hd + d;
#pragma unroll 8
    for (int j = 0; j < cnt; ++j) {
      const float wj = __shfl_sync(0xffffffffu, w, j);
      if (wj != 0.f && d < hd) {                                       // (a split without keys leaves its rows unwritten)
        const float2 v = *reinterpret_cast<const float2*>(op + (size_t)j * rows * hd);
        a0 = fmaf(v.x, wj, a0);
        a1 = fmaf(v.y, wj, a1);
      }
    }
  }
  L = warp_sum(L) + (sinks ? att_exp<PRECISE>(sinks[h] - M) : 0.f);
  if (d >= hd) return;
  const float inv = L > 0.f ? 1.f / L : 0.f;
  a0 *= inv;
  a1 *= inv;
  if (turn.cos && d / 2 < turn.half) {
    const int t = r / n_q;
    int b = 0;
    while (b + 1 < turn.B && turn.cu_q[b + 1] <= t) ++b;
    const int pos = turn.seq_lens[b] - (turn.cu_q[b + 1] - t);
    const size_t at = (size_t)min(pos, turn.n - 1) * turn.half + d / 2;
    const float u = a0, v = a1, c = __ldg(turn.cos + at), s = __ldg(turn.sin + at);
    a0 = turn_back(u, v, 0, c, s);
    a1 = turn_back(v, u, 1, c, s);
  }
  if (gate) {
    const T* gr = gate + (size_t)(r / n_q) * gate_ld;
    const float2 g = gate_heads ? make_float2(to_f32(gr[h]), to_f32(gr[h])) : load2(gr + (size_t)h * hd + d);
    a0 *= sigmoid_f<PRECISE>(g.x);
    a1 *= sigmoid_f<PRECISE>(g.y);
  }
  store2(out + (size_t)r * hd + d, a0, a1);
}

// Tickets of the fused merge: zero at load, and every launch leaves its counters at zero again.  Consecutive launches rotate
// through the slots, so that two launches that overlap (programmatic dependent launch lets the next kernel's CTAs start while
// this one drains) never count on the same words.
constexpr int ATT_TICKET_SLOTS = 8, ATT_TICKETS_PER_SLOT = 2048;
static __device__ int g_attn_tickets[ATT_TICKET_SLOTS * ATT_TICKETS_PER_SLOT];

constexpr size_t ATT_SMEM_MAX = 226 * 1024;           // (the kernel also has a few static bytes)
static size_t att_smem(const AttnParams& p, int ppw, int elem, int kpad) {
  return (size_t)ATT_WARPS * ppw * p.dk * 4 + (size_t)ATT_TILE * (p.dk + kpad) * elem + (p.v_cache ? (size_t)ATT_TILE * p.dv * elem : 0);
}

template <typename T, int HD, int PPW, bool EXACT, bool EXT>
static int launch_partial(const AttnExtParams& p, cudaStream_t st) {
  constexpr size_t SMEM_MAX = ATT_SMEM_MAX;
  const size_t smem = att_smem(p, PPW, sizeof(T), att_kpad<T>());
  if (smem > SMEM_MAX) return -112;
  auto kern = attn_partial_kernel<T, HD, PPW, EXACT, EXT>;
  static DeviceOnce configured;
  if (configured.pending()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, EXACT ? (int)smem : (int)SMEM_MAX);
    if (e != cudaSuccess) return (int)e;
    configured.mark();
  }
  dim3 grid(p.B * p.max_q_tiles, p.n_kv, p.n_splits);
  const typename AttnArgs<EXT>::T args = p;
  launch_pdl(kern, dim3(grid), dim3(ATT_WARPS * 32), smem, st, args);
  return (int)cudaGetLastError();
}

}  // namespace mx

using namespace mx;

// pairs per warp (1 for decode-sized work, 4 when there are many query tokens), query tokens per CTA, query tiles per sequence
static void att_tiling(int max_q_len, int gqa, int& ppw, int& q_tile, int& max_q_tiles, int max_ppw = 4) {
  ppw = (max_q_len * gqa > ATT_WARPS * 2) ? 4 : (max_q_len * gqa > ATT_WARPS ? 2 : 1);
  if (ppw > max_ppw) ppw = max_ppw;
  const int pairs = ATT_WARPS * ppw;
  q_tile = pairs / gqa > 0 ? pairs / gqa : 1;
  if (q_tile > max_q_len) q_tile = max_q_len;
  max_q_tiles = (max_q_len + q_tile - 1) / q_tile;
}

// Kernels one attention call launches: 1 when the split merge runs inside the partial kernel, 2 with the separate combine.
MX_HOST_API int mx_attention_launches(int B, int max_q_len, int n_q, int n_kv) {
  int ppw, q_tile, max_q_tiles;
  att_tiling(max_q_len, n_q / (n_kv > 0 ? n_kv : 1), ppw, q_tile, max_q_tiles);
  return (long long)B * max_q_tiles * n_kv <= ATT_TICKETS_PER_SLOT ? 1 : 2;
}

// Scratch: o_part needs n_splits*Tq*n_q*hd floats, ml_part n_splits*Tq*n_q*2 floats.
// max_q_len is the longest query segment of the batch (host knows it from cu_q).
struct AttnShape {            // what the plain entry points leave at its default
  int dk, dv, q_ld;           // q_ld: elements between the query rows
  const void* gate = nullptr;
  int gate_ld = 0;
  const float* q_scale = nullptr;
  int q_scale_n = 0;
  int elem_f32 = 0;           // queries, cache, gate and output in fp32
  int gate_heads = 0, keep_first = 0;
  const void* pk = nullptr;
  const void* pv = nullptr;
  int pool = 0, pool_rows = 0;
  const float* out_cos = nullptr;
  const float* out_sin = nullptr;
  int out_n = 0, out_half = 0;
};
static int attention_impl(const void* q, const void* k_cache, const void* v_cache, const float* k_scale, const float* v_scale,
                          const int* block_table, const int* seq_lens, const int* cu_q, const float* sinks, void* out, float* o_part,
                          float* ml_part, int B, int Tq, int max_q_len, int n_q, int n_kv, const AttnShape& sh, int max_blocks, int block_size,
                          int window, float scale, float softcap, int n_splits, cudaStream_t st) {
  if (B <= 0 || Tq <= 0) return 0;
  if (block_size % ATT_TILE) return -110;
  if (n_q % n_kv) return -111;
  const int gqa = n_q / n_kv;
  AttnExtParams p;
  p.q = q; p.k_cache = k_cache; p.v_cache = v_cache;
  p.dk = sh.dk; p.dv = sh.dv; p.q_ld = sh.q_ld; p.gate = sh.gate; p.gate_ld = sh.gate_ld; p.gate_heads = sh.gate_heads; p.keep_first = window > 0 ? sh.keep_first : 0; p.q_scale = sh.q_scale; p.q_scale_n = sh.q_scale_n;
  p.pk = window > 0 && sh.pool > 0 ? sh.pk : nullptr; p.pv = sh.pv; p.pool = sh.pool; p.pool_rows = sh.pool_rows;
  p.out_cos = sh.out_cos; p.out_sin = sh.out_sin; p.out_n = sh.out_n; p.out_half = sh.out_half;
  if (p.pk && (k_scale || !v_cache)) return -112;
  p.k_scale = k_scale; p.v_scale = k_scale ? v_scale : nullptr;
  p.block_table = block_table; p.seq_lens = seq_lens; p.cu_q = cu_q; p.o_part = o_part; p.ml_part = ml_part;
  p.B = B; p.n_q = n_q; p.n_kv = n_kv; p.max_blocks = max_blocks; p.block_size = block_size;
  p.n_splits = n_splits < 1 ? 1 : n_splits; p.Tq = Tq; p.window = window; p.scale = scale; p.softcap = softcap;
  int ppw;
  int max_ppw = 4;                                    // wide rows: fewer queries at a time, so that they fit beside the key tile
  while (max_ppw > 1 && att_smem(p, max_ppw, sh.elem_f32 ? 4 : 2, 2) > ATT_SMEM_MAX) max_ppw /= 2;
  att_tiling(max_q_len, gqa, ppw, p.q_tile, p.max_q_tiles, max_ppw);
  p.tickets = nullptr; p.sinks = sinks; p.out = out;
  const long long groups = (long long)B * p.max_q_tiles * n_kv;
  if (groups <= ATT_TICKETS_PER_SLOT) {
    static int* base[64] = {nullptr};
    static unsigned turn[64] = {0};
    int dev = 0;
    cudaGetDevice(&dev);
    dev &= 63;
    if (!base[dev]) {
      void* a = nullptr;
      if (cudaGetSymbolAddress(&a, g_attn_tickets) != cudaSuccess) return -115;
      base[dev] = (int*)a;
    }
    p.tickets = base[dev] + (size_t)(turn[dev]++ % ATT_TICKET_SLOTS) * ATT_TICKETS_PER_SLOT;
  }
  int rc;
  const bool ext = p.pk || p.out_cos;
#define MX_ATT_E(T_, HD_, EX_, XT_) \
  (ppw == 4 ? launch_partial<T_, HD_, 4, EX_, XT_>(p, st) : ppw == 2 ? launch_partial<T_, HD_, 2, EX_, XT_>(p, st) : launch_partial<T_, HD_, 1, EX_, XT_>(p, st))
#define MX_ATT(T_, HD_, EX_) (ext ? MX_ATT_E(T_, HD_, EX_, true) : MX_ATT_E(T_, HD_, EX_, false))
  const int dk = sh.dk, dv = sh.dv, ve = sh.elem_f32 ? 4 : 8;
  if (dk < 1 || dv < 1 || dk > (v_cache ? 512 : 1024) || dv > 512 || dk % ve || dv % ve || (!v_cache && dv > dk)) return -112;
  if (!sh.elem_f32 && v_cache && dk == dv && (dk == 64 || dk == 128 || dk == 256 || dk == 512)) {
    switch (dk) {
      case 64: rc = MX_ATT(__nv_bfloat16, 64, true); break;
      case 128: rc = MX_ATT(__nv_bfloat16, 128, true); break;
      case 256: rc = MX_ATT(__nv_bfloat16, 256, true); break;
      default: rc = MX_ATT(__nv_bfloat16, 512, true); break;      // Gemma-4 global layers
    }
  } else if (k_scale) {
    return -112;                                                  // int8 rows: instances with fixed widths only
  } else if (sh.elem_f32) {
    rc = dv <= 64 ? MX_ATT(float, 64, false) : dv <= 128 ? MX_ATT(float, 128, false) : dv <= 256 ? MX_ATT(float, 256, false) : MX_ATT(float, 512, false);
  } else {
    rc = dv <= 64 ? MX_ATT(__nv_bfloat16, 64, false) : dv <= 128 ? MX_ATT(__nv_bfloat16, 128, false)
         : dv <= 256 ? MX_ATT(__nv_bfloat16, 256, false) : MX_ATT(__nv_bfloat16, 512, false);
  }
#undef MX_ATT
#undef MX_ATT_E
  if (rc || p.tickets) return rc;
  const dim3 cgrid(Tq * n_q, (dv + CMB_COLS - 1) / CMB_COLS);
  const AttnTurn turn{p.out_cos, p.out_sin, seq_lens, cu_q, p.out_n, p.out_half, B};
  if (sh.elem_f32)
    launch_pdl(attn_combine_kernel<float>, cgrid, dim3(CMB_COLS / 2), 0, st, o_part, ml_part, sinks, (const float*)sh.gate, sh.gate_ld, sh.gate_heads, (float*)out, Tq, n_q, dv, p.n_splits, turn);
  else
    launch_pdl(attn_combine_kernel<__nv_bfloat16>, cgrid, dim3(CMB_COLS / 2), 0, st, o_part, ml_part, sinks, (const __nv_bfloat16*)sh.gate, sh.gate_ld, sh.gate_heads,
               (__nv_bfloat16*)out, Tq, n_q, dv, p.n_splits, turn);
  return (int)cudaGetLastError();
}

// Merge of split partials (o_part un-normalised, ml_part (maximum, denominator) per row): out bf16 [Tq][n_q][dv].
MX_HOST_API int mx_attention_combine(const float* o_part, const float* ml_part, void* out, int Tq, int n_q, int dv, int n_splits, cudaStream_t st) {
  if (Tq <= 0) return 0;
  const float* no_sinks = nullptr;
  const __nv_bfloat16* no_gate = nullptr;
  launch_pdl(attn_combine_kernel<__nv_bfloat16>, dim3(Tq * n_q, (dv + CMB_COLS - 1) / CMB_COLS), dim3(CMB_COLS / 2), 0, st, o_part, ml_part, no_sinks, no_gate, 0, 0, (__nv_bfloat16*)out, Tq, n_q, dv,
             n_splits, AttnTurn{});
  return (int)cudaGetLastError();
}

static AttnShape plain_shape(int n_q, int hd) {
  AttnShape sh;
  sh.dk = sh.dv = hd;
  sh.q_ld = n_q * hd;
  return sh;
}

// Queries [Tq] rows of [n_q][dk] (q_ld elements apart), cache pages of dk- / dv-wide rows, out [Tq][n_q][dv]; optional gate (rows of
// [n_q][dv], or with gate_heads of [n_q], gate_ld apart; out *= sigmoid(gate)) and per-position score factors q_scale [q_scale_n].  elem_f32: everything in
// fp32.  With a window the first keep_first keys of a sequence stay visible.
// o_part needs n_splits*Tq*n_q*dv floats.  Rows, widths and strides are multiples of 16 bytes.  v_cache null: a value is the first dv elements of
// its key row.  pk / pv: pool pages of `pool` tokens per block and pool_rows rows per page (window > 0); out_cos / out_sin [out_n][out_half]: the output turned
// by minus its position in neighbouring pairs.
MX_HOST_API int mx_attention_ext(const void* q, int q_ld, const void* k_cache, const void* v_cache, const int* block_table, const int* seq_lens,
                                 const int* cu_q, const float* sinks, const void* gate, int gate_ld, const float* q_scale, int q_scale_n, void* out,
                                 float* o_part, float* ml_part, int B, int Tq, int max_q_len, int n_q, int n_kv, int dk, int dv, int max_blocks,
                                 int block_size, int window, int keep_first, int gate_heads, float scale, float softcap, int n_splits, int elem_f32,
                                 const void* pk, const void* pv, int pool, int pool_rows, const float* out_cos, const float* out_sin, int out_n, int out_half,
                                 cudaStream_t st) {
  AttnShape sh;
  sh.pk = pk; sh.pv = pv; sh.pool = pool; sh.pool_rows = pool_rows; sh.out_cos = out_cos; sh.out_sin = out_sin; sh.out_n = out_n; sh.out_half = out_half;
  sh.gate_heads = gate_heads; sh.keep_first = keep_first;
  sh.dk = dk; sh.dv = dv; sh.q_ld = q_ld; sh.gate = gate; sh.gate_ld = gate_ld; sh.q_scale = q_scale; sh.q_scale_n = q_scale_n; sh.elem_f32 = elem_f32;
  return attention_impl(q, k_cache, v_cache, nullptr, nullptr, block_table, seq_lens, cu_q, sinks, out, o_part, ml_part, B, Tq, max_q_len, n_q, n_kv,
                        sh, max_blocks, block_size, window, scale, softcap, n_splits, st);
}

MX_HOST_API int mx_attention(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* seq_lens,
                             const int* cu_q, const float* sinks, void* out, float* o_part, float* ml_part, int B, int Tq, int max_q_len,
                             int n_q, int n_kv, int hd, int max_blocks, int block_size, int window, float scale, float softcap,
                             int n_splits, cudaStream_t st) {
  return attention_impl(q, k_cache, v_cache, nullptr, nullptr, block_table, seq_lens, cu_q, sinks, out, o_part, ml_part, B, Tq, max_q_len, n_q,
                        n_kv, plain_shape(n_q, hd), max_blocks, block_size, window, scale, softcap, n_splits, st);
}

// The same over an int8 cache with per-row scales (see the layout note at the top of this file).
MX_HOST_API int mx_attention_kv8(const void* q, const void* k_cache, const void* v_cache, const float* k_scale, const float* v_scale,
                                 const int* block_table, const int* seq_lens, const int* cu_q, const float* sinks, void* out, float* o_part,
                                 float* ml_part, int B, int Tq, int max_q_len, int n_q, int n_kv, int hd, int max_blocks, int block_size,
                                 int window, float scale, float softcap, int n_splits, cudaStream_t st) {
  if (!k_scale || !v_scale) return -113;
  return attention_impl(q, k_cache, v_cache, k_scale, v_scale, block_table, seq_lens, cu_q, sinks, out, o_part, ml_part, B, Tq, max_q_len, n_q,
                        n_kv, plain_shape(n_q, hd), max_blocks, block_size, window, scale, softcap, n_splits, st);
}

// dst_k / dst_v: bf16 [B * nb][n_kv][block_size][hd]; page (b, j) is filled when j * block_size < seq_lens[b].
MX_HOST_API int mx_kv_dequant_pages(const void* k8, const void* v8, const float* k_scale, const float* v_scale, const int* block_table,
                                    const int* seq_lens, void* dst_k, void* dst_v, int B, int n_kv, int block_size, int hd, int max_blocks,
                                    int nb, cudaStream_t st) {
  if (B <= 0 || nb <= 0) return 0;
  if (hd % 8) return -114;
  launch_pdl(kv_dequant_pages_kernel, dim3(nb, B, n_kv), dim3(256), 0, st, (const int8_t*)k8, (const int8_t*)v8, k_scale, v_scale, block_table,
             seq_lens, (__nv_bfloat16*)dst_k, (__nv_bfloat16*)dst_v, n_kv, block_size, hd, max_blocks, nb);
  return (int)cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------
// Allocation-free variant (see mx_noalloc.h): the split-KV partials live in this fixed device array.
// In host code the array's name is only a handle for cudaGetSymbolAddress; the kernels are given the
// device address that call returns.
static __device__ __align__(256) float g_noalloc_scratch[MX_NOALLOC_SCRATCH_FLOATS];

namespace {
float* g_noalloc_ptr[64] = {nullptr};        // per device, resolved on first use
thread_local char g_noalloc_err[256] = "";
}  // namespace

MX_HOST_API const char* mx_attention_noalloc_error(void) { return g_noalloc_err; }

MX_HOST_API int mx_attention_noalloc(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* seq_lens,
                                     const int* cu_q, const float* sinks, void* out, int B, int Tq, int max_q_len, int n_q, int n_kv, int hd,
                                     int max_blocks, int block_size, int window, float scale, float softcap, int n_splits,
                                     cudaStream_t stream) {
  g_noalloc_err[0] = 0;
  if (B <= 0 || Tq <= 0) return 0;
  const int splits = n_splits < 1 ? 1 : n_splits;
  const unsigned long long need = (unsigned long long)splits * Tq * n_q * (unsigned long long)(hd + 2);
  if (need > MX_NOALLOC_SCRATCH_FLOATS) {
    snprintf(g_noalloc_err, sizeof g_noalloc_err,
             "mx_attention_noalloc: needs %llu scratch floats (n_splits %d x Tq %d x n_q %d x (head_dim %d + 2)) but the built-in scratch holds %u; "
             "use fewer splits / tokens or call mx_attention with caller-provided scratch",
             need, splits, Tq, n_q, hd, (unsigned)MX_NOALLOC_SCRATCH_FLOATS);
    return MX_NOALLOC_E_TOO_LARGE;
  }
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess || dev < 0 || dev >= 64) {
    snprintf(g_noalloc_err, sizeof g_noalloc_err, "mx_attention_noalloc: cannot identify the current device (%s)", cudaGetErrorString(e));
    return MX_NOALLOC_E_SYMBOL;
  }
  if (!g_noalloc_ptr[dev]) {
    // once per device, with that device current: turn the symbol into a device address
    float* ptr = nullptr;
    e = cudaGetSymbolAddress((void**)&ptr, g_noalloc_scratch);
    if (e != cudaSuccess || !ptr) {
      snprintf(g_noalloc_err, sizeof g_noalloc_err, "mx_attention_noalloc: cudaGetSymbolAddress failed on device %d (%s)", dev, cudaGetErrorString(e));
      return MX_NOALLOC_E_SYMBOL;
    }
    g_noalloc_ptr[dev] = ptr;
  }
  float* o_part = g_noalloc_ptr[dev];
  float* ml_part = o_part + (size_t)splits * Tq * n_q * hd;
  return mx_attention(q, k_cache, v_cache, block_table, seq_lens, cu_q, sinks, out, o_part, ml_part, B, Tq, max_q_len, n_q, n_kv, hd, max_blocks,
                      block_size, window, scale, softcap, splits, stream);
}
