// Latent attention around the attention kernels: every token caches one row [c | r] (normed latent, rotated key part) that serves all heads.
//   latent_post   : latent RMS norm, rotation of the shared key part and of every head's rotated query part (interleaved pairs), cache row
//   head_linear   : every head its own small matrix (queries into the latent space, latent outputs to values), optional sigmoid gate; few rows
//                   or 32-bit activations -- many 16-bit rows run on the tensor cores (gemm_tcgen05.cu)
//   latent_plan   : the cache pages in reach of the long queries of a batch, as one list, and the page table of their expanded form
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

// ------------------------------------------------------------------ latent_post
struct LatentPostParams {
  const void* q;               // rotated query parts: row t of head h at t * q_ld + h * q_hs, r elements
  void* q_out;                 // the same, rotated: t * qo_ld + h * qo_hs (may be q)
  const void* ckv;             // rows of [R | r] elements, ckv_ld apart
  const float* norm_w;         // [R], zero past rank
  const int* positions;        // [T]
  const float* rope_cos;       // [max_pos][half]
  const float* rope_sin;
  const long long* slot_map;   // [T], < 0: no cache row
  void* cache;                 // [blocks][block_size][R + r] (a slot is a row)
  int q_ld, q_hs, qo_ld, qo_hs, ckv_ld;
  int H, R, r, rank, half, max_pos;
  float eps;
};

// 8 consecutive elements (pointer aligned to 16 bytes of bf16 / 32 of fp32)
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 t = *reinterpret_cast<const uint4*>(p);
  v[0] = bf16_lo(t.x); v[1] = bf16_hi(t.x); v[2] = bf16_lo(t.y); v[3] = bf16_hi(t.y); v[4] = bf16_lo(t.z); v[5] = bf16_hi(t.z); v[6] = bf16_lo(t.w); v[7] = bf16_hi(t.w);
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

// One CTA per token.  Warp 0 norms the latent and writes it (a lane keeps up to 16 of its elements in registers); the others rotate four pairs per
// thread of the H query parts and of the key part.
constexpr int LP_THREADS = 192;
template <typename T>
__global__ void __launch_bounds__(LP_THREADS) latent_post_kernel(const LatentPostParams p) {
  pdl_prologue();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* ckv = reinterpret_cast<const T*>(p.ckv) + (size_t)t * p.ckv_ld;
  const long long slot = p.slot_map[t];
  T* row = slot < 0 ? nullptr : reinterpret_cast<T*>(p.cache) + (size_t)slot * (p.R + p.r);
  if (warp == 0) {
    if (!row) return;
    const int n8 = p.R / 8;
    float v[2][8], ss = 0.f;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = lane + 32 * j;
      if (c < n8) {
        load8(ckv + 8 * c, v[j]);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = 8 * c + e < p.rank ? fmaf(v[j][e], v[j][e], ss) : ss;
      }
    }
    for (int i = 512 + lane; i < p.rank; i += 32) {                       // latents wider than what the lanes keep
      const float x = to_f32(ckv[i]);
      ss = fmaf(x, x, ss);
    }
    const float inv = rsqrtf(warp_sum(ss) / (float)p.rank + p.eps);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = lane + 32 * j;
      if (c < n8) {
        float w[8];
        load8(p.norm_w + 8 * c, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] = 8 * c + e < p.rank ? v[j][e] * inv * w[e] : 0.f;
        store8(row + 8 * c, w);
      }
    }
    for (int i = 512 + lane; i < p.R; i += 32) row[i] = from_f32<T>(i < p.rank ? to_f32(ckv[i]) * inv * p.norm_w[i] : 0.f);
    return;
  }
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
  const float* cs = p.rope_cos + (size_t)pos * p.half;
  const float* sn = p.rope_sin + (size_t)pos * p.half;
  const T* q = reinterpret_cast<const T*>(p.q) + (size_t)t * p.q_ld;
  T* qo = reinterpret_cast<T*>(p.q_out) + (size_t)t * p.qo_ld;
  const int per = p.r / 8;
  for (int i = threadIdx.x - 32; i < (p.H + 1) * per; i += LP_THREADS - 32) {
    const int h = i / per, c = i - h * per;
    const T* src = h < p.H ? q + (size_t)h * p.q_hs : ckv + p.R;
    T* dst = h < p.H ? qo + (size_t)h * p.qo_hs : (row ? row + p.R : nullptr);
    if (!dst) continue;
    float v[8];
    load8(src + 8 * c, v);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int j = 4 * c + e;                     // pairs past `half` are padding and only move
      if (j < p.half) {
        const float a = v[2 * e], b = v[2 * e + 1], co = cs[j], si = sn[j];
        v[2 * e] = a * co - b * si;
        v[2 * e + 1] = b * co + a * si;
      }
    }
    store8(dst + 8 * c, v);
  }
}

// ------------------------------------------------------------------ head_linear
struct HeadLinearParams {
  const void* x;               // row t of head h at t * x_ld + h * x_hs, K elements
  const __nv_bfloat16* w;      // [H][N][K]
  const void* gate;            // out *= sigmoid(gate[t * gate_ld + h * N + n]), or null
  void* out;                   // t * o_ld + h * o_hs, N elements
  long long x_ld, o_ld;
  int x_hs, o_hs, gate_ld;
  int T, N, K, lpr;            // lpr: lanes per weight row (a power of two)
  int out_f32;                 // out is fp32 whatever x is
};
constexpr int HL_WARPS = 4, HL_ROWS = 2;           // weight rows in flight per lane group

// blockIdx: (run of output features, head, tile of TT tokens).  A weight row is read once per token tile, 16 bytes per lane.
template <typename T, int TT>
__global__ void __launch_bounds__(HL_WARPS * 32) head_linear_kernel(const HeadLinearParams p) {
  extern __shared__ float hl_x[];                  // [TT][K]
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, t0 = blockIdx.z * TT, nt = min(TT, p.T - t0);
  const int groups = 32 / p.lpr, sub = lane & (p.lpr - 1), grp = lane / p.lpr, k8 = p.K / 8;
  const int n0 = (blockIdx.x * HL_WARPS + warp) * groups * HL_ROWS + grp * HL_ROWS;
  const uint4* wr = reinterpret_cast<const uint4*>(p.w + (size_t)h * p.N * p.K);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 w4[2][HL_ROWS];                            // two pieces of every row in flight; the first ones before the activations exist
#pragma unroll
  for (int u = 0; u < 2; ++u)
#pragma unroll
    for (int r = 0; r < HL_ROWS; ++r) w4[u][r] = (n0 + r < p.N && sub + u * p.lpr < k8) ? __ldg(wr + (size_t)(n0 + r) * k8 + sub + u * p.lpr) : zero;
  pdl_wait();
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    const T* xr = reinterpret_cast<const T*>(p.x) + (size_t)(t0 + min(t, nt - 1)) * p.x_ld + (size_t)h * p.x_hs;
    for (int k = threadIdx.x * 2; k < p.K; k += HL_WARPS * 64) {
      const float2 v = t < nt ? load2(xr + k) : make_float2(0.f, 0.f);
      *reinterpret_cast<float2*>(hl_x + t * p.K + k) = v;
    }
  }
  __syncthreads();
  float acc[HL_ROWS][TT];
#pragma unroll
  for (int r = 0; r < HL_ROWS; ++r)
#pragma unroll
    for (int t = 0; t < TT; ++t) acc[r][t] = 0.f;
  for (int c = sub; c < k8; c += 2 * p.lpr) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int cu = c + u * p.lpr;
      if (cu < k8) {
#pragma unroll
        for (int t = 0; t < TT; ++t) {
          const float4 a = *reinterpret_cast<const float4*>(hl_x + t * p.K + cu * 8), b = *reinterpret_cast<const float4*>(hl_x + t * p.K + cu * 8 + 4);
#pragma unroll
          for (int r = 0; r < HL_ROWS; ++r) {
            float s = acc[r][t];
            s = fmaf(bf16_lo(w4[u][r].x), a.x, s); s = fmaf(bf16_hi(w4[u][r].x), a.y, s);
            s = fmaf(bf16_lo(w4[u][r].y), a.z, s); s = fmaf(bf16_hi(w4[u][r].y), a.w, s);
            s = fmaf(bf16_lo(w4[u][r].z), b.x, s); s = fmaf(bf16_hi(w4[u][r].z), b.y, s);
            s = fmaf(bf16_lo(w4[u][r].w), b.z, s); s = fmaf(bf16_hi(w4[u][r].w), b.w, s);
            acc[r][t] = s;
          }
        }
      }
      const int cn = cu + 2 * p.lpr;
      if (cn < k8) {
#pragma unroll
        for (int r = 0; r < HL_ROWS; ++r) w4[u][r] = n0 + r < p.N ? __ldg(wr + (size_t)(n0 + r) * k8 + cn) : zero;
      }
    }
  }
#pragma unroll
  for (int r = 0; r < HL_ROWS; ++r)
#pragma unroll
    for (int t = 0; t < TT; ++t)
      for (int o = p.lpr / 2; o > 0; o >>= 1) acc[r][t] += __shfl_xor_sync(0xffffffffu, acc[r][t], o);
  if (sub != 0) return;
#pragma unroll
  for (int t = 0; t < TT; ++t) {
    if (t >= nt) break;
#pragma unroll
    for (int r = 0; r < HL_ROWS; ++r) {
      const int n = n0 + r;
      if (n >= p.N) break;
      float v = acc[r][t];
      if (p.gate) v *= sigmoid_f<sizeof(T) == 4>(to_f32(reinterpret_cast<const T*>(p.gate)[(size_t)(t0 + t) * p.gate_ld + (size_t)h * p.N + n]));
      const size_t at = (size_t)(t0 + t) * p.o_ld + (size_t)h * p.o_hs + n;
      if (p.out_f32) reinterpret_cast<float*>(p.out)[at] = v;
      else reinterpret_cast<T*>(p.out)[at] = from_f32<T>(v);
    }
  }
}

template <typename T>
static int launch_head_linear(const HeadLinearParams& p, int H, cudaStream_t st) {
  const int per_cta = HL_WARPS * (32 / p.lpr) * HL_ROWS;
  const unsigned gx = (unsigned)((p.N + per_cta - 1) / per_cta);
  if (p.T == 1) launch_pdl(head_linear_kernel<T, 1>, dim3(gx, H, 1), dim3(HL_WARPS * 32), (size_t)p.K * 4, st, p);
  else if (p.T == 2) launch_pdl(head_linear_kernel<T, 2>, dim3(gx, H, 1), dim3(HL_WARPS * 32), (size_t)p.K * 8, st, p);
  else if (p.T <= 4) launch_pdl(head_linear_kernel<T, 4>, dim3(gx, H, 1), dim3(HL_WARPS * 32), (size_t)p.K * 16, st, p);
  else launch_pdl(head_linear_kernel<T, 8>, dim3(gx, H, (unsigned)((p.T + 7) / 8)), dim3(HL_WARPS * 32), (size_t)p.K * 32, st, p);
  return (int)cudaGetLastError();
}

// ------------------------------------------------------------------ latent_plan
// Sequence b's queries see keys from max(0, start - window + 1) to its end: pages first .. last of its table.  The pages of all sequences form one
// list (pages[i] = cache page), and table[b][page] says where a page stands in it.  num[0] = pages in the list, at most max_pages (the host's bound).
__global__ void __launch_bounds__(256) latent_plan_kernel(const int* __restrict__ block_table, const int* __restrict__ seq_lens, const int* __restrict__ cu_q,
                                                          int B, int max_blocks, int block_size, int window, int max_pages, int* __restrict__ pages,
                                                          int* __restrict__ table, int* __restrict__ num) {
  pdl_prologue();
  __shared__ int s_first, s_count, s_base;
  if (threadIdx.x == 0) s_base = 0;
  for (int b = 0; b < B; ++b) {
    __syncthreads();
    if (threadIdx.x == 0) {
      const int len = seq_lens[b], start = len - (cu_q[b + 1] - cu_q[b]);
      const int lo = window > 0 ? max(0, start - window + 1) : 0;
      s_first = lo / block_size;
      s_count = len > 0 ? min((len - 1) / block_size, max_blocks - 1) - s_first + 1 : 0;
    }
    __syncthreads();
    const int first = s_first, count = s_count, base = s_base;
    for (int i = threadIdx.x; i < count; i += blockDim.x) {
      const int at = min(base + i, max_pages - 1);
      pages[at] = block_table[(size_t)b * max_blocks + first + i];
      table[(size_t)b * max_blocks + first + i] = at;
    }
    __syncthreads();
    if (threadIdx.x == 0) s_base = base + count;
  }
  __syncthreads();
  if (threadIdx.x == 0) num[0] = min(s_base, max_pages);
}

}  // namespace mx

using namespace mx;

// See LatentPostParams.  Strides in elements; rows, widths and strides are multiples of 8 elements.  elem_f32: q, ckv, cache and q_out hold fp32.
MX_HOST_API int mx_latent_post(const void* q, int q_ld, int q_hs, void* q_out, int qo_ld, int qo_hs, const void* ckv, int ckv_ld, const float* norm_w, int rank,
                               float eps, const int* positions, const float* rope_cos, const float* rope_sin, int half, int max_pos, const long long* slot_map,
                               void* cache, int T, int H, int R, int r, int elem_f32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (R % 8 || r % 8 || rank < 1 || rank > R || half < 0 || half > r / 2 || q_ld % 8 || q_hs % 8 || qo_ld % 8 || qo_hs % 8 || ckv_ld % 8) return -108;
  if (((uintptr_t)q | (uintptr_t)q_out | (uintptr_t)ckv | (uintptr_t)cache | (uintptr_t)norm_w) & 15) return -108;
  LatentPostParams p;
  p.q = q; p.q_out = q_out; p.ckv = ckv; p.norm_w = norm_w; p.positions = positions; p.rope_cos = rope_cos; p.rope_sin = rope_sin; p.slot_map = slot_map;
  p.cache = cache; p.q_ld = q_ld; p.q_hs = q_hs; p.qo_ld = qo_ld; p.qo_hs = qo_hs; p.ckv_ld = ckv_ld; p.H = H; p.R = R; p.r = r; p.rank = rank; p.half = half;
  p.max_pos = max_pos; p.eps = eps;
  if (elem_f32) launch_pdl(latent_post_kernel<float>, dim3(T), dim3(LP_THREADS), 0, st, p);
  else launch_pdl(latent_post_kernel<__nv_bfloat16>, dim3(T), dim3(LP_THREADS), 0, st, p);
  return (int)cudaGetLastError();
}

// out[t][h][:] = W[h] x[t][h][:] (* sigmoid(gate)), fp32 with out_f32; see HeadLinearParams.  K a multiple of 8, at most 1536; w on a 16-byte boundary.
MX_HOST_API int mx_head_linear(const void* x, long long x_ld, int x_hs, const void* w, const void* gate, int gate_ld, void* out, long long o_ld, int o_hs, int T,
                               int H, int N, int K, int elem_f32, int out_f32, cudaStream_t st) {
  if (T <= 0 || H <= 0 || N <= 0) return 0;
  if (K % 8 || K < 8 || K > 1536 || x_ld % 2 || x_hs % 2 || ((uintptr_t)w & 15) || ((uintptr_t)x & 7)) return -101;
  HeadLinearParams p;
  p.x = x; p.w = (const __nv_bfloat16*)w; p.gate = gate; p.out = out; p.x_ld = x_ld; p.o_ld = o_ld; p.x_hs = x_hs; p.o_hs = o_hs; p.gate_ld = gate_ld;
  p.T = T; p.N = N; p.K = K; p.out_f32 = out_f32 || elem_f32;
  p.lpr = 1;
  while (p.lpr < 32 && p.lpr * 8 < K) p.lpr *= 2;
  return elem_f32 ? launch_head_linear<float>(p, H, st) : launch_head_linear<__nv_bfloat16>(p, H, st);
}

// See latent_plan_kernel.  pages [max_pages], table [B][max_blocks], num [1].
MX_HOST_API int mx_latent_plan(const int* block_table, const int* seq_lens, const int* cu_q, int B, int max_blocks, int block_size, int window, int max_pages,
                               int* pages, int* table, int* num, cudaStream_t st) {
  if (B <= 0 || max_pages <= 0) return 0;
  launch_pdl(latent_plan_kernel, dim3(1), dim3(256), 0, st, block_table, seq_lens, cu_q, B, max_blocks, block_size, window, max_pages, pages, table, num);
  return (int)cudaGetLastError();
}
