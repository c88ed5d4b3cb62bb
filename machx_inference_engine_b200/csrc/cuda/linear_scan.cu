// Recurrences with a matrix per head and no delta rule, and the element-wise kernels around them.
//   token_shift      : every row mixed with the row of the sequence's previous token, several mixes at once
//   decay_scan       : S <- w S + k v^T, o = S^T q per head, with a fixed decay per head (lightning attention; q, k, v through SiLU) or one per token and
//                      key channel, w = exp(-exp(z)), with a bonus for the current token (RWKV-style time mixing)
//   gated_group_norm : norm(o) * w * act(gate) over equal runs of a row
//
// decay_scan: the state is fp32 and so is everything that enters it after the projections.  One CTA owns 32 value columns of one head of one sequence;
// a warp holds 8 of them, spread over 8 lanes along the keys, so that a lane keeps dk / 8 x 2 elements of S in registers for the whole step.  Tokens come
// in chunks of 16: the CTA stages them in shared memory as fp32 (decays formed once), with the next chunk's rows already on their way in registers; a
// token costs a lane three multiply-adds per state element and one 8-lane reduction, which does not sit on the recurrence's own dependency chain.
// Single tokens take the same kernel: it then reads and writes the state once, in 32-byte runs.
// A sequence whose step begins at position 0 starts from zeros, so a state slot needs no reset before it is used again.
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

// ------------------------------------------------------------------ token_shift
// x fp32 [T][W]; mu [n][W]; out [n][T][W].  A CTA walks `rows` consecutive rows, a thread four columns of them.  The CTA with a sequence's first row reads
// the state and replaces it by the sequence's last row, so that no other CTA touches it.
struct TokenShiftParams {
  const float* x;
  const float* mu;
  float* state;                // [slots][W]
  const int* slots;            // [B]
  const int* cu_q;             // [B+1]
  const int* seq_lens;         // [B]
  void* out;
  int T, W, B, rows;
};

template <typename OT, int N>
__global__ void __launch_bounds__(256) token_shift_kernel(const TokenShiftParams p) {
  pdl_prologue();
  const int t0 = blockIdx.x * p.rows, t1 = min(p.T, t0 + p.rows);
  int lo = 0, hi = p.B - 1;                              // the last sequence that begins at or before t0
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (p.cu_q[mid] <= t0) lo = mid; else hi = mid - 1;
  }
  for (int c = (blockIdx.y * 256 + threadIdx.x) * 4; c < p.W; c += gridDim.y * 1024) {
    float mu[N][4], prev[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int n = 0; n < N; ++n) loadv<4>(p.mu + (size_t)n * p.W + c, mu[n]);
    int b = lo;
    if (t0 > p.cu_q[b]) loadv<4>(p.x + (size_t)(t0 - 1) * p.W + c, prev);
    for (int t = t0; t < t1; ++t) {
      while (b + 1 < p.B && p.cu_q[b + 1] <= t) ++b;
      float x[4];
      loadv<4>(p.x + (size_t)t * p.W + c, x);
      const int first = p.cu_q[b];
      if (t == first) {
        const int len = p.cu_q[b + 1] - first;
        float* st = p.state + (size_t)p.slots[b] * p.W + c;
        if (p.seq_lens[b] == len) prev[0] = prev[1] = prev[2] = prev[3] = 0.f;
        else loadv<4>(st, prev);
        float last[4];
        loadv<4>(p.x + (size_t)(first + len - 1) * p.W + c, last);
        storev<4>(st, last);
      }
#pragma unroll
      for (int n = 0; n < N; ++n) {
        float o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) o[e] = fmaf(prev[e] - x[e], mu[n][e], x[e]);
        storev<4>(reinterpret_cast<OT*>(p.out) + ((size_t)n * p.T + t) * p.W + c, o);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) prev[e] = x[e];
    }
  }
}

// ------------------------------------------------------------------ decay_scan
struct DecayScanParams {
  const void* q;               // row t of head h at t * ld + h * dk
  const void* k;
  const void* v;               // t * v_ld + h * dv
  const float* z;              // [T][H * dk], or null (fixed decays)
  const float* u;              // [H][dk] (with z)
  const float* decay;          // [H] (without z)
  float* state;                // [slots][H][dk][dv]
  const int* slots;
  const int* cu_q;
  const int* seq_lens;
  float* out;                  // [T][H * dv]
  int q_ld, k_ld, v_ld, H, dk, dv, silu;
};
constexpr int DS_CHUNK = 16, DS_VT = 32;

template <typename T> struct Raw4;
template <> struct Raw4<__nv_bfloat16> { using type = uint2; };
template <> struct Raw4<float> { using type = float4; };
__device__ __forceinline__ float4 widen(uint2 r) { return make_float4(bf16_lo(r.x), bf16_hi(r.x), bf16_lo(r.y), bf16_hi(r.y)); }
__device__ __forceinline__ float4 widen(float4 r) { return r; }
template <bool PRECISE> __device__ __forceinline__ float4 silu4(float4 a) {
  return make_float4(a.x * sigmoid_f<PRECISE>(a.x), a.y * sigmoid_f<PRECISE>(a.y), a.z * sigmoid_f<PRECISE>(a.z), a.w * sigmoid_f<PRECISE>(a.w));
}

// NJ: groups of four keys per lane (dk <= 32 NJ); lane seg of eight holds keys 4 (seg + 8 j) .. + 3.  DATA: decays and bonus from the data.
template <typename T, int NJ, bool DATA>
__global__ void __launch_bounds__(128) decay_scan_kernel(const DecayScanParams p) {
  using R4 = typename Raw4<T>::type;
  constexpr bool PRECISE = sizeof(T) == 4;
  constexpr int DKP = 32 * NJ;
  pdl_prologue();
  extern __shared__ float4 ds_smem[];
  float4* sq = ds_smem;                                  // [16][DKP / 4]
  float4* sk = sq + DS_CHUNK * DKP / 4;
  float4* sw = sk + DS_CHUNK * DKP / 4;                  // (DATA)
  __shared__ __align__(16) float sv[DS_CHUNK][DS_VT];
  __shared__ float sb[DS_CHUNK];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, seg = lane & 7, vl = warp * 8 + (lane >> 3) * 2;
  const int h = blockIdx.y, b = blockIdx.z, v0 = blockIdx.x * DS_VT;
  const int t_begin = p.cu_q[b], len = p.cu_q[b + 1] - t_begin;
  if (len <= 0) return;
  const int dk = p.dk, dv = p.dv;
  const bool live = v0 + vl < dv;                        // (dv is a multiple of 8, vl even)
  float* sp = p.state + (((size_t)p.slots[b] * p.H + h) * dk) * dv + v0 + vl;
  float S[4 * NJ][2];
  const bool fresh = p.seq_lens[b] == len;
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int kk = 4 * (seg + 8 * j) + e;
      float2 s = make_float2(0.f, 0.f);
      if (!fresh && live && kk < dk) s = *reinterpret_cast<const float2*>(sp + (size_t)kk * dv);
      S[4 * j + e][0] = s.x;
      S[4 * j + e][1] = s.y;
    }
  const float d = DATA ? 0.f : p.decay[h];

  // a thread stages row tid / 8 of the chunk: key groups (tid % 8) + 8 j, and four of the tile's value columns
  const int lr = tid >> 3, vc = (tid & 7) * 4;
  R4 rq[NJ], rk[NJ], rv;
  float4 rz[NJ];
  float4 u4[DATA ? NJ : 1];
  if constexpr (DATA) {
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = 4 * (seg + 8 * j);
      u4[j] = c < dk ? *reinterpret_cast<const float4*>(p.u + (size_t)h * dk + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  auto fetch = [&](int c0) {
    const int r = c0 + lr;
    const bool ok = r < len;
    const size_t t = (size_t)(t_begin + (ok ? r : 0));
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = 4 * (seg + 8 * j);
      rq[j] = R4{}; rk[j] = R4{};
      if (ok && c < dk) {
        rq[j] = *reinterpret_cast<const R4*>(reinterpret_cast<const T*>(p.q) + t * p.q_ld + (size_t)h * dk + c);
        rk[j] = *reinterpret_cast<const R4*>(reinterpret_cast<const T*>(p.k) + t * p.k_ld + (size_t)h * dk + c);
        if constexpr (DATA) rz[j] = *reinterpret_cast<const float4*>(p.z + (t * p.H + h) * dk + c);
      }
    }
    rv = R4{};
    if (ok && v0 + vc < dv) rv = *reinterpret_cast<const R4*>(reinterpret_cast<const T*>(p.v) + t * p.v_ld + (size_t)h * dv + v0 + vc);
  };
  fetch(0);
  for (int c0 = 0; c0 < len; c0 += DS_CHUNK) {
    const int n = min(DS_CHUNK, len - c0);
    if (c0) __syncthreads();                             // every reader of the previous chunk is done
    {
      float bonus = 0.f;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int at = lr * (DKP / 4) + seg + 8 * j;
        float4 q = widen(rq[j]), k = widen(rk[j]);
        if (!DATA && p.silu) { q = silu4<PRECISE>(q); k = silu4<PRECISE>(k); }
        sq[at] = q;
        sk[at] = k;
        if constexpr (DATA) {
          float4 w = make_float4(0.f, 0.f, 0.f, 0.f);
          if (4 * (seg + 8 * j) < dk && c0 + lr < len) w = make_float4(expf(-expf(rz[j].x)), expf(-expf(rz[j].y)), expf(-expf(rz[j].z)), expf(-expf(rz[j].w)));
          sw[at] = w;
          bonus += q.x * u4[j].x * k.x + q.y * u4[j].y * k.y + q.z * u4[j].z * k.z + q.w * u4[j].w * k.w;
        }
      }
      float4 v = widen(rv);
      if (!DATA && p.silu) v = silu4<PRECISE>(v);
      *reinterpret_cast<float4*>(&sv[lr][vc]) = v;
      if constexpr (DATA) {
        bonus += __shfl_xor_sync(0xffffffffu, bonus, 1);
        bonus += __shfl_xor_sync(0xffffffffu, bonus, 2);
        bonus += __shfl_xor_sync(0xffffffffu, bonus, 4);
        if (seg == 0) sb[lr] = bonus;
      }
    }
    __syncthreads();
    if (c0 + DS_CHUNK < len) fetch(c0 + DS_CHUNK);       // travels while this chunk is worked on
    float* orow = p.out + ((size_t)(t_begin + c0) * p.H + h) * dv + v0 + vl + (seg >> 2);
#pragma unroll 4
    for (int t = 0; t < n; ++t) {
      const float2 v = *reinterpret_cast<const float2*>(&sv[t][vl]);
      float o0 = 0.f, o1 = 0.f;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const int at = t * (DKP / 4) + seg + 8 * j;
        const float4 q4 = sq[at], k4 = sk[at];
        const float qa[4] = {q4.x, q4.y, q4.z, q4.w}, ka[4] = {k4.x, k4.y, k4.z, k4.w};
        float wa[4];
        if constexpr (DATA) { const float4 w4 = sw[at]; wa[0] = w4.x; wa[1] = w4.y; wa[2] = w4.z; wa[3] = w4.w; }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float* s = S[4 * j + e];
          if constexpr (DATA) {
            o0 = fmaf(qa[e], s[0], o0);
            o1 = fmaf(qa[e], s[1], o1);
            s[0] = fmaf(wa[e], s[0], ka[e] * v.x);
            s[1] = fmaf(wa[e], s[1], ka[e] * v.y);
          } else {
            s[0] = fmaf(d, s[0], ka[e] * v.x);
            s[1] = fmaf(d, s[1], ka[e] * v.y);
            o0 = fmaf(qa[e], s[0], o0);
            o1 = fmaf(qa[e], s[1], o1);
          }
        }
      }
      // sum over the eight lanes: the lower four end up with column 0, the upper four with column 1
      const bool up = seg & 4;
      float o = (up ? o1 : o0) + __shfl_xor_sync(0xffffffffu, up ? o0 : o1, 4);
      o += __shfl_xor_sync(0xffffffffu, o, 2);
      o += __shfl_xor_sync(0xffffffffu, o, 1);
      if (DATA) o = fmaf(sb[t], up ? v.y : v.x, o);
      if ((seg & 3) == 0 && live) orow[(size_t)t * p.H * dv] = o;
    }
  }
#pragma unroll
  for (int j = 0; j < NJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int kk = 4 * (seg + 8 * j) + e;
      if (live && kk < dk) *reinterpret_cast<float2*>(sp + (size_t)kk * dv) = make_float2(S[4 * j + e][0], S[4 * j + e][1]);
    }
}

template <typename T, int NJ, bool DATA>
static int launch_decay_scan(const DecayScanParams& p, int B, cudaStream_t st) {
  const size_t smem = (size_t)DS_CHUNK * 32 * NJ * 4 * (DATA ? 3 : 2);
  auto kern = decay_scan_kernel<T, NJ, DATA>;
  static DeviceOnce configured;
  if (configured.pending()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured.mark();
  }
  launch_pdl(kern, dim3((unsigned)((p.dv + DS_VT - 1) / DS_VT), (unsigned)p.H, (unsigned)B), dim3(128), smem, st, p);
  return (int)cudaGetLastError();
}

// ------------------------------------------------------------------ gated_group_norm
// o fp32 [T][G * gs]; a team of `wpg` warps owns one (row, group) and keeps NV pieces of four elements per lane (NV == 0: reads them again).
struct GatedNormParams {
  const float* o;
  const void* gate;            // rows gate_ld apart
  const float* w;              // [G * gs]
  void* out;                   // [T][G * gs]
  float eps, inv_n;            // 1 / live elements of a group
  int T, G, gs, gate_ld, wpg, lpg, silu;       // lpg: lanes per group (32, or 16 / 8 for short groups of one warp's team)
};
constexpr int GG_WARPS = 8;

template <typename T, int NV>
__global__ void __launch_bounds__(GG_WARPS * 32) gated_group_norm_kernel(const GatedNormParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  pdl_prologue();
  __shared__ float red[GG_WARPS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wpg = p.wpg;
  const int lpg = p.lpg, gl = lane & (lpg - 1);
  const long long unit = ((long long)blockIdx.x * (GG_WARPS / wpg) + warp / wpg) * (32 / lpg) + lane / lpg;
  const bool some = unit < (long long)p.T * p.G;
  if (lpg == 32 ? !some : !__any_sync(0xffffffffu, some)) return;        // a whole team (or warp) leaves
  const long long t = some ? unit / p.G : 0;
  const int g = some ? (int)(unit - t * p.G) : 0, base = g * p.gs;
  const float* o = p.o + (size_t)t * p.G * p.gs + base;
  const T* gate = reinterpret_cast<const T*>(p.gate) + (size_t)t * p.gate_ld + base;
  const float* w = p.w + base;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)t * p.G * p.gs + base;
  const int first = some ? ((warp % wpg) * 32 + gl) * 4 : p.gs, step = wpg * 128;
  float x[NV > 0 ? NV : 1][4], gv[NV > 0 ? NV : 1][4], ss = 0.f;
  if constexpr (NV > 0) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = first + j * step;
      if (c < p.gs) {
        loadv<4>(o + c, x[j]);
        loadv<4>(gate + c, gv[j]);
#pragma unroll
        for (int e = 0; e < 4; ++e) ss = fmaf(x[j][e], x[j][e], ss);
      }
    }
  } else {
    for (int c = first; c < p.gs; c += step) {
      loadv<4>(o + c, x[0]);
#pragma unroll
      for (int e = 0; e < 4; ++e) ss = fmaf(x[0][e], x[0][e], ss);
    }
  }
  for (int o = lpg >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (wpg > 1) {
    const int team = warp / wpg;
    if (lane == 0) red[warp] = ss;
    asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "r"(wpg * 32) : "memory");
    ss = 0.f;
    for (int i = 0; i < wpg; ++i) ss += red[team * wpg + i];
  }
  const float inv = rsqrtf(ss * p.inv_n + p.eps);
  auto finish = [&](int c, const float (&xv)[4], const float (&gt)[4]) {
    float wv[4];
    loadv<4>(w + c, wv);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float s = sigmoid_f<PRECISE>(gt[e]);
      wv[e] *= xv[e] * inv * (p.silu ? gt[e] * s : s);
    }
    storev<4>(out + c, wv);
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = first + j * step;
      if (c < p.gs) finish(c, x[j], gv[j]);
    }
  } else {
    for (int c = first; c < p.gs; c += step) {
      loadv<4>(o + c, x[0]);
      loadv<4>(gate + c, gv[0]);
      finish(c, x[0], gv[0]);
    }
  }
}

template <typename T>
static int launch_gated_norm(GatedNormParams p, cudaStream_t st) {
  const long long units = (long long)p.T * p.G;
  p.wpg = 1;
  while (p.wpg < GG_WARPS && (p.gs > 512 * p.wpg || (units * p.wpg < 16ll * sm_count() && p.gs > 128 * p.wpg))) p.wpg *= 2;
  p.lpg = p.gs <= 32 ? 8 : p.gs <= 64 ? 16 : 32;
  const long long per_cta = (long long)(GG_WARPS / p.wpg) * (32 / p.lpg);
  const dim3 grid((unsigned)((units + per_cta - 1) / per_cta)), block(GG_WARPS * 32);
  const int pieces = (p.gs + 128 * p.wpg - 1) / (128 * p.wpg);
  if (pieces <= 1) launch_pdl(gated_group_norm_kernel<T, 1>, grid, block, 0, st, p);
  else if (pieces <= 2) launch_pdl(gated_group_norm_kernel<T, 2>, grid, block, 0, st, p);
  else if (pieces <= 4) launch_pdl(gated_group_norm_kernel<T, 4>, grid, block, 0, st, p);
  else launch_pdl(gated_group_norm_kernel<T, 0>, grid, block, 0, st, p);
  return (int)cudaGetLastError();
}

}  // namespace mx

using namespace mx;

// See token_shift_kernel; W a multiple of 4, n from 1 to 8.
MX_HOST_API int mx_token_shift(const float* x, const float* mu, float* state, const int* slots, const int* cu_q, const int* seq_lens, void* out, int out_is_f32,
                               int T, int W, int n, int B, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (W < 4 || W % 4 || n < 1 || n > 8) return -107;
  TokenShiftParams p;
  p.x = x; p.mu = mu; p.state = state; p.slots = slots; p.cu_q = cu_q; p.seq_lens = seq_lens; p.out = out; p.T = T; p.W = W; p.B = B;
  p.rows = T >= 1024 ? 4 : 1;
  const dim3 grid((unsigned)((T + p.rows - 1) / p.rows), (unsigned)((W + 1023) / 1024)), block(256);
#define MX_TS(N_) \
  case N_: \
    if (out_is_f32) launch_pdl(token_shift_kernel<float, N_>, grid, block, 0, st, p); \
    else launch_pdl(token_shift_kernel<__nv_bfloat16, N_>, grid, block, 0, st, p); \
    break;
  switch (n) { MX_TS(1) MX_TS(2) MX_TS(3) MX_TS(4) MX_TS(5) MX_TS(6) MX_TS(7) MX_TS(8) }
#undef MX_TS
  return (int)cudaGetLastError();
}

// See decay_scan_kernel.  z and u, or decay; widths multiples of 8, dk up to 256; rows, bases and strides on four-element boundaries.
MX_HOST_API int mx_decay_scan(const void* q, int q_ld, const void* k, int k_ld, const void* v, int v_ld, const float* z, const float* u, const float* decay,
                              float* state, const int* slots, const int* cu_q, const int* seq_lens, float* out, int B, int H, int dk, int dv, int silu,
                              int elem_f32, cudaStream_t st) {
  if (B <= 0 || H <= 0) return 0;
  if (dk < 8 || dk > 256 || dk % 8 || dv < 8 || dv % 8 || q_ld % 4 || k_ld % 4 || v_ld % 4 || H > 65535 || B > 65535) return -112;
  if ((z != nullptr) == (decay != nullptr) || (z && !u)) return -109;
  const uintptr_t mask = elem_f32 ? 15 : 7;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & mask) return -112;
  DecayScanParams p;
  p.q = q; p.k = k; p.v = v; p.z = z; p.u = u; p.decay = decay; p.state = state; p.slots = slots; p.cu_q = cu_q; p.seq_lens = seq_lens; p.out = out;
  p.q_ld = q_ld; p.k_ld = k_ld; p.v_ld = v_ld; p.H = H; p.dk = dk; p.dv = dv; p.silu = silu;
  using bf = __nv_bfloat16;
#define MX_DS(T_, D_) \
  (dk <= 32 ? launch_decay_scan<T_, 1, D_>(p, B, st) : dk <= 64 ? launch_decay_scan<T_, 2, D_>(p, B, st) : dk <= 128 ? launch_decay_scan<T_, 4, D_>(p, B, st) \
                                                                                                          : launch_decay_scan<T_, 8, D_>(p, B, st))
  if (elem_f32) return z ? MX_DS(float, true) : MX_DS(float, false);
  return z ? MX_DS(bf, true) : MX_DS(bf, false);
#undef MX_DS
}

// See gated_group_norm_kernel.  o fp32 [T][groups * gs], gate / out in bf16 or fp32; `live` elements of a group count (the others are zero); gs a multiple of 4.
MX_HOST_API int mx_gated_group_norm(const float* o, const void* gate, int gate_ld, const float* w, void* out, int elem_f32, float eps, int T, int groups, int gs,
                                    int live, int silu, cudaStream_t st) {
  if (T <= 0) return 0;
  if (groups < 1 || gs < 4 || gs % 4 || gate_ld % 4 || live < 1 || ((uintptr_t)gate & (elem_f32 ? 15 : 7))) return -107;
  GatedNormParams p;
  p.o = o; p.gate = gate; p.w = w; p.out = out; p.eps = eps; p.inv_n = 1.f / (float)live; p.T = T; p.G = groups; p.gs = gs; p.gate_ld = gate_ld; p.silu = silu;
  return elem_f32 ? launch_gated_norm<float>(p, st) : launch_gated_norm<__nv_bfloat16>(p, st);
}
