// Real-gated linear recurrent unit (RG-LRU) behind a causal convolution:
//     u_t = sum_j w_j x_(t - taps + 1 + j) + b                            per channel, zeros before the start
//     r, i = sigmoid(W_r u + b_r), sigmoid(W_i u + b_i)                   per block of n channels (the products are GEMMs of their own in prompts)
//     log a = c r (c = -8 softplus(lam), formed by the caller);   S_t = a S_(t-1) + sqrt(1 - a^2) i u;   y_t = S_t gelu(g)
// Gates, decays and state are fp32; a sequence whose step starts at position 0 starts from zeros (inputs and state), whatever its slot holds.
//
// Prompts: causal_conv (a thread walks a strip of tokens with the taps in registers), a per-block GEMM with fp32 results, rglru_scan: the recurrence is
// linear in S, so a run of tokens acts as S -> A S + B.  A cluster of CTAs owns 32 channels of one sequence and walks its tokens in rounds: every CTA takes
// the next tile, every thread eight consecutive tokens of two channels, one warp chains the runs of the CTA, the cluster exchanges the CTAs' totals through
// distributed shared memory, and the threads replay their runs from the right start.
// Decode: rglru_step is one kernel from the projection to the recurrence's output.  A cluster owns a block of channels, a CTA of it a slice: every CTA forms
// u of the whole block, streams its rows of the two gate matrices against it and advances its channels; the convolution's inputs move on behind a cluster
// barrier, since all CTAs of the block read them.
#include "act.cuh"
#include "cluster.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

// a and b of S <- a S + b, through e = e^(log a) - 1: a long memory multiplies by a hundreds of times, and a rounding that leans one way in an exponential
// near 1 would add up over them.  sqrt(1 - a^2) = sqrt(-e (2 + e)) does not cancel.
template <bool PRECISE>
__device__ __forceinline__ void rglru_gates(float rp, float ip, float u, float c, float& a, float& b) {
  const float la = c * sigmoid_f<PRECISE>(rp);
  const float iu = sigmoid_f<PRECISE>(ip) * u;
  if constexpr (PRECISE) {
    const float e = expm1f(la);
    a = 1.f + e;
    b = sqrtf(-e * (2.f + e)) * iu;
  } else {
    float x, q;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(x) : "f"(la * 1.4426950408889634f));
    const float near = la * fmaf(0.5f * la, fmaf(la, 0.33333333f * fmaf(0.25f, la, 1.f), 1.f), 1.f);       // the series, for small steps
    const float e = la > -0.0625f ? near : x - 1.f;
    a = 1.f + e;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(q) : "f"(-e * (2.f + e)));
    b = q * iu;
  }
}

// ------------------------------------------------------------------ causal_conv
struct ConvParams {
  const void* x;               // [T] rows, ld elements apart
  const float* w;              // [C][taps]
  const float* b;              // [C]
  void* state;                 // [slots][taps - 1][C]
  const int* slots;
  const int* cu_q;
  const int* seq_lens;
  void* y;                     // [T][C]
  int ld, C, B, T, taps;
};
constexpr int RC_STRIP = 16, RC_MAX_TAPS = 8;

template <typename T, int KC>
__global__ void __launch_bounds__(128) causal_conv_kernel(const ConvParams p) {
  pdl_prologue();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  if (c >= p.C) return;
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  const T* state = reinterpret_cast<const T*>(p.state) + c;
  T* y = reinterpret_cast<T*>(p.y) + c;
  const int t_lo = blockIdx.y * RC_STRIP, t_hi = min(p.T, t_lo + RC_STRIP);
  float w[KC][4], win[KC][4], bias[4];
#pragma unroll
  for (int j = 0; j < KC; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) w[j][e] = p.w[(size_t)(c + e) * KC + j];
  loadv<4>(p.b + c, bias);
  float cur[RC_STRIP][4];                                // the strip's own inputs, fetched together
#pragma unroll
  for (int i = 0; i < RC_STRIP; ++i) {
    if (t_lo + i < t_hi) loadv<4>(x + (size_t)(t_lo + i) * p.ld, cur[i]);
  }
  int b = 0;
  while (b + 1 < p.B && p.cu_q[b + 1] <= t_lo) ++b;
  int t_start = p.cu_q[b], t_next = p.cu_q[b + 1];
  bool reload = true;                                    // first token of the strip or of a sequence
#pragma unroll
  for (int i = 0; i < RC_STRIP; ++i) {
    const int t = t_lo + i;
    if (t >= t_hi) break;
    while (t >= t_next && b + 1 < p.B) { ++b; t_start = p.cu_q[b]; t_next = p.cu_q[b + 1]; reload = true; }
    if (reload) {
      const bool fresh = p.seq_lens[b] == t_next - t_start;
      const int slot = p.slots[b];
#pragma unroll
      for (int j = 0; j < KC - 1; ++j) {
        const int src = t - (KC - 1) + j;
        if (src >= t_start) loadv<4>(x + (size_t)src * p.ld, win[j]);
        else if (!fresh) loadv<4>(state + ((size_t)slot * (KC - 1) + (KC - 1 + src - t_start)) * p.C, win[j]);
        else win[j][0] = win[j][1] = win[j][2] = win[j][3] = 0.f;
      }
      reload = false;
    }
    float a[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      win[KC - 1][e] = cur[i][e];
      a[e] = 0.f;
#pragma unroll
      for (int j = 0; j < KC; ++j) a[e] = fmaf(w[j][e], win[j][e], a[e]);
      a[e] += bias[e];
    }
    storev<4>(y + (size_t)t * p.C, a);
#pragma unroll
    for (int j = 0; j < KC - 1; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) win[j][e] = win[j + 1][e];
  }
}

// The inputs in front of every sequence's next token.  A thread owns two channels of a sequence and walks upwards: an old entry is read before it is
// overwritten.
template <typename T>
__global__ void __launch_bounds__(128) causal_conv_state_kernel(const ConvParams p) {
  pdl_prologue();
  const int b = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * 2, n1 = p.taps - 1;
  if (c >= p.C) return;
  const int t_start = p.cu_q[b], t_end = p.cu_q[b + 1], n = t_end - t_start;
  if (n <= 0) return;
  const bool fresh = p.seq_lens[b] == n;
  T* st = reinterpret_cast<T*>(p.state) + (size_t)p.slots[b] * n1 * p.C + c;
  for (int i = 0; i < n1; ++i) {
    const int src = t_end - n1 + i;
    float2 v = make_float2(0.f, 0.f);
    if (src >= t_start) v = load2(reinterpret_cast<const T*>(p.x) + (size_t)src * p.ld + c);
    else if (!fresh) v = load2(st + (size_t)(i + n) * p.C);
    store2(st + (size_t)i * p.C, v.x, v.y);
  }
}

template <typename T>
static int launch_conv(const ConvParams& p, cudaStream_t st) {
  const dim3 grid((p.C / 4 + 127) / 128, (p.T + RC_STRIP - 1) / RC_STRIP), block(128);
  switch (p.taps) {
    case 1: launch_pdl(causal_conv_kernel<T, 1>, grid, block, 0, st, p); return (int)cudaGetLastError();
    case 2: launch_pdl(causal_conv_kernel<T, 2>, grid, block, 0, st, p); break;
    case 3: launch_pdl(causal_conv_kernel<T, 3>, grid, block, 0, st, p); break;
    case 4: launch_pdl(causal_conv_kernel<T, 4>, grid, block, 0, st, p); break;
    case 5: launch_pdl(causal_conv_kernel<T, 5>, grid, block, 0, st, p); break;
    case 6: launch_pdl(causal_conv_kernel<T, 6>, grid, block, 0, st, p); break;
    case 7: launch_pdl(causal_conv_kernel<T, 7>, grid, block, 0, st, p); break;
    default: launch_pdl(causal_conv_kernel<T, 8>, grid, block, 0, st, p); break;
  }
  launch_pdl(causal_conv_state_kernel<T>, dim3((p.C / 2 + 127) / 128, p.B), block, 0, st, p);
  return (int)cudaGetLastError();
}

// ------------------------------------------------------------------ rglru_scan
struct RglruParams {
  const float* gates;          // [T][blocks][2 n]: pre-activations of r, then of i
  const float* bias;           // [blocks][2 n]
  const float* coef;           // [W]
  const void* u;               // [T] rows, u_ld apart
  const void* g;               // [T] rows, g_ld apart
  float* state;                // [slots][W]
  const int* state_slots;
  const int* cu_q;
  const int* seq_lens;
  void* y;                     // [T][W]
  int B, W, n, u_ld, g_ld;
};
constexpr int RG_THREADS = 256, RG_MAX_CLUSTER = 8;

template <typename T, int CP, int TPS>
__global__ void __launch_bounds__(RG_THREADS, 2) rglru_scan_kernel(const RglruParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  constexpr int CH = 2 * CP, SL = RG_THREADS / CP, TILE = SL * TPS;
  static_assert(CH <= RG_THREADS, "one chaining thread per channel");
  __shared__ float sA[SL][CH], sB[SL][CH];              // run (A, B), then their running composition from the CTA's first run
  __shared__ float2 s_tot[2][CH];                       // (A, B) of the whole CTA tile, by parity of the round; read by the cluster
  __shared__ float s_in[CH];                            // state in front of this CTA's tile
  const int b = blockIdx.y;
  const int t_begin = p.cu_q[b], n = p.cu_q[b + 1] - t_begin;
  if (n <= 0) return;                                    // the same for every CTA of the cluster
  const bool fresh = p.seq_lens[b] - n == 0;
  const uint32_t rank = cluster_rank(), csize = cluster_size();
  const int ch0 = (blockIdx.x / csize) * CH;
  const int slice = threadIdx.x / CP, cp = threadIdx.x % CP;
  const int ch = ch0 + 2 * cp;
  const bool ch_ok = ch < p.W;                           // W and n are even
  const int blk = ch_ok ? ch / p.n : 0;
  const size_t gate_row = 2 * (size_t)p.W, gc0 = (size_t)blk * 2 * p.n + (ch - blk * p.n);
  const float* rr = p.gates + (size_t)t_begin * gate_row + gc0;
  const T* ur = reinterpret_cast<const T*>(p.u) + (size_t)t_begin * p.u_ld + ch;
  const T* gr = reinterpret_cast<const T*>(p.g) + (size_t)t_begin * p.g_ld + ch;
  T* yr = reinterpret_cast<T*>(p.y) + (size_t)t_begin * p.W + ch;
  float2 rb = make_float2(0.f, 0.f), ib = rb, co = rb;
  if (ch_ok) { rb = load2(p.bias + gc0); ib = load2(p.bias + gc0 + p.n); co = load2(p.coef + ch); }
  float* st = p.state + (size_t)p.state_slots[b] * p.W + ch0;
  const bool chain = threadIdx.x < CH;                   // thread i carries the state of channel i in front of the round
  float S = (chain && ch0 + (int)threadIdx.x < p.W && !fresh) ? st[threadIdx.x] : 0.f;

  int par = 0;
  for (int r0 = 0; r0 < n; r0 += TILE * csize, par ^= 1) {
    const int t0 = r0 + (int)rank * TILE + slice * TPS;                  // first token of this run
    const int mine = ch_ok ? min(TPS, n - t0) : 0;                       // its live tokens (may be <= 0)
    RawPair<float> rc[TPS], ic[TPS];
    RawPair<T> uc[TPS], gc[TPS];
    float A0 = 1.f, A1 = 1.f, B0 = 0.f, B1 = 0.f;
    auto load = [&](int j) {
      const size_t t = t0 + j;
      rc[j].load(rr + t * gate_row);
      ic[j].load(rr + t * gate_row + p.n);
      uc[j].load(ur + t * p.u_ld);
      gc[j].load(gr + t * p.g_ld);
    };
    auto compose = [&](int j) {                          // (a, b) take the gates' place
      const float2 rv = rc[j].v, iv = ic[j].v, uv = uc[j].get();
      rglru_gates<PRECISE>(rv.x + rb.x, iv.x + ib.x, uv.x, co.x, rc[j].v.x, ic[j].v.x);
      rglru_gates<PRECISE>(rv.y + rb.y, iv.y + ib.y, uv.y, co.y, rc[j].v.y, ic[j].v.y);
      A0 *= rc[j].v.x; B0 = fmaf(rc[j].v.x, B0, ic[j].v.x);
      A1 *= rc[j].v.y; B1 = fmaf(rc[j].v.y, B1, ic[j].v.y);
    };
    if (mine >= TPS) {
#pragma unroll
      for (int j = 0; j < TPS; ++j) load(j);
#pragma unroll
      for (int j = 0; j < TPS; ++j) compose(j);
    } else {
#pragma unroll
      for (int j = 0; j < TPS; ++j)
        if (j < mine) load(j);
#pragma unroll
      for (int j = 0; j < TPS; ++j)
        if (j < mine) compose(j);
    }
    *reinterpret_cast<float2*>(&sA[slice][2 * cp]) = make_float2(A0, A1);
    *reinterpret_cast<float2*>(&sB[slice][2 * cp]) = make_float2(B0, B1);
    __syncthreads();
    if (chain) {
      float A = 1.f, B = 0.f;
#pragma unroll 8
      for (int s = 0; s < SL; ++s) {
        const float a = sA[s][threadIdx.x], bb = sB[s][threadIdx.x];
        sA[s][threadIdx.x] = A;
        sB[s][threadIdx.x] = B;
        A *= a;
        B = fmaf(a, B, bb);
      }
      s_tot[par][threadIdx.x] = make_float2(A, B);
    }
    // a round's totals are overwritten two rounds later, behind the next round's barrier, so one barrier per round is enough
    cluster_sync_all();
    if (chain) {
      const uint32_t addr = smem_u32(&s_tot[par][threadIdx.x]);
      float2 tot[RG_MAX_CLUSTER];
#pragma unroll
      for (uint32_t r = 0; r < RG_MAX_CLUSTER; ++r)
        if (r < csize) tot[r] = cluster_ld2(addr, r);
#pragma unroll
      for (uint32_t r = 0; r < RG_MAX_CLUSTER; ++r) {
        if (r == rank) s_in[threadIdx.x] = S;
        if (r < csize) S = fmaf(tot[r].x, S, tot[r].y);
      }
    }
    __syncthreads();
    float S0 = fmaf(sA[slice][2 * cp], s_in[2 * cp], sB[slice][2 * cp]);
    float S1 = fmaf(sA[slice][2 * cp + 1], s_in[2 * cp + 1], sB[slice][2 * cp + 1]);
    auto replay = [&](int j) {
      const float2 gv = gc[j].get();
      S0 = fmaf(rc[j].v.x, S0, ic[j].v.x);
      S1 = fmaf(rc[j].v.y, S1, ic[j].v.y);
      store2(yr + (size_t)(t0 + j) * p.W, S0 * gelu_tanh<PRECISE>(gv.x), S1 * gelu_tanh<PRECISE>(gv.y));
    };
    if (mine >= TPS) {
#pragma unroll
      for (int j = 0; j < TPS; ++j) replay(j);
    } else {
#pragma unroll
      for (int j = 0; j < TPS; ++j)
        if (j < mine) replay(j);
    }
    __syncthreads();                                     // sA / sB / s_in are read before the next round writes them
  }
  if (chain && rank == 0 && ch0 + (int)threadIdx.x < p.W) st[threadIdx.x] = S;
  cluster_sync_all();                                    // no CTA leaves while another still reads its totals
}

static int g_rglru_cluster = 0;      // 0: by the length of the longest sequence; otherwise the cluster size (A/B timing)

template <typename T>
static int launch_rglru_scan(const RglruParams& p, int max_q_len, cudaStream_t st) {
  constexpr int CP = 16, TPS = 8, CH = 2 * CP, TILE = RG_THREADS / CP * TPS;
  int c = 1;                         // CTAs along the tokens: no more than the longest sequence fills, and no more than fit the chip at once
  const long long base = (long long)p.B * ((p.W + CH - 1) / CH);
  while (c < RG_MAX_CLUSTER && c * TILE < max_q_len && 2 * c * base <= 2ll * sm_count()) c *= 2;
  if (g_rglru_cluster > 0) c = g_rglru_cluster;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(c * ((p.W + CH - 1) / CH)), p.B);
  cfg.blockDim = dim3(RG_THREADS);
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = c; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr; cfg.numAttrs = 1;
  return (int)cudaLaunchKernelEx(&cfg, rglru_scan_kernel<T, CP, TPS>, p);
}

// ------------------------------------------------------------------ rglru_step
struct RglruStepParams {
  const void* x;               // [T] rows, x_ld apart: the convolution's input
  const void* g;               // [T] rows, g_ld apart
  const float* conv_w;         // [W][taps]
  const float* conv_b;         // [W]
  const __nv_bfloat16* w;      // [blocks][2 n][n]
  const float* bias;           // [blocks][2 n]
  const float* coef;           // [W]
  void* conv_state;            // [slots][taps - 1][W]
  float* state;                // [slots][W]
  const int* slots;
  const int* cu_q;
  const int* seq_lens;
  void* y;                     // [T][W]
  int B, W, n, taps, x_ld, g_ld, slice;
};
constexpr int RS_THREADS = 256;

// sums of V values over the warp (V a power of two up to 32): lane l ends up with the sum of value l / (32 / V)
template <int V>
__device__ __forceinline__ float warp_sums(float (&v)[V], int lane) {
#pragma unroll
  for (int h = V / 2, o = 16; h > 0; h /= 2, o /= 2) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < h; ++i) {
      const float send = up ? v[i] : v[i + h], keep = up ? v[i + h] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
#pragma unroll
  for (int o = 16 / V; o > 0; o /= 2) v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
  return v[0];
}

// TT: sequences per pass.  Grid (slices per block as one cluster, blocks).
template <typename T, int TT>
__global__ void __launch_bounds__(RS_THREADS) rglru_step_kernel(const RglruStepParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  extern __shared__ float rs_smem[];
  float* su = rs_smem;                                   // [TT][n]
  float* sg = su + TT * p.n;                             // [2][TT][slice]
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = p.n;
  const int blk = blockIdx.y, c0 = blockIdx.x * p.slice, c1 = min(n, c0 + p.slice), base = blk * n;
  const __nv_bfloat16* w = p.w + (size_t)blk * 2 * n * n;
  for (int i = threadIdx.x * 64; i < (c1 - c0) * n; i += RS_THREADS * 64) {              // 128 bytes each, before the inputs exist
    asm volatile("prefetch.global.L2 [%0];" ::"l"(w + (size_t)c0 * n + i));
    asm volatile("prefetch.global.L2 [%0];" ::"l"(w + (size_t)(n + c0) * n + i));
  }
  pdl_wait();
  const int n1 = p.taps - 1;
  for (int b0 = 0; b0 < p.B; b0 += TT) {
    const int nb = min(TT, p.B - b0);
    for (int i = threadIdx.x; i < TT * n; i += RS_THREADS) {
      const int k = i / n, c = i - k * n, b = b0 + k;
      float u = 0.f;
      if (k < nb) {
        const float* cw = p.conv_w + (size_t)(base + c) * p.taps;
        const T* st = reinterpret_cast<const T*>(p.conv_state) + (size_t)p.slots[b] * n1 * p.W + base + c;
        const bool fresh = p.seq_lens[b] == 1;
        for (int j = 0; j < n1; ++j) u = fmaf(cw[j], fresh ? 0.f : to_f32(st[(size_t)j * p.W]), u);
        u = fmaf(cw[n1], to_f32(reinterpret_cast<const T*>(p.x)[(size_t)p.cu_q[b] * p.x_ld + base + c]), u) + p.conv_b[base + c];
        u = to_f32(from_f32<T>(u));
      }
      su[i] = u;
    }
    cluster_sync_all();                                  // all of the block's CTAs have read the convolution's inputs (and su is written)
    for (int i = threadIdx.x; i < nb * (c1 - c0); i += RS_THREADS) {
      const int k = i / (c1 - c0), c = base + c0 + i - k * (c1 - c0), b = b0 + k;
      T* st = reinterpret_cast<T*>(p.conv_state) + (size_t)p.slots[b] * n1 * p.W + c;
      const bool fresh = p.seq_lens[b] == 1;
      for (int j = 0; j < n1; ++j)
        st[(size_t)j * p.W] = j + 1 < n1 ? (fresh ? from_f32<T>(0.f) : st[(size_t)(j + 1) * p.W]) : reinterpret_cast<const T*>(p.x)[(size_t)p.cu_q[b] * p.x_ld + c];
    }
    for (int c = c0 + warp; c < c1; c += RS_THREADS / 32) {
      const uint4* w0 = reinterpret_cast<const uint4*>(w + (size_t)c * n);
      const uint4* w1 = reinterpret_cast<const uint4*>(w + (size_t)(n + c) * n);
      float acc[2 * TT];
#pragma unroll
      for (int i = 0; i < 2 * TT; ++i) acc[i] = 0.f;
      for (int e = lane; e < n / 8; e += 32) {
        const uint4 a = __ldg(w0 + e), q = __ldg(w1 + e);
        const uint32_t aw[4] = {a.x, a.y, a.z, a.w}, qw[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
        for (int k = 0; k < TT; ++k) {
          const float4 v0 = *reinterpret_cast<const float4*>(su + k * n + e * 8), v1 = *reinterpret_cast<const float4*>(su + k * n + e * 8 + 4);
          const float uv[8] = {v0.x, v0.y, v0.z, v0.w, v1.x, v1.y, v1.z, v1.w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            acc[k] = fmaf(bf16_lo(aw[j]), uv[2 * j], acc[k]);
            acc[k] = fmaf(bf16_hi(aw[j]), uv[2 * j + 1], acc[k]);
            acc[TT + k] = fmaf(bf16_lo(qw[j]), uv[2 * j], acc[TT + k]);
            acc[TT + k] = fmaf(bf16_hi(qw[j]), uv[2 * j + 1], acc[TT + k]);
          }
        }
      }
      const float v = warp_sums<2 * TT>(acc, lane);
      constexpr int PER = 32 / (2 * TT);
      if (lane % PER == 0) sg[(lane / PER) * p.slice + c - c0] = v;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nb * (c1 - c0); i += RS_THREADS) {
      const int k = i / (c1 - c0), c = c0 + i - k * (c1 - c0), b = b0 + k;
      float* st = p.state + (size_t)p.slots[b] * p.W + base + c;
      const float* bias = p.bias + (size_t)blk * 2 * n + c;
      float a, bb;
      rglru_gates<PRECISE>(sg[k * p.slice + c - c0] + bias[0], sg[(TT + k) * p.slice + c - c0] + bias[n], su[k * n + c], p.coef[base + c], a, bb);
      const float S = fmaf(a, p.seq_lens[b] == 1 ? 0.f : *st, bb);
      *st = S;
      const size_t t = p.cu_q[b];
      reinterpret_cast<T*>(p.y)[t * p.W + base + c] =
          from_f32<T>(S * gelu_tanh<PRECISE>(to_f32(reinterpret_cast<const T*>(p.g)[t * p.g_ld + base + c])));
    }
    __syncthreads();                                     // su and sg are written again
  }
}

template <typename T, int TT>
static int launch_rglru_step(const RglruStepParams& p, int blocks, cudaStream_t st) {
  const int slices = (p.n + p.slice - 1) / p.slice;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)slices, (unsigned)blocks);
  cfg.blockDim = dim3(RS_THREADS);
  cfg.dynamicSmemBytes = ((size_t)TT * p.n + 2 * TT * p.slice) * 4;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = slices; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = pdl_enabled() ? 1 : 0;
  cfg.attrs = attr; cfg.numAttrs = 2;
  return (int)cudaLaunchKernelEx(&cfg, rglru_step_kernel<T, TT>, p);
}
template <typename T>
static int dispatch_rglru_step(const RglruStepParams& p, int blocks, cudaStream_t st) {
  if (p.B == 1) return launch_rglru_step<T, 1>(p, blocks, st);
  if (p.B == 2) return launch_rglru_step<T, 2>(p, blocks, st);
  if (p.B <= 4 || p.n > 1024) return launch_rglru_step<T, 4>(p, blocks, st);
  return launch_rglru_step<T, 8>(p, blocks, st);
}

}  // namespace mx

using namespace mx;

// cluster size of the prompt kernel: 1, 2, 4 or 8; 0 = chosen per call (the default)
MX_HOST_API void mx_rglru_set_cluster(int c) { mx::g_rglru_cluster = (c == 1 || c == 2 || c == 4 || c == 8) ? c : 0; }

// elem_f32: x, y and the state are fp32 instead of bf16.  C and ld multiples of 4; taps 1 .. 8.  With more than one tap the state is advanced (second launch).
MX_HOST_API int mx_causal_conv(const void* x, int ld, const float* w, const float* b, void* state, const int* slots, const int* cu_q, const int* seq_lens, void* y,
                               int B, int T, int C, int taps, int elem_f32, cudaStream_t st) {
  if (B <= 0 || T <= 0) return 0;
  const uintptr_t al = elem_f32 ? 15 : 7;
  if (C % 4 || ld % 4 || taps < 1 || taps > RC_MAX_TAPS || (((uintptr_t)x | (uintptr_t)y | (uintptr_t)state) & al) || ((uintptr_t)b & 15)) return -161;
  ConvParams p{x, w, b, state, slots, cu_q, seq_lens, y, ld, C, B, T, taps};
  return elem_f32 ? launch_conv<float>(p, st) : launch_conv<__nv_bfloat16>(p, st);
}

// elem_f32: u / g / y are fp32 instead of bf16.  W a multiple of n, n even; pointers and strides aligned to element pairs.
MX_HOST_API int mx_rglru_scan(const float* gates, const float* bias, const float* coef, const void* u, int u_ld, const void* g, int g_ld, float* state,
                              const int* state_slots, const int* cu_q, const int* seq_lens, void* y, int B, int W, int n, int max_q_len, int elem_f32, cudaStream_t st) {
  if (B <= 0 || W <= 0 || max_q_len <= 0) return 0;
  const uintptr_t al = elem_f32 ? 7 : 3;
  if (n < 2 || n % 2 || W % n || u_ld % 2 || g_ld % 2 || (((uintptr_t)u | (uintptr_t)g | (uintptr_t)y) & al) ||
      (((uintptr_t)gates | (uintptr_t)bias | (uintptr_t)coef | (uintptr_t)state) & 7)) return -162;
  RglruParams p{gates, bias, coef, u, g, state, state_slots, cu_q, seq_lens, y, B, W, n, u_ld, g_ld};
  return elem_f32 ? launch_rglru_scan<float>(p, max_q_len, st) : launch_rglru_scan<__nv_bfloat16>(p, max_q_len, st);
}

// One token per sequence.  n a multiple of 8 up to 1536; elem_f32: x, g, y and the convolution's state are fp32 instead of bf16.
MX_HOST_API int mx_rglru_step(const void* x, int x_ld, const void* g, int g_ld, const float* conv_w, const float* conv_b, const void* w, const float* bias,
                              const float* coef, void* conv_state, float* state, const int* slots, const int* cu_q, const int* seq_lens, void* y, int B, int W, int n,
                              int taps, int elem_f32, cudaStream_t st) {
  if (B <= 0 || W <= 0) return 0;
  if (n < 8 || n % 8 || n > 1536 || W % n || taps < 1 || taps > RC_MAX_TAPS || ((uintptr_t)w & 15)) return -163;
  int slice = (n + 7) / 8;                                 // eight CTAs per block at most, at least a channel per warp
  slice = slice < 8 ? 8 : (slice + 7) / 8 * 8;
  RglruStepParams p{x, g, conv_w, conv_b, (const __nv_bfloat16*)w, bias, coef, conv_state, state, slots, cu_q, seq_lens, y, B, W, n, taps, x_ld, g_ld, slice};
  return elem_f32 ? dispatch_rglru_step<float>(p, W / n, st) : dispatch_rglru_step<__nv_bfloat16>(p, W / n, st);
}
