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
// Decode, a few sequences: rglru_step is one kernel from the projection to the recurrence's output.  A cluster owns a block of channels, a CTA of it a slice:
// every CTA forms u of the whole block, multiplies its rows of the two gate matrices -- the first ones fetched before the preceding kernel has ended -- with it
// and advances its channels; the convolution's inputs move on behind a cluster barrier, since all CTAs of the block read them.  With more sequences the
// products go to the tensor cores and convolution and recurrence are step kernels, a thread per channel pair and sequence.
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

// one token per sequence: the thread that owns two channels of a sequence also moves its inputs on
template <typename T>
__global__ void __launch_bounds__(128) causal_conv_step_kernel(const ConvParams p) {
  pdl_prologue();
  const int b = blockIdx.y, c = (blockIdx.x * 128 + threadIdx.x) * 2, n1 = p.taps - 1;
  if (c >= p.C) return;
  const int t = p.cu_q[b];
  if (p.cu_q[b + 1] == t) return;
  const bool fresh = p.seq_lens[b] == 1;
  T* st = reinterpret_cast<T*>(p.state) + (size_t)p.slots[b] * n1 * p.C + c;
  const float2 x = load2(reinterpret_cast<const T*>(p.x) + (size_t)t * p.ld + c), bias = load2(p.b + c);
  const float* w0 = p.w + (size_t)c * p.taps;
  const float* w1 = w0 + p.taps;
  float2 v[RC_MAX_TAPS - 1];
#pragma unroll
  for (int j = 0; j < RC_MAX_TAPS - 1; ++j) v[j] = j < n1 && !fresh ? load2(st + (size_t)j * p.C) : make_float2(0.f, 0.f);
  float a0 = 0.f, a1 = 0.f;
#pragma unroll
  for (int j = 0; j < RC_MAX_TAPS - 1; ++j) {
    if (j >= n1) break;
    a0 = fmaf(w0[j], v[j].x, a0);
    a1 = fmaf(w1[j], v[j].y, a1);
    const float2 next = j + 1 < n1 ? v[(j + 1) % (RC_MAX_TAPS - 1)] : x;
    store2(st + (size_t)j * p.C, next.x, next.y);
  }
  a0 = fmaf(w0[n1], x.x, a0) + bias.x;
  a1 = fmaf(w1[n1], x.y, a1) + bias.y;
  store2(reinterpret_cast<T*>(p.y) + (size_t)t * p.C + c, a0, a1);
}

template <typename T>
static int launch_conv(const ConvParams& p, int max_q_len, cudaStream_t st) {
  if (max_q_len == 1) {
    launch_pdl(causal_conv_step_kernel<T>, dim3((p.C / 2 + 127) / 128, p.B), dim3(128), 0, st, p);
    return (int)cudaGetLastError();
  }
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

// one token per sequence
template <typename T>
__global__ void __launch_bounds__(128) rglru_scan_step_kernel(const RglruParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  pdl_prologue();
  const int b = blockIdx.y, ch = 2 * (blockIdx.x * blockDim.x + threadIdx.x);
  const int t = p.cu_q[b];
  if (ch >= p.W || p.cu_q[b + 1] == t) return;
  const int blk = ch / p.n;
  const size_t gc = (size_t)blk * 2 * p.n + (ch - blk * p.n);
  const float* gr = p.gates + (size_t)t * 2 * p.W + gc;
  const float2 r = load2(gr), i = load2(gr + p.n), rb = load2(p.bias + gc), ib = load2(p.bias + gc + p.n), co = load2(p.coef + ch);
  const float2 u = load2(reinterpret_cast<const T*>(p.u) + (size_t)t * p.u_ld + ch), g = load2(reinterpret_cast<const T*>(p.g) + (size_t)t * p.g_ld + ch);
  float* st = p.state + (size_t)p.state_slots[b] * p.W + ch;
  float2 S = p.seq_lens[b] == 1 ? make_float2(0.f, 0.f) : load2(st);
  float a0, b0, a1, b1;
  rglru_gates<PRECISE>(r.x + rb.x, i.x + ib.x, u.x, co.x, a0, b0);
  rglru_gates<PRECISE>(r.y + rb.y, i.y + ib.y, u.y, co.y, a1, b1);
  S.x = fmaf(a0, S.x, b0);
  S.y = fmaf(a1, S.y, b1);
  store2(st, S.x, S.y);
  store2(reinterpret_cast<T*>(p.y) + (size_t)t * p.W + ch, S.x * gelu_tanh<PRECISE>(g.x), S.y * gelu_tanh<PRECISE>(g.y));
}

static int g_rglru_cluster = 0;      // 0: by the length of the longest sequence; otherwise the cluster size (A/B timing)

template <typename T>
static int launch_rglru_scan(const RglruParams& p, int max_q_len, cudaStream_t st) {
  if (max_q_len == 1) {
    launch_pdl(rglru_scan_step_kernel<T>, dim3((p.W / 2 + 127) / 128, p.B), dim3(128), 0, st, p);
    return (int)cudaGetLastError();
  }
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

// TT: sequences per pass.  Grid (slices per block as one cluster, blocks).  A warp owns every eighth channel of the slice and takes RS_GROUP of them at a time.
constexpr int RS_GROUP = 4;
template <typename T, int TT>
__global__ void __launch_bounds__(RS_THREADS) rglru_step_kernel(const RglruStepParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  constexpr int WARPS = RS_THREADS / 32;
  extern __shared__ float rs_smem[];
  float* su = rs_smem;                                   // [TT][n]
  float* sg = su + TT * p.n;                             // [2][TT][slice]
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = p.n, n8 = n / 8;
  const int blk = blockIdx.y, c0 = blockIdx.x * p.slice, c1 = min(n, c0 + p.slice), width = c1 - c0, base = blk * n;
  const uint4* w = reinterpret_cast<const uint4*>(p.w + (size_t)blk * 2 * n * n);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 wr[RS_GROUP], wi[RS_GROUP];                      // rows of r and of i of a group, one piece per lane; the first ones before the inputs exist
  auto fetch = [&](int first, int e) {
#pragma unroll
    for (int q = 0; q < RS_GROUP; ++q) {
      const int c = first + q * WARPS;
      const bool ok = c < c1 && e < n8;
      wr[q] = ok ? __ldg(w + (size_t)c * n8 + e) : zero;
      wi[q] = ok ? __ldg(w + (size_t)(n + c) * n8 + e) : zero;
    }
  };
  fetch(c0 + warp, lane);
  const int n1 = p.taps - 1;
  float cw[RC_MAX_TAPS], cb = 0.f;                       // the thread's first channel
#pragma unroll
  for (int j = 0; j < RC_MAX_TAPS; ++j) cw[j] = j <= n1 && (int)threadIdx.x < n ? __ldg(p.conv_w + (size_t)(base + threadIdx.x) * p.taps + j) : 0.f;
  if ((int)threadIdx.x < n) cb = __ldg(p.conv_b + base + threadIdx.x);
  pdl_wait();
  for (int b0 = 0; b0 < p.B; b0 += TT) {
    const int nb = min(TT, p.B - b0);
    for (int c = threadIdx.x; c < n; c += RS_THREADS) {
      if (c >= RS_THREADS) {
#pragma unroll
        for (int j = 0; j < RC_MAX_TAPS; ++j) cw[j] = j <= n1 ? __ldg(p.conv_w + (size_t)(base + c) * p.taps + j) : 0.f;
        cb = __ldg(p.conv_b + base + c);
      }
#pragma unroll
      for (int k = 0; k < TT; ++k) {
        float u = 0.f;
        if (k < nb) {
          const int b = b0 + k;
          const T* st = reinterpret_cast<const T*>(p.conv_state) + (size_t)p.slots[b] * n1 * p.W + base + c;
          const bool fresh = p.seq_lens[b] == 1;
          const float x = to_f32(reinterpret_cast<const T*>(p.x)[(size_t)p.cu_q[b] * p.x_ld + base + c]);
#pragma unroll
          for (int j = 0; j < RC_MAX_TAPS; ++j) {
            if (j > n1) break;
            u = fmaf(cw[j], j == n1 ? x : fresh ? 0.f : to_f32(st[(size_t)j * p.W]), u);
          }
          u = to_f32(from_f32<T>(u + cb));
        }
        su[k * n + c] = u;
      }
    }
    // what the recurrence wants, for the thread's first channel
    float S0 = 0.f, g0 = 0.f, co = 0.f, rb = 0.f, ib = 0.f;
    auto operands = [&](int i) {
      const int k = i / width, c = c0 + i - k * width, b = b0 + k;
      S0 = p.seq_lens[b] == 1 ? 0.f : p.state[(size_t)p.slots[b] * p.W + base + c];
      g0 = to_f32(reinterpret_cast<const T*>(p.g)[(size_t)p.cu_q[b] * p.g_ld + base + c]);
      co = p.coef[base + c];
      rb = p.bias[(size_t)blk * 2 * n + c];
      ib = p.bias[(size_t)blk * 2 * n + n + c];
    };
    if ((int)threadIdx.x < nb * width) operands(threadIdx.x);
    cluster_sync_all();                                  // all of the block's CTAs have read the convolution's inputs (and su is written)
    for (int i = threadIdx.x; i < nb * width; i += RS_THREADS) {
      const int k = i / width, c = base + c0 + i - k * width, b = b0 + k;
      T* st = reinterpret_cast<T*>(p.conv_state) + (size_t)p.slots[b] * n1 * p.W + c;
      const bool fresh = p.seq_lens[b] == 1;
      for (int j = 0; j < n1; ++j)
        st[(size_t)j * p.W] = j + 1 < n1 ? (fresh ? from_f32<T>(0.f) : st[(size_t)(j + 1) * p.W]) : reinterpret_cast<const T*>(p.x)[(size_t)p.cu_q[b] * p.x_ld + c];
    }
    for (int first = c0 + warp; first < c1; first += RS_GROUP * WARPS) {
      float acc[RS_GROUP][2 * TT];
#pragma unroll
      for (int q = 0; q < RS_GROUP; ++q)
#pragma unroll
        for (int i = 0; i < 2 * TT; ++i) acc[q][i] = 0.f;
      for (int e0 = 0; e0 < n8; e0 += 32) {
        const int e = e0 + lane;
        if (b0 || e0 || first != c0 + warp) fetch(first, e);
        if (e < n8) {
#pragma unroll
          for (int k = 0; k < TT; ++k) {
            const float4 v0 = *reinterpret_cast<const float4*>(su + k * n + e * 8), v1 = *reinterpret_cast<const float4*>(su + k * n + e * 8 + 4);
            const float uv[8] = {v0.x, v0.y, v0.z, v0.w, v1.x, v1.y, v1.z, v1.w};
#pragma unroll
            for (int q = 0; q < RS_GROUP; ++q) {
              const uint32_t a[4] = {wr[q].x, wr[q].y, wr[q].z, wr[q].w}, d[4] = {wi[q].x, wi[q].y, wi[q].z, wi[q].w};
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                acc[q][k] = fmaf(bf16_lo(a[j]), uv[2 * j], acc[q][k]);
                acc[q][k] = fmaf(bf16_hi(a[j]), uv[2 * j + 1], acc[q][k]);
                acc[q][TT + k] = fmaf(bf16_lo(d[j]), uv[2 * j], acc[q][TT + k]);
                acc[q][TT + k] = fmaf(bf16_hi(d[j]), uv[2 * j + 1], acc[q][TT + k]);
              }
            }
          }
        }
      }
      constexpr int PER = 32 / (2 * TT);
#pragma unroll
      for (int q = 0; q < RS_GROUP; ++q) {
        const int c = first + q * WARPS;
        const float v = warp_sums<2 * TT>(acc[q], lane);
        if (c < c1 && lane % PER == 0) sg[(lane / PER) * p.slice + c - c0] = v;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nb * width; i += RS_THREADS) {
      const int k = i / width, c = i - k * width, b = b0 + k;
      if (i >= RS_THREADS) operands(i);
      float a, bb;
      rglru_gates<PRECISE>(sg[k * p.slice + c] + rb, sg[(TT + k) * p.slice + c] + ib, su[k * n + c0 + c], co, a, bb);
      const float S = fmaf(a, S0, bb);
      p.state[(size_t)p.slots[b] * p.W + base + c0 + c] = S;
      reinterpret_cast<T*>(p.y)[(size_t)p.cu_q[b] * p.W + base + c0 + c] = from_f32<T>(S * gelu_tanh<PRECISE>(g0));
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
  return launch_rglru_step<T, 4>(p, blocks, st);
}

}  // namespace mx

using namespace mx;

// cluster size of the prompt kernel: 1, 2, 4 or 8; 0 = chosen per call (the default)
MX_HOST_API void mx_rglru_set_cluster(int c) { mx::g_rglru_cluster = (c == 1 || c == 2 || c == 4 || c == 8) ? c : 0; }

// elem_f32: x, y and the state are fp32 instead of bf16.  C and ld multiples of 4; taps 1 .. 8.  With more than one tap the state is advanced (in steps of more
// than one token by a second launch).
MX_HOST_API int mx_causal_conv(const void* x, int ld, const float* w, const float* b, void* state, const int* slots, const int* cu_q, const int* seq_lens, void* y,
                               int B, int T, int C, int taps, int max_q_len, int elem_f32, cudaStream_t st) {
  if (B <= 0 || T <= 0) return 0;
  const uintptr_t al = elem_f32 ? 15 : 7;
  if (C % 4 || ld % 4 || taps < 1 || taps > RC_MAX_TAPS || (((uintptr_t)x | (uintptr_t)y | (uintptr_t)state) & al) || ((uintptr_t)b & 15)) return -161;
  ConvParams p{x, w, b, state, slots, cu_q, seq_lens, y, ld, C, B, T, taps};
  return elem_f32 ? launch_conv<float>(p, max_q_len, st) : launch_conv<__nv_bfloat16>(p, max_q_len, st);
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
