// minGRU recurrence (element-wise gated linear recurrence whose gates read only the current token), fused with its gate activations and
// its output gate:
//     z = sigmoid(zp + zb);  u = up + ub;  c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0)
//     S_t = (1 - z) S_(t-1) + z c;        y = S_t * silu(g)
// zp, up, g are column ranges of one projection [T][ld]; the biases are added here in fp32 (a bias far from zero would otherwise push
// the 16-bit rounding of the sum above the size of the projection's own signal).  The state is fp32 [slots][W]; a sequence whose step
// starts at position 0 starts from zeros, whatever its slot holds.
//
// Prompts: the recurrence is linear in S, so a run of tokens acts as S -> A S + B.  A CTA owns CH channels of one sequence and walks its
// tokens in tiles: every thread takes TPS consecutive tokens of two channels (a slice), composes (A, B) of its slice, one warp chains
// the slices of the tile, and the threads replay their slices from the right start; the next tile's loads are issued before that.
// Every input is read once and there is no pass over partial results.  Decode: one thread per (sequence, channel pair).
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

struct MinGruParams {
  const void* z;               // [T] rows, ld elements apart
  const void* u;
  const void* g;
  const float* zb;             // [W]
  const float* ub;
  float* state;                // [slots][W]
  const int* state_slots;      // [B]
  const int* cu_q;             // [B + 1]
  const int* seq_lens;         // [B] tokens of the sequence after this step
  void* y;                     // [T][W]
  int B, W, ld;
};

template <bool PRECISE>
__device__ __forceinline__ void mingru_gates(float zp, float u, float& a, float& b) {
  const float z = sigmoid_f<PRECISE>(zp);
  const float c = u >= 0.f ? u + 0.5f : sigmoid_f<PRECISE>(u);
  a = 1.f - z;
  b = z * c;
}
template <bool PRECISE>
__device__ __forceinline__ float silu_f(float g) { return g * sigmoid_f<PRECISE>(g); }

constexpr int MG_WARPS = 16;

// a channel pair as it was loaded: converted where it is used, so that the loads of the next tile stay in flight
template <typename T> struct RawPair;
template <> struct RawPair<__nv_bfloat16> {
  uint32_t v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = __ldg(reinterpret_cast<const uint32_t*>(p)); }
  __device__ __forceinline__ float2 get() const { return make_float2(bf16_lo(v), bf16_hi(v)); }
};
template <> struct RawPair<float> {
  float2 v;
  __device__ __forceinline__ void load(const float* p) { v = __ldg(reinterpret_cast<const float2*>(p)); }
  __device__ __forceinline__ float2 get() const { return v; }
};

// CP: channel pairs per CTA (16 or 8); TPS: tokens per slice
template <typename T, int CP, int TPS>
__global__ void __launch_bounds__(MG_WARPS * 32) mingru_scan_kernel(const MinGruParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  constexpr int CH = 2 * CP, SL = MG_WARPS * (32 / CP), TILE = SL * TPS;
  pdl_prologue();
  __shared__ float sA[SL][CH + 2], sB[SL][CH + 2];      // slice aggregates; sB is overwritten with the state at the slice's start
  const int b = blockIdx.y;
  const int t_begin = p.cu_q[b], n = p.cu_q[b + 1] - t_begin;
  if (n <= 0) return;
  const bool fresh = p.seq_lens[b] - n == 0;
  const int ch0 = blockIdx.x * CH;
  const int slice = threadIdx.x / CP, cp = threadIdx.x % CP;
  const int ch = ch0 + 2 * cp;
  const bool ch_ok = ch < p.W;                           // W is even
  const T* zr = reinterpret_cast<const T*>(p.z) + (size_t)t_begin * p.ld + ch;
  const T* ur = reinterpret_cast<const T*>(p.u) + (size_t)t_begin * p.ld + ch;
  const T* gr = reinterpret_cast<const T*>(p.g) + (size_t)t_begin * p.ld + ch;
  T* yr = reinterpret_cast<T*>(p.y) + (size_t)t_begin * p.W + ch;
  float2 zb = make_float2(0.f, 0.f), ub = zb;
  if (ch_ok) { zb = load2(p.zb + ch); ub = load2(p.ub + ch); }
  float* st = p.state + (size_t)p.state_slots[b] * p.W + ch0;
  // the chaining warp carries the running state of channel `lane` (lanes past the CTA's channels idle)
  const bool chain = threadIdx.x < CH && ch0 + (int)threadIdx.x < p.W;
  float S = (chain && !fresh) ? st[threadIdx.x] : 0.f;

  RawPair<T> zc[TPS], uc[TPS], gc[TPS];
  auto load_tile = [&](int t0) {
#pragma unroll
    for (int j = 0; j < TPS; ++j) {
      const int t = t0 + slice * TPS + j;
      if (ch_ok && t < n) {
        zc[j].load(zr + (size_t)t * p.ld);
        uc[j].load(ur + (size_t)t * p.ld);
        gc[j].load(gr + (size_t)t * p.ld);
      }
    }
  };
  load_tile(0);
  for (int t0 = 0; t0 < n; t0 += TILE) {
    const int mine = ch_ok ? min(TPS, n - (t0 + slice * TPS)) : 0;       // live tokens of this slice (may be <= 0)
    float2 av[TPS], bv[TPS];
    float2 gs[TPS];
    float A0 = 1.f, A1 = 1.f, B0 = 0.f, B1 = 0.f;
#pragma unroll
    for (int j = 0; j < TPS; ++j) {
      if (j < mine) {
        const float2 zv = zc[j].get(), uv = uc[j].get(), gv = gc[j].get();
        mingru_gates<PRECISE>(zv.x + zb.x, uv.x + ub.x, av[j].x, bv[j].x);
        mingru_gates<PRECISE>(zv.y + zb.y, uv.y + ub.y, av[j].y, bv[j].y);
        gs[j] = make_float2(silu_f<PRECISE>(gv.x), silu_f<PRECISE>(gv.y));
        A0 *= av[j].x; B0 = fmaf(av[j].x, B0, bv[j].x);
        A1 *= av[j].y; B1 = fmaf(av[j].y, B1, bv[j].y);
      }
    }
    if (t0 + TILE < n) load_tile(t0 + TILE);
    __syncthreads();                                     // the previous tile's starts have been read
    sA[slice][2 * cp] = A0; sA[slice][2 * cp + 1] = A1;
    sB[slice][2 * cp] = B0; sB[slice][2 * cp + 1] = B1;
    __syncthreads();
    if (threadIdx.x < CH) {
      const int live = min(SL, (n - t0 + TPS - 1) / TPS);
#pragma unroll 8
      for (int s = 0; s < live; ++s) {
        const float A = sA[s][threadIdx.x], Bs = sB[s][threadIdx.x];
        sB[s][threadIdx.x] = S;
        S = fmaf(A, S, Bs);
      }
    }
    __syncthreads();
    float S0 = sB[slice][2 * cp], S1 = sB[slice][2 * cp + 1];
#pragma unroll
    for (int j = 0; j < TPS; ++j) {
      if (j < mine) {
        S0 = fmaf(av[j].x, S0, bv[j].x);
        S1 = fmaf(av[j].y, S1, bv[j].y);
        store2(yr + (size_t)(t0 + slice * TPS + j) * p.W, S0 * gs[j].x, S1 * gs[j].y);
      }
    }
  }
  if (chain) st[threadIdx.x] = S;
}

// one token per sequence
template <typename T>
__global__ void __launch_bounds__(128) mingru_step_kernel(const MinGruParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  pdl_prologue();
  const int b = blockIdx.y, ch = 2 * (blockIdx.x * blockDim.x + threadIdx.x);
  const int t = p.cu_q[b];
  if (ch >= p.W || p.cu_q[b + 1] == t) return;
  const size_t row = (size_t)t * p.ld + ch;
  const float2 zp = load2(reinterpret_cast<const T*>(p.z) + row), up = load2(reinterpret_cast<const T*>(p.u) + row);
  const float2 g = load2(reinterpret_cast<const T*>(p.g) + row);
  const float2 zb = load2(p.zb + ch), ub = load2(p.ub + ch);
  float* st = p.state + (size_t)p.state_slots[b] * p.W + ch;
  float2 S = p.seq_lens[b] == 1 ? make_float2(0.f, 0.f) : load2(st);
  float a0, b0, a1, b1;
  mingru_gates<PRECISE>(zp.x + zb.x, up.x + ub.x, a0, b0);
  mingru_gates<PRECISE>(zp.y + zb.y, up.y + ub.y, a1, b1);
  S.x = fmaf(a0, S.x, b0);
  S.y = fmaf(a1, S.y, b1);
  store2(st, S.x, S.y);
  store2(reinterpret_cast<T*>(p.y) + (size_t)t * p.W + ch, S.x * silu_f<PRECISE>(g.x), S.y * silu_f<PRECISE>(g.y));
}

template <typename T>
static int launch_mingru(const MinGruParams& p, int max_q_len, cudaStream_t st) {
  if (max_q_len == 1) {
    launch_pdl(mingru_step_kernel<T>, dim3((p.W / 2 + 127) / 128, p.B), dim3(128), 0, st, p);
    return (int)cudaGetLastError();
  }
  // narrow channel ranges when the wide ones would leave SMs without work
  const bool narrow = (long long)p.B * ((p.W + 31) / 32) < sm_count();
  if (narrow) launch_pdl(mingru_scan_kernel<T, 8, 8>, dim3((p.W + 15) / 16, p.B), dim3(MG_WARPS * 32), 0, st, p);
  else launch_pdl(mingru_scan_kernel<T, 16, 8>, dim3((p.W + 31) / 32, p.B), dim3(MG_WARPS * 32), 0, st, p);
  return (int)cudaGetLastError();
}

}  // namespace mx

using namespace mx;

// elem_f32: z / u / g / y are fp32 instead of bf16.  W even; pointers and ld aligned to element pairs.
MX_HOST_API int mx_mingru_scan(const void* z, const void* u, const void* g, int ld, const float* zb, const float* ub, float* state, const int* state_slots,
                               const int* cu_q, const int* seq_lens, void* y, int B, int W, int max_q_len, int elem_f32, cudaStream_t st) {
  if (B <= 0 || W <= 0 || max_q_len <= 0) return 0;
  const uintptr_t al = elem_f32 ? 7 : 3;
  if (W % 2 || ld % 2 || (((uintptr_t)z | (uintptr_t)u | (uintptr_t)g | (uintptr_t)y) & al) || (((uintptr_t)zb | (uintptr_t)ub | (uintptr_t)state) & 7)) return -160;
  MinGruParams p{z, u, g, zb, ub, state, state_slots, cu_q, seq_lens, y, B, W, ld};
  return elem_f32 ? launch_mingru<float>(p, max_q_len, st) : launch_mingru<__nv_bfloat16>(p, max_q_len, st);
}
