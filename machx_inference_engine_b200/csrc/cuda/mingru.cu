// minGRU recurrence (element-wise gated linear recurrence whose gates read only the current token), fused with its gate activations and
// its output gate:
//     z = sigmoid(zp + zb);  u = up + ub;  c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0)
//     S_t = (1 - z) S_(t-1) + z c;        y = S_t * silu(g)
// zp, up, g are column ranges of one projection [T][ld]; the biases are added here in fp32 (a bias far from zero would otherwise push
// the 16-bit rounding of the sum above the size of the projection's own signal).  The state is fp32 [slots][W]; a sequence whose step
// starts at position 0 starts from zeros, whatever its slot holds.
//
// Prompts: the recurrence is linear in S, so a run of tokens acts as S -> A S + B.  A cluster of CTAs owns CH channels of one sequence
// and walks its tokens in rounds: every CTA of the cluster takes the next TILE tokens, every thread of it TPS consecutive tokens of two
// channels (a slice).  A thread composes (A, B) of its slice, one warp chains the slices of the CTA, the cluster exchanges the CTAs'
// totals through distributed shared memory, and the threads replay their slices from the right start.  Every input is read once and
// nothing but the result is written.  Decode: one thread per (sequence, channel pair).
#include "act.cuh"
#include "cluster.cuh"
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

constexpr int MG_THREADS = 256;
constexpr int MG_MAX_CLUSTER = 8;

// CP: channel pairs per CTA; TPS: tokens per slice.  Cluster: (size, 1, 1), along the tokens.
template <typename T, int CP, int TPS>
__global__ void __launch_bounds__(MG_THREADS, sizeof(T) == 2 ? 3 : 2) mingru_scan_kernel(const MinGruParams p) {
  constexpr bool PRECISE = sizeof(T) == 4;
  constexpr int CH = 2 * CP, SL = MG_THREADS / CP, TILE = SL * TPS;
  static_assert(CH <= MG_THREADS, "one chaining thread per channel");
  __shared__ float sA[SL][CH], sB[SL][CH];              // slice (A, B), then their running composition from the CTA's first slice
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
  const bool ch_ok = ch < p.W;                           // W is even
  const T* zr = reinterpret_cast<const T*>(p.z) + (size_t)t_begin * p.ld + ch;
  const T* ur = reinterpret_cast<const T*>(p.u) + (size_t)t_begin * p.ld + ch;
  const T* gr = reinterpret_cast<const T*>(p.g) + (size_t)t_begin * p.ld + ch;
  T* yr = reinterpret_cast<T*>(p.y) + (size_t)t_begin * p.W + ch;
  float2 zb = make_float2(0.f, 0.f), ub = zb;
  if (ch_ok) { zb = load2(p.zb + ch); ub = load2(p.ub + ch); }
  float* st = p.state + (size_t)p.state_slots[b] * p.W + ch0;
  // chaining threads: thread i carries the state of channel i in front of the round
  const bool chain = threadIdx.x < CH;
  float S = (chain && ch0 + (int)threadIdx.x < p.W && !fresh) ? st[threadIdx.x] : 0.f;

  int par = 0;
  for (int r0 = 0; r0 < n; r0 += TILE * csize, par ^= 1) {
    const int t0 = r0 + (int)rank * TILE + slice * TPS;                  // first token of this slice
    const int mine = ch_ok ? min(TPS, n - t0) : 0;                       // its live tokens (may be <= 0)
    RawPair<T> zc[TPS], uc[TPS], gc[TPS];
    float2 av[TPS], bv[TPS];
    float A0 = 1.f, A1 = 1.f, B0 = 0.f, B1 = 0.f;
    auto load = [&](int j) {
      const size_t at = (size_t)(t0 + j) * p.ld;
      zc[j].load(zr + at);
      uc[j].load(ur + at);
      gc[j].load(gr + at);
    };
    auto compose = [&](int j) {
      const float2 zv = zc[j].get(), uv = uc[j].get();
      mingru_gates<PRECISE>(zv.x + zb.x, uv.x + ub.x, av[j].x, bv[j].x);
      mingru_gates<PRECISE>(zv.y + zb.y, uv.y + ub.y, av[j].y, bv[j].y);
      A0 *= av[j].x; B0 = fmaf(av[j].x, B0, bv[j].x);
      A1 *= av[j].y; B1 = fmaf(av[j].y, B1, bv[j].y);
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
      float2 tot[MG_MAX_CLUSTER];
#pragma unroll
      for (uint32_t r = 0; r < MG_MAX_CLUSTER; ++r)
        if (r < csize) tot[r] = cluster_ld2(addr, r);
#pragma unroll
      for (uint32_t r = 0; r < MG_MAX_CLUSTER; ++r) {
        if (r == rank) s_in[threadIdx.x] = S;
        if (r < csize) S = fmaf(tot[r].x, S, tot[r].y);
      }
    }
    __syncthreads();
    float S0 = fmaf(sA[slice][2 * cp], s_in[2 * cp], sB[slice][2 * cp]);
    float S1 = fmaf(sA[slice][2 * cp + 1], s_in[2 * cp + 1], sB[slice][2 * cp + 1]);
    auto replay = [&](int j) {
      const float2 gv = gc[j].get();
      S0 = fmaf(av[j].x, S0, bv[j].x);
      S1 = fmaf(av[j].y, S1, bv[j].y);
      store2(yr + (size_t)(t0 + j) * p.W, S0 * silu_f<PRECISE>(gv.x), S1 * silu_f<PRECISE>(gv.y));
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

static int g_mingru_cluster = 0;      // 0: by the length of the longest sequence; otherwise the cluster size (A/B timing)

template <typename T, int CP, int TPS>
static int launch_scan(const MinGruParams& p, int max_q_len, cudaStream_t st) {
  constexpr int CH = 2 * CP, TILE = MG_THREADS / CP * TPS;
  // CTAs along the tokens: no more than the longest sequence fills, and no more than fit the chip at once (three per SM).  Measured for
  // 4096 channels, one sequence of 512 tokens: 10.9 us with 2 (the choice), 15.8 with 1, 19.0 with 8; 6144 channels x 4096 tokens: 82 us
  // with 2, 130 with 1, 92 with 8; 2048 x 2048: 19.3 us with 4, 54.6 with 1, 22.6 with 8.
  int c = 1;
  const long long base = (long long)p.B * ((p.W + CH - 1) / CH);
  while (c < MG_MAX_CLUSTER && c * TILE < max_q_len && 2 * c * base <= 3ll * sm_count()) c *= 2;
  if (g_mingru_cluster > 0) c = g_mingru_cluster;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(c * ((p.W + CH - 1) / CH)), p.B);
  cfg.blockDim = dim3(MG_THREADS);
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = c; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr; cfg.numAttrs = 1;
  return (int)cudaLaunchKernelEx(&cfg, mingru_scan_kernel<T, CP, TPS>, p);
}

template <typename T>
static int launch_mingru(const MinGruParams& p, int max_q_len, cudaStream_t st) {
  if (max_q_len == 1) {
    launch_pdl(mingru_step_kernel<T>, dim3((p.W / 2 + 127) / 128, p.B), dim3(128), 0, st, p);
    return (int)cudaGetLastError();
  }
  return launch_scan<T, 16, 8>(p, max_q_len, st);       // 64-byte runs per token, tiles of 128 tokens
}

}  // namespace mx

using namespace mx;

// cluster size of the prompt kernel: 1, 2, 4 or 8; 0 = chosen per call (the default)
MX_HOST_API void mx_mingru_set_cluster(int c) { mx::g_mingru_cluster = (c == 1 || c == 2 || c == 4 || c == 8) ? c : 0; }

// elem_f32: z / u / g / y are fp32 instead of bf16.  W even; pointers and ld aligned to element pairs.
MX_HOST_API int mx_mingru_scan(const void* z, const void* u, const void* g, int ld, const float* zb, const float* ub, float* state, const int* state_slots,
                               const int* cu_q, const int* seq_lens, void* y, int B, int W, int max_q_len, int elem_f32, cudaStream_t st) {
  if (B <= 0 || W <= 0 || max_q_len <= 0) return 0;
  const uintptr_t al = elem_f32 ? 7 : 3;
  if (W % 2 || ld % 2 || (((uintptr_t)z | (uintptr_t)u | (uintptr_t)g | (uintptr_t)y) & al) || (((uintptr_t)zb | (uintptr_t)ub | (uintptr_t)state) & 7)) return -160;
  MinGruParams p{z, u, g, zb, ub, state, state_slots, cu_q, seq_lens, y, B, W, ld};
  return elem_f32 ? launch_mingru<float>(p, max_q_len, st) : launch_mingru<__nv_bfloat16>(p, max_q_len, st);
}
