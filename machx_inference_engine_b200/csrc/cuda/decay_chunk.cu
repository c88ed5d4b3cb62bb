// Linear attention with decaying state (see linear_scan.cu) in chunked form on the tensor cores: prompts.
//
// Over a chunk of C = 64 tokens, with G_i the sum of the log decays of its tokens 0 .. i (per key channel, or one number per head),
//     O = Q'' S0 + M V,      Q''_i = q_i e^{G_i}       M_ij = (q_i e^{G_i}) . (k_j e^{-G_j}), j <= i                 (fixed decay, current token included)
//                            Q''_i = q_i e^{G_{i-1}}   M_ij = (q_i e^{G_{i-1}}) . (k_j e^{-G_j}), j < i, M_ii = q_i . (u k_i)   (decay from the data)
//     S = diag(e^{G_last}) S0 + KD^T V,                KD_j = k_j e^{G_last - G_j}
// so that only Q'' S0 waits for the running state.  Two kernels:
//
//   *_prep_kernel      one CTA per (chunk, head), all chunks in parallel: decays in fp32, M through one tcgen05.mma batch, and the operands Q'', KD, M, V as
//       ready-made shared-memory images (rows of 128 bytes, 128-byte swizzle).  With a fixed decay M is (Q K^T) times a table.  With decays from the data
//       the exponents are split so that no factor grows: the chunk falls into four blocks of 16 tokens, a query's factor runs from the start of its own
//       block (or pair of blocks), and the keys of earlier ones are decayed up to that start.  Inside a block the keys' factor does grow, by less than
//       e^80 -- inside the range of bf16, whose relative precision does not depend on size; a chunk in which it would grow further forms those 16 x 16
//       products one by one in fp32.
//   decay_chunk_scan_kernel  one CTA per (sequence, head, 64 value columns), chunks in order.  The state slice stays in registers (thread = key channel);
//       once per chunk it goes to shared memory as a bf16 high + low pair for Q'' S0.  KD is a high + low pair too, so that what a state gathers over
//       thousands of tokens is not rounded to 16 bits on its way in.
//
// Rows past a sequence's end are zero in every image and leave the state as it is.  A operands have 64 rows: the MMA's other 64 rows read whatever image
// follows in shared memory, and their results are never read.  Every wait is bounded (status word).
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

using bf16 = __nv_bfloat16;

constexpr int CC = 64;                 // chunk length
constexpr int CA = CC * 128;           // bytes of one image atom: 64 rows of 64 bf16
constexpr int CV = 64;                 // value columns of a scan CTA

struct DecayChunkParams {
  const bf16* q; const bf16* k; const bf16* v;     // row t of head h at t * ld + h * dk (dv)
  const float* z;                                  // [T][H * dk], or null: fixed decays
  const float* u;                                  // [H][dk]
  const float* decay;                              // [H], positive
  const int* cu_q; const int* seq_lens; const int* slots;
  float* state;                                    // [slots][H][dk][dv]
  float* out;                                      // [T][H * dv]
  uint8_t* ws;                                     // per (chunk, head): Q'' | KD high, low | M | V
  float* gl;                                       // [chunk][head][64 KA]: e^{G_last}
  int q_ld, k_ld, v_ld, B, H, dk, dv, silu, va;    // va: 64-column slices of V
  int* status;
};

__device__ __forceinline__ bool chunk_locate(const int* __restrict__ cu_q, int B, int ci, int& t0, int& n) {
  int base = 0;
  for (int b = 0; b < B; ++b) {
    const int first = cu_q[b], len = cu_q[b + 1] - first, nc = (len + CC - 1) / CC;
    if (ci < base + nc) {
      t0 = first + (ci - base) * CC;
      n = min(CC, len - (ci - base) * CC);
      return true;
    }
    base += nc;
  }
  return false;
}
__host__ __device__ constexpr int ws_bytes(int ka, int va) { return (3 * ka + 1 + va) * CA; }

__device__ __forceinline__ void unpack8(uint4 r, float (&v)[8]) {
  v[0] = bf16_lo(r.x); v[1] = bf16_hi(r.x); v[2] = bf16_lo(r.y); v[3] = bf16_hi(r.y); v[4] = bf16_lo(r.z); v[5] = bf16_hi(r.z); v[6] = bf16_lo(r.w); v[7] = bf16_hi(r.w);
}
__device__ __forceinline__ uint4 pack8(const float (&v)[8]) {
  return make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}
__device__ __forceinline__ void silu8(float (&v)[8]) {
#pragma unroll
  for (int i = 0; i < 8; ++i) v[i] *= sigmoid_f<false>(v[i]);
}
// image address of (row, 16-byte piece) in a run of atoms
__device__ __forceinline__ uint32_t atom_offset(int row, int piece) { return (uint32_t)(piece >> 3) * CA + sw128_offset(row, piece & 7); }

// V rows of the chunk -> image (shared by both prep kernels)
__device__ __forceinline__ void value_image(const DecayChunkParams& p, uint8_t* ws_v, int h, int t0, int n, int tid, int threads) {
  for (int i = tid; i < CC * p.va * 8; i += threads) {
    const int r = i / (p.va * 8), c = i % (p.va * 8);
    uint4 x = make_uint4(0, 0, 0, 0);
    if (r < n && 8 * c < p.dv) {
      x = *reinterpret_cast<const uint4*>(p.v + (size_t)(t0 + r) * p.v_ld + (size_t)h * p.dv + 8 * c);
      if (p.silu) {
        float f[8];
        unpack8(x, f);
        silu8(f);
        x = pack8(f);
      }
    }
    *reinterpret_cast<uint4*>(ws_v + atom_offset(r, c)) = x;
  }
}

// ------------------------------------------------------------------------------------------------ prep, fixed decay
template <int KA>
struct FixedSmem {
  static constexpr int Q = 0, K = KA * CA, MISC = 2 * KA * CA + CA, TOTAL = MISC + 64 + 1024;      // (the last atom of K is followed by room for its over-read)
};

template <int KA>
__global__ void __launch_bounds__(256) decay_fixed_prep_kernel(const DecayChunkParams p) {
  using L = FixedSmem<KA>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  uint64_t* bar = reinterpret_cast<uint64_t*>(smem + L::MISC);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  __shared__ float pw[CC + 1];                           // decay^e
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  pdl_prologue();
  int t0, n;
  if (!chunk_locate(p.cu_q, p.B, blockIdx.x, t0, n)) return;            // whole CTA, before any barrier / TMEM use
  if (tid == 0) { mbar_init(smem_u32(bar), 1); *abort_flag = 0; fence_mbar_init(); }
  if (warp == 0) { tmem_alloc(smem_u32(tmem_slot), 64); tmem_relinquish(); }
  if (tid <= CC) pw[tid] = exp2f((float)tid * log2f(p.decay[h]));
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  uint8_t* ws = p.ws + ((size_t)blockIdx.x * p.H + h) * ws_bytes(KA, p.va);
  for (int i = tid; i < CC * KA * 8; i += 256) {
    const int r = i / (KA * 8), c = i % (KA * 8);
    uint4 xq = make_uint4(0, 0, 0, 0), xk = xq, xq2 = xq, xk2 = xq, xk3 = xq;
    if (r < n && 8 * c < p.dk) {
      xq = *reinterpret_cast<const uint4*>(p.q + (size_t)(t0 + r) * p.q_ld + (size_t)h * p.dk + 8 * c);
      xk = *reinterpret_cast<const uint4*>(p.k + (size_t)(t0 + r) * p.k_ld + (size_t)h * p.dk + 8 * c);
      float q[8], k[8];
      unpack8(xq, q);
      unpack8(xk, k);
      if (p.silu) { silu8(q); silu8(k); xq = pack8(q); xk = pack8(k); }
      const float eq = pw[r + 1], ek = pw[n - 1 - r];
#pragma unroll
      for (int e = 0; e < 8; ++e) { q[e] *= eq; k[e] *= ek; }
      xq2 = pack8(q);
      xk2 = pack8(k);
      float hi[8];
      unpack8(xk2, hi);
#pragma unroll
      for (int e = 0; e < 8; ++e) k[e] -= hi[e];
      xk3 = pack8(k);
    }
    const uint32_t at = atom_offset(r, c);
    *reinterpret_cast<uint4*>(smem + L::Q + at) = xq;
    *reinterpret_cast<uint4*>(smem + L::K + at) = xk;
    *reinterpret_cast<uint4*>(ws + at) = xq2;
    *reinterpret_cast<uint4*>(ws + KA * CA + at) = xk2;
    *reinterpret_cast<uint4*>(ws + 2 * KA * CA + at) = xk3;
  }
  fence_proxy_async();
  __syncthreads();
  const uint32_t mbar = smem_u32(bar);
  if (tid == 0) {
    constexpr uint32_t idesc = umma_idesc_bf16(128, CC, 0, 0);
#pragma unroll
    for (int kk = 0; kk < KA * 4; ++kk) {
      const uint32_t off = (kk >> 2) * CA + (kk & 3) * 32;
      umma_bf16(tmem, umma_desc_k_sw128(sbase + L::Q + off), umma_desc_k_sw128(sbase + L::K + off), idesc, kk != 0);
    }
    umma_commit(mbar);
  }
  value_image(p, ws + (3 * KA + 1) * CA, h, t0, n, tid, 256);
  if (tid < 64 * KA) p.gl[((size_t)blockIdx.x * p.H + h) * 64 * KA + tid] = pw[n];
  const bool ok = mbar_wait(mbar, 0, p.status, ERR_MBAR_TIMEOUT_EPILOGUE, abort_flag, 32);
  tc_fence_after();
  if (ok && (warp & 3) < 2) {                            // accumulator rows 0 .. 63; warps w and w + 4 take half the columns each
    const int i = (warp & 3) * 32 + lane, col0 = (warp >> 2) * 32;
    uint32_t c[32];
    tmem_ld_32x32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + col0, c);
    tmem_ld_wait();
#pragma unroll
    for (int ch = 0; ch < 4; ++ch) {
      float m[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int j = col0 + 8 * ch + e;
        m[e] = j <= i ? pw[i - j < 0 ? 0 : i - j] * __uint_as_float(c[8 * ch + e]) : 0.f;
      }
      *reinterpret_cast<uint4*>(ws + 3 * KA * CA + sw128_offset(i, (col0 >> 3) + ch)) = pack8(m);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 64);
}

// ------------------------------------------------------------------------------------------------ prep, decays from the data
// Blocks of 16 tokens 0 .. 3.  A: queries against the start of their own block; A2: block 3 against the start of block 2 instead (block 2 as in A).
// B operand rows: K'' (0 .. 63: keys against the start of their own block, a growing factor), K_1 (64 .. 79: block 0 decayed to its end, for block 1),
// K_3 (80 .. 95: block 2 decayed to its end, for block 3), K_H (96 .. 127: blocks 0 and 1 decayed to the end of block 1, for A2's blocks 2 and 3).
constexpr int WB_ROWS = 128, WB_K1 = 64, WB_K3 = 80, WB_KH = 96;
constexpr float WKV_MAX_GROWTH = -80.f;
template <int KA>
struct DataSmem {
  static constexpr int A = 0, A2 = KA * CA, B = 2 * KA * CA, BA = WB_ROWS * 128;      // BA: bytes of a B atom
  static constexpr int LOGS = B + KA * BA;                               // cumulative logs inside the blocks, fp32 [64][64 KA + 1] (slow path only)
  static constexpr int DIAG = LOGS + CC * (64 * KA + 1) * 4;             // [64][16] fp32 (slow path only)
  static constexpr int MISC = DIAG + CC * 16 * 4;
  static constexpr int TOTAL = MISC + 64 + 1024;
};
__device__ __forceinline__ void sts32(uint32_t addr, uint32_t v) { asm volatile("st.shared.b32 [%0], %1;" ::"r"(addr), "r"(v) : "memory"); }
__device__ __forceinline__ void sts128(uint32_t addr, uint32_t a, uint32_t b, uint32_t c, uint32_t d) {
  asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(addr), "r"(a), "r"(b), "r"(c), "r"(d) : "memory");
}

template <int KA>
__global__ void __launch_bounds__(128 * KA, 4 / KA) decay_data_prep_kernel(const DecayChunkParams p) {
  using L = DataSmem<KA>;
  constexpr int W = 64 * KA, LS = W + 1, THREADS = 128 * KA;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  __shared__ __align__(8) float tot[4][W];               // sums of the logs of the blocks
  __shared__ float bonus[KA][CC];                        // r . (u k) of the tokens, one part per warp of a block
  uint64_t* bar = reinterpret_cast<uint64_t*>(smem + L::MISC);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* logs = reinterpret_cast<float*>(smem + L::LOGS);
  float* diag = reinterpret_cast<float*>(smem + L::DIAG);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  const int c = (tid % (32 * KA)) * 2, J = tid / (32 * KA);              // two key channels, a block
  pdl_prologue();
  int t0, n;
  if (!chunk_locate(p.cu_q, p.B, blockIdx.x, t0, n)) return;            // whole CTA, before any barrier / TMEM use
  if (tid == 0) { mbar_init(smem_u32(bar), 1); *abort_flag = 0; fence_mbar_init(); }
  if (warp == 0) { tmem_alloc(smem_u32(tmem_slot), 128); tmem_relinquish(); }
  const bool live = c < p.dk;
  uint32_t r2[16], k2[16];                               // bf16 pairs
  float lg[16][2];                                       // cumulative log decays inside the block
#pragma unroll
  for (int t = 0; t < 16; ++t) {
    const int row = 16 * J + t;
    const size_t tt = (size_t)(t0 + row);
    r2[t] = k2[t] = 0u;
    lg[t][0] = lg[t][1] = -INFINITY;                     // (rows past the end: log decay 0)
    if (live && row < n) {
      r2[t] = *reinterpret_cast<const uint32_t*>(p.q + tt * p.q_ld + (size_t)h * p.dk + c);
      k2[t] = *reinterpret_cast<const uint32_t*>(p.k + tt * p.k_ld + (size_t)h * p.dk + c);
      const float2 z = *reinterpret_cast<const float2*>(p.z + (tt * p.H + h) * p.dk + c);
      lg[t][0] = z.x;
      lg[t][1] = z.y;
    }
  }
  float2 u = make_float2(0.f, 0.f);
  if (live) u = *reinterpret_cast<const float2*>(p.u + (size_t)h * p.dk + c);
  {
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int t = 0; t < 16; ++t) {                       // (a decay of e^-104 and less is zero in fp32; larger sums would cost the others their digits)
      s0 -= fminf(expf(lg[t][0]), 110.f);
      s1 -= fminf(expf(lg[t][1]), 110.f);
      lg[t][0] = s0;
      lg[t][1] = s1;
    }
  }
  *reinterpret_cast<float2*>(&tot[J][c]) = make_float2(lg[15][0], lg[15][1]);
  {
    float v[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) v[t] = bf16_lo(r2[t]) * u.x * bf16_lo(k2[t]) + bf16_hi(r2[t]) * u.y * bf16_hi(k2[t]);
    // sum over the lanes, halving the values that a lane keeps: lane l ends with token l / 2
#pragma unroll
    for (int m = 8; m > 0; m >>= 1) {
      const bool up = lane & (2 * m);
#pragma unroll
      for (int i = 0; i < m; ++i) {
        const float give = up ? v[i] : v[i + m], keep = up ? v[i + m] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, give, 2 * m);
      }
    }
    v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
    if (!(lane & 1)) bonus[KA == 1 ? 0 : warp & 1][16 * J + (lane >> 1)] = v[0];
  }
  tc_fence_before();
  const bool slow = __syncthreads_or(fminf(lg[15][0], lg[15][1]) < WKV_MAX_GROWTH);
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  uint8_t* ws = p.ws + ((size_t)blockIdx.x * p.H + h) * ws_bytes(KA, p.va);
  float eb[2], ea[2], eh[2], e2[2], after[2] = {0.f, 0.f};              // e^{logs of the blocks before; after; to the end of block 1; of block 2}
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    float before = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float v = tot[i][c + x];
      if (i < J) before += v;
      if (i > J) after[x] += v;
    }
    eb[x] = __expf(before);
    ea[x] = __expf(after[x]);
    eh[x] = J == 0 ? __expf(tot[1][c + x]) : 1.f;
    e2[x] = J == 3 ? __expf(tot[2][c + x]) : 1.f;
  }
  {
    // the low bits of 16 J + t and of every image's first row come from t alone
    const uint32_t piece = (c & 63) >> 3, sub = (c & 7) * 2, atom = c >> 6;
    const uint32_t sa = sbase + L::A + atom * CA + J * 2048 + sub, sa2 = sa + (L::A2 - L::A);
    const uint32_t sb = sbase + L::B + atom * L::BA + J * 2048 + sub;
    const uint32_t side = J == 0 ? (WB_K1 >> 3) * 1024 : J == 2 ? ((WB_K3 >> 3) - 4) * 1024 : 0;       // from the K'' row of the block to its K_1 / K_3 row
    uint8_t* gq = ws + atom * CA + J * 2048 + sub;
    float ep[2] = {1.f, 1.f};                            // e^{sum of the block's logs before t}
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const uint32_t at = (t >> 3) * 1024 + (t & 7) * 128 + ((piece ^ (t & 7)) << 4);
      const float r0 = bf16_lo(r2[t]) * ep[0], r1 = bf16_hi(r2[t]) * ep[1], k0 = bf16_lo(k2[t]), k1 = bf16_hi(k2[t]);
      const float d0 = k0 * __expf(lg[15][0] - lg[t][0]), d1 = k1 * __expf(lg[15][1] - lg[t][1]);      // decayed to the block's end
      sts32(sa + at, pack_bf16(r0, r1));
      if (J >= 2) sts32(sa2 + at, pack_bf16(r0 * e2[0], r1 * e2[1]));
      sts32(sb + at, pack_bf16(k0 * __expf(-lg[t][0]), k1 * __expf(-lg[t][1])));
      if (side) sts32(sb + side + at, pack_bf16(d0, d1));
      if (J < 2) sts32(sb + (WB_KH >> 3) * 1024 + at, pack_bf16(d0 * eh[0], d1 * eh[1]));
      *reinterpret_cast<uint32_t*>(gq + at) = pack_bf16(r0 * eb[0], r1 * eb[1]);
      const uint32_t kd = pack_bf16(d0 * ea[0], d1 * ea[1]);
      *reinterpret_cast<uint32_t*>(gq + KA * CA + at) = kd;
      *reinterpret_cast<uint32_t*>(gq + 2 * KA * CA + at) = pack_bf16(d0 * ea[0] - bf16_lo(kd), d1 * ea[1] - bf16_hi(kd));
      if (slow) {
        logs[(16 * J + t) * LS + c] = lg[t][0];
        logs[(16 * J + t) * LS + c + 1] = lg[t][1];
      }
      ep[0] = __expf(lg[t][0]);
      ep[1] = __expf(lg[t][1]);
    }
  }
  if (J == 0)
    *reinterpret_cast<float2*>(p.gl + ((size_t)blockIdx.x * p.H + h) * W + c) = make_float2(__expf(lg[15][0] + after[0]), __expf(lg[15][1] + after[1]));
  fence_proxy_async();
  __syncthreads();
  const uint32_t mbar = smem_u32(bar);
  if (tid == 0) {
    constexpr uint32_t idesc = umma_idesc_bf16(128, WB_KH, 0, 0), idesc_h = umma_idesc_bf16(128, WB_ROWS - WB_KH, 0, 0);
#pragma unroll
    for (int kk = 0; kk < KA * 4; ++kk) {
      const uint32_t ao = (kk >> 2) * CA + (kk & 3) * 32, bo = sbase + L::B + (kk >> 2) * L::BA + (kk & 3) * 32;
      umma_bf16(tmem, umma_desc_k_sw128(sbase + L::A + ao), umma_desc_k_sw128(bo), idesc, kk != 0);
      umma_bf16(tmem + WB_KH, umma_desc_k_sw128(sbase + L::A2 + ao), umma_desc_k_sw128(bo + WB_KH * 128), idesc_h, kk != 0);
    }
    umma_commit(mbar);
  }
  value_image(p, ws + (3 * KA + 1) * CA, h, t0, n, tid, THREADS);
  if (slow) {                                            // products inside the blocks one by one: no factor is formed that could leave fp32's range
    for (int e = tid; e < CC * 16; e += THREADS) {
      const int i = e >> 4, j = (i & ~15) + (e & 15);
      float s = 0.f;
      if (j < i && i < n) {
        const bf16* ri = p.q + (size_t)(t0 + i) * p.q_ld + (size_t)h * p.dk;
        const bf16* kj = p.k + (size_t)(t0 + j) * p.k_ld + (size_t)h * p.dk;
        for (int x = 0; x < p.dk; ++x)
          s = fmaf(__bfloat162float(ri[x]) * __expf(logs[(i - 1) * LS + x] - logs[j * LS + x]), __bfloat162float(kj[x]), s);
      }
      diag[e] = s;
    }
    __syncthreads();
  }
  const bool ok = mbar_wait(mbar, 0, p.status, ERR_MBAR_TIMEOUT_EPILOGUE, abort_flag, 32);
  tc_fence_after();
  if (ok && warp < 2) {                                  // rows 32 warp + lane: blocks 2 warp and 2 warp + 1
    const int i = warp * 32 + lane, at = lane & 15;
    const bool lo = lane < 16;                           // the warp's first block
    const uint32_t ta = tmem + ((uint32_t)(warp * 32) << 16);
    uint32_t d[32], x[32], y[32];
    tmem_ld_32x32(ta + warp * 32, d);                    // own columns of both blocks
    tmem_ld_32x32(ta + WB_K1, x);                        // K_1 | K_3
    if (warp) tmem_ld_32x32(ta + WB_KH, y);
    tmem_ld_wait();
    const float b = KA == 1 ? bonus[0][i] : bonus[0][i] + bonus[KA - 1][i];
    float own[16];
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      own[j] = j < at ? __uint_as_float(lo ? d[j] : d[16 + j]) : j == at ? b : 0.f;
      if (slow && j < at) own[j] = diag[i * 16 + j];
    }
    uint8_t* wm = ws + 3 * KA * CA;
    auto store16 = [&](int Jc, const float (&v)[16]) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float m[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) m[e] = v[8 * half + e];
        *reinterpret_cast<uint4*>(wm + sw128_offset(i, 2 * Jc + half)) = pack8(m);
      }
    };
    float a[16], e[16];                                  // columns of the warp's first and second block
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      a[j] = lo ? own[j] : __uint_as_float(warp ? x[16 + j] : x[j]);
      e[j] = lo ? 0.f : own[j];
    }
    store16(2 * warp, a);
    store16(2 * warp + 1, e);
#pragma unroll
    for (int j = 0; j < 16; ++j) {                       // the other half of the columns
      a[j] = warp ? __uint_as_float(y[j]) : 0.f;
      e[j] = warp ? __uint_as_float(y[16 + j]) : 0.f;
    }
    store16(2 - 2 * warp, a);
    store16(3 - 2 * warp, e);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 128);
}

// ------------------------------------------------------------------------------------------------ scan
// Eight warps:  0 - 3  state (thread = key channel): S as a bf16 pair to shared memory, increment from TMEM, S <- decay S + increment
//               4, 5   output rows from TMEM to memory (row = token)
//               6      MMAs:  KD^T V (high and low part of KD) into one of two increments; M V + Q'' [S_high | S_low] into one of two outputs
//               7      bulk copies of the images, three chunks in flight
// The increment of a chunk does not depend on the state, so it is issued behind the previous chunk's output product and is there when the state warps
// want it; their conversion of the next state overlaps it.
template <int KA>
struct ChunkScanSmem {
  static constexpr int NS = 3;
  static constexpr int Q = 0, KD = KA * CA, KL = 2 * KA * CA, M = 3 * KA * CA, V = M + CA, STAGE = V + CA;
  static constexpr int SHI = NS * STAGE, SLO = SHI + KA * CA;            // state slice: [64 KA keys][64 values] high and low part
  static constexpr int BARS = SLO + KA * CA;
  static constexpr int TOTAL = BARS + 128 + 1024;
  static_assert(TOTAL <= 232448, "shared memory plan exceeds 227 KB");
};
constexpr int SCAN_THREADS = 256, TM_INC = 256;          // TMEM: outputs at 0 and 128 (high | low), increments at 256 and 320
__device__ __forceinline__ void chunk_bulk(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
__device__ __forceinline__ void stg256(float* p, const float (&v)[8]) {
  asm volatile("st.global.v8.f32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(p), "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]),
               "f"(v[7]) : "memory");
}

template <int KA>
__global__ void __launch_bounds__(SCAN_THREADS) decay_chunk_scan_kernel(const DecayChunkParams p) {
  using L = ChunkScanSmem<KA>;
  constexpr int NS = L::NS;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::BARS);
  const uint32_t b_load = smem_u32(bars), b_free = b_load + 8 * NS, b_inc = b_free + 8 * NS, b_out = b_inc + 16, b_ofree = b_out + 16, b_state = b_ofree + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * NS + 7);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, vs = blockIdx.x, b = blockIdx.z;
  pdl_prologue();
  const int t_begin = p.cu_q[b], len = p.cu_q[b + 1] - t_begin;
  if (len <= 0) return;                                  // whole CTA, before any barrier / TMEM use
  const int nc = (len + CC - 1) / CC;
  int cb = 0;                                            // index of this sequence's first chunk
  for (int i = 0; i < b; ++i) cb += (p.cu_q[i + 1] - p.cu_q[i] + CC - 1) / CC;
  if (tid == 0) {
    for (int s = 0; s < 2 * NS + 4; ++s) mbar_init(b_load + 8 * s, 1);   // load, free, inc, out
    mbar_init(b_ofree, 2); mbar_init(b_ofree + 8, 2);
    mbar_init(b_state, 2 * KA);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) { tmem_alloc(smem_u32(tmem_slot), 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot, tm_lane = (uint32_t)((warp & 3) * 32) << 16;
  const int dv = p.dv, v0 = vs * CV, nv = min(CV, dv - v0);              // (nv is a multiple of 8)
  bool ok = true;

  if (warp == 7) {
    if (lane == 0) {
      for (int c = 0; c < nc && ok; ++c) {
        const int s = c % NS;
        if (c >= NS && !(ok = mbar_wait(b_free + 8 * s, (c / NS - 1) & 1, p.status, ERR_MBAR_TIMEOUT_PRODUCER, abort_flag, 32))) break;
        const uint8_t* ws = p.ws + ((size_t)(cb + c) * p.H + h) * ws_bytes(KA, p.va);
        const uint32_t dst = sbase + s * L::STAGE, bar = b_load + 8 * s;
        mbar_expect_tx(bar, L::STAGE);
        chunk_bulk(dst, ws, L::V, bar);
        chunk_bulk(dst + L::V, ws + L::V + vs * CA, CA, bar);
      }
    }
  } else if (warp == 6) {
    if (lane == 0) {
      constexpr uint32_t idesc = umma_idesc_bf16(128, CV, 0, 1), idesc2 = umma_idesc_bf16(128, 2 * CV, 0, 1), idesc_t = umma_idesc_bf16(128, CV, 1, 1);
      auto increment = [&](int c) -> bool {
        if (!mbar_wait(b_load + 8 * (c % NS), (c / NS) & 1, p.status, ERR_MBAR_TIMEOUT_PRODUCER, abort_flag)) return false;
        tc_fence_after();
        const uint32_t st = sbase + (c % NS) * L::STAGE;
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < CC / 16; ++kk)
            umma_bf16(tmem + TM_INC + (c & 1) * CV, umma_desc_mn_sw128(st + (part ? L::KL : L::KD) + kk * 2048, CA, 1024),
                      umma_desc_mn_sw128(st + L::V + kk * 2048, CA, 1024), idesc_t, (part | kk) != 0);
        umma_commit(b_inc + 8 * (c & 1));
        return true;
      };
      ok = increment(0);
      for (int c = 0; c < nc && ok; ++c) {
        const uint32_t st = sbase + (c % NS) * L::STAGE, out = tmem + (c & 1) * 128;
        if (!(ok = mbar_wait(b_state, c & 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag))) break;
        if (c >= 2 && !(ok = mbar_wait(b_ofree + 8 * (c & 1), (c / 2 - 1) & 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag))) break;
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < KA * 4; ++kk)              // (the stage has been waited for by its increment)
          umma_bf16(out, umma_desc_k_sw128(st + L::Q + (kk >> 2) * CA + (kk & 3) * 32), umma_desc_mn_sw128(sbase + L::SHI + kk * 2048, KA * CA, 1024), idesc2, kk != 0);
#pragma unroll
        for (int kk = 0; kk < CC / 16; ++kk)
          umma_bf16(out, umma_desc_k_sw128(st + L::M + kk * 32), umma_desc_mn_sw128(st + L::V + kk * 2048, CA, 1024), idesc, 1);
        umma_commit(b_out + 8 * (c & 1));
        umma_commit(b_free + 8 * (c % NS));
        // (the state warps have read the increment of chunk c - 1: they have delivered the state of chunk c)
        if (c + 1 < nc) ok = increment(c + 1);
      }
    }
  } else if (warp >= 4) {
    const int row = (warp - 4) * 32 + lane;              // token of the chunk == TMEM lane
    for (int c = 0; c < nc && ok; ++c) {
      if (!(ok = mbar_wait(b_out + 8 * (c & 1), (c >> 1) & 1, p.status, ERR_MBAR_TIMEOUT_EPILOGUE, abort_flag, 32))) break;
      tc_fence_after();
      const uint32_t ta = tmem + tm_lane + (c & 1) * 128;
      uint32_t d0[32], d1[32], e0[32], e1[32];
      tmem_ld_32x32(ta, d0);
      tmem_ld_32x32(ta + 32, d1);
      tmem_ld_32x32(ta + 64, e0);
      tmem_ld_32x32(ta + 96, e1);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(b_ofree + 8 * (c & 1));
      if (row < min(CC, len - c * CC)) {
        float* o = p.out + ((size_t)(t_begin + c * CC + row) * p.H + h) * dv + v0;
#pragma unroll
        for (int j = 0; j < CV; j += 8) {
          float v[8];
#pragma unroll
          for (int e = 0; e < 8; ++e)
            v[e] = j < 32 ? __uint_as_float(d0[(j & 31) + e]) + __uint_as_float(e0[(j & 31) + e]) : __uint_as_float(d1[(j & 31) + e]) + __uint_as_float(e1[(j & 31) + e]);
          if (j < nv) stg256(o + j, v);
        }
      }
    }
  } else if (warp < 2 * KA) {
    // thread = key channel; S[j] = its state against value column 64 vs + j
    const bool live = tid < p.dk;
    float S[CV];
    float* sp = p.state + (((size_t)p.slots[b] * p.H + h) * p.dk + tid) * dv + v0;
    const bool fresh = p.seq_lens[b] == len;
#pragma unroll
    for (int j = 0; j < CV; j += 4) {
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && !fresh && j < nv) s = *reinterpret_cast<const float4*>(sp + j);
      S[j] = s.x; S[j + 1] = s.y; S[j + 2] = s.z; S[j + 3] = s.w;
    }
    const float* gl = p.gl + ((size_t)cb * p.H + h) * 64 * KA + tid;
    const size_t gl_step = (size_t)p.H * 64 * KA;
    float decay = gl[0];
    for (int c = 0; c < nc && ok; ++c) {
      if (c && !(ok = mbar_wait(b_out + 8 * ((c - 1) & 1), ((c - 1) >> 1) & 1, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag))) break;      // its reader is done
#pragma unroll
      for (int ch = 0; ch < 8; ++ch) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = S[8 * ch + 2 * e], y = S[8 * ch + 2 * e + 1];
          hi[e] = pack_bf16(x, y);
          lo[e] = pack_bf16(x - bf16_lo(hi[e]), y - bf16_hi(hi[e]));
        }
        sts128(sbase + L::SHI + sw128_offset(tid, ch), hi[0], hi[1], hi[2], hi[3]);
        sts128(sbase + L::SLO + sw128_offset(tid, ch), lo[0], lo[1], lo[2], lo[3]);
      }
      fence_proxy_async();
      tc_fence_before();                                 // (the previous increment's TMEM reads too)
      __syncwarp();
      if (lane == 0) mbar_arrive(b_state);
      const float decay_next = c + 1 < nc ? gl[(c + 1) * gl_step] : 0.f;
      if (!(ok = mbar_wait(b_inc + 8 * (c & 1), (c >> 1) & 1, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag))) break;
      tc_fence_after();
      uint32_t d0[32], d1[32];
      const uint32_t ta = tmem + tm_lane + TM_INC + (c & 1) * CV;
      tmem_ld_32x32(ta, d0);
      tmem_ld_32x32(ta + 32, d1);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        S[j] = fmaf(decay, S[j], __uint_as_float(d0[j]));
        S[32 + j] = fmaf(decay, S[32 + j], __uint_as_float(d1[j]));
      }
      decay = decay_next;
    }
    if (ok) {
#pragma unroll
      for (int j = 0; j < CV; j += 4)
        if (live && j < nv) *reinterpret_cast<float4*>(sp + j) = make_float4(S[j], S[j + 1], S[j + 2], S[j + 3]);
    }
  }
  if (*abort_flag)
    for (int i = 0; i < 200; ++i) __nanosleep(1000);     // a wait ran out: let copies in flight land before shared memory is released
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 512);
}

template <int KA>
static int launch_decay_chunk(const DecayChunkParams& p, int T, cudaStream_t st) {
  static DeviceOnce configured;
  if (configured.pending()) {
    cudaError_t e = cudaFuncSetAttribute(decay_fixed_prep_kernel<KA>, cudaFuncAttributeMaxDynamicSharedMemorySize, FixedSmem<KA>::TOTAL);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_data_prep_kernel<KA>, cudaFuncAttributeMaxDynamicSharedMemorySize, DataSmem<KA>::TOTAL);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_chunk_scan_kernel<KA>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkScanSmem<KA>::TOTAL);
    if (e != cudaSuccess) return (int)e;
    configured.mark();
  }
  const dim3 grid((unsigned)(T / CC + p.B), (unsigned)p.H);
  if (p.z) launch_pdl(decay_data_prep_kernel<KA>, grid, dim3(128 * KA), (size_t)DataSmem<KA>::TOTAL, st, p);
  else launch_pdl(decay_fixed_prep_kernel<KA>, grid, dim3(256), (size_t)FixedSmem<KA>::TOTAL, st, p);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  launch_pdl(decay_chunk_scan_kernel<KA>, dim3((unsigned)p.va, (unsigned)p.H, (unsigned)p.B), dim3(SCAN_THREADS), (size_t)ChunkScanSmem<KA>::TOTAL, st, p);
  return (int)cudaGetLastError();
}

}  // namespace mx

using namespace mx;

// Bytes of workspace (16-byte aligned) and floats of chunk decays for T tokens in B sequences (chunks <= T / 64 + B).
MX_HOST_API long long mx_decay_chunk_ws_bytes(int T, int B, int H, int dk, int dv) {
  return (long long)(T / CC + B) * H * ws_bytes(dk <= 64 ? 1 : 2, (dv + CV - 1) / CV);
}
MX_HOST_API long long mx_decay_chunk_gl_floats(int T, int B, int H, int dk) { return (long long)(T / CC + B) * H * (dk <= 64 ? 64 : 128); }

// Chunked form of mx_decay_scan: bf16 rows, dk up to 128, positive fixed decays; rows, bases and strides on 8-element boundaries.
MX_HOST_API int mx_decay_scan_chunked(const void* q, int q_ld, const void* k, int k_ld, const void* v, int v_ld, const float* z, const float* u, const float* decay,
                                      float* state, const int* slots, const int* cu_q, const int* seq_lens, float* out, int B, int T, int H, int dk, int dv,
                                      int silu, void* ws, float* gl, cudaStream_t st) {
  if (B <= 0 || H <= 0 || T <= 0) return 0;
  if (dk < 8 || dk > 128 || dk % 8 || dv < 8 || dv % 8 || q_ld % 8 || k_ld % 8 || v_ld % 8 || H > 65535 || B > 65535) return -112;
  if ((z != nullptr) == (decay != nullptr) || (z && (!u || silu))) return -109;
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)ws | (uintptr_t)state) & 15) return -112;
  if ((uintptr_t)out & 31) return -112;
  DecayChunkParams p;
  p.q = (const bf16*)q; p.k = (const bf16*)k; p.v = (const bf16*)v; p.z = z; p.u = u; p.decay = decay; p.cu_q = cu_q; p.seq_lens = seq_lens; p.slots = slots;
  p.state = state; p.out = out; p.ws = (uint8_t*)ws; p.gl = gl; p.q_ld = q_ld; p.k_ld = k_ld; p.v_ld = v_ld; p.B = B; p.H = H; p.dk = dk; p.dv = dv;
  p.silu = silu; p.va = (dv + CV - 1) / CV; p.status = status_word();
  return dk <= 64 ? launch_decay_chunk<1>(p, T, st) : launch_decay_chunk<2>(p, T, st);
}
