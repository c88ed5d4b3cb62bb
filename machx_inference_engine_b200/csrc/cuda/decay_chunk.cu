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
//       block, and every later block has its own copy of the keys, decayed up to its start (rows K'_1 .. K'_3 of the B operand).  Inside a block the keys'
//       factor does grow, by less than e^80 -- inside the range of bf16, whose relative precision does not depend on size; a chunk in which it would grow
//       further forms those 16 x 16 products one by one in fp32.
//   decay_chunk_scan_kernel  one CTA per (sequence, head, 64 value columns), chunks in order.  The state slice stays in registers (thread = key channel);
//       once per chunk it goes to shared memory as a bf16 high + low pair, Q'' S0 + M V and KD^T V run as one MMA batch, and the next chunk's images
//       arrive by bulk copies meanwhile.
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
  uint8_t* ws;                                     // per (chunk, head): Q'' | KD | M | V
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
__host__ __device__ constexpr int ws_bytes(int ka, int va) { return (2 * ka + 1 + va) * CA; }

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
    uint4 xq = make_uint4(0, 0, 0, 0), xk = xq, xq2 = xq, xk2 = xq;
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
    }
    const uint32_t at = atom_offset(r, c);
    *reinterpret_cast<uint4*>(smem + L::Q + at) = xq;
    *reinterpret_cast<uint4*>(smem + L::K + at) = xk;
    *reinterpret_cast<uint4*>(ws + at) = xq2;
    *reinterpret_cast<uint4*>(ws + KA * CA + at) = xk2;
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
  value_image(p, ws + (2 * KA + 1) * CA, h, t0, n, tid, 256);
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
      *reinterpret_cast<uint4*>(ws + 2 * KA * CA + sw128_offset(i, (col0 >> 3) + ch)) = pack8(m);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 64);
}

// ------------------------------------------------------------------------------------------------ prep, decays from the data
// B operand rows: K'' (0 .. 63: keys against the start of their own block), U (64 .. 127: u k against the query's factor, for the diagonal), K'_1 (128 ..),
// K'_2 (144 ..), K'_3 (176 .. 223).
constexpr int WB_ROWS = 224;
constexpr float WKV_MAX_GROWTH = -80.f;
template <int KA>
struct DataSmem {
  static constexpr int A = 0, B = KA * CA, BA = WB_ROWS * 128;          // BA: bytes of a B atom
  static constexpr int LOGS = B + KA * BA;                               // cumulative logs inside the blocks, fp32 [64][64 KA + 1] (slow path only)
  static constexpr int DIAG = LOGS + CC * (64 * KA + 1) * 4;             // [64][16] fp32 (slow path only)
  static constexpr int TOT = DIAG + CC * 16 * 4;                         // block totals [4][64 KA]
  static constexpr int MISC = TOT + 4 * 64 * KA * 4;
  static constexpr int TOTAL = MISC + 64 + 1024;
  static_assert(KA * CA + CA <= LOGS, "A over-read stays inside the images");
};
__device__ __forceinline__ int kprime_row(int I) { return I == 1 ? 128 : I == 2 ? 144 : 176; }

template <int KA>
__global__ void __launch_bounds__(256 * KA, 2 / KA) decay_data_prep_kernel(const DecayChunkParams p) {
  using L = DataSmem<KA>;
  constexpr int W = 64 * KA, LS = W + 1, THREADS = 256 * KA;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  uint64_t* bar = reinterpret_cast<uint64_t*>(smem + L::MISC);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* tot = reinterpret_cast<float*>(smem + L::TOT);
  float* logs = reinterpret_cast<float*>(smem + L::LOGS);
  float* diag = reinterpret_cast<float*>(smem + L::DIAG);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y;
  const int c = tid % W, J = tid / W;                    // key channel, block of 16 tokens
  pdl_prologue();
  int t0, n;
  if (!chunk_locate(p.cu_q, p.B, blockIdx.x, t0, n)) return;            // whole CTA, before any barrier / TMEM use
  if (tid == 0) { mbar_init(smem_u32(bar), 1); *abort_flag = 0; fence_mbar_init(); }
  if (warp == 0) { tmem_alloc(smem_u32(tmem_slot), 256); tmem_relinquish(); }
  float lg[16], r[16], k[16];                            // cumulative log decays inside the block
  const bool live = c < p.dk;
  const float uc = live ? p.u[(size_t)h * p.dk + c] : 0.f;
  {
    float z[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const int row = 16 * J + t;
      const size_t tt = (size_t)(t0 + row);
      r[t] = k[t] = 0.f;
      z[t] = -INFINITY;                                  // (rows past the end: log decay 0)
      if (live && row < n) {
        r[t] = __bfloat162float(p.q[tt * p.q_ld + (size_t)h * p.dk + c]);
        k[t] = __bfloat162float(p.k[tt * p.k_ld + (size_t)h * p.dk + c]);
        z[t] = p.z[(tt * p.H + h) * p.dk + c];
      }
    }
    float s = 0.f;
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      s -= fminf(expf(z[t]), 110.f);                     // (a decay of e^-104 and less is zero in fp32; larger sums would cost the others their digits)
      lg[t] = s;
    }
  }
  tot[J * W + c] = lg[15];
  tc_fence_before();
  const bool slow = __syncthreads_or(lg[15] < WKV_MAX_GROWTH);
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  uint8_t* ws = p.ws + ((size_t)blockIdx.x * p.H + h) * ws_bytes(KA, p.va);
  float before = 0.f, after = 0.f, step[3] = {0.f, 0.f, 0.f};            // logs of the blocks before and after; of those between J and block J + 1 + i
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float x = tot[i * W + c];
    if (i < J) before += x;
    if (i > J) { after += x; }
  }
  step[1] = J + 1 < 4 ? tot[(J + 1) * W + c] : 0.f;
  step[2] = J + 2 < 4 ? step[1] + tot[(J + 2) * W + c] : 0.f;
  const float e_before = __expf(before), e_after = __expf(after), e_step[3] = {1.f, __expf(step[1]), __expf(step[2])};
  {
    const uint32_t piece = (c & 63) >> 3, sub = (c & 7) * 2, atom = c >> 6;
    auto put = [&](uint8_t* base, int stride, int row, float x) {
      *reinterpret_cast<bf16*>(base + atom * stride + sw128_offset(row, piece) + sub) = __float2bfloat16(x);
    };
    float e_prev = 1.f, l_prev = 0.f;                    // e^{sum of the block's logs before t}
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const int row = 16 * J + t;
      const float e_t = __expf(lg[t]), to_end = __expf(lg[15] - lg[t]);
      put(smem + L::A, CA, row, r[t] * e_prev);
      put(smem + L::B, L::BA, row, k[t] * __expf(-lg[t]));
      put(smem + L::B, L::BA, 64 + row, uc * k[t] * __expf(-l_prev));
#pragma unroll
      for (int i = 0; i < 3; ++i)
        if (J + 1 + i < 4) put(smem + L::B, L::BA, kprime_row(J + 1 + i) + row, k[t] * to_end * e_step[i]);
      put(ws, CA, row, r[t] * e_prev * e_before);
      put(ws + KA * CA, CA, row, k[t] * to_end * e_after);
      if (slow) logs[row * LS + c] = lg[t];
      e_prev = e_t;
      l_prev = lg[t];
    }
  }
  if (J == 0) p.gl[((size_t)blockIdx.x * p.H + h) * W + c] = __expf(lg[15] + after);
  fence_proxy_async();
  __syncthreads();
  const uint32_t mbar = smem_u32(bar);
  if (tid == 0) {
    constexpr uint32_t idesc = umma_idesc_bf16(128, WB_ROWS, 0, 0);
#pragma unroll
    for (int kk = 0; kk < KA * 4; ++kk)
      umma_bf16(tmem, umma_desc_k_sw128(sbase + L::A + (kk >> 2) * CA + (kk & 3) * 32), umma_desc_k_sw128(sbase + L::B + (kk >> 2) * L::BA + (kk & 3) * 32), idesc,
                kk != 0);
    umma_commit(mbar);
  }
  value_image(p, ws + (2 * KA + 1) * CA, h, t0, n, tid, THREADS);
  if (slow) {                                            // products inside the blocks one by one: no factor is formed that could leave fp32's range
    for (int e = tid; e < CC * 16; e += THREADS) {
      const int i = e >> 4, j = (i & ~15) + (e & 15);
      float s = 0.f;
      if (j <= i && i < n) {
        const bf16* ri = p.q + (size_t)(t0 + i) * p.q_ld + (size_t)h * p.dk;
        const bf16* kj = p.k + (size_t)(t0 + j) * p.k_ld + (size_t)h * p.dk;
        for (int x = 0; x < p.dk; ++x) {
          const float d = j == i ? p.u[(size_t)h * p.dk + x] : __expf(logs[(i - 1) * LS + x] - logs[j * LS + x]);
          s = fmaf(__bfloat162float(ri[x]) * d, __bfloat162float(kj[x]), s);
        }
      }
      diag[e] = s;
    }
    __syncthreads();
  }
  const bool ok = mbar_wait(mbar, 0, p.status, ERR_MBAR_TIMEOUT_EPILOGUE, abort_flag, 32);
  tc_fence_after();
  if (ok && warp < 2) {                                  // rows 32 warp + lane: blocks 2 warp and 2 warp + 1
    const int i = warp * 32 + lane;
    const bool lo = lane < 16;                           // the warp's first block
    const uint32_t ta = tmem + ((uint32_t)(warp * 32) << 16);
    float own[16];                                       // the block's own 16 columns, diagonal included
    {
      uint32_t d[32], g[32];
      tmem_ld_32x32(ta + warp * 32, d);
      tmem_ld_32x32(ta + 64 + warp * 32, g);
      tmem_ld_wait();
      uint32_t bonus = 0;
#pragma unroll
      for (int x = 0; x < 32; ++x) bonus = lane == x ? g[x] : bonus;
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        const int at = lane & 15;
        own[j] = j < at ? __uint_as_float(lo ? d[j] : d[16 + j]) : j == at ? __uint_as_float(bonus) : 0.f;
        if (slow) own[j] = diag[i * 16 + j];
      }
    }
    auto store16 = [&](int Jc, const float (&x)[16]) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float m[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) m[e] = x[8 * half + e];
        *reinterpret_cast<uint4*>(ws + 2 * KA * CA + sw128_offset(i, 2 * Jc + half)) = pack8(m);
      }
    };
    float x0[16], x1[16], x2[16], x3[16];
    if (warp == 0) {
      uint32_t a[32];
      tmem_ld_32x32(ta + 128, a);                        // K'_1 in its first 16 columns
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        x0[j] = lo ? own[j] : __uint_as_float(a[j]);
        x1[j] = lo ? 0.f : own[j];
        x2[j] = x3[j] = 0.f;
      }
    } else {
      uint32_t a[32], b[32], e[32];
      tmem_ld_32x32(ta + 144, a);                        // K'_2
      tmem_ld_32x32(ta + 176, b);                        // K'_3, columns 0 .. 31
      tmem_ld_32x32(ta + 192, e);                        // ... 16 .. 47
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        x0[j] = __uint_as_float(lo ? a[j] : b[j]);
        x1[j] = __uint_as_float(lo ? a[16 + j] : b[16 + j]);
        x2[j] = lo ? own[j] : __uint_as_float(e[16 + j]);
        x3[j] = lo ? 0.f : own[j];
      }
    }
    store16(0, x0); store16(1, x1); store16(2, x2); store16(3, x3);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 256);
}

// ------------------------------------------------------------------------------------------------ scan
template <int KA>
struct ChunkScanSmem {
  static constexpr int Q = 0, KD = KA * CA, M = 2 * KA * CA, V = M + CA, STAGE = V + CA;
  static constexpr int SHI = 2 * STAGE, SLO = SHI + 2 * CA, BARS = SLO + 2 * CA;      // state slice: [128 keys][64 values] high and low part
  static constexpr int TOTAL = BARS + 64 + 1024;
  static_assert(TOTAL <= 232448, "shared memory plan exceeds 227 KB");
};
__device__ __forceinline__ void chunk_bulk(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

template <int KA>
__global__ void __launch_bounds__(128) decay_chunk_scan_kernel(const DecayChunkParams p) {
  using L = ChunkScanSmem<KA>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::BARS);
  const uint32_t bar_load = smem_u32(bars), bar_inc = bar_load + 16, bar_o = bar_load + 24;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int tid = threadIdx.x, warp = tid >> 5, h = blockIdx.y, vs = blockIdx.x, b = blockIdx.z;
  pdl_prologue();
  const int t_begin = p.cu_q[b], len = p.cu_q[b + 1] - t_begin;
  if (len <= 0) return;                                  // whole CTA, before any barrier / TMEM use
  const int nc = (len + CC - 1) / CC;
  int cb = 0;                                            // index of this sequence's first chunk
  for (int i = 0; i < b; ++i) cb += (p.cu_q[i + 1] - p.cu_q[i] + CC - 1) / CC;
  if (tid == 0) {
    mbar_init(bar_load, 1); mbar_init(bar_load + 8, 1); mbar_init(bar_inc, 1); mbar_init(bar_o, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) { tmem_alloc(smem_u32(tmem_slot), 128); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot, tm_lane = (uint32_t)(warp * 32) << 16;

  // thread = key channel; S[j] = its state against value column 64 vs + j
  const int dv = p.dv, v0 = vs * CV, nv = min(CV, dv - v0);              // (nv is a multiple of 8)
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
  auto issue_load = [&](int c) {
    const int stg = c & 1;
    const uint8_t* ws = p.ws + ((size_t)(cb + c) * p.H + h) * ws_bytes(KA, p.va);
    const uint32_t dst = sbase + stg * L::STAGE, bar = bar_load + 8 * stg;
    mbar_expect_tx(bar, L::STAGE);
    chunk_bulk(dst, ws, L::V, bar);
    chunk_bulk(dst + L::V, ws + L::V + vs * CA, CA, bar);
  };
  if (tid == 0) issue_load(0);
  constexpr uint32_t idesc = umma_idesc_bf16(128, CV, 0, 1), idesc_t = umma_idesc_bf16(128, CV, 1, 1);
  bool ok = true;
  for (int c = 0; c < nc && ok; ++c) {
    const uint32_t st = sbase + (c & 1) * L::STAGE;
    const float decay = tid < 64 * KA ? p.gl[((size_t)(cb + c) * p.H + h) * 64 * KA + tid] : 0.f;
    if (tid < 64 * KA) {
#pragma unroll
      for (int ch = 0; ch < 8; ++ch) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float x = S[8 * ch + 2 * e], y = S[8 * ch + 2 * e + 1];
          hi[e] = pack_bf16(x, y);
          lo[e] = pack_bf16(x - bf16_lo(hi[e]), y - bf16_hi(hi[e]));
        }
        *reinterpret_cast<uint4*>(smem + L::SHI + sw128_offset(tid, ch)) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(smem + L::SLO + sw128_offset(tid, ch)) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    if (tid == 0) {
      if (c + 1 < nc) issue_load(c + 1);                 // that stage's readers (the MMAs of chunk c - 1) have completed
      if (mbar_wait(bar_load + 8 * (c & 1), (c >> 1) & 1, p.status, ERR_MBAR_TIMEOUT_PRODUCER, abort_flag)) {
        tc_fence_after();
#pragma unroll
        for (int kk = 0; kk < CC / 16; ++kk)             // state increment [key][value]
          umma_bf16(tmem + CV, umma_desc_mn_sw128(st + L::KD + kk * 2048, CA, 1024), umma_desc_mn_sw128(st + L::V + kk * 2048, CA, 1024), idesc_t, kk != 0);
        umma_commit(bar_inc);
#pragma unroll
        for (int kk = 0; kk < CC / 16; ++kk)
          umma_bf16(tmem, umma_desc_k_sw128(st + L::M + kk * 32), umma_desc_mn_sw128(st + L::V + kk * 2048, CA, 1024), idesc, kk != 0);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < KA * 4; ++kk)
            umma_bf16(tmem, umma_desc_k_sw128(st + L::Q + (kk >> 2) * CA + (kk & 3) * 32), umma_desc_mn_sw128(sbase + (part ? L::SLO : L::SHI) + kk * 2048, 2 * CA, 1024),
                      idesc, 1);
        umma_commit(bar_o);
      }
    }
    if (!(ok = mbar_wait(bar_inc, c & 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag))) break;
    tc_fence_after();
    if (warp < 2 * KA) {
      uint32_t d0[32], d1[32];
      tmem_ld_32x32(tmem + tm_lane + CV, d0);
      tmem_ld_32x32(tmem + tm_lane + CV + 32, d1);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 32; ++j) {
        S[j] = fmaf(decay, S[j], __uint_as_float(d0[j]));
        S[32 + j] = fmaf(decay, S[32 + j], __uint_as_float(d1[j]));
      }
    }
    if (!(ok = mbar_wait(bar_o, c & 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag))) break;
    tc_fence_after();
    if (warp < 2) {
      uint32_t d0[32], d1[32];
      tmem_ld_32x32(tmem + tm_lane, d0);
      tmem_ld_32x32(tmem + tm_lane + 32, d1);
      tmem_ld_wait();
      if (tid < min(CC, len - c * CC)) {
        float* o = p.out + ((size_t)(t_begin + c * CC + tid) * p.H + h) * dv + v0;
#pragma unroll
        for (int j = 0; j < CV; j += 4) {
          const uint32_t* s = j < 32 ? d0 : d1;
          if (j < nv)
            *reinterpret_cast<float4*>(o + j) = make_float4(__uint_as_float(s[j & 31]), __uint_as_float(s[(j & 31) + 1]), __uint_as_float(s[(j & 31) + 2]),
                                                            __uint_as_float(s[(j & 31) + 3]));
        }
      }
    }
  }
  if (ok) {
#pragma unroll
    for (int j = 0; j < CV; j += 4)
      if (live && j < nv) *reinterpret_cast<float4*>(sp + j) = make_float4(S[j], S[j + 1], S[j + 2], S[j + 3]);
  } else {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);     // a wait ran out: let copies in flight land before shared memory is released
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, 128);
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
  if (p.z) launch_pdl(decay_data_prep_kernel<KA>, grid, dim3(256 * KA), (size_t)DataSmem<KA>::TOTAL, st, p);
  else launch_pdl(decay_fixed_prep_kernel<KA>, grid, dim3(256), (size_t)FixedSmem<KA>::TOTAL, st, p);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  launch_pdl(decay_chunk_scan_kernel<KA>, dim3((unsigned)p.va, (unsigned)p.H, (unsigned)p.B), dim3(128), (size_t)ChunkScanSmem<KA>::TOTAL, st, p);
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
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)ws | (uintptr_t)state | (uintptr_t)out) & 15) return -112;
  DecayChunkParams p;
  p.q = (const bf16*)q; p.k = (const bf16*)k; p.v = (const bf16*)v; p.z = z; p.u = u; p.decay = decay; p.cu_q = cu_q; p.seq_lens = seq_lens; p.slots = slots;
  p.state = state; p.out = out; p.ws = (uint8_t*)ws; p.gl = gl; p.q_ld = q_ld; p.k_ld = k_ld; p.v_ld = v_ld; p.B = B; p.H = H; p.dk = dk; p.dv = dv;
  p.silu = silu; p.va = (dv + CV - 1) / CV; p.status = status_word();
  return dk <= 64 ? launch_decay_chunk<1>(p, T, st) : launch_decay_chunk<2>(p, T, st);
}
