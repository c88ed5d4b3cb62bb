// Prefill FlashAttention on the sm_100a tensor cores: paged KV, causal, sliding window with whole-tile skipping, attention sinks,
// logit soft-cap, GQA, score factors per query position (query temperature), sigmoid output gate.  Keys and values may have different
// widths (multiples of 8 up to 256): the shared tiles are 64 / 128 / 256 columns wide and the tensor maps, whose rows end at the real
// width, fill the rest with zeros, so the cache itself is not padded.
//
// Keys in two parts (ROT = 1; latent attention over expanded keys): the first DK - 64 columns of a head come from expanded pages [row][head][dim],
// the last 64 from a part that all heads share, at its place in the latent cache; each part has its own tensor maps (and page table).  The values
// are expanded pages too.
//
// Pooled blocks (MODE 2): means of whole runs of `pool` tokens before the window are keys and values too, read from dense pages [sequence][page][kv head]
// [128] that pool_blocks (pooled.cu) has written for the step, as tiles in front of the window's.  This mode also takes the soft-cap as a parameter, through
// an accurate tanh, and may turn the output back by the query's position (a rotation of neighbouring pairs, before the gate).
//
// One CTA owns 128 query tokens of one query head and walks the key tiles of its range (128 keys per tile, 64 for
// head_dim 256 so that two K and two V tiles still fit in shared memory):
//   warp 0  : TMA loads of the K and V tiles (two-stage rings) and, once, of the Q tile
//   warp 1  : tcgen05.mma  S(j) = Q K_j^T  into one of two S buffers in TMEM, so that S(j+1) is computed while the softmax
//             threads work on S(j);  O += P_j V_j  accumulates in TMEM over all tiles
//   warps 2-5 (one thread per query row = TMEM lane): read S, mask, online softmax, write P (bf16) into a 128-byte-swizzled
//             shared tile for the PV MMA.  The output row is NOT kept in registers: O stays in TMEM and is rescaled in place
//             (tcgen05.ld / tcgen05.st) only when the running maximum has grown by more than 2^8 since the last rescale;
//             until then P is formed against the old reference maximum (it stays far inside bf16's range) and O and the
//             denominator remain consistent.  That removes the per-tile fold of O and is what lets head_dim 256 fit.
// The per-head sink joins the denominator once, at the end.  Every wait is bounded.
//
// Reference parity: src/ops/attention.cpp:2456-2815 (fa2_tile_wide_impl<HD,Bc,REGDOT,SG,SINK> for HD 64..512 and its
// dispatcher: causal and window masks per key, whole-tile skip outside the window, sink folded at row end); the soft-cap
// of src/model/gemma4.cpp's attention is applied to the scores here.
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

constexpr int FA_BQ = 128;     // query rows per CTA
constexpr int FA_PAGE = 128;   // KV page size

struct FaParams {
  const int* block_table;  // [B][max_blocks]
  const int* rot_table;    // ROT: [B][max_blocks] pages of the shared key part (block_table: the expanded pages)
  const int* seq_lens;     // [B]
  const int* cu_q;         // [B+1]
  const float* sinks;      // [n_q] or null
  const float* q_scale;    // [q_scale_n] factor on the scores of a query at that position, or null
  const __nv_bfloat16* gate;   // out *= sigmoid(gate): [Tq] rows of [n_q][dv], gate_ld elements apart, or null
  __nv_bfloat16* out;      // [Tq][n_q][dv]
  int q_scale_n, gate_ld, dk, dv, q_ld;
  int gate_heads, keep_first;   // one gate number per head; with a window: the first keys that stay visible
  int n_q, n_kv, max_blocks, max_q_tiles, window;
  float scale, softcap;
  int* status;
};

// MODE 2 alone carries these (a longer argument block alone made the other modes spill registers)
struct FaPoolParams : FaParams {
  int pool, pool_pages;    // tokens per pooled block (0: none), dense pages per sequence
  const float* out_cos;    // [out_n][out_half] or null: the output is turned by minus its position
  const float* out_sin;
  int out_n, out_half;
};
template <int MODE> struct FaArgs { using T = FaParams; };
template <> struct FaArgs<2> { using T = FaPoolParams; };

template <int DK, int DV>
struct FaCfg {
  static constexpr int BKV = (DK <= 128 && DV <= 128) ? 128 : 64;   // keys per tile
  static constexpr int NS = 2;                                 // S buffers in TMEM
  static constexpr int CTAS = 1;                               // one CTA per SM: its softmax threads keep a whole S row in registers
  static constexpr uint32_t TMEM_COLS = 512;
  static constexpr int KATOMS = DK / 64, VATOMS = DV / 64;     // 64-column (128-byte) swizzle atoms per row of Q / K and of V
  static constexpr int Q_BYTES = FA_BQ * DK * 2;
  static constexpr int K_BYTES = BKV * DK * 2, V_BYTES = BKV * DV * 2;
  static constexpr int KS = 2, VS = 2;                         // tiles in flight
  static constexpr int P_BYTES = FA_BQ * BKV * 2;
  static constexpr int Q_OFF = 0;
  static constexpr int K_OFF = Q_OFF + Q_BYTES;
  static constexpr int V_OFF = K_OFF + KS * K_BYTES;
  static constexpr int P_OFF = V_OFF + VS * V_BYTES;
  static constexpr int BAR_OFF = P_OFF + P_BYTES;
  static constexpr int TOTAL = BAR_OFF + 256 + 1024;
  static_assert(TOTAL <= 232448, "shared memory plan exceeds 227 KB");
  static_assert(NS * BKV + DV <= (int)TMEM_COLS, "TMEM plan");
};

__device__ __forceinline__ void tmem_st_32x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
        "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]),
        "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float tanh_fast(float x) {
  float y;
  asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// two fp32 operations in one instruction
__device__ __forceinline__ uint64_t pack2(float a, float b) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(a), "f"(b));
  return d;
}
__device__ __forceinline__ void unpack2(uint64_t d, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(d)); }
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// v x P(v^2) over a run, P of degree D with the coefficients c (of rising powers)
template <int D, int N>
__device__ __forceinline__ void odd_series_run(float (&v)[N], const float (&c)[D + 1]) {
  uint64_t k[D + 1];
#pragma unroll
  for (int d = 0; d <= D; ++d) k[d] = pack2(c[d], c[d]);
#pragma unroll
  for (int i = 0; i < N; i += 2) {
    const uint64_t x = pack2(v[i], v[i + 1]), w = mul2(x, x);
    uint64_t t = k[D];
#pragma unroll
    for (int d = D - 1; d >= 0; --d) t = fma2(w, t, k[d]);
    unpack2(mul2(x, t), v[i], v[i + 1]);
  }
}

// cap * tanh(x / cap) over a run of raw scores, without the hardware's 11-bit tanh: the power series of tanh y where all of the run is small
//     y (1 - z / 3 + 2 z^2 / 15 - 17 z^3 / 315 + 62 z^4 / 2835 - 1382 z^5 / 155925 + 21844 z^6 / 6081075 - ...), z = y^2
// (three terms up to |y| = 1/8, seven up to 1/2: relative error below 1e-6), otherwise 1 - 2 / (1 + e^2y).  in: factor to y = x / cap; out_c: factor on the
// result.
template <int N>
__device__ __forceinline__ void softcap_run(float (&v)[N], float in, float out_c) {
  float big = 0.f;
#pragma unroll
  for (int i = 0; i < N; i += 2) big = fmaxf(fmaxf(big, fabsf(v[i])), fabsf(v[i + 1]));
  big *= fabsf(in);
  const float s = in * in, lin = in * out_c;
  if (!__any_sync(0xffffffffu, big > 0.125f)) {
    const float c[3] = {lin, lin * s * -3.3333333e-1f, lin * s * s * 1.3333333e-1f};
    odd_series_run<2>(v, c);
  } else if (!__any_sync(0xffffffffu, big > 0.5f)) {
    const float s2 = s * s, s3 = s2 * s;
    const float c[7] = {lin, lin * s * -3.3333333e-1f, lin * s2 * 1.3333333e-1f, lin * s3 * -5.3968254e-2f, lin * s2 * s2 * 2.1869489e-2f,
                        lin * s2 * s3 * -8.8632355e-3f, lin * s3 * s3 * 3.5921280e-3f};
    odd_series_run<6>(v, c);
  } else {
    const float in2 = in * 2.8853900817779268f;        // 2 / ln 2
#pragma unroll
    for (int i = 0; i < N; ++i) {
      float r;
      asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + ex2_fast(v[i] * in2)));
      v[i] = fmaf(-2.f * out_c, r, out_c);
    }
  }
}

// MODE: 0 plain, 1 keys in two parts, 2 pooled blocks
template <int DK, int DV, bool CAP, int MODE>
__global__ void __launch_bounds__(192, FaCfg<DK, DV>::CTAS)
fa_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                  const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_qr,
                  const __grid_constant__ CUtensorMap tmap_kr, const typename FaArgs<MODE>::T p) {
  using L = FaCfg<DK, DV>;
  constexpr int ROT = MODE == 1 ? 1 : 0;         // key atoms of the shared part
  constexpr int BKV = L::BKV, NS = L::NS, KS = L::KS, VS = L::VS;
  constexpr float LOG2E = 1.4426950408889634f;
  constexpr float RESCALE_STEP = 8.f;            // in log2 units: O is rescaled when the maximum has grown by a factor of 256
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::BAR_OFF);
  // barriers: q_full, k_full[2], v_full[2], k_empty[2], v_empty[2], s_full[2], s_empty[2], p_full, pv_done
  const uint32_t b_qfull = smem_u32(bars), b_kfull = b_qfull + 8, b_vfull = b_kfull + 16, b_kempty = b_vfull + 16, b_vempty = b_kempty + 16;
  const uint32_t b_sfull = b_vempty + 16, b_sempty = b_sfull + 16, b_pfull = b_sempty + 16, b_pvdone = b_pfull + 8;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.x / p.max_q_tiles, qt = blockIdx.x % p.max_q_tiles;
  const int head = blockIdx.y;
  const int kvh = head / (p.n_q / p.n_kv);
  const int q_begin = p.cu_q[b], q_len = p.cu_q[b + 1] - q_begin;
  const int t0 = qt * FA_BQ;
  if (t0 >= q_len) return;                       // whole CTA leaves before any barrier / TMEM use
  const int seq_len = p.seq_lens[b];
  const int pos0 = seq_len - q_len + t0;         // absolute position of query row 0 of this tile
  const int rows = min(FA_BQ, q_len - t0);
  const int kv_hi = min(seq_len, pos0 + rows);   // exclusive
  const int kv_lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;
  const int tile_lo = kv_lo / BKV, tile_hi = (kv_hi + BKV - 1) / BKV;
  const int n_keep = min((p.keep_first + BKV - 1) / BKV, tile_lo);            // kept tiles before the window's
  auto blocks_seen = [&](int pos) {
    if constexpr (MODE == 2) return pos >= p.window ? (pos - p.window + 1) / p.pool : 0;
    return 0;
  };
  int n_pool = 0;                                                             // tiles of pooled blocks, the first ones
  if constexpr (MODE == 2) {
    if (p.pool) n_pool = (blocks_seen(pos0 + rows - 1) + BKV - 1) / BKV;
  }
  const int n_tiles = n_pool + n_keep + tile_hi - tile_lo;
  auto first_key = [&](int j) {                  // (of a pooled tile: its first block)
    if constexpr (MODE == 2) {
      if (j < n_pool) return j * BKV;
      j -= n_pool;
    }
    return (j < n_keep ? j : tile_lo + j - n_keep) * BKV;
  };

  if (threadIdx.x == 0) {
    mbar_init(b_qfull, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(b_kfull + 8 * s, 1); mbar_init(b_vfull + 8 * s, 1); mbar_init(b_kempty + 8 * s, 1); mbar_init(b_vempty + 8 * s, 1);
      mbar_init(b_sfull + 8 * s, 1); mbar_init(b_sempty + 8 * s, 4);
    }
    mbar_init(b_pfull, 4); mbar_init(b_pvdone, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) { tmem_alloc(smem_u32(tmem_slot), L::TMEM_COLS); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + NS * BKV;

  if (warp == 0) {
    if (lane == 0) {
      prefetch_tmap(&tmap_q); prefetch_tmap(&tmap_k); prefetch_tmap(&tmap_v);
      mbar_expect_tx(b_qfull, L::Q_BYTES);
#pragma unroll
      for (int a = 0; a < L::KATOMS; ++a)
        if (a < L::KATOMS - ROT) tma_load_3d(sbase + L::Q_OFF + a * (FA_BQ * 128), &tmap_q, b_qfull, a * 64, head, q_begin + t0);
        else tma_load_3d(sbase + L::Q_OFF + a * (FA_BQ * 128), &tmap_qr, b_qfull, 0, head, q_begin + t0);
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const uint32_t sk = j % KS, phk = (j / KS) & 1, sv = j % VS, phv = (j / VS) & 1;
        const int key0 = first_key(j);
        bool pooled = false;
        int blk = 0;
        if constexpr (MODE == 2) pooled = j < n_pool;
        if constexpr (MODE == 2) {
          if (pooled) blk = b * p.pool_pages + key0 / FA_PAGE;
        }
        if (!pooled) blk = p.block_table[(size_t)b * p.max_blocks + key0 / FA_PAGE];
        const int krow = key0 % FA_PAGE;
        int rblk = 0;
        if constexpr (ROT != 0) rblk = p.rot_table[(size_t)b * p.max_blocks + key0 / FA_PAGE];
        if (!(ok = mbar_wait(b_kempty + 8 * sk, phk ^ 1, p.status, ERR_MBAR_TIMEOUT_PRODUCER, abort_flag))) break;
        mbar_expect_tx(b_kfull + 8 * sk, L::K_BYTES);
#pragma unroll
        for (int a = 0; a < L::KATOMS; ++a)
          if (a < L::KATOMS - ROT) tma_load_4d(sbase + L::K_OFF + sk * L::K_BYTES + a * (BKV * 128), pooled ? &tmap_qr : &tmap_k, b_kfull + 8 * sk, a * 64, krow, kvh, blk);
          else tma_load_3d(sbase + L::K_OFF + sk * L::K_BYTES + a * (BKV * 128), &tmap_kr, b_kfull + 8 * sk, 0, krow, rblk);
        if (!(ok = mbar_wait(b_vempty + 8 * sv, phv ^ 1, p.status, ERR_MBAR_TIMEOUT_PRODUCER, abort_flag))) break;
        mbar_expect_tx(b_vfull + 8 * sv, L::V_BYTES);
#pragma unroll
        for (int a = 0; a < L::VATOMS; ++a)
          tma_load_4d(sbase + L::V_OFF + sv * L::V_BYTES + a * (BKV * 128), pooled ? &tmap_kr : &tmap_v, b_vfull + 8 * sv, a * 64, krow, kvh, blk);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(FA_BQ, BKV, 0, 0);
      constexpr uint32_t idesc_o = umma_idesc_bf16(FA_BQ, DV, 0, 1);      // B = V is MN-major (head_dim contiguous)
      bool ok = mbar_wait(b_qfull, 0, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag);
      // S(j) = Q K_j^T into S buffer j % NS (waits for K_j and for the softmax threads to have released that buffer)
      auto issue_s = [&](int j) -> bool {
        const uint32_t sk = j % KS, phk = (j / KS) & 1, sb = j % NS, phs = (j / NS) & 1;
        if (!mbar_wait(b_kfull + 8 * sk, phk, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag)) return false;
        if (!mbar_wait(b_sempty + 8 * sb, phs ^ 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag)) return false;
        tc_fence_after();
        const uint32_t qa = sbase + L::Q_OFF, ka = sbase + L::K_OFF + sk * L::K_BYTES;
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint64_t ad = umma_desc_k_sw128(qa + (kk >> 2) * (FA_BQ * 128) + (kk & 3) * 32);
          const uint64_t bd = umma_desc_k_sw128(ka + (kk >> 2) * (BKV * 128) + (kk & 3) * 32);
          umma_bf16(tmem_base + sb * BKV, ad, bd, idesc_s, kk != 0);
        }
        umma_commit(b_sfull + 8 * sb);
        umma_commit(b_kempty + 8 * sk);
        return true;
      };
      if (ok && n_tiles > 0) ok = issue_s(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (NS == 2 && j + 1 < n_tiles && !(ok = issue_s(j + 1))) break;       // the next score tile runs while softmax(j) works
        const uint32_t sv = j % VS, phv = (j / VS) & 1;
        if (!(ok = mbar_wait(b_pfull, j & 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag))) break;
        if (!(ok = mbar_wait(b_vfull + 8 * sv, phv, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag))) break;
        tc_fence_after();
        const uint32_t pa = sbase + L::P_OFF, va = sbase + L::V_OFF + sv * L::V_BYTES;
#pragma unroll
        for (int kk = 0; kk < BKV / 16; ++kk) {
          const uint64_t ad = umma_desc_k_sw128(pa + (kk >> 2) * (FA_BQ * 128) + (kk & 3) * 32);
          const uint64_t bd = umma_desc_mn_sw128(va + kk * 2048, BKV * 128, 1024);
          umma_bf16(tmem_o, ad, bd, idesc_o, (j | kk) != 0);
        }
        umma_commit(b_pvdone);
        umma_commit(b_vempty + 8 * sv);
        if (NS == 1 && j + 1 < n_tiles && !(ok = issue_s(j + 1))) break;
      }
    }
  } else {
    // ------------------------------------------------ softmax, one thread per query row
    // Per score: one max, one fused multiply-add, one ex2, half a pack and one add.  The whole S row of the tile sits in
    // registers, so the S buffer goes back to the MMA thread before the exponentials start.
    const int q4 = warp & 3;
    const int r = q4 * 32 + lane;                  // row inside the tile == TMEM lane
    const int qpos = pos0 + r;
    const bool row_ok = r < rows;
    const float qs = p.scale * (p.q_scale ? p.q_scale[min(qpos, p.q_scale_n - 1)] : 1.f);
    // c: factor from the stored score to log2 units, applied after the maximum.  That needs c > 0: a row whose factor is not (a
    // temperature law may change sign) multiplies its scores first and goes on with 1.
    bool cap = CAP;
    if constexpr (MODE == 2) cap = p.softcap > 0.f;
    const bool early = !cap && !(qs > 0.f);
    const float c = (cap || early) ? 1.f : qs * LOG2E;
    const float cap_c = p.softcap * LOG2E, inv_cap = cap ? qs / p.softcap : 0.f;
    int seen = 0;
    if constexpr (MODE == 2) {
      if (p.pool) seen = blocks_seen(qpos);
    }
    if (p.gate && !p.gate_heads && row_ok) {       // bring the row's gate into L2 while the keys are walked
      const __nv_bfloat16* g0 = p.gate + (size_t)(q_begin + t0 + r) * p.gate_ld + (size_t)head * p.dv;
      for (int i = 0; i < p.dv; i += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(g0 + i));
    }
    float m = -1e30f, l = 0.f;                     // reference maximum (log2 units) and running denominator
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const uint32_t sb = j % NS, phs = (j / NS) & 1;
      if (!(ok = mbar_wait(b_sfull + 8 * sb, phs, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag))) break;
      tc_fence_after();
      const uint32_t ts = tmem_base + lane_addr + sb * BKV;
      float sv[BKV];
#pragma unroll
      for (int cb = 0; cb < BKV; cb += 32) tmem_ld_32x32(ts + cb, *reinterpret_cast<uint32_t(*)[32]>(&sv[cb]));
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(b_sempty + 8 * sb);
      const int key0 = first_key(j);
      bool capped = false;
      if constexpr (MODE == 2) {
        if (cap) softcap_run(sv, inv_cap, cap_c);
        capped = cap;
      }
      if (capped) {
      } else if (CAP) {
#pragma unroll
        for (int i = 0; i < BKV; ++i) sv[i] = cap_c * tanh_fast(sv[i] * inv_cap);
      } else if (early) {
#pragma unroll
        for (int i = 0; i < BKV; ++i) sv[i] *= qs * LOG2E;
      }
      // a tile needs per-key masking only at the diagonal, at the window edge and at the sequence end
      bool pooled = false;
      if constexpr (MODE == 2) {
        pooled = j < n_pool;
        if (pooled && key0 + BKV > blocks_seen(pos0)) {
#pragma unroll
          for (int i = 0; i < BKV; ++i) sv[i] = key0 + i < seen ? sv[i] : -INFINITY;
        }
      }
      if (pooled) {
      } else if ((key0 + BKV - 1 > pos0) || (p.window > 0 && key0 <= pos0 + FA_BQ - 1 - p.window) || (key0 + BKV > seq_len)) {
        if (key0 < p.keep_first) {
#pragma unroll
          for (int i = 0; i < BKV; ++i) {
            const int kpos = key0 + i;
            const bool keep = kpos <= qpos && kpos < seq_len && (kpos > qpos - p.window || kpos < p.keep_first);
            sv[i] = keep ? sv[i] : -INFINITY;
          }
        } else {
#pragma unroll
          for (int i = 0; i < BKV; ++i) {
            const int kpos = key0 + i;
            const bool keep = kpos <= qpos && kpos < seq_len && (p.window <= 0 || kpos > qpos - p.window);
            sv[i] = keep ? sv[i] : -INFINITY;
          }
        }
      }
      float tmax = sv[0];
#pragma unroll
      for (int i = 1; i < BKV; ++i) tmax = fmaxf(tmax, sv[i]);
      tmax *= c;                                   // c > 0
      // P(j) overwrites the shared tile PV(j-1) reads, and a rescale touches the accumulator PV(j-1) writes: both wait for it
      if (j > 0 && !(ok = mbar_wait(b_pvdone, (j - 1) & 1, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag))) break;
      // tcgen05.ld / tcgen05.st are warp-wide instructions: the decision to rescale is taken per warp, and a row whose own
      // maximum has not grown simply rescales by 1
      const bool grow = tmax > m + RESCALE_STEP || j == 0;
      const float m_new = grow ? fmaxf(m, tmax) : m;
      if (j > 0 && __any_sync(0xffffffffu, grow)) {
        const float alpha = ex2_fast(m - m_new);
        l *= alpha;
        tc_fence_after();
#pragma unroll 1
        for (int cb = 0; cb < DV; cb += 32) {
          uint32_t ov[32];
          tmem_ld_32x32(tmem_o + lane_addr + cb, ov);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * alpha);
          tmem_st_32x32(tmem_o + lane_addr + cb, ov);
        }
        tmem_st_wait();
      }
      m = m_new;
      float psum = 0.f;
      const float neg_m = -m;
#pragma unroll
      for (int cb = 0; cb < BKV; cb += 32) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float p0 = ex2_fast(fmaf(sv[cb + i], c, neg_m)), p1 = ex2_fast(fmaf(sv[cb + i + 1], c, neg_m));
          psum += p0 + p1;
          pk[i >> 1] = pack_bf16(p0, p1);
        }
        // 32 keys = 64 bytes = 4 chunks of this row, in atom (cb / 64), chunks (cb % 64) / 8 ..
        uint8_t* prow = smem + L::P_OFF + (cb >> 6) * (FA_BQ * 128);
        const int ch0 = (cb & 63) >> 3;
#pragma unroll
        for (int ch = 0; ch < 4; ++ch)
          *reinterpret_cast<uint4*>(prow + sw128_offset(r, ch0 + ch)) = make_uint4(pk[4 * ch], pk[4 * ch + 1], pk[4 * ch + 2], pk[4 * ch + 3]);
      }
      l += psum;
      tc_fence_before();            // a rescale's TMEM stores, before the MMA thread is told to accumulate into O again
      fence_proxy_async();          // the P tile, written through the generic proxy, before the MMA reads it
      __syncwarp();
      if (lane == 0) mbar_arrive(b_pfull);
    }
    const int dv = p.dv;
    const __nv_bfloat16* grow = p.gate && !p.gate_heads && row_ok ? p.gate + (size_t)(q_begin + t0 + r) * p.gate_ld + (size_t)head * dv : nullptr;
    // the first GPRE columns of the row's gate travel while the last PV runs (the score registers are free here)
    constexpr int GPRE = DV < 128 ? DV : 128;
    uint4 gpre[GPRE / 8];
    if (grow) {
#pragma unroll
      for (int i = 0; i < GPRE / 8; ++i)
        if (8 * i < dv) gpre[i] = __ldg(reinterpret_cast<const uint4*>(grow + 8 * i));
    }
    if (ok && n_tiles > 0) ok = mbar_wait(b_pvdone, (n_tiles - 1) & 1, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag);
    if (ok) {
      tc_fence_after();
      if (p.sinks) l += ex2_fast(p.sinks[head] * LOG2E - m);
      float inv = l > 0.f ? 1.f / l : 0.f;
      if (p.gate && p.gate_heads && row_ok) inv *= sigmoid_f<false>(__bfloat162float(p.gate[(size_t)(q_begin + t0 + r) * p.gate_ld + head]));
      __nv_bfloat16* orow = p.out + ((size_t)(q_begin + t0 + r) * p.n_q + head) * dv;
#pragma unroll
      for (int cb = 0; cb < DV; cb += 32) {
        if (cb >= dv) break;
        uint32_t ov[32];
        if (n_tiles > 0) {
          tmem_ld_32x32(tmem_o + lane_addr + cb, ov);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) ov[i] = 0u;
        }
        if (row_ok) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (cb + i >= dv) break;
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = __uint_as_float(ov[i + e]) * inv;
            if constexpr (MODE == 2) if (p.out_cos) {
              const size_t at = (size_t)min(qpos, p.out_n - 1) * p.out_half;
              const int m = (cb + i) / 2;
              float co[4], si[4];
              if ((p.out_half & 3) == 0 && m < p.out_half) {             // (rows of whole vectors)
                loadv<4>(p.out_cos + at + m, co);
                loadv<4>(p.out_sin + at + m, si);
              } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  co[e] = m + e < p.out_half ? __ldg(p.out_cos + at + m + e) : 1.f;
                  si[e] = m + e < p.out_half ? __ldg(p.out_sin + at + m + e) : 0.f;
                }
              }
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const float u = o[2 * e], v = o[2 * e + 1];
                o[2 * e] = u * co[e] + v * si[e];
                o[2 * e + 1] = v * co[e] - u * si[e];
              }
            }
            if (grow) {
              const uint4 g4 = cb + i < GPRE ? gpre[(cb + i) < GPRE ? (cb + i) / 8 : 0] : __ldg(reinterpret_cast<const uint4*>(grow + cb + i));
              const uint32_t gw[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                o[2 * e] *= sigmoid_f<false>(bf16_lo(gw[e]));
                o[2 * e + 1] *= sigmoid_f<false>(bf16_hi(gw[e]));
              }
            }
            *reinterpret_cast<uint4*>(orow + cb + i) = make_uint4(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]), pack_bf16(o[4], o[5]), pack_bf16(o[6], o[7]));
          }
        }
      }
    }
  }

  if (*abort_flag) {
    for (int i = 0; i < 200; ++i) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, L::TMEM_COLS);
}

template <int DK, int DV, bool CAP>
static int launch_fa(const void* q, const void* k_cache, const void* v_cache, const FaParams& p, int B, int Tq, int n_blocks, cudaStream_t st) {
  using L = FaCfg<DK, DV>;
  CUtensorMap tq, tk, tv;
  {
    uint64_t dims[3] = {(uint64_t)p.dk, (uint64_t)p.n_q, (uint64_t)Tq};
    uint64_t strides[2] = {(uint64_t)p.dk * 2, (uint64_t)p.q_ld * 2};
    uint32_t box[3] = {64, 1, FA_BQ};
    int r = make_tmap_bf16(&tq, q, 3, dims, strides, box, 1);
    if (r) return r;
  }
  {
    auto page_map = [&](CUtensorMap* m, const void* base, uint64_t d) {
      uint64_t dims[4] = {d, (uint64_t)FA_PAGE, (uint64_t)p.n_kv, (uint64_t)n_blocks};
      uint64_t strides[3] = {d * 2, d * 2 * FA_PAGE, d * 2 * FA_PAGE * p.n_kv};
      uint32_t box[4] = {64, (uint32_t)L::BKV, 1, 1};
      return make_tmap_bf16(m, base, 4, dims, strides, box, 1);
    };
    int r = page_map(&tk, k_cache, (uint64_t)p.dk);
    if (r) return r;
    r = page_map(&tv, v_cache, (uint64_t)p.dv);
    if (r) return r;
  }
  auto kern = fa_prefill_kernel<DK, DV, CAP, 0>;
  static DeviceOnce configured;
  if (configured.pending()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) return (int)e;
    configured.mark();
  }
  dim3 grid(B * p.max_q_tiles, p.n_q);
  kern<<<grid, 192, L::TOTAL, st>>>(tq, tk, tv, tq, tk, p);
  return (int)cudaGetLastError();
}

// Keys in two parts: `kv` holds expanded pages of 128 rows [n_q][dim] | [n_q][vdim] (kv_ld elements per row), `cache` the latent pages with the shared
// key part (rot elements from column `rank`, rows cache_ld elements apart).  Queries: rows of [n_q][dim | rot].
struct FaSplit { const void* kv; const void* cache; int dim, rot, rank, kv_ld, cache_ld, n_pages; };
template <int DK, int DV>
static int launch_fa_split(const void* q, const FaSplit& x, const FaParams& p, int B, int Tq, int n_blocks, cudaStream_t st) {
  using L = FaCfg<DK, DV>;
  using bf = __nv_bfloat16;
  CUtensorMap tq, tqr, tk, tkr, tv;
  int r = 0;
  auto q_map = [&](CUtensorMap* m, const void* base, int width) {
    uint64_t dims[3] = {(uint64_t)width, (uint64_t)p.n_q, (uint64_t)Tq};
    uint64_t strides[2] = {(uint64_t)(x.dim + x.rot) * 2, (uint64_t)p.q_ld * 2};
    uint32_t box[3] = {64, 1, FA_BQ};
    return make_tmap_bf16(m, base, 3, dims, strides, box, 1);
  };
  auto page_map = [&](CUtensorMap* m, const void* base, int width) {
    uint64_t dims[4] = {(uint64_t)width, (uint64_t)FA_PAGE, (uint64_t)p.n_q, (uint64_t)x.n_pages};
    uint64_t strides[3] = {(uint64_t)x.kv_ld * 2, (uint64_t)width * 2, (uint64_t)x.kv_ld * 2 * FA_PAGE};
    uint32_t box[4] = {64, (uint32_t)L::BKV, 1, 1};
    return make_tmap_bf16(m, base, 4, dims, strides, box, 1);
  };
  if ((r = q_map(&tq, q, x.dim)) || (r = q_map(&tqr, (const bf*)q + x.dim, x.rot))) return r;
  if ((r = page_map(&tk, x.kv, x.dim)) || (r = page_map(&tv, (const bf*)x.kv + (size_t)p.n_q * x.dim, p.dv))) return r;
  {
    uint64_t dims[3] = {(uint64_t)x.rot, (uint64_t)FA_PAGE, (uint64_t)n_blocks};
    uint64_t strides[2] = {(uint64_t)x.cache_ld * 2, (uint64_t)x.cache_ld * 2 * FA_PAGE};
    uint32_t box[3] = {64, (uint32_t)L::BKV, 1};
    if ((r = make_tmap_bf16(&tkr, (const bf*)x.cache + x.rank, 3, dims, strides, box, 1))) return r;
  }
  auto kern = fa_prefill_kernel<DK, DV, false, 1>;
  static DeviceOnce configured;
  if (configured.pending()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) return (int)e;
    configured.mark();
  }
  kern<<<dim3(B * p.max_q_tiles, p.n_q), 192, L::TOTAL, st>>>(tq, tk, tv, tqr, tkr, p);
  return (int)cudaGetLastError();
}

// MODE 2: the plain pages and, for the pooled blocks, dense pages [n_dense][n_kv][128][dk / dv].
struct FaPooled { const void* pk; const void* pv; int n_dense; };
template <int DK, int DV>
static int launch_fa_pooled(const void* q, const void* k_cache, const void* v_cache, const FaPooled& x, const FaPoolParams& p, int B, int Tq, int n_blocks,
                            cudaStream_t st) {
  using L = FaCfg<DK, DV>;
  CUtensorMap tq, tk, tv, tpk, tpv;
  uint64_t qd[3] = {(uint64_t)p.dk, (uint64_t)p.n_q, (uint64_t)Tq};
  uint64_t qs[2] = {(uint64_t)p.dk * 2, (uint64_t)p.q_ld * 2};
  uint32_t qb[3] = {64, 1, FA_BQ};
  auto page_map = [&](CUtensorMap* m, const void* base, uint64_t d, int pages) {
    uint64_t dims[4] = {d, (uint64_t)FA_PAGE, (uint64_t)p.n_kv, (uint64_t)pages};
    uint64_t strides[3] = {d * 2, d * 2 * FA_PAGE, d * 2 * FA_PAGE * p.n_kv};
    uint32_t box[4] = {64, (uint32_t)L::BKV, 1, 1};
    return make_tmap_bf16(m, base, 4, dims, strides, box, 1);
  };
  int r = 0;
  if ((r = make_tmap_bf16(&tq, q, 3, qd, qs, qb, 1)) || (r = page_map(&tk, k_cache, p.dk, n_blocks)) || (r = page_map(&tv, v_cache, p.dv, n_blocks))) return r;
  tpk = tk;
  tpv = tv;
  if (p.pool && ((r = page_map(&tpk, x.pk, p.dk, x.n_dense)) || (r = page_map(&tpv, x.pv, p.dv, x.n_dense)))) return r;
  auto kern = fa_prefill_kernel<DK, DV, false, 2>;
  static DeviceOnce configured;
  if (configured.pending()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) return (int)e;
    configured.mark();
  }
  kern<<<dim3(B * p.max_q_tiles, p.n_q), 192, L::TOTAL, st>>>(tq, tk, tv, tpk, tpv, p);
  return (int)cudaGetLastError();
}

// the instance whose tiles are the key / value widths rounded up to 64, 128 or 256 columns
static int dispatch_fa(const void* q, const void* k_cache, const void* v_cache, const FaParams& p, int B, int Tq, int n_blocks, cudaStream_t st) {
  if (p.dk < 8 || p.dv < 8 || p.dk > 256 || p.dv > 256 || p.dk % 8 || p.dv % 8 || p.q_ld % 8) return -112;
  if (p.gate && !p.gate_heads && (p.gate_ld % 8 || ((uintptr_t)p.gate & 15))) return -112;
  const int a = p.dk <= 64 ? 64 : p.dk <= 128 ? 128 : 256, b = p.dv <= 64 ? 64 : p.dv <= 128 ? 128 : 256;
#define MX_FA(DK_, DV_, CAP_) launch_fa<DK_, DV_, CAP_>(q, k_cache, v_cache, p, B, Tq, n_blocks, st)
  if (p.softcap > 0.f) {
    if (a != b) return -112;
    return a == 64 ? MX_FA(64, 64, true) : a == 128 ? MX_FA(128, 128, true) : MX_FA(256, 256, true);
  }
  switch (a * 1000 + b) {
    case 64064: return MX_FA(64, 64, false);
    case 64128: return MX_FA(64, 128, false);
    case 64256: return MX_FA(64, 256, false);
    case 128064: return MX_FA(128, 64, false);
    case 128128: return MX_FA(128, 128, false);
    case 128256: return MX_FA(128, 256, false);
    case 256064: return MX_FA(256, 64, false);
    case 256128: return MX_FA(256, 128, false);
    default: return MX_FA(256, 256, false);
  }
#undef MX_FA
}

}  // namespace mx

using namespace mx;

// Tensor-core prefill attention over pages of 128 tokens.  Queries: [Tq] rows of [n_q][dk], q_ld elements apart; out [Tq][n_q][dv];
// optional gate (rows of [n_q][dv], or with gate_heads of [n_q], gate_ld apart; out *= sigmoid(gate)) and per-position score factors q_scale
// [q_scale_n].  With a window the first keep_first keys of a sequence stay visible.  softcap > 0
// applies cap * tanh(score / cap) to the scaled scores.  n_blocks is the number of pages in the cache tensors (their leading dimension).
MX_HOST_API int mx_attention_prefill_tc_ext(const void* q, int q_ld, const void* k_cache, const void* v_cache, const int* block_table,
                                            const int* seq_lens, const int* cu_q, const float* sinks, const void* gate, int gate_ld,
                                            const float* q_scale, int q_scale_n, void* out, int B, int Tq, int max_q_len, int n_q, int n_kv, int dk,
                                            int dv, int max_blocks, int n_blocks, int block_size, int window, int keep_first, int gate_heads, float scale,
                                            float softcap, cudaStream_t st) {
  if (B <= 0 || Tq <= 0) return 0;
  if (block_size != FA_PAGE) return -110;
  if (n_q % n_kv) return -111;
  FaParams p;
  p.block_table = block_table; p.rot_table = nullptr; p.seq_lens = seq_lens; p.cu_q = cu_q; p.sinks = sinks; p.out = (__nv_bfloat16*)out;
  p.gate = (const __nv_bfloat16*)gate; p.gate_ld = gate ? gate_ld : 0; p.q_scale = q_scale; p.q_scale_n = q_scale_n;
  p.dk = dk; p.dv = dv; p.q_ld = q_ld; p.gate_heads = gate_heads; p.keep_first = window > 0 ? keep_first : 0;
  p.n_q = n_q; p.n_kv = n_kv; p.max_blocks = max_blocks; p.window = window; p.scale = scale; p.softcap = softcap;
  p.max_q_tiles = (max_q_len + FA_BQ - 1) / FA_BQ;
  p.status = status_word();
  return dispatch_fa(q, k_cache, v_cache, p, B, Tq, n_blocks, st);
}

// The plain form: dense queries, head_dim 64, 128 or 256 for keys and values.
MX_HOST_API int mx_attention_prefill_tc(const void* q, const void* k_cache, const void* v_cache, const int* block_table, const int* seq_lens,
                                        const int* cu_q, const float* sinks, void* out, int B, int Tq, int max_q_len, int n_q, int n_kv,
                                        int hd, int max_blocks, int n_blocks, int block_size, int window, float scale, float softcap,
                                        cudaStream_t st) {
  if (hd != 64 && hd != 128 && hd != 256) return -112;
  return mx_attention_prefill_tc_ext(q, n_q * hd, k_cache, v_cache, block_table, seq_lens, cu_q, sinks, nullptr, 0, nullptr, 0, out, B, Tq, max_q_len,
                                     n_q, n_kv, hd, hd, max_blocks, n_blocks, block_size, window, 0, 0, scale, softcap, st);
}

// Attention over a window and pooled blocks before it (MODE 2).  pk / pv: dense pages [B * pool_pages][n_kv][128][dk / dv] of the blocks of `pool` tokens
// that each sequence's last query sees, rows past them zero up to a whole page (pool 0: none); out_cos / out_sin [out_n][out_half] (or null): the output is
// turned by minus its position in neighbouring pairs, before the gate (rows of [n_q][dv]).  softcap 0: none.
MX_HOST_API int mx_attention_prefill_pooled(const void* q, int q_ld, const void* k_cache, const void* v_cache, const int* block_table, const int* seq_lens,
                                            const int* cu_q, const float* sinks, const void* gate, int gate_ld, void* out, int B, int Tq, int max_q_len, int n_q,
                                            int n_kv, int dk, int dv, int max_blocks, int n_blocks, int block_size, int window, float scale, float softcap,
                                            const void* pk, const void* pv, int pool, int pool_pages, const float* out_cos, const float* out_sin, int out_n,
                                            int out_half, cudaStream_t st) {
  if (B <= 0 || Tq <= 0) return 0;
  if (block_size != FA_PAGE) return -110;
  if (n_kv < 1 || n_q % n_kv) return -111;
  if (dk < 8 || dv < 8 || dk > 256 || dv > 256 || dk % 8 || dv % 8 || q_ld % 8 || out_half > dv / 2 || pool < 0 || (((uintptr_t)out_cos | (uintptr_t)out_sin) & 15)) return -112;
  if (pool && (window < 1 || !pk || !pv || pool_pages < 1)) return -112;
  if ((gate && (gate_ld % 8 || ((uintptr_t)gate & 15))) || (((uintptr_t)q | (uintptr_t)pk | (uintptr_t)pv) & 15)) return -112;
  FaPoolParams p;
  p.block_table = block_table; p.rot_table = nullptr; p.seq_lens = seq_lens; p.cu_q = cu_q; p.sinks = sinks; p.out = (__nv_bfloat16*)out;
  p.gate = (const __nv_bfloat16*)gate; p.gate_ld = gate ? gate_ld : 0; p.q_scale = nullptr; p.q_scale_n = 0; p.gate_heads = p.keep_first = 0;
  p.dk = dk; p.dv = dv; p.q_ld = q_ld; p.n_q = n_q; p.n_kv = n_kv; p.max_blocks = max_blocks; p.window = window; p.scale = scale; p.softcap = softcap;
  p.pool = pool; p.pool_pages = pool_pages; p.out_cos = out_cos; p.out_sin = out_sin; p.out_n = out_n; p.out_half = out_half;
  p.max_q_tiles = (max_q_len + FA_BQ - 1) / FA_BQ;
  p.status = status_word();
  const FaPooled x{pk, pv, B * pool_pages};
  const int a = dk <= 64 ? 64 : dk <= 128 ? 128 : 256, b = dv <= 64 ? 64 : dv <= 128 ? 128 : 256;
#define MX_FAP(DK_, DV_) launch_fa_pooled<DK_, DV_>(q, k_cache, v_cache, x, p, B, Tq, n_blocks, st)
  if (a == 64 && b == 64) return MX_FAP(64, 64);
  if (a == 64 && b == 128) return MX_FAP(64, 128);
  if (a == 128 && b == 64) return MX_FAP(128, 64);
  if (a == 128 && b == 128) return MX_FAP(128, 128);
  return MX_FAP(256, 256);
#undef MX_FAP
}

// Latent attention over expanded pages (see FaSplit).  q: [Tq] rows of [n_q][dim | rot], q_ld elements apart, rotated; kv: [n_pages * 128][n_q * (dim +
// vdim)], its pages listed by kv_table; cache: [n_blocks][128][rank + rot], its pages listed by block_table (both tables [B][max_blocks]); gate (rows of
// [n_q][vdim], gate_ld apart; out *= sigmoid(gate)); out [Tq][n_q][vdim].  Widths are multiples of 8: dim up to 192, rot up to 64, vdim up to 256.
MX_HOST_API int mx_attention_prefill_latent(const void* q, int q_ld, const void* kv, int n_pages, const int* kv_table, const void* cache, int n_blocks,
                                            const int* block_table, int max_blocks, const int* seq_lens, const int* cu_q, const void* gate, int gate_ld,
                                            void* out, int B, int Tq, int max_q_len, int n_q, int dim, int rot, int vdim, int rank, int window, float scale,
                                            cudaStream_t st) {
  if (B <= 0 || Tq <= 0) return 0;
  if (dim < 8 || dim > 192 || rot < 8 || rot > 64 || vdim < 8 || vdim > 256 || dim % 8 || rot % 8 || vdim % 8 || rank % 8 || q_ld % 8 || gate_ld % 8) return -112;
  if (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)cache | (uintptr_t)gate | (uintptr_t)out) & 15) return -112;
  FaParams p;
  p.block_table = kv_table; p.rot_table = block_table; p.seq_lens = seq_lens; p.cu_q = cu_q; p.sinks = nullptr; p.out = (__nv_bfloat16*)out;
  p.gate = (const __nv_bfloat16*)gate; p.gate_ld = gate ? gate_ld : 0; p.q_scale = nullptr; p.q_scale_n = 0; p.gate_heads = p.keep_first = 0;
  p.dk = dim + rot; p.dv = vdim; p.q_ld = q_ld; p.n_q = n_q; p.n_kv = n_q; p.max_blocks = max_blocks; p.window = window; p.scale = scale; p.softcap = 0.f;
  p.max_q_tiles = (max_q_len + FA_BQ - 1) / FA_BQ;
  p.status = status_word();
  FaSplit x{kv, cache, dim, rot, rank, n_q * (dim + vdim), rank + rot, n_pages};
#define MX_FAS(DK_, DV_) launch_fa_split<DK_, DV_>(q, x, p, B, Tq, n_blocks, st)
  const int a = dim <= 64 ? 0 : dim <= 128 ? 1 : 2, b = vdim <= 64 ? 0 : vdim <= 128 ? 1 : 2;
  switch (a * 3 + b) {
    case 0: return MX_FAS(128, 64);
    case 1: return MX_FAS(128, 128);
    case 2: return MX_FAS(128, 256);
    case 3: return MX_FAS(192, 64);
    case 4: return MX_FAS(192, 128);
    case 5: return MX_FAS(192, 256);
    case 6: return MX_FAS(256, 64);
    case 7: return MX_FAS(256, 128);
    default: return MX_FAS(256, 256);
  }
#undef MX_FAS
}
