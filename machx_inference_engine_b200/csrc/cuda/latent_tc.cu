// Attention in the latent space on the sm_100a tensor cores: decoding and short query segments of latent attention.  All heads share one cached row
// per token, [c | r]; a key is the whole row and its value is c, so a tile of rows is fetched once and multiplied twice.
//
// A CTA owns NR query rows (row = token of the segment x head) of one sequence and a range of its 128-row pages, and works on transposed tiles: the
// cached rows are the wide M operand, the few query rows the N operand --
//   S^T [128 keys][NR]      = tile [128][rank + rot]  Q^T            (K-major operands)
//   O^T [rank][NR]         += tile[:, :rank]^T [rank][128]  P^T      (the tile read MN-major: no transpose is made)
// so that 16 or 32 heads cost no padding to 128 rows, and the accumulator of a 512-wide latent takes 4 x NR TMEM columns.
//   warp 0  : TMA, with the next tile on its way into L2 while this one is loaded.  The rotated part of a tile goes to a ring of its own and is free again after S^T; the latent part travels in pairs of
//             64-column atoms (128 latent rows of O^T) through a ring whose slots are held until their O^T product is done
//   warp 1  : tcgen05.mma.  As much of the next tile's S^T as there is room for runs ahead of O^T of this tile
//   warps 2-5: one thread per key (TMEM lane).  Scores -> mask -> maximum over the keys by a transposing butterfly (lane n of every warp ends up
//             with row n), exchanged over the four warps; P is formed against a reference maximum that moves only when a row has grown by 2^8
//             (then O^T is rescaled in place) and stored as bf16 into the swizzled operand tile; denominators stay per thread until the end
// With several ranges per sequence each writes an un-normalised fp32 partial and (maximum, denominator) per row for the merge in attention.cu; a
// range without keys writes a zero weight only.  Every wait is bounded.
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

constexpr int LA_PAGE = 128;                  // cached rows per tile = page size
constexpr int LA_ATOM = LA_PAGE * 128;        // bytes of a 64-column atom of a tile
constexpr int LA_MAX_SLOTS = 8;

struct LaParams {
  const int* block_table;  // [B][max_blocks]
  const int* seq_lens;     // [B]
  const int* cu_q;         // [B+1]
  float* o_part;           // [splits][Tq * heads][rank]; null: one range per sequence, out is written
  float* ml_part;          // [splits][Tq * heads][2]
  __nv_bfloat16* out;      // [Tq * heads][rank]
  int heads, max_blocks, row_tiles, n_splits, window, rank;
  long long rows_all;      // Tq * heads
  int catoms, ratoms, nslots, rslots;
  int q_off, r_off, c_off, p_off, x_off;      // shared-memory offsets
  float scale_log2;
  int* status;
};

// a[] holds, in every lane, a value for each of 32 columns; lane n returns the reduction of column n over the lanes (a is used up)
template <bool MAX>
__device__ __forceinline__ float reduce_columns(float (&a)[32], int lane) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? a[i] : a[i + o], keep = up ? a[i + o] : a[i];
      const float got = __shfl_xor_sync(0xffffffffu, send, o);
      a[i] = MAX ? fmaxf(keep, got) : keep + got;
    }
  }
  return a[0];
}

__device__ __forceinline__ void la_tmem_st_32x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
        "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]),
        "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}
__device__ __forceinline__ float la_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// barrier of the four softmax warps that also tells all of them whether any has given up a wait
__device__ __forceinline__ bool la_bar_all(bool ok) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %1, 0;\n\t"
      "bar.red.and.pred q, 1, 128, p;\n\t"
      "selp.u32 %0, 1, 0, q;\n\t}\n"
      : "=r"(r)
      : "r"((uint32_t)ok)
      : "memory");
  return r != 0;
}

template <int NR>
__global__ void __launch_bounds__(192, 1)
latent_attn_kernel(const __grid_constant__ CUtensorMap tmap_qc, const __grid_constant__ CUtensorMap tmap_qr, const __grid_constant__ CUtensorMap tmap_c,
                   const __grid_constant__ CUtensorMap tmap_r, const LaParams p) {
  constexpr int G = NR / 32;                     // groups of 32 query rows
  constexpr int QATOM = NR * 128;                // bytes of a 64-column atom of the query rows
  constexpr float RESCALE_STEP = 8.f;
  pdl_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  const uint32_t sbase = smem_u32(smem);
  __shared__ uint64_t bars[2 * LA_MAX_SLOTS + 12];
  __shared__ uint32_t tmem_slot;
  __shared__ int abort_word;
  __shared__ int s_pos[NR];                      // position of every query row
  volatile int* abort_flag = &abort_word;
  const uint32_t b_qfull = smem_u32(bars), b_rfull = b_qfull + 8, b_rempty = b_rfull + 16, b_sfull = b_rempty + 16, b_sempty = b_sfull + 16;
  const uint32_t b_pfull = b_sempty + 16, b_pvdone = b_pfull + 8, b_cfull = b_pvdone + 8, b_cempty = b_cfull + 8 * LA_MAX_SLOTS;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.x / p.row_tiles, rt = blockIdx.x % p.row_tiles, split = blockIdx.y;
  const int q_begin = p.cu_q[b], q_len = p.cu_q[b + 1] - q_begin;
  const int r0 = rt * NR, total = q_len * p.heads;
  if (r0 >= total) return;                       // whole CTA leaves before any barrier / TMEM use
  const int rows = min(NR, total - r0);
  const int seq_len = p.seq_lens[b], first_pos = seq_len - q_len;
  const int pos_lo = first_pos + r0 / p.heads, pos_hi = first_pos + (r0 + rows - 1) / p.heads;
  const int kv_lo = p.window > 0 ? max(0, pos_lo - p.window + 1) : 0;
  const int all_lo = kv_lo / LA_PAGE, all_n = pos_hi / LA_PAGE - all_lo + 1;
  const int per = (all_n + p.n_splits - 1) / p.n_splits;
  const int tile_lo = all_lo + split * per, n_tiles = min(per, all_lo + all_n - tile_lo);
  const long long out_row0 = (long long)q_begin * p.heads + r0;
  if (n_tiles <= 0) {                            // (only with several ranges)
    pdl_wait();
    if (p.o_part && threadIdx.x < rows) {
      float* ml = p.ml_part + ((long long)split * p.rows_all + out_row0 + threadIdx.x) * 2;
      ml[0] = -1e30f; ml[1] = 0.f;
    }
    return;
  }
  const int catoms = p.catoms, ratoms = p.ratoms, cpairs = (catoms + 1) / 2, nslots = p.nslots, rslots = p.rslots;

  if (threadIdx.x == 0) {
    mbar_init(b_qfull, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(b_rfull + 8 * s, 1); mbar_init(b_rempty + 8 * s, 1); mbar_init(b_sfull + 8 * s, 1); mbar_init(b_sempty + 8 * s, 4);
    }
    mbar_init(b_pfull, 4); mbar_init(b_pvdone, 1);
    for (int s = 0; s < LA_MAX_SLOTS; ++s) { mbar_init(b_cfull + 8 * s, 1); mbar_init(b_cempty + 8 * s, 1); }
    abort_word = 0;
    fence_mbar_init();
  }
  for (int i = threadIdx.x; i < NR; i += blockDim.x) s_pos[i] = first_pos + min(r0 + i, total - 1) / p.heads;
  uint32_t tmem_cols = 32;
  while (tmem_cols < (uint32_t)((2 + cpairs) * NR)) tmem_cols *= 2;
  if (warp == 1) { tmem_alloc(smem_u32(&tmem_slot), tmem_cols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_slot, tmem_o = tmem_base + 2 * NR;
  pdl_wait();                                    // queries and the newest cache rows come from the kernels before

  if (warp == 0) {
    if (lane == 0) {
      prefetch_tmap(&tmap_qc); prefetch_tmap(&tmap_qr); prefetch_tmap(&tmap_c); prefetch_tmap(&tmap_r);
      mbar_expect_tx(b_qfull, (catoms + ratoms) * QATOM);
      for (int a = 0; a < catoms; ++a) tma_load_2d(sbase + p.q_off + a * QATOM, &tmap_qc, b_qfull, a * 64, (int)out_row0);
      for (int a = 0; a < ratoms; ++a) tma_load_2d(sbase + p.q_off + (catoms + a) * QATOM, &tmap_qr, b_qfull, a * 64, (int)out_row0);
      bool ok = true;
      int it = 0;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int blk = p.block_table[(size_t)b * p.max_blocks + tile_lo + j];
        if (j + 1 < n_tiles) {
          const int nb = p.block_table[(size_t)b * p.max_blocks + tile_lo + j + 1];
          for (int a = 0; a < ratoms; ++a) tma_prefetch_3d(&tmap_r, a * 64, 0, nb);
          for (int a = 0; a < catoms; ++a) tma_prefetch_3d(&tmap_c, a * 64, 0, nb);
        }
        const int rs = j % rslots, rph = (j / rslots) & 1;
        if (!(ok = mbar_wait(b_rempty + 8 * rs, rph ^ 1, p.status, ERR_MBAR_TIMEOUT_PRODUCER, abort_flag))) break;
        mbar_expect_tx(b_rfull + 8 * rs, ratoms * LA_ATOM);
        for (int a = 0; a < ratoms; ++a) tma_load_3d(sbase + p.r_off + (rs * ratoms + a) * LA_ATOM, &tmap_r, b_rfull + 8 * rs, a * 64, 0, blk);
        for (int c = 0; c < cpairs; ++c, ++it) {
          const int s = it % nslots, ph = (it / nslots) & 1, na = min(2, catoms - 2 * c);
          if (!(ok = mbar_wait(b_cempty + 8 * s, ph ^ 1, p.status, ERR_MBAR_TIMEOUT_PRODUCER, abort_flag))) break;
          mbar_expect_tx(b_cfull + 8 * s, na * LA_ATOM);
          for (int a = 0; a < na; ++a) tma_load_3d(sbase + p.c_off + (2 * s + a) * LA_ATOM, &tmap_c, b_cfull + 8 * s, (2 * c + a) * 64, 0, blk);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(128, NR, 0, 0);
      constexpr uint32_t idesc_o = umma_idesc_bf16(128, NR, 1, 0);       // A = tile^T is MN-major (latent columns contiguous)
      bool ok = mbar_wait(b_qfull, 0, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag);
      // descriptors differ in their address field only (16-byte units): the constant part is formed once
      const uint64_t dk = umma_desc_k_sw128(0), dm = umma_desc_mn_sw128(0, LA_ATOM, 1024);
      const uint64_t q0 = dk + ((sbase + p.q_off) >> 4), p0 = dk + ((sbase + p.p_off) >> 4), r_0 = dk + ((sbase + p.r_off) >> 4);
      const uint64_t ck0 = dk + ((sbase + p.c_off) >> 4), cm0 = dm + ((sbase + p.c_off) >> 4);
      constexpr int A16 = LA_ATOM >> 4, Q16 = QATOM >> 4;
      auto atom = [&](uint32_t d, uint64_t tile, uint64_t q, bool acc) {
        umma_bf16(d, tile, q, idesc_s, acc);
#pragma unroll
        for (int kk = 1; kk < 4; ++kk) umma_bf16(d, tile + 2 * kk, q + 2 * kk, idesc_s, 1);
      };
      // latent pairs [c_lo, c_hi) of S^T(j); the first call of a tile (c_lo == 0) brings the rotated part, the last one hands S^T over
      auto issue_s = [&](int j, int c_lo, int c_hi) -> bool {
        const int sb = j & 1;
        const uint32_t d = tmem_base + sb * NR;
        if (c_lo == 0) {
          const int rs = j % rslots, rph = (j / rslots) & 1;
          if (!mbar_wait(b_sempty + 8 * sb, ((j >> 1) & 1) ^ 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag)) return false;
          if (!mbar_wait(b_rfull + 8 * rs, rph, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag)) return false;
          tc_fence_after();
          for (int a = 0; a < ratoms; ++a) atom(d, r_0 + (rs * ratoms + a) * A16, q0 + (catoms + a) * Q16, a != 0);
          umma_commit(b_rempty + 8 * rs);
        }
        for (int c = c_lo; c < c_hi; ++c) {
          const int it = j * cpairs + c, s = it % nslots, ph = (it / nslots) & 1;
          if (!mbar_wait(b_cfull + 8 * s, ph, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag)) return false;
          tc_fence_after();
          atom(d, ck0 + 2 * s * A16, q0 + 2 * c * Q16, true);
          if (2 * c + 1 < catoms) atom(d, ck0 + (2 * s + 1) * A16, q0 + (2 * c + 1) * Q16, true);
        }
        if (c_hi == cpairs) umma_commit(b_sfull + 8 * sb);
        return true;
      };
      const int early = min(cpairs, nslots - cpairs);      // pairs of the next tile that fit beside this tile
      if (ok) ok = issue_s(0, 0, cpairs);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (early > 0 && j + 1 < n_tiles && !(ok = issue_s(j + 1, 0, early))) break;
        if (!(ok = mbar_wait(b_pfull, j & 1, p.status, ERR_MBAR_TIMEOUT_MMA, abort_flag))) break;
        tc_fence_after();
        for (int c = 0; c < cpairs; ++c) {
          const int s = (j * cpairs + c) % nslots;
          const uint64_t va = cm0 + 2 * s * A16;
          const uint32_t d = tmem_o + c * NR;
          umma_bf16(d, va, p0, idesc_o, j != 0);
#pragma unroll
          for (int kk = 1; kk < LA_PAGE / 16; ++kk) umma_bf16(d, va + kk * 128, p0 + (kk >> 2) * Q16 + (kk & 3) * 2, idesc_o, 1);
          umma_commit(b_cempty + 8 * s);
        }
        umma_commit(b_pvdone);
        if (early < cpairs && j + 1 < n_tiles && !(ok = issue_s(j + 1, early, cpairs))) break;
      }
    }
  } else {
    // ------------------------------------------------ softmax, one thread per key
    const int q4 = warp & 3, key = q4 * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    float* s_max = reinterpret_cast<float*>(smem + p.x_off);             // [2][4][NR] per-warp maxima, then sums
    float* s_ref = s_max + 8 * NR + q4 * 2 * NR;                          // this warp's copy: [NR] reference maxima, [NR] factors
    const int chunk = (key & 63) >> 3;
    uint8_t* pbase = smem + p.p_off + (key >> 6) * QATOM + (key & 7) * 2;
    float m[G], l[NR];                                                     // m: row 32 g + lane
#pragma unroll
    for (int g = 0; g < G; ++g) m[g] = -1e30f;
#pragma unroll
    for (int n = 0; n < NR; ++n) l[n] = 0.f;
    bool ok = true, left = false;                  // left: the four warps gave up together
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j & 1;
      float* wmax = s_max + sb * 4 * NR;
      float v[NR];
      if (ok) ok = __all_sync(0xffffffffu, mbar_wait(b_sfull + 8 * sb, (j >> 1) & 1, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag));
      if (ok) {
        tc_fence_after();
#pragma unroll
        for (int g = 0; g < G; ++g) tmem_ld_32x32(tmem_base + lane_addr + sb * NR + 32 * g, *reinterpret_cast<uint32_t(*)[32]>(&v[32 * g]));
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(b_sempty + 8 * sb);
        const int k0 = (tile_lo + j) * LA_PAGE, kpos = k0 + key;
#pragma unroll
        for (int n = 0; n < NR; ++n) v[n] *= p.scale_log2;
        if (k0 + LA_PAGE - 1 > pos_lo || (p.window > 0 && k0 <= pos_hi - p.window)) {       // the diagonal or a window's edge crosses the tile
#pragma unroll
          for (int n = 0; n < NR; ++n) {
            const int qpos = s_pos[n];
            v[n] = (kpos <= qpos && (p.window <= 0 || kpos > qpos - p.window)) ? v[n] : -INFINITY;
          }
        }
#pragma unroll
        for (int g = 0; g < G; ++g) {
          float a[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) a[i] = v[32 * g + i];
          wmax[q4 * NR + 32 * g + lane] = reduce_columns<true>(a, lane);
        }
      }
      if (!la_bar_all(ok)) { ok = false; left = true; break; }
      bool grew = false;
#pragma unroll
      for (int g = 0; g < G; ++g) {
        const float* w4 = wmax + 32 * g + lane;
        const float tmax = fmaxf(fmaxf(w4[0], w4[NR]), fmaxf(w4[2 * NR], w4[3 * NR]));
        const bool up = j == 0 || tmax > m[g] + RESCALE_STEP;
        const float mn = up ? fmaxf(m[g], tmax) : m[g];
        s_ref[32 * g + lane] = mn;
        s_ref[NR + 32 * g + lane] = la_ex2(m[g] - mn);
        m[g] = mn;
        grew |= up;
      }
      const bool rescale = j > 0 && __any_sync(0xffffffffu, grew);       // the same in every warp: all saw the same maxima
      __syncwarp();
      // P(j) overwrites the operand tile that O^T(j-1) reads, and a rescale touches what it writes: both wait for it
      if (j > 0) ok = __all_sync(0xffffffffu, mbar_wait(b_pvdone, (j - 1) & 1, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag));
      if (!ok) continue;                           // the next barrier tells the others
      if (rescale) {
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < cpairs; ++c) {
#pragma unroll
          for (int g = 0; g < G; ++g) {
            uint32_t ov[32];
            tmem_ld_32x32(tmem_o + lane_addr + c * NR + 32 * g, ov);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * s_ref[NR + 32 * g + i]);
            la_tmem_st_32x32(tmem_o + lane_addr + c * NR + 32 * g, ov);
          }
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
#pragma unroll
        for (int n = 0; n < NR; ++n) l[n] *= s_ref[NR + n];
      }
#pragma unroll
      for (int n = 0; n < NR; n += 4) {
        const float4 ref = *reinterpret_cast<const float4*>(s_ref + n);
        const float e[4] = {la_ex2(v[n] - ref.x), la_ex2(v[n + 1] - ref.y), la_ex2(v[n + 2] - ref.z), la_ex2(v[n + 3] - ref.w)};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          l[n + i] += e[i];
          *reinterpret_cast<__nv_bfloat16*>(pbase + sw128_offset(n + i, chunk)) = __float2bfloat16(e[i]);
        }
      }
      tc_fence_before();            // a rescale's TMEM stores, before the MMA thread accumulates into O^T again
      fence_proxy_async();          // P, written through the generic proxy, before the MMA reads it
      __syncwarp();
      if (lane == 0) mbar_arrive(b_pfull);
    }
    // denominators: over the lanes of a warp, then over the warps.  The sums go to the half of the exchange buffer that the last tile left alone
    float* wsum = s_max + (n_tiles & 1) * 4 * NR;
#pragma unroll
    for (int g = 0; g < G; ++g) {
      float a[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) a[i] = l[32 * g + i];
      wsum[q4 * NR + 32 * g + lane] = reduce_columns<false>(a, lane);
    }
    if (!left) ok = la_bar_all(ok);
#pragma unroll
    for (int g = 0; g < G; ++g) {
      const float* w4 = wsum + 32 * g + lane;
      const float L = (w4[0] + w4[NR]) + (w4[2 * NR] + w4[3 * NR]);
      s_ref[32 * g + lane] = p.o_part ? 1.f : (L > 0.f ? 1.f / L : 0.f);
      if (p.o_part && q4 == 0 && 32 * g + lane < rows) {
        float* ml = p.ml_part + ((long long)split * p.rows_all + out_row0 + 32 * g + lane) * 2;
        ml[0] = m[g] * 0.6931471805599453f;      // natural units
        ml[1] = L;
      }
    }
    __syncwarp();
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(b_pvdone, (n_tiles - 1) & 1, p.status, ERR_MBAR_TIMEOUT_SOFTMAX, abort_flag));
    if (ok) {
      tc_fence_after();
      for (int c = 0; c < cpairs; ++c) {
        const int d = c * 128 + key;               // latent element of this thread
#pragma unroll
        for (int g = 0; g < G; ++g) {
          uint32_t ov[32];
          tmem_ld_32x32(tmem_o + lane_addr + c * NR + 32 * g, ov);
          tmem_ld_wait();
          if (d < p.rank) {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const int n = 32 * g + i;
              if (n < rows) {
                const float o = __uint_as_float(ov[i]) * s_ref[n];
                if (p.o_part) p.o_part[((long long)split * p.rows_all + out_row0 + n) * p.rank + d] = o;
                else p.out[(out_row0 + n) * p.rank + d] = __float2bfloat16(o);
              }
            }
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
  if (warp == 1) tmem_dealloc(tmem_base, tmem_cols);
}

constexpr int LA_SMEM = 227 * 1024 - 1024;         // dynamic bytes: 227 KB less the static words

// Shared-memory plan for NR query rows; false when the shape does not fit.
static bool la_plan(LaParams& p, int nr, int& smem) {
  constexpr int LIMIT = LA_SMEM - 1024;
  const int cpairs = (p.catoms + 1) / 2;
  if ((2 + cpairs) * nr > 512) return false;
  const int q = (p.catoms + p.ratoms) * nr * 128, pb = 2 * nr * 128, x = 16 * nr * 4;
  for (p.rslots = 2; p.rslots >= 1; --p.rslots) {
    const int left = LIMIT - q - pb - x - p.rslots * p.ratoms * LA_ATOM;
    p.nslots = left / (2 * LA_ATOM);
    if (p.nslots > 2 * cpairs) p.nslots = 2 * cpairs;
    if (p.nslots > LA_MAX_SLOTS) p.nslots = LA_MAX_SLOTS;
    if (p.nslots >= cpairs + (p.rslots == 2 ? 1 : 0) || (p.rslots == 1 && p.nslots >= cpairs)) break;
  }
  if (p.rslots < 1) return false;
  p.q_off = 0;
  p.r_off = q;
  p.c_off = p.r_off + p.rslots * p.ratoms * LA_ATOM;
  p.p_off = p.c_off + p.nslots * 2 * LA_ATOM;
  p.x_off = p.p_off + pb;
  smem = p.x_off + x + 1024;
  return true;
}

template <int NR>
static int launch_latent(const void* q, const void* cache, LaParams& p, int smem, int rot, int B, int n_blocks, cudaStream_t st) {
  using bf = __nv_bfloat16;
  const int width = p.rank + rot;
  CUtensorMap qc, qr, tc, tr;
  auto q_map = [&](CUtensorMap* m, const void* base, int w) {
    uint64_t dims[2] = {(uint64_t)w, (uint64_t)p.rows_all};
    uint64_t strides[1] = {(uint64_t)width * 2};
    uint32_t box[2] = {64, NR};
    return make_tmap_bf16(m, base, 2, dims, strides, box, 1);
  };
  auto page_map = [&](CUtensorMap* m, const void* base, int w) {
    uint64_t dims[3] = {(uint64_t)w, (uint64_t)LA_PAGE, (uint64_t)n_blocks};
    uint64_t strides[2] = {(uint64_t)width * 2, (uint64_t)width * 2 * LA_PAGE};
    uint32_t box[3] = {64, LA_PAGE, 1};
    return make_tmap_bf16(m, base, 3, dims, strides, box, 1);
  };
  int r;
  if ((r = q_map(&qc, q, p.rank)) || (r = q_map(&qr, (const bf*)q + p.rank, rot))) return r;
  if ((r = page_map(&tc, cache, p.rank)) || (r = page_map(&tr, (const bf*)cache + p.rank, rot))) return r;
  auto kern = latent_attn_kernel<NR>;
  static DeviceOnce configured;
  if (configured.pending()) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LA_SMEM);
    if (e != cudaSuccess) return (int)e;
    configured.mark();
  }
  launch_pdl(kern, dim3(B * p.row_tiles, p.n_splits), dim3(192), (size_t)smem, st, qc, qr, tc, tr, p);
  return (int)cudaGetLastError();
}

}  // namespace mx

using namespace mx;

// q bf16 [Tq][heads][rank + rot] (dense); cache bf16 [n_blocks][128][rank + rot]; rank and rot multiples of 8, rank at most 512.  n_splits == 1: out bf16
// [Tq][heads][rank]; otherwise partials for mx_attention_combine in o_part (n_splits * Tq * heads * rank floats) and ml_part (n_splits * Tq * heads * 2).
MX_HOST_API int mx_latent_attention(const void* q, const void* cache, int n_blocks, const int* block_table, int max_blocks, const int* seq_lens, const int* cu_q,
                                    void* out, float* o_part, float* ml_part, int B, int Tq, int max_q_len, int heads, int rank, int rot, int window, float scale,
                                    int n_splits, cudaStream_t st) {
  if (B <= 0 || Tq <= 0 || max_q_len <= 0) return 0;
  if (rank < 8 || rank > 512 || rot < 8 || rank % 8 || rot % 8 || heads < 1 || n_splits < 1 || (n_splits > 1 && (!o_part || !ml_part))) return -112;
  if (((uintptr_t)q | (uintptr_t)cache) & 15) return -112;
  LaParams p;
  p.block_table = block_table; p.seq_lens = seq_lens; p.cu_q = cu_q; p.out = (__nv_bfloat16*)out;
  p.o_part = n_splits > 1 ? o_part : nullptr; p.ml_part = n_splits > 1 ? ml_part : nullptr;
  p.heads = heads; p.max_blocks = max_blocks; p.n_splits = n_splits; p.window = window; p.rank = rank; p.rows_all = (long long)Tq * heads;
  p.catoms = (rank + 63) / 64; p.ratoms = (rot + 63) / 64;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = status_word();
  int smem = 0;
  const long long rows = (long long)max_q_len * heads;
  const bool wide = rows > 32 && la_plan(p, 64, smem);
  if (!wide && !la_plan(p, 32, smem)) return -112;
  p.row_tiles = (int)((rows + (wide ? 63 : 31)) / (wide ? 64 : 32));
  return wide ? launch_latent<64>(q, cache, p, smem, rot, B, n_blocks, st) : launch_latent<32>(q, cache, p, smem, rot, B, n_blocks, st);
}
