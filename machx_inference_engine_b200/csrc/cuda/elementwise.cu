// Memory-bound glue kernels, each fusing what the reference ran as separate submits:
//   embed           : dequantising row gather into the fp32 residual stream
//   rmsnorm         : residual add (+bias) + RMSNorm (+ "1+w" form) -> bf16, one pass
//   qkv_post        : bias + per-head QK RMSNorm + NEOX RoPE (table driven: llama3 factors and
//                     YaRN are baked into the cos/sin tables) + Q|gate split + paged KV write
//   glu             : SwiGLU / clamped OAI SwiGLU / GeGLU over 16-column interleaved gate|up
//   group_norm      : RMSNorm over equal groups of a row; one pass norms a branch output, adds it to the residual and norms the
//                     sum for the next branch (norms on both sides of a sublayer)
//   dyt_norm        : residual add (branch output or expert combine, plus a vector of the row) + tanh(alpha x) w + b, one pass
//   kv_store        : K / V columns of a projection (own widths, no rotation) into the paged cache
//   gated_rmsnorm   : y = w * x / rms(x) * silu(z) per head (DeltaNet output norm)
//   misc            : sigmoid gate multiply, scaled add, casts
// Reference parity: src/ops/elementwise.cpp:29-786, src/ops/embedding.cpp:45-206,
// src/core/kv_cache.cpp:107-133, src/ops/deltanet.cpp:41-81.
#include "act.cuh"
#include "common.cuh"
#include "dequant.cuh"
#include "host_util.h"

namespace mx {

// ------------------------------------------------------------------ embed
template <int FMT>
__global__ void embed_kernel(WeightRef w, const int* __restrict__ ids, float* __restrict__ out, int H, int vocab, float scale) {
  pdl_prologue();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const RowPtrs rp = row_ptrs<FMT>(w, id, H);
  for (int kb = threadIdx.x; kb < H / 32; kb += blockDim.x) {
    float v[32];
    decode32_f32<FMT>(rp, kb, v);
    float4* o = reinterpret_cast<float4*>(out + (size_t)t * H + kb * 32);
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i] = make_float4(v[4 * i] * scale, v[4 * i + 1] * scale, v[4 * i + 2] * scale, v[4 * i + 3] * scale);
  }
}

// ------------------------------------------------------------------ rmsnorm
// x (fp32, [T,H]) += delta (bf16 or fp32, optional) + dbias (optional); out = norm(x) * w.
// delta_scale multiplies delta (Granite residual scale).  If out_f32 != null the normalised row
// is also written in fp32 (final norm feeding an fp32 consumer).
template <typename DT>
__global__ void __launch_bounds__(256) rmsnorm_kernel(float* __restrict__ x, const DT* __restrict__ delta, const float* __restrict__ dbias,
                                                      const float* __restrict__ w, __nv_bfloat16* __restrict__ out, float eps, int H,
                                                      int one_plus_w, float delta_scale, int write_x) {
  pdl_prologue();
  const int t = blockIdx.x;
  float* xr = x + (size_t)t * H;
  __shared__ float red[8];
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    float4 v = *reinterpret_cast<const float4*>(xr + i);
    if (delta) {
      float d0, d1, d2, d3;
      if constexpr (sizeof(DT) == 2) {
        const uint2 dv = *reinterpret_cast<const uint2*>(delta + (size_t)t * H + i);
        d0 = bf16_lo(dv.x); d1 = bf16_hi(dv.x); d2 = bf16_lo(dv.y); d3 = bf16_hi(dv.y);
      } else {
        const float4 dv = *reinterpret_cast<const float4*>(delta + (size_t)t * H + i);
        d0 = dv.x; d1 = dv.y; d2 = dv.z; d3 = dv.w;
      }
      if (dbias) { d0 += dbias[i]; d1 += dbias[i + 1]; d2 += dbias[i + 2]; d3 += dbias[i + 3]; }
      v.x += d0 * delta_scale; v.y += d1 * delta_scale; v.z += d2 * delta_scale; v.w += d3 * delta_scale;
      if (write_x) *reinterpret_cast<float4*>(xr + i) = v;
    }
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  if (threadIdx.x < 32) {
    float v = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.f;
    v = warp_sum(v);
    if (threadIdx.x == 0) red[0] = rsqrtf(v / H + eps);
  }
  __syncthreads();
  const float inv = red[0];
  if (!out) return;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    // when the sum was not written back (write_x == 0 with delta) recompute it
    float4 v = *reinterpret_cast<const float4*>(xr + i);
    if (delta && !write_x) {
      float d0, d1, d2, d3;
      if constexpr (sizeof(DT) == 2) {
        const uint2 dv = *reinterpret_cast<const uint2*>(delta + (size_t)t * H + i);
        d0 = bf16_lo(dv.x); d1 = bf16_hi(dv.x); d2 = bf16_lo(dv.y); d3 = bf16_hi(dv.y);
      } else {
        const float4 dv = *reinterpret_cast<const float4*>(delta + (size_t)t * H + i);
        d0 = dv.x; d1 = dv.y; d2 = dv.z; d3 = dv.w;
      }
      if (dbias) { d0 += dbias[i]; d1 += dbias[i + 1]; d2 += dbias[i + 2]; d3 += dbias[i + 3]; }
      v.x += d0 * delta_scale; v.y += d1 * delta_scale; v.z += d2 * delta_scale; v.w += d3 * delta_scale;
    }
    float4 g = *reinterpret_cast<const float4*>(w + i);
    if (one_plus_w) { g.x += 1.f; g.y += 1.f; g.z += 1.f; g.w += 1.f; }
    uint2 o;
    o.x = pack_bf16(v.x * inv * g.x, v.y * inv * g.y);
    o.y = pack_bf16(v.z * inv * g.z, v.w * inv * g.w);
    *reinterpret_cast<uint2*>(out + (size_t)t * H + i) = o;
  }
}

// Residual add + RMSNorm whose delta is the expert combine: delta[t] = sum_k cw[t,k] * yp[pair_to_packed[t*K+k]] (slot order,
// pairs with a negative position contribute nothing), so that the weighted sum of the expert outputs never exists as a tensor.
__global__ void __launch_bounds__(256) rmsnorm_combine_kernel(float* __restrict__ x, const __nv_bfloat16* __restrict__ yp, const int* __restrict__ pair_to_packed,
                                                              const float* __restrict__ cw, int K, const float* __restrict__ w,
                                                              __nv_bfloat16* __restrict__ out, float eps, int H, int one_plus_w, float delta_scale) {
  pdl_prologue();
  const int t = blockIdx.x;
  float* xr = x + (size_t)t * H;
  __shared__ float red[8];
  __shared__ int s_pos[32];
  __shared__ float s_w[32];
  if (threadIdx.x < K) {
    s_pos[threadIdx.x] = pair_to_packed[(size_t)t * K + threadIdx.x];
    s_w[threadIdx.x] = cw[(size_t)t * K + threadIdx.x];
  }
  __syncthreads();
  float ss = 0.f;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    float4 v = *reinterpret_cast<const float4*>(xr + i);
    float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < K; ++k) {
      const int pos = s_pos[k];
      if (pos < 0) continue;
      const uint2 yv = *reinterpret_cast<const uint2*>(yp + (size_t)pos * H + i);
      const float ww = s_w[k];
      d.x = fmaf(ww, bf16_lo(yv.x), d.x); d.y = fmaf(ww, bf16_hi(yv.x), d.y);
      d.z = fmaf(ww, bf16_lo(yv.y), d.z); d.w = fmaf(ww, bf16_hi(yv.y), d.w);
    }
    v.x += d.x * delta_scale; v.y += d.y * delta_scale; v.z += d.z * delta_scale; v.w += d.w * delta_scale;
    *reinterpret_cast<float4*>(xr + i) = v;
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  if (threadIdx.x < 32) {
    float v = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.f;
    v = warp_sum(v);
    if (threadIdx.x == 0) red[0] = rsqrtf(v / H + eps);
  }
  __syncthreads();
  const float inv = red[0];
  if (!out) return;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    const float4 v = *reinterpret_cast<const float4*>(xr + i);
    float4 g = *reinterpret_cast<const float4*>(w + i);
    if (one_plus_w) { g.x += 1.f; g.y += 1.f; g.z += 1.f; g.w += 1.f; }
    *reinterpret_cast<uint2*>(out + (size_t)t * H + i) = make_uint2(pack_bf16(v.x * inv * g.x, v.y * inv * g.y), pack_bf16(v.z * inv * g.z, v.w * inv * g.w));
  }
}

// ------------------------------------------------------------------ group_norm
// A row of H elements is `groups` equal parts, each normalised by its own root mean square.  In one pass over a row:
//   x  (fp32 residual) = (FRESH ? 0 : x) + norm(delta) * delta_w      (delta null: x is only read)
//   out               = norm(x) * w                                   (out null: skipped)
// Rows have ld elements (ld >= H, multiple of 4); columns H.. are padding: written as zeros in out (and in x when it starts fresh).
// A team of `wpg` warps owns one (row, group); a CTA holds 8 / wpg teams, which work on consecutive groups and never wait for each other.
struct GroupNormParams {
  float* x;
  const void* delta;
  const float* delta_w;
  const float* w;
  void* out;
  float eps;
  int T, H, ld, groups, gs, wpg, fresh;   // gs = H / groups
};
constexpr int GN_WARPS = 8;
constexpr int GN_LANE_MAX = 16;          // elements of a group that a lane holds, before the team gets more warps

// sum over the warps of a team (a team of several warps meets at its own named barrier)
__device__ __forceinline__ float team_sum(float v, float* red, int warp, int wpg) {
  v = warp_sum(v);
  if (wpg == 1) return v;
  const int team = warp / wpg, first = team * wpg;
  asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "r"(wpg * 32) : "memory");     // readers of the previous use are done
  if ((threadIdx.x & 31) == 0) red[warp] = v;
  asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "r"(wpg * 32) : "memory");
  float t = 0.f;
  for (int i = 0; i < wpg; ++i) t += red[first + i];
  return t;
}

// V elements per access; NV > 0: a lane keeps its NV pieces of x in registers; NV == 0: any size, x is re-read
template <typename DT, typename OT, int V, int NV>
__global__ void __launch_bounds__(GN_WARPS * 32) group_norm_kernel(const GroupNormParams p) {
  pdl_prologue();
  __shared__ float red[GN_WARPS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wpg = p.wpg;
  const unsigned unit = blockIdx.x * (GN_WARPS / wpg) + warp / wpg;      // (T * groups fits 32 bits: checked by the host)
  if (unit >= (unsigned)p.T * p.groups) return;            // a whole team leaves
  const unsigned t = unit / (unsigned)p.groups;
  const int g = (int)(unit - t * p.groups);
  const size_t row = (size_t)t * p.ld;
  float* xr = p.x + row;
  const DT* dr = reinterpret_cast<const DT*>(p.delta) + row;
  OT* orow = reinterpret_cast<OT*>(p.out) + row;
  const int first = (warp % wpg) * 32 + lane, step = wpg * 32, n = p.gs / V, base = g * p.gs;
  const float inv_n = 1.f / (float)p.gs;
  {
    if constexpr (NV > 0) {
      float xv[NV][V];
      float ss = 0.f;
      if (p.delta) {
        float dv[NV][V];
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const int i = first + j * step;
          if (i < n) {
            loadv<V>(dr + base + i * V, dv[j]);
            if (!p.fresh) loadv<V>(xr + base + i * V, xv[j]);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(dv[j][e], dv[j][e], ss);
          }
        }
        const float dinv = rsqrtf(team_sum(ss, red, warp, wpg) * inv_n + p.eps);
        ss = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const int i = first + j * step;
          if (i < n) {
            float wv[V];
            loadv<V>(p.delta_w + base + i * V, wv);
#pragma unroll
            for (int e = 0; e < V; ++e) {
              const float add = dv[j][e] * dinv * wv[e];
              xv[j][e] = p.fresh ? add : xv[j][e] + add;
              ss = fmaf(xv[j][e], xv[j][e], ss);
            }
            storev<V>(xr + base + i * V, xv[j]);
          }
        }
      } else {
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const int i = first + j * step;
          if (i < n) {
            loadv<V>(xr + base + i * V, xv[j]);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(xv[j][e], xv[j][e], ss);
          }
        }
      }
      if (p.out) {
        const float inv = rsqrtf(team_sum(ss, red, warp, wpg) * inv_n + p.eps);
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          const int i = first + j * step;
          if (i < n) {
            float wv[V];
            loadv<V>(p.w + base + i * V, wv);
#pragma unroll
            for (int e = 0; e < V; ++e) wv[e] *= xv[j][e] * inv;
            storev<V>(orow + base + i * V, wv);
          }
        }
      }
    } else {
      float ss = 0.f;
      if (p.delta) {
        for (int i = first; i < n; i += step) {
          float dv[V];
          loadv<V>(dr + base + i * V, dv);
#pragma unroll
          for (int e = 0; e < V; ++e) ss = fmaf(dv[e], dv[e], ss);
        }
        const float dinv = rsqrtf(team_sum(ss, red, warp, wpg) * inv_n + p.eps);
        ss = 0.f;
        for (int i = first; i < n; i += step) {
          float dv[V], wv[V], xv[V];
          loadv<V>(dr + base + i * V, dv);
          loadv<V>(p.delta_w + base + i * V, wv);
          if (!p.fresh) loadv<V>(xr + base + i * V, xv);
#pragma unroll
          for (int e = 0; e < V; ++e) {
            const float add = dv[e] * dinv * wv[e];
            xv[e] = p.fresh ? add : xv[e] + add;
            ss = fmaf(xv[e], xv[e], ss);
          }
          storev<V>(xr + base + i * V, xv);
        }
      } else {
        for (int i = first; i < n; i += step) {
          float xv[V];
          loadv<V>(xr + base + i * V, xv);
#pragma unroll
          for (int e = 0; e < V; ++e) ss = fmaf(xv[e], xv[e], ss);
        }
      }
      if (p.out) {
        const float inv = rsqrtf(team_sum(ss, red, warp, wpg) * inv_n + p.eps);
        for (int i = first; i < n; i += step) {           // a lane reads back the elements it wrote itself
          float xv[V], wv[V];
          loadv<V>(xr + base + i * V, xv);
          loadv<V>(p.w + base + i * V, wv);
#pragma unroll
          for (int e = 0; e < V; ++e) wv[e] *= xv[e] * inv;
          storev<V>(orow + base + i * V, wv);
        }
      }
    }
  }
  if (g == p.groups - 1)
    for (int i = p.H + first; i < p.ld; i += step) {
      if (p.out) orow[i] = from_f32<OT>(0.f);
      if (p.fresh) xr[i] = 0.f;
    }
}

// ------------------------------------------------------------------ sublayer_norm
// Norms on a sublayer's output.  In one pass over a row, the branch d formed as it is read:
//   x (fp32 residual) += norm(d) * delta_w          (delta_w null: += d; KIND 0: x is only read)
//   out                = x, or norm(x) * w when w is given   (out null: skipped)
// d: a row (KIND 1); the sum of the rows pos[t * K + k] of a, k < K, each times pw[t * K + k] when there are weights, and of row t of b when there is one,
// times the sigmoid of b_gate[t * b_gate_ld] when there is a gate (KIND 2: a token's experts and the expert that every token uses); the mean of norm(a) * a_w and norm(b) * b_w (KIND 3: two mixers side by side).
// Rows have ld elements (a multiple of 4) of which the first H count; the others are zero in a, b and the weights and stay zero.
// A team of `wpg` warps owns a row and keeps NV pieces of four elements per lane; NV == 0: any width, memory is read again.
struct SublayerNormParams {
  float* x;
  const void* a;
  const void* b;
  const int* pos;
  const float* pw;
  const float* b_gate;
  const float* a_w;
  const float* b_w;
  const float* delta_w;
  const float* w;
  void* out;
  float eps, inv_h;
  int T, ld, K, wpg, b_gate_ld;
  long long out_ld;
};

template <int KIND, typename DT, typename OT, int NV>
__global__ void __launch_bounds__(GN_WARPS * 32) sublayer_norm_kernel(const SublayerNormParams p) {
  pdl_prologue();
  __shared__ float red[GN_WARPS], red2[GN_WARPS];
  constexpr int N = NV > 0 ? NV : 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wpg = p.wpg;
  const int t = blockIdx.x * (GN_WARPS / wpg) + warp / wpg;
  if (t >= p.T) return;                                  // a whole team leaves
  const size_t row = (size_t)t * p.ld;
  float* xr = p.x + row;
  const DT* ar = reinterpret_cast<const DT*>(p.a) + row;
  const DT* br = reinterpret_cast<const DT*>(p.b) + row;
  OT* orow = reinterpret_cast<OT*>(p.out) + t * p.out_ld;
  const int first = ((warp % wpg) * 32 + lane) * 4, step = wpg * 128;
  const float b_factor = KIND == 2 && p.b && p.b_gate ? sigmoid_f<sizeof(DT) == 4>(p.b_gate[(size_t)t * p.b_gate_ld]) : 1.f;
  float x[N][4], d[N][4], e2[KIND == 3 ? N : 1][4];

  auto fetch = [&](int c, float (&dv)[4], float (&ev)[4]) {
    if constexpr (KIND == 1) loadv<4>(ar + c, dv);
    if constexpr (KIND == 2) {
      if (p.b) loadv<4>(br + c, dv);
      else dv[0] = dv[1] = dv[2] = dv[3] = 0.f;
      if (p.b_gate) {
#pragma unroll
        for (int e = 0; e < 4; ++e) dv[e] *= b_factor;
      }
      for (int k = 0; k < p.K; ++k) {
        float v[4];
        loadv<4>(reinterpret_cast<const DT*>(p.a) + (size_t)p.pos[(size_t)t * p.K + k] * p.ld + c, v);
        const float w = p.pw ? p.pw[(size_t)t * p.K + k] : 1.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) dv[e] = fmaf(w, v[e], dv[e]);
      }
    }
    if constexpr (KIND == 3) { loadv<4>(ar + c, dv); loadv<4>(br + c, ev); }
  };
  auto mean = [&](int c, float (&dv)[4], const float (&ev)[4], float ia, float ib) {
    float wa[4], wb[4];
    loadv<4>(p.a_w + c, wa);
    loadv<4>(p.b_w + c, wb);
#pragma unroll
    for (int e = 0; e < 4; ++e) dv[e] = 0.5f * (dv[e] * ia * wa[e] + ev[e] * ib * wb[e]);
  };
  auto square = [](const float (&v)[4], float s) {
#pragma unroll
    for (int e = 0; e < 4; ++e) s = fmaf(v[e], v[e], s);
    return s;
  };
  // every piece of the row that this lane owns: body(column, index of its registers)
  auto each = [&](auto&& body) {
    if constexpr (NV > 0) {
#pragma unroll
      for (int j = 0; j < NV; ++j)
        if (first + j * step < p.ld) body(first + j * step, j);
    } else {
      for (int c = first; c < p.ld; c += step) body(c, 0);
    }
  };
  float ia = 0.f, ib = 0.f, ss = 0.f;
  if constexpr (KIND != 0) {
    float sa = 0.f, sb = 0.f;
    each([&](int c, int j) {
      if (NV > 0) loadv<4>(xr + c, x[j]);
      fetch(c, d[j], e2[KIND == 3 ? j : 0]);
      sa = square(d[j], sa);
      if (KIND == 3) sb = square(e2[KIND == 3 ? j : 0], sb);
    });
    if constexpr (KIND == 3) {
      ia = rsqrtf(team_sum(sa, red, warp, wpg) * p.inv_h + p.eps);
      ib = rsqrtf(team_sum(sb, red2, warp, wpg) * p.inv_h + p.eps);
      sa = 0.f;
      each([&](int c, int j) {
        if (NV == 0) fetch(c, d[j], e2[j]);
        mean(c, d[j], e2[j], ia, ib);
        sa = square(d[j], sa);
      });
    }
    const bool plain = p.delta_w == nullptr;
    const float dinv = plain ? 1.f : rsqrtf(team_sum(sa, red, warp, wpg) * p.inv_h + p.eps);
    each([&](int c, int j) {
      if (NV == 0) {
        loadv<4>(xr + c, x[j]);
        fetch(c, d[j], e2[KIND == 3 ? j : 0]);
        if constexpr (KIND == 3) mean(c, d[j], e2[j], ia, ib);
      }
      float wv[4] = {1.f, 1.f, 1.f, 1.f};
      if (!plain) loadv<4>(p.delta_w + c, wv);
#pragma unroll
      for (int e = 0; e < 4; ++e) x[j][e] = fmaf(d[j][e] * dinv, wv[e], x[j][e]);
      storev<4>(xr + c, x[j]);
      ss = square(x[j], ss);
    });
  } else {
    each([&](int c, int j) {
      loadv<4>(xr + c, x[j]);
      ss = square(x[j], ss);
    });
  }
  if (!p.out) return;
  const float inv = p.w ? rsqrtf(team_sum(ss, red2, warp, wpg) * p.inv_h + p.eps) : 1.f;
  each([&](int c, int j) {
    if (NV == 0) loadv<4>(xr + c, x[j]);                 // (a lane reads back what it wrote itself)
    float o[4] = {x[j][0], x[j][1], x[j][2], x[j][3]};
    if (p.w) {
      float wv[4];
      loadv<4>(p.w + c, wv);
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] *= inv * wv[e];
    }
    storev<4>(orow + c, o);
  });
}

// ------------------------------------------------------------------ dyt_norm
// A norm without statistics: every element on its own, so a thread needs no other thread.
//   x (fp32 residual) += delta + step;   out = tanh(alpha x) w + b
// delta: rows of DT (KIND 1), the weighted sum of expert outputs (KIND 2: rows pair_to_packed[t * K + k] of delta times cw[t * K + k]), or
// none (KIND 0).  Four columns per thread; ld is a multiple of 4; padded columns are zero in w, b, delta and step and stay zero.
struct DytParams {
  float* x;
  const void* delta;
  const int* pair_to_packed;
  const float* cw;
  const float* step;          // [ld] or null
  const float* w;
  const float* b;
  void* out;
  float alpha;
  int K, ld4;                 // ld4 = ld / 4
  long long n4;               // rows * ld4
};

template <int KIND, typename DT, typename OT>
__global__ void __launch_bounds__(256) dyt_norm_kernel(const DytParams p) {
  pdl_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= p.n4) return;
  const long long t = i / p.ld4;
  const int c = (int)(i - t * p.ld4) * 4;
  float x[4];
  loadv<4>(p.x + i * 4, x);
  if constexpr (KIND == 1) {
    float d[4];
    loadv<4>(reinterpret_cast<const DT*>(p.delta) + i * 4, d);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] += d[e];
  } else if constexpr (KIND == 2) {
    float a[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k = 0; k < p.K; ++k) {
      const int pos = p.pair_to_packed[t * p.K + k];
      if (pos < 0) continue;
      const float cw = p.cw[t * p.K + k];
      float d[4];
      loadv<4>(reinterpret_cast<const DT*>(p.delta) + (size_t)pos * (p.ld4 * 4) + c, d);
#pragma unroll
      for (int e = 0; e < 4; ++e) a[e] = fmaf(cw, d[e], a[e]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] += a[e];
  }
  if (p.step) {
    float s[4];
    loadv<4>(p.step + c, s);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[e] += s[e];
  }
  if (KIND != 0 || p.step) storev<4>(p.x + i * 4, x);
  if (!p.out) return;
  float w[4], b[4];
  loadv<4>(p.w + c, w);
  loadv<4>(p.b + c, b);
#pragma unroll
  for (int e = 0; e < 4; ++e) w[e] = fmaf(tanhf(p.alpha * x[e]), w[e], b[e]);
  storev<4>(reinterpret_cast<OT*>(p.out) + i * 4, w);
}

// ------------------------------------------------------------------ kv_store
// Columns of a projection row ([n_kv][dk] keys, [n_kv][dv] values; any row stride) -> paged cache rows, 16 bytes per thread.
__global__ void __launch_bounds__(256) kv_store_kernel(const uint4* __restrict__ k, const uint4* __restrict__ v, int k_ld, int v_ld,
                                                       const long long* __restrict__ slot_map, uint4* __restrict__ k_cache, uint4* __restrict__ v_cache,
                                                       int T, int n_kv, int pk, int pv, int block_size) {   // pk, pv: 16-byte pieces per row of a head
  pdl_prologue();
  const int per_tok = n_kv * (pk + pv);
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)T * per_tok) return;
  const int t = (int)(i / per_tok);
  int c = (int)(i - (long long)t * per_tok);
  const long long slot = slot_map[t];
  if (slot < 0) return;
  const long long blk = slot / block_size, off = slot % block_size;
  const bool is_v = c >= n_kv * pk;
  if (is_v) c -= n_kv * pk;
  const int per = is_v ? pv : pk, h = c / per, e = c - h * per;
  const size_t dst = ((size_t)(blk * n_kv + h) * block_size + off) * per + e;
  if (is_v) v_cache[dst] = v[(size_t)t * v_ld + c];
  else k_cache[dst] = k[(size_t)t * k_ld + c];
}

// ------------------------------------------------------------------ qkv_post
struct QkvPostParams {
  const __nv_bfloat16* qkv;   // [T][q_cols + 2*n_kv*hd]
  const float* bias;          // [q_cols + 2*n_kv*hd] or null
  const float* q_norm_w;      // [hd] or null
  const float* k_norm_w;      // [hd] or null
  const int* positions;       // [T]
  const float* rope_cos;      // [max_pos][n_rot/2]
  const float* rope_sin;
  const long long* slot_map;  // [T] slot = block*block_size + offset, <0: do not store
  __nv_bfloat16* q_out;       // [T][n_q][hd]
  __nv_bfloat16* gate_out;    // [T][n_q][hd] when q_gate != 0
  __nv_bfloat16* k_cache;     // [blocks][n_kv][block_size][hd]
  __nv_bfloat16* v_cache;
  float* k_scale;             // non-null: the caches hold int8, one fp32 scale per (block, kv head, token) row
  float* v_scale;
  int T, n_q, n_kv, hd, n_rot, block_size;
  int q_gate;                 // 1: q columns hold per-head [q(hd) | gate(hd)]
  int norm_one_plus_w;
  int v_norm;                 // 1: V rows get a weightless RMS norm (Gemma-4)
  float eps;
  int max_pos;
};

__global__ void __launch_bounds__(128) qkv_post_kernel(const QkvPostParams p) {
  pdl_prologue();
  __shared__ float sh[4][512];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads_total = p.n_q + 2 * p.n_kv;
  const int unit = blockIdx.x * 4 + warp;
  if (unit >= p.T * heads_total) return;
  const int t = unit / heads_total, h = unit % heads_total;
  const int hd = p.hd;
  const int q_stride = p.q_gate ? 2 * hd : hd;
  const int q_cols = p.n_q * q_stride;
  const int row_cols = q_cols + 2 * p.n_kv * hd;
  int kind, hh, col0;   // kind 0 q, 1 k, 2 v
  if (h < p.n_q) { kind = 0; hh = h; col0 = h * q_stride; }
  else if (h < p.n_q + p.n_kv) { kind = 1; hh = h - p.n_q; col0 = q_cols + hh * hd; }
  else { kind = 2; hh = h - p.n_q - p.n_kv; col0 = q_cols + p.n_kv * hd + hh * hd; }
  const __nv_bfloat16* src = p.qkv + (size_t)t * row_cols + col0;
  float* v = sh[warp];
  float ss = 0.f;
  for (int i = lane; i < hd; i += 32) {
    float x = __bfloat162float(src[i]);
    if (p.bias) x += p.bias[col0 + i];
    v[i] = x;
    ss += x * x;
  }
  if (kind == 0 && p.q_gate) {
    for (int i = lane; i < hd; i += 32) {
      float g = __bfloat162float(src[hd + i]);
      if (p.bias) g += p.bias[col0 + hd + i];
      p.gate_out[((size_t)t * p.n_q + hh) * hd + i] = __float2bfloat16(g);
    }
  }
  const float* nw = kind == 0 ? p.q_norm_w : (kind == 1 ? p.k_norm_w : nullptr);
  if (nw) {
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / hd + p.eps);
    for (int i = lane; i < hd; i += 32) v[i] = v[i] * inv * (p.norm_one_plus_w ? 1.f + nw[i] : nw[i]);
  } else if (kind == 2 && p.v_norm) {
    ss = warp_sum(ss);
    const float inv = rsqrtf(ss / hd + p.eps);
    for (int i = lane; i < hd; i += 32) v[i] *= inv;
  }
  __syncwarp();
  if (kind != 2 && p.n_rot > 0) {
    const int half = p.n_rot / 2;
    int pos = p.positions[t];
    pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
    const float* cs = p.rope_cos + (size_t)pos * half;
    const float* sn = p.rope_sin + (size_t)pos * half;
    for (int i = lane; i < half; i += 32) {
      const float a = v[i], b = v[i + half], c = cs[i], s = sn[i];
      v[i] = a * c - b * s;
      v[i + half] = a * s + b * c;
    }
    __syncwarp();
  }
  __nv_bfloat16* dst;
  if (kind == 0) dst = p.q_out + ((size_t)t * p.n_q + hh) * hd;
  else {
    const long long slot = p.slot_map[t];
    if (slot < 0) return;
    const long long blk = slot / p.block_size, off = slot % p.block_size;
    __nv_bfloat16* cache = kind == 1 ? p.k_cache : p.v_cache;
    const long long row = (blk * p.n_kv + hh) * p.block_size + off;
    if (p.k_scale) {          // symmetric int8 per row: scale = max|x| / 127
      float amax = 0.f;
      for (int i = lane; i < hd; i += 32) amax = fmaxf(amax, fabsf(v[i]));
      amax = warp_max(amax);
      const float sc = amax > 0.f ? amax / 127.f : 1.f, inv = 1.f / sc;
      int8_t* d8 = reinterpret_cast<int8_t*>(cache) + row * hd;
      for (int i = lane; i < hd; i += 32) d8[i] = (int8_t)max(-127, min(127, __float2int_rn(v[i] * inv)));
      if (lane == 0) (kind == 1 ? p.k_scale : p.v_scale)[row] = sc;
      return;
    }
    dst = cache + row * hd;
  }
  for (int i = lane; i < hd; i += 32) dst[i] = __float2bfloat16(v[i]);
}

// Prefill form of the same epilogue: one CTA per token.  The token's position, cache slot and rope row are fetched once (the
// rope row into shared memory) and the warps walk the token's heads, a lane holding HD / 32 consecutive elements of a head (one
// vector load) and reaching its rotation partner with one shuffle.  The per-head math is that of qkv_post_kernel; the host picks
// this form for batches of many tokens when n_rot / 2 is a multiple of the lane's element count (every model so far).
template <int HD>
__global__ void __launch_bounds__(128) qkv_post_token_kernel(const QkvPostParams p) {
  constexpr int EPL = HD / 32;                 // elements per lane
  pdl_prologue();
  __shared__ float s_cos[256], s_sin[256];
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int half = p.n_rot / 2;
  if (half > 0) {
    int pos = p.positions[t];
    pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      s_cos[i] = p.rope_cos[(size_t)pos * half + i];
      s_sin[i] = p.rope_sin[(size_t)pos * half + i];
    }
  }
  const long long slot = p.slot_map[t];
  __syncthreads();
  const int heads_total = p.n_q + 2 * p.n_kv;
  const int q_stride = p.q_gate ? 2 * HD : HD;
  const int q_cols = p.n_q * q_stride;
  const int row_cols = q_cols + 2 * p.n_kv * HD;
  const __nv_bfloat16* row = p.qkv + (size_t)t * row_cols;
  const int e0 = lane * EPL;                   // first element of this lane
  const int dl = half / EPL;                   // lane distance to the rotation partner
  for (int h = warp; h < heads_total; h += 4) {
    int kind, hh, col0;                        // kind 0 q, 1 k, 2 v
    if (h < p.n_q) { kind = 0; hh = h; col0 = h * q_stride; }
    else if (h < p.n_q + p.n_kv) { kind = 1; hh = h - p.n_q; col0 = q_cols + hh * HD; }
    else { kind = 2; hh = h - p.n_q - p.n_kv; col0 = q_cols + p.n_kv * HD + hh * HD; }
    if (kind != 0 && slot < 0) continue;       // this token's K/V rows are not stored
    float v[EPL];
    {
      uint32_t raw[EPL / 2];
      if constexpr (EPL == 2) raw[0] = *reinterpret_cast<const uint32_t*>(row + col0 + e0);
      else if constexpr (EPL == 4) { const uint2 r2 = *reinterpret_cast<const uint2*>(row + col0 + e0); raw[0] = r2.x; raw[1] = r2.y; }
      else {
#pragma unroll
        for (int c = 0; c < EPL / 8; ++c) {
          const uint4 r4 = *reinterpret_cast<const uint4*>(row + col0 + e0 + 8 * c);
          raw[4 * c] = r4.x; raw[4 * c + 1] = r4.y; raw[4 * c + 2] = r4.z; raw[4 * c + 3] = r4.w;
        }
      }
#pragma unroll
      for (int j = 0; j < EPL / 2; ++j) { v[2 * j] = bf16_lo(raw[j]); v[2 * j + 1] = bf16_hi(raw[j]); }
    }
    if (p.bias) {
#pragma unroll
      for (int j = 0; j < EPL; ++j) v[j] += p.bias[col0 + e0 + j];
    }
    if (kind == 0 && p.q_gate) {
#pragma unroll
      for (int j = 0; j < EPL; ++j) {
        float g = __bfloat162float(row[col0 + HD + e0 + j]);
        if (p.bias) g += p.bias[col0 + HD + e0 + j];
        p.gate_out[((size_t)t * p.n_q + hh) * HD + e0 + j] = __float2bfloat16(g);
      }
    }
    const float* nw = kind == 0 ? p.q_norm_w : (kind == 1 ? p.k_norm_w : nullptr);
    if (nw || (kind == 2 && p.v_norm)) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < EPL; ++j) ss += v[j] * v[j];
      const float inv = rsqrtf(warp_sum(ss) / HD + p.eps);
#pragma unroll
      for (int j = 0; j < EPL; ++j) v[j] *= nw ? inv * (p.norm_one_plus_w ? 1.f + nw[e0 + j] : nw[e0 + j]) : inv;
    }
    if (kind != 2 && half > 0) {
      const bool lo = e0 < half, in = e0 < p.n_rot;
#pragma unroll
      for (int j = 0; j < EPL; ++j) {
        const float other = __shfl_xor_sync(0xffffffffu, v[j], dl);
        if (in) {
          const int f = (lo ? e0 : e0 - half) + j;
          v[j] = lo ? v[j] * s_cos[f] - other * s_sin[f] : other * s_sin[f] + v[j] * s_cos[f];
        }
      }
    }
    if (kind == 0) {
      __nv_bfloat16* dst = p.q_out + ((size_t)t * p.n_q + hh) * HD + e0;
#pragma unroll
      for (int j = 0; j < EPL; j += 2) *reinterpret_cast<uint32_t*>(dst + j) = pack_bf16(v[j], v[j + 1]);
      continue;
    }
    const long long blk = slot / p.block_size, off = slot % p.block_size;
    const long long crow = (blk * p.n_kv + hh) * p.block_size + off;
    __nv_bfloat16* cache = kind == 1 ? p.k_cache : p.v_cache;
    if (p.k_scale) {          // symmetric int8 per row: scale = max|x| / 127
      float amax = 0.f;
#pragma unroll
      for (int j = 0; j < EPL; ++j) amax = fmaxf(amax, fabsf(v[j]));
      amax = warp_max(amax);
      const float sc = amax > 0.f ? amax / 127.f : 1.f, inv = 1.f / sc;
      int8_t* d8 = reinterpret_cast<int8_t*>(cache) + crow * HD + e0;
#pragma unroll
      for (int j = 0; j < EPL; ++j) d8[j] = (int8_t)max(-127, min(127, __float2int_rn(v[j] * inv)));
      if (lane == 0) (kind == 1 ? p.k_scale : p.v_scale)[crow] = sc;
    } else {
      __nv_bfloat16* dst = cache + crow * HD + e0;
#pragma unroll
      for (int j = 0; j < EPL; j += 2) *reinterpret_cast<uint32_t*>(dst + j) = pack_bf16(v[j], v[j + 1]);
    }
  }
}

// ------------------------------------------------------------------ qk_post
// Head epilogue of attention whose values are its projected keys: per-head RMS norm with a weight, rotation of the first `rot` elements (interleaved pairs or
// half splits), optional RMS norm without a weight behind it; queries in place, keys and raw keys (the values) into the cache pages.  A warp holds a head, a
// lane groups of G consecutive elements of it, group g at g * 32 G.
struct QkPostParams {
  void* q;                     // row t of head h at t * q_ld + h * dp
  const void* k;
  const float* q_norm;         // [dp] or null
  const float* k_norm;
  const int* positions;        // [T]
  const float* rope_cos;       // [max_pos][rot / 2]
  const float* rope_sin;
  const long long* slot_map;   // [T], < 0: no cache row
  void* k_cache;               // [blocks][n_kv][block_size][dp]
  void* v_cache;
  int q_ld, k_ld, T, n_q, n_kv, dp, dim, rot, interleaved, norm_after, block_size, max_pos, hpw;
  float eps;
  const float* q_scale;        // [n_q] factor on the finished queries of a head, or null
  // values of their own (null: the keys as they came are the values): row t of head h at t * v_ld + h * dv, turned in neighbouring pairs
  const void* v;
  const float* v_cos;          // [v_max_pos][v_half]
  const float* v_sin;
  int v_ld, dv, v_half, v_max_pos;
  // pooled blocks of a step with one token per sequence (null: none): layout as in pooled.cu
  void* pk;                    // [blocks][n_kv][pool_rows][dp]
  void* pv;
  const int* block_table;      // [T][max_blocks]
  int pool, pool_rows, window, max_blocks;
};
constexpr int QK_WARPS = 4;

template <int G, typename T> __device__ __forceinline__ void load_group(const T* p, float (&v)[G]) {
  if constexpr (G == 2) { const float2 a = load2(p); v[0] = a.x; v[1] = a.y; }
  else if constexpr (G == 4) loadv<4>(p, v);
  else { loadv<4>(p, *reinterpret_cast<float(*)[4]>(&v[0])); loadv<4>(p + 4, *reinterpret_cast<float(*)[4]>(&v[4])); }
}
template <int G, typename T> __device__ __forceinline__ void store_group(T* p, const float (&v)[G]) {
  if constexpr (G == 2) store2(p, v[0], v[1]);
  else if constexpr (G == 4) storev<4>(p, v);
  else { storev<4>(p, *reinterpret_cast<const float(*)[4]>(&v[0])); storev<4>(p + 4, *reinterpret_cast<const float(*)[4]>(&v[4])); }
}

// A warp takes `hpw` heads of one token (1 for few tokens; then the rotation's factors are fetched once per warp and the next head's row travels while
// this one is worked on).
template <typename T, int G, int NG>
__global__ void __launch_bounds__(QK_WARPS * 32) qk_post_kernel(const QkPostParams p) {
  pdl_prologue();
  __shared__ float sh[QK_WARPS][NG == 1 ? 32 * G : 32 * G * NG];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // units of a token: query and key heads, then value heads, then pooled rows
  const int qk_heads = p.n_q + p.n_kv, qk_units = (qk_heads + p.hpw - 1) / p.hpw, v_units = p.v ? (p.n_kv + p.hpw - 1) / p.hpw : 0;
  const int all = qk_units + v_units + (p.pk ? p.n_kv : 0);
  const long long unit = (long long)blockIdx.x * QK_WARPS + warp;
  if (unit >= (long long)p.T * all) return;
  const int t = (int)(unit / all);
  int h0 = (int)(unit - (long long)t * all);
  const long long slot = p.slot_map[t];
  if (h0 >= qk_units + v_units) {                                          // the block that this token is the first to see, if there is one
    const int h = h0 - qk_units - v_units, end = p.positions[t] + 1 - p.window, b = end / p.pool - 1;
    if (slot < 0 || end < p.pool || end % p.pool) return;
    const int* table = p.block_table + (size_t)t * p.max_blocks;
    const int page = (end - 1) / p.block_size;
    const size_t at = ((size_t)table[page] * p.n_kv + h) * p.pool_rows + (b - page * p.block_size / p.pool);
    for (int which = 0; which < 2; ++which) {
      const int width = which ? p.dv : p.dp;
      const T* cache = reinterpret_cast<const T*>(which ? p.v_cache : p.k_cache);
      T* out = reinterpret_cast<T*>(which ? p.pv : p.pk) + at * width;
      for (int c = lane * 4; c < width; c += 128) {
        float a[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
        for (int j = 0; j < p.pool; ++j) {
          const int i = b * p.pool + j;
          float v[4];
          loadv<4>(cache + (((size_t)table[i / p.block_size] * p.n_kv + h) * p.block_size + i % p.block_size) * width + c, v);
#pragma unroll
          for (int e = 0; e < 4; ++e) a[e] += v[e];
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) a[e] /= (float)p.pool;
        storev<4>(out + c, a);
      }
    }
    return;
  }
  const bool vals = h0 >= qk_units;
  if (vals) h0 -= qk_units;
  const int heads = vals ? p.n_kv : qk_heads, per_tok = vals ? v_units : qk_units;           // heads h0, h0 + per_tok, ...
  const int dp = vals ? p.dv : p.dp, half = vals ? p.v_half : p.rot / 2, rot = 2 * half, max_pos = vals ? p.v_max_pos : p.max_pos;
  const bool interleaved = vals || p.interleaved;
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= max_pos ? max_pos - 1 : pos);
  const float* cs = (vals ? p.v_cos : p.rope_cos) + (size_t)pos * half;
  const float* sn = (vals ? p.v_sin : p.rope_sin) + (size_t)pos * half;
  // element i turns into v_i c_i + v_partner s_i
  float c[NG][G], s[NG][G];
#pragma unroll
  for (int g = 0; g < NG; ++g)
#pragma unroll
    for (int e = 0; e < G; ++e) {
      const int i = (g * 32 + lane) * G + e;
      const bool first = interleaved ? !(i & 1) : i < half;
      const int f = interleaved ? i >> 1 : first ? i : i - half;
      c[g][e] = i < rot ? __ldg(cs + f) : 1.f;
      s[g][e] = i < rot ? (first ? -__ldg(sn + f) : __ldg(sn + f)) : 0.f;
    }
  const bool by_shuffle = NG == 1 && half % G == 0;                      // a lane's partners sit in one other lane
  const int partner = lane * G < half ? lane + half / G : lane - half / G;
  auto source = [&](int h) {
    return vals ? reinterpret_cast<const T*>(p.v) + (size_t)t * p.v_ld + (size_t)h * dp
           : h < p.n_q ? reinterpret_cast<const T*>(p.q) + (size_t)t * p.q_ld + (size_t)h * dp
                     : reinterpret_cast<const T*>(p.k) + (size_t)t * p.k_ld + (size_t)(h - p.n_q) * dp;
  };
  float next[NG][G];
  auto fetch = [&](int h) {
    const T* src = source(h);
#pragma unroll
    for (int g = 0; g < NG; ++g) {
      const int e0 = (g * 32 + lane) * G;
      if (e0 < dp) load_group<G>(src + e0, next[g]);
      else {
#pragma unroll
        for (int e = 0; e < G; ++e) next[g][e] = 0.f;
      }
    }
  };
  fetch(h0);
  for (int h = h0; h < heads; h += per_tok) {
    const bool is_q = !vals && h < p.n_q;
    if (!is_q && slot < 0) break;                                        // (key heads come last)
    const int kh = vals ? h : h - p.n_q;
    const long long crow = is_q ? 0 : (((slot / p.block_size) * p.n_kv + kh) * p.block_size + slot % p.block_size) * dp;
    float v[NG][G], ss = 0.f;
#pragma unroll
    for (int g = 0; g < NG; ++g) {
      const int e0 = (g * 32 + lane) * G;
#pragma unroll
      for (int e = 0; e < G; ++e) { v[g][e] = next[g][e]; ss = fmaf(v[g][e], v[g][e], ss); }
      if (!is_q && !p.v && e0 < dp) store_group<G>(reinterpret_cast<T*>(p.v_cache) + crow + e0, v[g]);
    }
    if (h + per_tok < heads) fetch(h + per_tok);
    const float* nw = vals ? nullptr : is_q ? p.q_norm : p.k_norm;
    if (nw) {
      const float inv = rsqrtf(warp_sum(ss) / (float)p.dim + p.eps);
#pragma unroll
      for (int g = 0; g < NG; ++g) {
        const int e0 = (g * 32 + lane) * G;
        if (e0 < dp) {
          float w[G];
          load_group<G>(nw + e0, w);
#pragma unroll
          for (int e = 0; e < G; ++e) v[g][e] *= inv * w[e];
        }
      }
    }
    if (interleaved) {
#pragma unroll
      for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int e = 0; e < G; e += 2) {
          const float a = v[g][e], b = v[g][e + 1];
          v[g][e] = fmaf(b, s[g][e], a * c[g][e]);
          v[g][e + 1] = fmaf(a, s[g][e + 1], b * c[g][e + 1]);
        }
    } else if (by_shuffle) {
#pragma unroll
      for (int e = 0; e < G; ++e) {
        const float o = __shfl_sync(0xffffffffu, v[0][e], partner & 31);
        v[0][e] = fmaf(o, s[0][e], v[0][e] * c[0][e]);
      }
    } else {
      float* buf = sh[warp];
      __syncwarp();
#pragma unroll
      for (int g = 0; g < NG; ++g) store_group<G>(buf + (g * 32 + lane) * G, v[g]);
      __syncwarp();
#pragma unroll
      for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int e = 0; e < G; ++e) {
          const int i = (g * 32 + lane) * G + e;
          if (i < rot) v[g][e] = fmaf(buf[i < half ? i + half : i - half], s[g][e], v[g][e] * c[g][e]);
        }
    }
    if (p.norm_after && !vals) {
      ss = 0.f;
#pragma unroll
      for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int e = 0; e < G; ++e) ss = fmaf(v[g][e], v[g][e], ss);
      const float inv = rsqrtf(warp_sum(ss) / (float)p.dim + p.eps);
#pragma unroll
      for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int e = 0; e < G; ++e) v[g][e] *= inv;
    }
    if (is_q && p.q_scale) {
      const float f = p.q_scale[h];
#pragma unroll
      for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int e = 0; e < G; ++e) v[g][e] *= f;
    }
    T* dst = is_q ? reinterpret_cast<T*>(p.q) + (size_t)t * p.q_ld + (size_t)h * dp : reinterpret_cast<T*>(vals ? p.v_cache : p.k_cache) + crow;
#pragma unroll
    for (int g = 0; g < NG; ++g) {
      const int e0 = (g * 32 + lane) * G;
      if (e0 < dp) store_group<G>(dst + e0, v[g]);
    }
  }
}

// The same for many tokens where nothing is normed and all rotations are of neighbouring pairs: a CTA per token, eight elements per thread and pass.
template <typename T>
__global__ void __launch_bounds__(256) qk_pairs_kernel(const QkPostParams p) {
  pdl_prologue();
  const int t = blockIdx.x, dp = p.dp, dv = p.dv;
  const int cq = p.n_q * dp / 8, ck = cq + p.n_kv * dp / 8, all = ck + p.n_kv * dv / 8;
  const long long slot = p.slot_map[t];
  const int pos = max(p.positions[t], 0);
  const size_t page = slot < 0 ? 0 : (size_t)(slot / p.block_size) * p.n_kv, off = slot < 0 ? 0 : (size_t)(slot % p.block_size);
  const size_t at = (size_t)min(pos, p.max_pos - 1) * (p.rot / 2), vat = (size_t)min(pos, p.v_max_pos - 1) * p.v_half;
#pragma unroll 2
  for (int i = threadIdx.x; i < all; i += 256) {
    const bool is_q = i < cq, is_v = i >= ck;
    if (!is_q && slot < 0) break;
    const int j = is_q ? i : is_v ? i - ck : i - cq, width = is_v ? dv : dp, h = j / (width / 8), c = (j - h * (width / 8)) * 8;
    const int half = is_v ? p.v_half : p.rot / 2, m = c / 2;
    const T* src = is_q ? reinterpret_cast<const T*>(p.q) + (size_t)t * p.q_ld : is_v ? reinterpret_cast<const T*>(p.v) + (size_t)t * p.v_ld
                                                                                      : reinterpret_cast<const T*>(p.k) + (size_t)t * p.k_ld;
    float v[8], co[4] = {1.f, 1.f, 1.f, 1.f}, si[4] = {0.f, 0.f, 0.f, 0.f};
    load_group<8>(src + (size_t)j * 8, v);
    if (m < half) {
      const float* cs = is_v ? p.v_cos + vat + m : p.rope_cos + at + m;
      const float* sn = is_v ? p.v_sin + vat + m : p.rope_sin + at + m;
      if ((half & 3) == 0) {
        loadv<4>(cs, co);
        loadv<4>(sn, si);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (m + e < half) { co[e] = __ldg(cs + e); si[e] = __ldg(sn + e); }
      }
    }
    const float f = is_q && p.q_scale ? p.q_scale[h] : 1.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float a = v[2 * e], b = v[2 * e + 1];
      v[2 * e] = fmaf(-b, si[e], a * co[e]) * f;
      v[2 * e + 1] = fmaf(a, si[e], b * co[e]) * f;
    }
    T* dst = is_q ? reinterpret_cast<T*>(p.q) + (size_t)t * p.q_ld + (size_t)j * 8
                  : reinterpret_cast<T*>(is_v ? p.v_cache : p.k_cache) + ((page + h) * p.block_size + off) * width + c;
    store_group<8>(dst, v);
  }
}

// ------------------------------------------------------------------ GLU over interleaved-16 columns
__device__ __forceinline__ float glu_act(int act, float g, float u, float alpha, float limit) {
  if (act == 1) return g / (1.f + __expf(-g)) * u;
  if (act == 2) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + __expf(-alpha * g)) * (u + 1.f);
  }
  const float t = tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g));
  return 0.5f * g * (1.f + t) * u;
}
// (fp32 rows: SwiGLU and its clamped form through the full-precision exponential)
__device__ __forceinline__ float glu_act_precise(int act, float g, float u, float alpha, float limit) {
  if (act == 2) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_f<true>(alpha * g) * (u + 1.f);
  }
  return act == 1 ? g * sigmoid_f<true>(g) * u : glu_act(act, g, u, alpha, limit);
}
__global__ void glu_f32_kernel(const float* __restrict__ in, float* __restrict__ out, long long total_out, int F, int act, float alpha, float limit) {
  pdl_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total_out) return;
  const long long t = i / F;
  const int f = (int)(i % F);
  const float* row = in + t * 2 * F;
  const int g = 32 * (f >> 4) + (f & 15);
  out[i] = glu_act_precise(act, row[g], row[g + 16], alpha, limit);
}
__global__ void glu_kernel(const __nv_bfloat16* __restrict__ in, __nv_bfloat16* __restrict__ out, long long total_out, int F, int act,
                           float alpha, float limit) {
  pdl_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total_out) return;
  const long long t = i / F;
  const int f = (int)(i % F);
  const __nv_bfloat16* row = in + t * 2 * F;
  const int g = 32 * (f >> 4) + (f & 15);
  out[i] = __float2bfloat16(glu_act(act, __bfloat162float(row[g]), __bfloat162float(row[g + 16]), alpha, limit));
}

// y[i] = x[i] * sigmoid(g[i])   (gated attention output, shared-expert gate uses the scalar form below)
__global__ void sigmoid_mul_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ g, __nv_bfloat16* __restrict__ y, long long n) {
  pdl_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) y[i] = __float2bfloat16(__bfloat162float(x[i]) / (1.f + __expf(-__bfloat162float(g[i]))));
}
// out[t][:] (fp32) += scale_t * src[t][:], scale_t = sigmoid(gate_logit[t]) if gate_logit else 1
__global__ void scaled_add_kernel(float* __restrict__ out, const __nv_bfloat16* __restrict__ src, const float* __restrict__ gate_logit, int H, long long n) {
  pdl_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float s = gate_logit ? 1.f / (1.f + __expf(-gate_logit[i / H])) : 1.f;
  out[i] += s * __bfloat162float(src[i]);
}
__global__ void cast_f32_bf16_kernel(const float* __restrict__ a, __nv_bfloat16* __restrict__ b, long long n) {
  pdl_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) b[i] = __float2bfloat16(a[i]);
}

// y[t,h,:] = w * x / rms(x) * silu(z)  over head_dim (one warp per (t,h))
__global__ void __launch_bounds__(128) gated_rmsnorm_kernel(const float* __restrict__ x, const __nv_bfloat16* __restrict__ z, const float* __restrict__ w,
                                                            __nv_bfloat16* __restrict__ y, int rows, int hd, float eps) {
  pdl_prologue();
  const int r = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const float* xr = x + (size_t)r * hd;
  float ss = 0.f;
  for (int i = lane; i < hd; i += 32) ss += xr[i] * xr[i];
  ss = warp_sum(ss);
  const float inv = rsqrtf(ss / hd + eps);
  for (int i = lane; i < hd; i += 32) {
    const float zz = __bfloat162float(z[(size_t)r * hd + i]);
    y[(size_t)r * hd + i] = __float2bfloat16(xr[i] * inv * w[i] * (zz / (1.f + __expf(-zz))));
  }
}

// Decoder probe: every 32-bit word of `in` (eight E2M1 codes) is decoded twice, with the byte-permute
// table path (bf16) and with the hardware conversion path (fp16); out[w][0..7] and out[w][8..15].
__global__ void e2m1_probe_kernel(const uint32_t* __restrict__ in, float* __restrict__ out, int n) {
  pdl_prologue();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  uint32_t a[4], b[4];
  e2m1x8_to_bf16x2(in[i], a);
  e2m1x8_to_f16x2(in[i], b);
  for (int j = 0; j < 4; ++j) {
    out[(size_t)i * 16 + 2 * j] = bf16_lo(a[j]);
    out[(size_t)i * 16 + 2 * j + 1] = bf16_hi(a[j]);
    const __half2 h = *reinterpret_cast<const __half2*>(&b[j]);
    out[(size_t)i * 16 + 8 + 2 * j] = __low2float(h);
    out[(size_t)i * 16 + 8 + 2 * j + 1] = __high2float(h);
  }
}

}  // namespace mx

using namespace mx;

MX_HOST_API int mx_e2m1_probe(const void* in, float* out, int n, cudaStream_t st) {
  if (n <= 0) return 0;
  launch_pdl(e2m1_probe_kernel, dim3((n + 127) / 128), dim3(128), 0, st, (const uint32_t*)in, out, n);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_embed(int wfmt, const void* w0, const void* w1, const void* w2, const void* w3, const int* ids, float* out, int T,
                         int H, int vocab, float scale, cudaStream_t st) {
  if (T <= 0) return 0;
  if (H % 32) return -102;
  WeightRef w{w0, w1, w2, w3};
  const int threads = 128;
  switch (wfmt) {
    case WF_BF16: launch_pdl(embed_kernel<WF_BF16>, dim3(T), dim3(threads), 0, st, w, ids, out, H, vocab, scale); break;
    case WF_Q8: launch_pdl(embed_kernel<WF_Q8>, dim3(T), dim3(threads), 0, st, w, ids, out, H, vocab, scale); break;
    case WF_Q4K: launch_pdl(embed_kernel<WF_Q4K>, dim3(T), dim3(threads), 0, st, w, ids, out, H, vocab, scale); break;
    case WF_Q6K: launch_pdl(embed_kernel<WF_Q6K>, dim3(T), dim3(threads), 0, st, w, ids, out, H, vocab, scale); break;
    case WF_MXFP4: launch_pdl(embed_kernel<WF_MXFP4>, dim3(T), dim3(threads), 0, st, w, ids, out, H, vocab, scale); break;
    default: return -100;
  }
  return (int)cudaGetLastError();
}

// delta_is_f32: 0 -> bf16 delta, 1 -> fp32 delta.  write_x: store x+delta back into x.
MX_HOST_API int mx_rmsnorm(float* x, const void* delta, int delta_is_f32, const float* dbias, const float* w, void* out_bf16, float eps,
                           int T, int H, int one_plus_w, float delta_scale, int write_x, cudaStream_t st) {
  if (T <= 0) return 0;
  if (H % 4) return -107;
  if (delta_is_f32) launch_pdl(rmsnorm_kernel<float>, dim3(T), dim3(256), 0, st, x, (const float*)delta, dbias, w, (__nv_bfloat16*)out_bf16, eps, H, one_plus_w, delta_scale, write_x);
  else launch_pdl(rmsnorm_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, st, x, (const __nv_bfloat16*)delta, dbias, w, (__nv_bfloat16*)out_bf16, eps, H, one_plus_w, delta_scale, write_x);
  return (int)cudaGetLastError();
}

// x[t] += delta_scale * sum_k cw[t,k] * yp[pair_to_packed[t*K+k]];  out = rmsnorm(x) * w   (K <= 32)
MX_HOST_API int mx_rmsnorm_combine(float* x, const void* yp, const int* pair_to_packed, const float* cw, int K, const float* w, void* out_bf16,
                                   float eps, int T, int H, int one_plus_w, float delta_scale, cudaStream_t st) {
  if (T <= 0) return 0;
  if (H % 4 || K > 32 || K < 1) return -107;
  launch_pdl(rmsnorm_combine_kernel, dim3(T), dim3(256), 0, st, x, (const __nv_bfloat16*)yp, pair_to_packed, cw, K, w, (__nv_bfloat16*)out_bf16, eps, H,
             one_plus_w, delta_scale);
  return (int)cudaGetLastError();
}

namespace mx {
template <typename DT, typename OT>
static int launch_group_norm(GroupNormParams p, cudaStream_t st) {
  const bool v4 = p.gs % 4 == 0;
  const long long units = (long long)p.T * p.groups;
  // warps per group: enough that a lane holds at most 16 elements, then more while the chip has room for them (4096 rows of 2 x 2048:
  // 37 us with 16 elements per lane, 49 with 8, 58 with 32)
  p.wpg = 1;
  while (p.wpg < GN_WARPS && (p.gs > 32 * p.wpg * GN_LANE_MAX || (units * p.wpg < 16ll * sm_count() && p.gs > 32 * p.wpg * 4))) p.wpg *= 2;
  const dim3 grid((unsigned)((units + GN_WARPS / p.wpg - 1) / (GN_WARPS / p.wpg))), block(GN_WARPS * 32);
  const int lanes = 32 * p.wpg, per_lane = v4 ? (p.gs / 4 + lanes - 1) / lanes : 0;
  if (v4 && per_lane <= 2) launch_pdl(group_norm_kernel<DT, OT, 4, 2>, grid, block, 0, st, p);
  else if (v4 && per_lane <= 4) launch_pdl(group_norm_kernel<DT, OT, 4, 4>, grid, block, 0, st, p);
  else if (v4 && per_lane <= 8) launch_pdl(group_norm_kernel<DT, OT, 4, 8>, grid, block, 0, st, p);
  else if (v4) launch_pdl(group_norm_kernel<DT, OT, 4, 0>, grid, block, 0, st, p);
  else launch_pdl(group_norm_kernel<DT, OT, 1, 0>, grid, block, 0, st, p);
  return (int)cudaGetLastError();
}
}  // namespace mx

// See group_norm_kernel.  x [T][ld] fp32; delta [T][ld] bf16 / fp32 or null; out [T][ld] bf16 / fp32 or null; delta_w, w fp32 [H].
MX_HOST_API int mx_group_norm(float* x, const void* delta, int delta_is_f32, const float* delta_w, const float* w, void* out, int out_is_f32,
                              float eps, int T, int H, int ld, int groups, int fresh, cudaStream_t st) {
  if (T <= 0) return 0;
  if (groups < 1 || H < groups || H % groups || ld < H || ld % 4 || (long long)T * groups > 0x7fffffffll) return -107;
  if ((delta && !delta_w) || (out && !w) || (fresh && !delta)) return -109;
  GroupNormParams p;
  p.x = x; p.delta = delta; p.delta_w = delta_w; p.w = w; p.out = out; p.eps = eps; p.H = H; p.ld = ld; p.groups = groups; p.gs = H / groups;
  p.T = T; p.fresh = fresh;
  if (delta_is_f32) return out_is_f32 ? launch_group_norm<float, float>(p, st) : launch_group_norm<float, __nv_bfloat16>(p, st);
  return out_is_f32 ? launch_group_norm<__nv_bfloat16, float>(p, st) : launch_group_norm<__nv_bfloat16, __nv_bfloat16>(p, st);
}

namespace mx {
template <int KIND, typename DT, typename OT>
static int launch_sublayer_norm(SublayerNormParams p, cudaStream_t st) {
  // enough warps per row that a lane holds at most 16 elements (32 with eight), then more while the chip has room for them
  p.wpg = 1;
  while (p.wpg < GN_WARPS && (p.ld > 512 * p.wpg || ((long long)p.T * p.wpg < 16ll * sm_count() && p.ld > 128 * p.wpg))) p.wpg *= 2;
  const dim3 grid((unsigned)((p.T + GN_WARPS / p.wpg - 1) / (GN_WARPS / p.wpg))), block(GN_WARPS * 32);
  const int pieces = (p.ld + 128 * p.wpg - 1) / (128 * p.wpg);
  if (pieces <= 2) launch_pdl(sublayer_norm_kernel<KIND, DT, OT, 2>, grid, block, 0, st, p);
  else if (pieces <= 4) launch_pdl(sublayer_norm_kernel<KIND, DT, OT, 4>, grid, block, 0, st, p);
  else if (pieces <= 8) launch_pdl(sublayer_norm_kernel<KIND, DT, OT, 8>, grid, block, 0, st, p);
  else launch_pdl(sublayer_norm_kernel<KIND, DT, OT, 0>, grid, block, 0, st, p);
  return (int)cudaGetLastError();
}
template <typename DT, typename OT>
static int dispatch_sublayer_norm(int kind, const SublayerNormParams& p, cudaStream_t st) {
  switch (kind) {
    case 0: return launch_sublayer_norm<0, DT, OT>(p, st);
    case 1: return launch_sublayer_norm<1, DT, OT>(p, st);
    case 2: return launch_sublayer_norm<2, DT, OT>(p, st);
    default: return launch_sublayer_norm<3, DT, OT>(p, st);
  }
}
}  // namespace mx

// See sublayer_norm_kernel.  x fp32 [T][ld]; kind 0 nothing, 1 a row of a, 2 rows pos[t][K] of a (+ row t of b), 3 the mean of a and b normed; a and b are
// bf16, or fp32 when out is (out null: elem_f32 names the dtype of a and b).  pw [T][K], b_gate (stride b_gate_ld): factors of kind 2, or null.  out: rows
// out_ld elements apart (a multiple of 4).
MX_HOST_API int mx_sublayer_norm(int kind, float* x, const void* a, const void* b, const int* pos, int K, const float* pw, const float* b_gate, int b_gate_ld,
                                 const float* a_w, const float* b_w, const float* delta_w, const float* w, void* out, long long out_ld, int elem_f32, float eps,
                                 int T, int H, int ld, cudaStream_t st) {
  if (T <= 0) return 0;
  if (H < 1 || ld < H || ld % 4 || kind < 0 || kind > 3 || out_ld % 4 || (out && out_ld < ld)) return -107;
  if ((kind && !a) || (kind == 3 && !delta_w) || (kind == 2 && (!pos || K < 1)) || (kind == 3 && (!b || !a_w || !b_w))) return -109;
  SublayerNormParams p;
  p.x = x; p.a = a; p.b = b; p.pos = pos; p.a_w = a_w; p.b_w = b_w; p.delta_w = delta_w; p.w = w; p.out = out; p.eps = eps; p.inv_h = 1.f / (float)H;
  p.T = T; p.ld = ld; p.K = K; p.pw = pw; p.b_gate = b_gate; p.b_gate_ld = b_gate_ld; p.out_ld = out_ld;
  return elem_f32 ? dispatch_sublayer_norm<float, float>(kind, p, st) : dispatch_sublayer_norm<__nv_bfloat16, __nv_bfloat16>(kind, p, st);
}

// See qk_post_kernel.  dp (the padded head width) a multiple of 8 up to 512, dim <= dp its live elements, rot <= dim even; the same of dv and 2 v_half.
MX_HOST_API int mx_qk_post(void* q, int q_ld, const void* k, int k_ld, const float* q_norm, const float* k_norm, const int* positions, const float* rope_cos,
                           const float* rope_sin, int max_pos, const long long* slot_map, void* k_cache, void* v_cache, int T, int n_q, int n_kv, int dp, int dim,
                           int rot, int interleaved, int norm_after, int block_size, float eps, int elem_f32, const float* q_scale, const void* v, int v_ld, int dv,
                           const float* v_cos, const float* v_sin, int v_half, int v_max_pos, void* pk, void* pv, const int* block_table, int max_blocks, int pool,
                           int pool_rows, int window, cudaStream_t st) {
  if (T <= 0) return 0;
  if (v && (dv < 8 || dv > 512 || dv % 8 || v_half < 0 || 2 * v_half > dv || v_ld % 8 || ((uintptr_t)v & 15))) return -108;
  if (pk && (!pv || !v || !block_table || pool < 1 || window < 1 || pool_rows < (block_size + pool - 1) / pool)) return -108;
  if (dp < 8 || dp > 512 || dp % 8 || dim < 1 || dim > dp || rot < 0 || rot > dim || rot % 2 || q_ld % 8 || k_ld % 8 || (((uintptr_t)q | (uintptr_t)k) & 15)) return -108;
  QkPostParams p;
  p.q = q; p.k = k; p.q_norm = q_norm; p.k_norm = k_norm; p.positions = positions; p.rope_cos = rope_cos; p.rope_sin = rope_sin; p.slot_map = slot_map;
  p.k_cache = k_cache; p.v_cache = v_cache; p.q_ld = q_ld; p.k_ld = k_ld; p.T = T; p.n_q = n_q; p.n_kv = n_kv; p.dp = dp; p.dim = dim; p.rot = rot;
  p.interleaved = interleaved; p.norm_after = norm_after; p.block_size = block_size; p.max_pos = max_pos; p.eps = eps;
  p.q_scale = q_scale; p.v = v; p.v_ld = v_ld; p.dv = v ? dv : dp; p.v_cos = v_cos; p.v_sin = v_sin; p.v_half = v_half; p.v_max_pos = v_max_pos;
  p.pk = pk; p.pv = pv; p.block_table = block_table; p.max_blocks = max_blocks; p.pool = pool; p.pool_rows = pool_rows; p.window = window;
  const int heads = n_q + n_kv;
  p.hpw = (long long)T * heads >= 64ll * 64 * sm_count() / 8 ? 8 : 1;    // (many tokens: the chip is full with fewer, longer warps)
  if (p.hpw > heads) p.hpw = heads;
  const long long units = (long long)T * ((heads + p.hpw - 1) / p.hpw + (v ? (n_kv + p.hpw - 1) / p.hpw : 0) + (pk ? n_kv : 0));
  const int wide = v && dv > dp ? dv : dp;
  if (v && T >= 128 && interleaved && !norm_after && !q_norm && !k_norm && !pk &&
      (((uintptr_t)rope_cos | (uintptr_t)rope_sin | (uintptr_t)v_cos | (uintptr_t)v_sin) & 15) == 0) {
    if (elem_f32) launch_pdl(qk_pairs_kernel<float>, dim3(T), dim3(256), 0, st, p);
    else launch_pdl(qk_pairs_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, st, p);
    return (int)cudaGetLastError();
  }
  const dim3 grid((unsigned)((units + QK_WARPS - 1) / QK_WARPS)), block(QK_WARPS * 32);
#define MX_QK(T_)   (wide <= 64 ? launch_pdl(qk_post_kernel<T_, 2, 1>, grid, block, 0, st, p) : wide <= 128 ? launch_pdl(qk_post_kernel<T_, 4, 1>, grid, block, 0, st, p)    : wide <= 256 ? launch_pdl(qk_post_kernel<T_, 8, 1>, grid, block, 0, st, p) : launch_pdl(qk_post_kernel<T_, 8, 2>, grid, block, 0, st, p))
  if (elem_f32) MX_QK(float); else MX_QK(__nv_bfloat16);
#undef MX_QK
  return (int)cudaGetLastError();
}

// See dyt_norm_kernel.  x [T][ld] fp32; delta (null: none) [T][ld], or with pair_to_packed [rows][ld] combined with cw [T][K]; step, w, b [ld];
// out (null: skipped) [T][ld].
MX_HOST_API int mx_dyt_norm(float* x, const void* delta, int delta_is_f32, const int* pair_to_packed, const float* cw, int K, const float* step,
                            float alpha, const float* w, const float* b, void* out, int out_is_f32, int T, int ld, cudaStream_t st) {
  if (T <= 0) return 0;
  if (ld < 4 || ld % 4 || (pair_to_packed && (!delta || K < 1))) return -107;
  if (out && (!w || !b)) return -109;
  DytParams p;
  p.x = x; p.delta = delta; p.pair_to_packed = pair_to_packed; p.cw = cw; p.step = step; p.w = w; p.b = b; p.out = out; p.alpha = alpha; p.K = K;
  p.ld4 = ld / 4; p.n4 = (long long)T * p.ld4;
  const dim3 grid((unsigned)((p.n4 + 255) / 256)), block(256);
  using bf = __nv_bfloat16;
#define MX_DYT(KIND_, DT_) \
  (out_is_f32 ? launch_pdl(dyt_norm_kernel<KIND_, DT_, float>, grid, block, 0, st, p) : launch_pdl(dyt_norm_kernel<KIND_, DT_, bf>, grid, block, 0, st, p))
  if (!delta) MX_DYT(0, float);
  else if (pair_to_packed) { if (delta_is_f32) MX_DYT(2, float); else MX_DYT(2, bf); }
  else { if (delta_is_f32) MX_DYT(1, float); else MX_DYT(1, bf); }
#undef MX_DYT
  return (int)cudaGetLastError();
}

// k / v: rows of n_kv * dk / n_kv * dv elements, k_ld / v_ld elements apart; elem_bytes 2 or 4; every row, head and stride a multiple of 16 bytes.
MX_HOST_API int mx_kv_store(const void* k, const void* v, int k_ld, int v_ld, const long long* slot_map, void* k_cache, void* v_cache, int T, int n_kv,
                            int dk, int dv, int block_size, int elem_bytes, cudaStream_t st) {
  if (T <= 0 || n_kv <= 0) return 0;
  const int pe = 16 / elem_bytes;
  if ((elem_bytes != 2 && elem_bytes != 4) || dk % pe || dv % pe || k_ld % pe || v_ld % pe) return -108;
  if (((uintptr_t)k | (uintptr_t)v | (uintptr_t)k_cache | (uintptr_t)v_cache) & 15) return -108;
  const long long n = (long long)T * n_kv * (dk / pe + dv / pe);
  launch_pdl(kv_store_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, (const uint4*)k, (const uint4*)v, k_ld / pe, v_ld / pe, slot_map,
             (uint4*)k_cache, (uint4*)v_cache, T, n_kv, dk / pe, dv / pe, block_size);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_qkv_post_kv8(const void* qkv, const float* bias, const float* q_norm_w, const float* k_norm_w, const int* positions,
                                const float* rope_cos, const float* rope_sin, const long long* slot_map, void* q_out, void* gate_out,
                                void* k_cache, void* v_cache, float* k_scale, float* v_scale, int T, int n_q, int n_kv, int hd, int n_rot,
                                int block_size, int q_gate, int norm_one_plus_w, float eps, int max_pos, cudaStream_t st);

MX_HOST_API int mx_qkv_post(const void* qkv, const float* bias, const float* q_norm_w, const float* k_norm_w, const int* positions,
                            const float* rope_cos, const float* rope_sin, const long long* slot_map, void* q_out, void* gate_out,
                            void* k_cache, void* v_cache, int T, int n_q, int n_kv, int hd, int n_rot, int block_size, int q_gate,
                            int norm_one_plus_w, float eps, int max_pos, cudaStream_t st) {
  return mx_qkv_post_kv8(qkv, bias, q_norm_w, k_norm_w, positions, rope_cos, rope_sin, slot_map, q_out, gate_out, k_cache, v_cache, nullptr,
                         nullptr, T, n_q, n_kv, hd, n_rot, block_size, q_gate, norm_one_plus_w, eps, max_pos, st);
}

// k_scale / v_scale non-null: k_cache / v_cache are int8 [blocks][n_kv][block_size][hd] and the rows are quantised on the way in.
MX_HOST_API int mx_qkv_post_kv8(const void* qkv, const float* bias, const float* q_norm_w, const float* k_norm_w, const int* positions,
                                const float* rope_cos, const float* rope_sin, const long long* slot_map, void* q_out, void* gate_out,
                                void* k_cache, void* v_cache, float* k_scale, float* v_scale, int T, int n_q, int n_kv, int hd, int n_rot,
                                int block_size, int q_gate, int norm_one_plus_w, float eps, int max_pos, cudaStream_t st) {
  if (T <= 0) return 0;
  if (hd > 512) return -108;
  QkvPostParams p;
  p.qkv = (const __nv_bfloat16*)qkv; p.bias = bias; p.q_norm_w = q_norm_w; p.k_norm_w = k_norm_w; p.positions = positions;
  p.rope_cos = rope_cos; p.rope_sin = rope_sin; p.slot_map = slot_map; p.q_out = (__nv_bfloat16*)q_out; p.gate_out = (__nv_bfloat16*)gate_out;
  p.k_cache = (__nv_bfloat16*)k_cache; p.v_cache = (__nv_bfloat16*)v_cache;
  p.k_scale = k_scale; p.v_scale = k_scale ? v_scale : nullptr;
  p.T = T; p.n_q = n_q; p.n_kv = n_kv; p.hd = hd; p.n_rot = n_rot; p.block_size = block_size; p.q_gate = q_gate & 1;
  p.v_norm = (q_gate >> 1) & 1;           // flag word: bit 0 = q columns carry a gate, bit 1 = weightless RMS norm on V
  p.norm_one_plus_w = norm_one_plus_w; p.eps = eps; p.max_pos = max_pos;
  const int half = n_rot / 2, epl = hd / 32;
  const int row_cols = n_q * (p.q_gate ? 2 * hd : hd) + 2 * n_kv * hd;
  // many tokens: the token-major form (vector loads need the row start and every head start on an element-count boundary)
  if (T >= 64 && (hd == 64 || hd == 128 || hd == 256 || hd == 512) && half <= 256 && half % epl == 0 && ((half / epl) & (half / epl - 1)) == 0 &&
      n_rot <= hd && row_cols % 8 == 0 && ((uintptr_t)qkv & 15) == 0) {
    switch (hd) {
      case 64: launch_pdl(qkv_post_token_kernel<64>, dim3(T), dim3(128), 0, st, p); break;
      case 128: launch_pdl(qkv_post_token_kernel<128>, dim3(T), dim3(128), 0, st, p); break;
      case 256: launch_pdl(qkv_post_token_kernel<256>, dim3(T), dim3(128), 0, st, p); break;
      default: launch_pdl(qkv_post_token_kernel<512>, dim3(T), dim3(128), 0, st, p); break;
    }
    return (int)cudaGetLastError();
  }
  const int units = T * (n_q + 2 * n_kv);
  launch_pdl(qkv_post_kernel, dim3((units + 3) / 4), dim3(128), 0, st, p);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_glu(const void* in, void* out, long long T, int F, int act, float alpha, float limit, cudaStream_t st) {
  const long long total = T * F;
  if (total <= 0) return 0;
  if (F % 16) return -104;
  launch_pdl(glu_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st, (const __nv_bfloat16*)in, (__nv_bfloat16*)out, total, F, act, alpha, limit);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_glu_f32(const float* in, float* out, long long T, int F, int act, float alpha, float limit, cudaStream_t st) {
  const long long total = T * F;
  if (total <= 0) return 0;
  if (F % 16) return -104;
  launch_pdl(glu_f32_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, st, in, out, total, F, act, alpha, limit);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_sigmoid_mul(const void* x, const void* g, void* y, long long n, cudaStream_t st) {
  if (n <= 0) return 0;
  launch_pdl(sigmoid_mul_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, (const __nv_bfloat16*)x, (const __nv_bfloat16*)g, (__nv_bfloat16*)y, n);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_scaled_add(float* out, const void* src, const float* gate_logit, int H, long long n, cudaStream_t st) {
  if (n <= 0) return 0;
  launch_pdl(scaled_add_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, out, (const __nv_bfloat16*)src, gate_logit, H, n);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_cast_f32_bf16(const float* a, void* b, long long n, cudaStream_t st) {
  if (n <= 0) return 0;
  launch_pdl(cast_f32_bf16_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, a, (__nv_bfloat16*)b, n);
  return (int)cudaGetLastError();
}

MX_HOST_API int mx_gated_rmsnorm(const float* x, const void* z, const float* w, void* y, int rows, int hd, float eps, cudaStream_t st) {
  if (rows <= 0) return 0;
  launch_pdl(gated_rmsnorm_kernel, dim3((rows + 3) / 4), dim3(128), 0, st, x, (const __nv_bfloat16*)z, w, (__nv_bfloat16*)y, rows, hd, eps);
  return (int)cudaGetLastError();
}
