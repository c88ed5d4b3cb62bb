// Linear layers in full 32-bit: y[M][N] = act(x[M][K] W[N][K]^T + bias), fp32 activations against bf16 weights (exact in fp32), FMA on
// the CUDA cores -- no reduced-precision matrix mode.  This is the arithmetic of models that are run in 32-bit (checking, short jobs);
// the 16-bit path has its own GEMV and tensor-core kernels.
//
// A CTA of 256 threads owns a 64 x 64 tile (4 x 4 outputs per thread) and walks K in steps of 16 through shared memory; with few rows
// the tile is 16 x 64 so that more CTAs read the weights.  Grouped form (experts): every 128 rows of x belong to one expert, whose id and the
// number of live 128-row tiles come from device memory.
#include "act.cuh"
#include "common.cuh"
#include "host_util.h"

namespace mx {

constexpr int LF_BN = 64, LF_BK = 16;

template <int BM>
__global__ void __launch_bounds__(256) linear_f32_kernel(const float* __restrict__ x, const __nv_bfloat16* __restrict__ w, const float* __restrict__ bias,
                                                         float* __restrict__ y, int M, int N, int K, int ldy, int act, float act_a, float act_b,
                                                         const int* __restrict__ tile_expert, const int* __restrict__ num_tiles) {
  constexpr int RM = BM / 16;
  pdl_prologue();
  __shared__ float xs[LF_BK][BM + 1];
  __shared__ float ws[LF_BK][LF_BN + 1];
  const int m0 = blockIdx.y * BM, n0 = blockIdx.x * LF_BN;
  if (tile_expert) {
    if (m0 / 128 >= num_tiles[0]) return;
    w += (size_t)tile_expert[m0 / 128] * N * K;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[RM][4];
#pragma unroll
  for (int i = 0; i < RM; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += LF_BK) {
    for (int i = threadIdx.x; i < BM * LF_BK; i += 256) {
      const int r = i / LF_BK, c = i % LF_BK;
      xs[c][r] = (m0 + r < M && k0 + c < K) ? x[(size_t)(m0 + r) * K + k0 + c] : 0.f;
    }
    for (int i = threadIdx.x; i < LF_BN * LF_BK; i += 256) {
      const int r = i / LF_BK, c = i % LF_BK;
      ws[c][r] = (n0 + r < N && k0 + c < K) ? __bfloat162float(w[(size_t)(n0 + r) * K + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < LF_BK; ++c) {
      float xv[RM], wv[4];
#pragma unroll
      for (int i = 0; i < RM; ++i) xv[i] = xs[c][ty + 16 * i];
#pragma unroll
      for (int j = 0; j < 4; ++j) wv[j] = ws[c][tx + 16 * j];
#pragma unroll
      for (int i = 0; i < RM; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < RM; ++i) {
    const int m = m0 + ty + 16 * i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n < N) y[(size_t)m * ldy + n] = act_unary<true>(act, acc[i][j] + (bias ? bias[n] : 0.f), act_a, act_b);
    }
  }
}

}  // namespace mx

using namespace mx;

// act: 0 or a unary code (act.cuh).  x rows are K elements apart, y rows ldy.
MX_HOST_API int mx_linear_f32(const float* x, const void* w, const float* bias, float* y, int M, int N, int K, int ldy, int act, float act_a, float act_b,
                              cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (act_gated(act)) return -104;
  const unsigned gx = (unsigned)((N + LF_BN - 1) / LF_BN);
  const int* none = nullptr;
  if (M <= 16) launch_pdl(linear_f32_kernel<16>, dim3(gx, 1), dim3(256), 0, st, x, (const __nv_bfloat16*)w, bias, y, M, N, K, ldy, act, act_a, act_b, none, none);
  else launch_pdl(linear_f32_kernel<64>, dim3(gx, (unsigned)((M + 63) / 64)), dim3(256), 0, st, x, (const __nv_bfloat16*)w, bias, y, M, N, K, ldy, act, act_a, act_b, none, none);
  return (int)cudaGetLastError();
}

// Rows 128 t .. 128 t + 127 of x meet expert tile_expert[t] of w [experts][N][K], for t < num_tiles[0]; other rows of y are left unwritten.
MX_HOST_API int mx_grouped_linear_f32(const float* x, const void* w, float* y, int M, int N, int K, const int* tile_expert, const int* num_tiles, int act,
                                      float act_a, float act_b, cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (act_gated(act) || !tile_expert || !num_tiles || M % 128) return -104;
  const float* no_bias = nullptr;
  launch_pdl(linear_f32_kernel<64>, dim3((unsigned)((N + LF_BN - 1) / LF_BN), (unsigned)(M / 64)), dim3(256), 0, st, x, (const __nv_bfloat16*)w, no_bias, y, M, N, K,
             N, act, act_a, act_b, tile_expert, num_tiles);
  return (int)cudaGetLastError();
}
