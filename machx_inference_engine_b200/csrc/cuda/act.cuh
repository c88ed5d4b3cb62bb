// Element-wise activations that a projection's epilogue applies to its own output (unary), beside the gated ones that combine a gate
// and an up column (gated forms live with their kernels because they differ in how the pair is laid out).
#pragma once
#include "common.cuh"

namespace mx {

// activation codes: 0 none; 1 SwiGLU, 2 clamped SwiGLU, 3 GeGLU (gated: N columns become N / 2); 4 xIELU, 5 GELU (tanh form),
// 6 the square of ReLU, 7 tanh (unary)
constexpr int ACT_CODE_XIELU = 4, ACT_CODE_GELU_TANH = 5, ACT_CODE_RELU2 = 6, ACT_CODE_TANH = 7;
__host__ __device__ constexpr bool act_gated(int act) { return act >= 1 && act <= 3; }

// xIELU: a z^2 + z / 2 for z > 0, b (e^z - 1 - z) + z / 2 otherwise (a = softplus(p), b = 1/2 + softplus(q), formed by the caller).
// PRECISE: expm1f; otherwise the fast exponential, whose cancellation near 0 (about 1e-7 absolute) vanishes in a bf16 result.
template <bool PRECISE>
__device__ __forceinline__ float xielu(float z, float a, float b) {
  const float neg = fminf(z, 0.f);
  const float tail = PRECISE ? expm1f(neg) - neg : __expf(neg) - 1.f - neg;
  return fmaf(0.5f, z, z > 0.f ? a * z * z : b * tail);
}

// sigmoid with the full-precision exponential and division, or with the hardware's base-2 exponential and reciprocal (a few units in
// the last place of fp32; the exponential overflows to infinity below about -88 and the result is 0)
template <bool PRECISE>
__device__ __forceinline__ float sigmoid_f(float x) {
  if constexpr (PRECISE) return 1.f / (1.f + expf(-x));
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * -1.4426950408889634f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return r;
}

// GELU, tanh form: 0.5 z (1 + tanh u) = z sigmoid(2 u) with u = sqrt(2 / pi) (z + 0.044715 z^3)
template <bool PRECISE>
__device__ __forceinline__ float gelu_tanh(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  if constexpr (PRECISE) return 0.5f * z * (1.f + tanhf(u));
  return z * sigmoid_f<false>(2.f * u);
}
__device__ __forceinline__ float relu2(float z) {
  const float m = fmaxf(z, 0.f);
  return m * m;
}

template <bool PRECISE>
__device__ __forceinline__ float act_unary(int act, float z, float a, float b) {
  if (act == ACT_CODE_XIELU) return xielu<PRECISE>(z, a, b);
  if (act == ACT_CODE_GELU_TANH) return gelu_tanh<PRECISE>(z);
  if (act == ACT_CODE_TANH) return tanhf(z);
  return act == ACT_CODE_RELU2 ? relu2(z) : z;
}

// the same over a run of values: one branch for the run
template <bool PRECISE, int N>
__device__ __forceinline__ void act_unary_run(int act, float (&v)[N], float a, float b) {
  if (act == ACT_CODE_XIELU) {
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = xielu<PRECISE>(v[j], a, b);
  } else if (act == ACT_CODE_GELU_TANH) {
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = gelu_tanh<PRECISE>(v[j]);
  } else if (act == ACT_CODE_RELU2) {
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = relu2(v[j]);
  } else if (act == ACT_CODE_TANH) {
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = tanhf(v[j]);
  }
}

// ---------------------------------------------------------------- element types of activations (bf16 or fp32)
template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// two consecutive elements (pointer aligned to the pair)
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(bf16_lo(v), bf16_hi(v));
}
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16(a, b); }
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }

// V = 4 or 1 consecutive elements (pointer aligned to the group)
template <int V> __device__ __forceinline__ void loadv(const float* p, float (&v)[V]) {
  if constexpr (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
  else v[0] = *p;
}
template <int V> __device__ __forceinline__ void loadv(const __nv_bfloat16* p, float (&v)[V]) {
  if constexpr (V == 4) { const uint2 t = *reinterpret_cast<const uint2*>(p); v[0] = bf16_lo(t.x); v[1] = bf16_hi(t.x); v[2] = bf16_lo(t.y); v[3] = bf16_hi(t.y); }
  else v[0] = __bfloat162float(*p);
}
template <int V> __device__ __forceinline__ void storev(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <int V> __device__ __forceinline__ void storev(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
  else *p = __float2bfloat16(v[0]);
}

}  // namespace mx
