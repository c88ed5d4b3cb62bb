// Thread-block cluster helpers and raw element pairs, shared by the kernels that scan element-wise recurrences.
#pragma once
#include "common.cuh"

namespace mx {

__device__ __forceinline__ uint32_t cluster_rank() { uint32_t r; asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ uint32_t cluster_size() { uint32_t r; asm volatile("mov.u32 %0, %%cluster_nctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// two floats at the shared-memory address `addr` of this CTA's window, read from CTA `rank` of the cluster
__device__ __forceinline__ float2 cluster_ld2(uint32_t addr, uint32_t rank) {
  uint32_t remote;
  float2 v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(addr), "r"(rank));
  asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(remote) : "memory");
  return v;
}

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

}  // namespace mx
