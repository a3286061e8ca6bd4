// Activations and caches that are fp32 or bf16: loads and stores by type, and a few scalar functions
// that the row kernels share.
#pragma once
#include "common.cuh"

namespace ainfer {

template <typename T>
__device__ __forceinline__ float ld_val(const T *p);
template <>
__device__ __forceinline__ float ld_val<float>(const float *p) { return *p; }
template <>
__device__ __forceinline__ float ld_val<uint16_t>(const uint16_t *p) { return bf16_to_f32(*p); }
template <typename T>
__device__ __forceinline__ void st_val(T *p, float v);
template <>
__device__ __forceinline__ void st_val<float>(float *p, float v) { *p = v; }
template <>
__device__ __forceinline__ void st_val<uint16_t>(uint16_t *p, float v) { *p = f32_to_bf16(v); }

// Four consecutive values; p aligned to four of them.
__device__ __forceinline__ float4 ld_val4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 ld_val4(const uint16_t *p) {
  const uint2 v = *reinterpret_cast<const uint2 *>(p);
  return make_float4(u2f(v.x << 16), u2f(v.x & 0xFFFF0000u), u2f(v.y << 16), u2f(v.y & 0xFFFF0000u));
}
__device__ __forceinline__ void st_val4(float *p, const float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void st_val4(uint16_t *p, const float4 v) {
  *reinterpret_cast<uint2 *>(p) = make_uint2((uint32_t)f32_to_bf16(v.x) | ((uint32_t)f32_to_bf16(v.y) << 16),
                                             (uint32_t)f32_to_bf16(v.z) | ((uint32_t)f32_to_bf16(v.w) << 16));
}

__device__ __forceinline__ float logistic(float v) { return 1.0f / (1.0f + expf(-v)); }

// Block sum in fp32 (any number of warps up to 32); every thread gets the total. red: 33 floats.
__device__ __forceinline__ float block_sum(float v, float *red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_tree_sum(v);
  __syncthreads();   // earlier readers of red are done
  if (lane == 0) red[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nw ? red[lane] : 0.0f;
    t = warp_tree_sum(t);
    if (lane == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

}  // namespace ainfer
