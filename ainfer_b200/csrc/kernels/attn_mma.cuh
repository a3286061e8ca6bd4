// Attention on the tensor cores with mma.sync: tiles of 64 keys (or values) in shared memory as rows of
// DP + 8 bf16 values, fragments of 16 rows per warp, fp32 scores and sums. Shared by the attention
// kernels of the models with bf16 caches.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace ainfer {

constexpr int kCmKeys = 64;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ uint32_t cm_smem(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(a)
               : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t *>(&v);
}
__device__ __forceinline__ void cpa16(uint32_t dst, const void *src, bool in) {   // out of range: zero fill
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cpa_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cpa_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// 64 keys [slot, slot + 64) of one key head into a tile of rows of DP + 8 values.
template <int DP, int THREADS>
__device__ __forceinline__ void load_keys(uint32_t dst, const uint16_t *K, int slot, int KW, int D) {
  constexpr int P = DP / 8;
  for (int i = threadIdx.x; i < kCmKeys * P; i += THREADS) {
    const int r = i / P, c = i % P;
    const bool in = c * 8 < D;
    cpa16(dst + (uint32_t)(r * (DP + 8) + c * 8) * 2, K + (size_t)(slot + r) * KW + (in ? c * 8 : 0), in);
  }
}

// One warp, 16 rows against NK keys of a tile at `kt`: s[n] = products with keys 8n .. 8n+7.
template <int DP, int NK>
__device__ __forceinline__ void scores(float (&s)[NK / 8][4], const uint32_t (&q)[DP / 16][4], uint32_t kt, int lane) {
#pragma unroll
  for (int n = 0; n < NK / 8; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) s[n][i] = 0.0f;
  const uint32_t a = kt + (uint32_t)(((lane & 7) + ((lane >> 4) & 1) * 8) * (DP + 8) + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
  for (int kk = 0; kk < DP / 16; ++kk)
#pragma unroll
    for (int n = 0; n < NK / 16; ++n) {
      uint32_t b[4];
      ldm4(b, a + (uint32_t)(n * 16 * (DP + 8) + kk * 16) * 2);
      mma16816(s[2 * n], q[kk], b[0], b[1]);
      mma16816(s[2 * n + 1], q[kk], b[2], b[3]);
    }
}
// The same with the query fragments read from shared memory (qa: this lane's address in the warp's 16 rows).
template <int DP, int NK>
__device__ __forceinline__ void scores_smem(float (&s)[NK / 8][4], uint32_t qa, uint32_t kt, int lane) {
#pragma unroll
  for (int n = 0; n < NK / 8; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) s[n][i] = 0.0f;
  const uint32_t a = kt + (uint32_t)(((lane & 7) + ((lane >> 4) & 1) * 8) * (DP + 8) + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
  for (int kk = 0; kk < DP / 16; ++kk) {
    uint32_t q[4];
    ldm4(q, qa + (uint32_t)(kk * 32));
#pragma unroll
    for (int n = 0; n < NK / 16; ++n) {
      uint32_t b[4];
      ldm4(b, a + (uint32_t)(n * 16 * (DP + 8) + kk * 16) * 2);
      mma16816(s[2 * n], q, b[0], b[1]);
      mma16816(s[2 * n + 1], q, b[2], b[3]);
    }
  }
}
// o += weights (as the score fragments hold them) . keys of the tile
template <int DP, int NK>
__device__ __forceinline__ void values(float (&o)[DP / 8][4], const float (&p)[NK / 8][4], uint32_t kt, int lane) {
  const uint32_t a = kt + (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * (DP + 8) + ((lane >> 4) & 1) * 8) * 2;
#pragma unroll
  for (int j = 0; j < NK / 16; ++j) {
    const uint32_t w[4] = {pack2(p[2 * j][0], p[2 * j][1]), pack2(p[2 * j][2], p[2 * j][3]), pack2(p[2 * j + 1][0], p[2 * j + 1][1]),
                           pack2(p[2 * j + 1][2], p[2 * j + 1][3])};
#pragma unroll
    for (int d = 0; d < DP / 16; ++d) {
      uint32_t b[4];
      ldm4t(b, a + (uint32_t)(j * 16 * (DP + 8) + d * 16) * 2);
      mma16816(o[2 * d], w, b[0], b[1]);
      mma16816(o[2 * d + 1], w, b[2], b[3]);
    }
  }
}
__device__ __forceinline__ float fast_exp2(float x) {   // one instruction, 2 ulp, small results flushed to zero
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float quad_max(float v) {
  v = fmaxf(v, __shfl_xor_sync(kFull, v, 1));
  return fmaxf(v, __shfl_xor_sync(kFull, v, 2));
}
__device__ __forceinline__ float quad_sum(float v) {
  v = v + __shfl_xor_sync(kFull, v, 1);
  return v + __shfl_xor_sync(kFull, v, 2);
}

}  // namespace ainfer
