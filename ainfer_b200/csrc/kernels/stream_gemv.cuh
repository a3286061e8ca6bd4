// One fp32 row times a matrix of bf16 rows W [N][ldw] that crosses HBM once: the core of the decode
// step's GEMV kernels. A kernel prepares its row in shared memory in whatever way its model needs and
// hands it to these functions.
#pragma once
#include "common.cuh"
#include "weight_ring.cuh"

namespace ainfer {

enum { ACT_NONE = 0, ACT_RELU2 = 1, ACT_SOFTCAP = 2 };
__device__ __forceinline__ float apply_act(float v, int act, float cap) {
  if (act == ACT_RELU2) { v = v > 0.0f ? v : 0.0f; return v * v; }
  if (act == ACT_SOFTCAP) return cap * tanhf(v / cap);
  return v;
}

// The block's rows are one contiguous range of bytes: a producer warp brings them in tiles of whole rows
// (about 16 KB) through a ring of shared-memory stages with bulk copies, which start before the kernel's
// dependency wait (weights do not depend on it); 8 consumer warps multiply. Two blocks per SM: one
// block's copies complete at a rate that fills about half of an SM's share of the HBM bandwidth. Per tile a row is shared
// by wpr warps; the partial sums of all rows stay in shared memory until the block's last tile.
constexpr int kSgWarps = 8, kSgThreads = kSgWarps * 32 + 32, kSgRing = 65536;
constexpr uint32_t kSgSpin = 1u << 22;
struct GemvDims { int tile_rows, stage_bytes, nst, wpr; };
__host__ __device__ inline GemvDims gemv_dims(int ldw) {
  GemvDims d;
  d.tile_rows = 16384 / (ldw * 2);
  if (d.tile_rows < 1) d.tile_rows = 1;
  if (d.tile_rows > 64) d.tile_rows = 64;
  d.stage_bytes = d.tile_rows * ldw * 2;
  d.nst = kSgRing / d.stage_bytes;
  if (d.nst < 2) d.nst = 2;
  if (d.nst > 8) d.nst = 8;
  d.wpr = 1;
  while (d.wpr * 2 * d.tile_rows <= kSgWarps && d.wpr * 256 < ldw) d.wpr *= 2;
  return d;
}
// The vector in shared memory, split so that a lane's eight values come from two conflict-free
// 16-byte reads: element k of piece k / 8 lies in half (k / 4) % 2 at (k / 8) * 4 + k % 4.
__device__ __forceinline__ void sg_put(float *lo, float *hi, int k, float v) { ((k & 4) ? hi : lo)[(k >> 3) * 4 + (k & 3)] = v; }

struct GemvShape {
  const uint16_t *W;
  const float *Bias;
  float *Y;
  int32_t N, ldw, rows_pb, act;   // rows_pb: rows of a block
  float cap;
};
struct GemvShared {
  unsigned long long full[8], empty[8];
  uint32_t fail;
};
__device__ __forceinline__ bool sg_wait(GemvShared *s, unsigned long long *b, uint32_t parity) {
  if (mbar_try(b, parity)) return true;
  for (uint32_t i = 0; i < kSgSpin; ++i) {
    if (mbar_try(b, parity)) return true;
    if (*reinterpret_cast<volatile uint32_t *>(&s->fail)) return false;
  }
  *reinterpret_cast<volatile uint32_t *>(&s->fail) = 1;
  if (g_stream_fault_word) *reinterpret_cast<volatile unsigned int *>(g_stream_fault_word) = 1;
  return false;
}
__device__ __forceinline__ float dot8(const uint4 w, const float4 a, const float4 b, float s) {
  s = fmaf(u2f(w.x << 16), a.x, s); s = fmaf(u2f(w.x & 0xFFFF0000u), a.y, s);
  s = fmaf(u2f(w.y << 16), a.z, s); s = fmaf(u2f(w.y & 0xFFFF0000u), a.w, s);
  s = fmaf(u2f(w.z << 16), b.x, s); s = fmaf(u2f(w.z & 0xFFFF0000u), b.y, s);
  s = fmaf(u2f(w.w << 16), b.z, s); s = fmaf(u2f(w.w & 0xFFFF0000u), b.w, s);
  return s;
}
__device__ __forceinline__ void gemv_init(GemvShared *sh, int nst) {
  if (threadIdx.x == 0) {
    for (int i = 0; i < nst; ++i) { mbar_init(&sh->full[i], 1); mbar_init(&sh->empty[i], kSgWarps); }
    sh->fail = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
}
// Place in the ring: the producer starts at phase 1, the consumers at phase 0.
struct GemvCursor { uint32_t st, ph, issued; };
__device__ __forceinline__ void gemv_next(GemvCursor &r, const GemvDims &d) {
  if (++r.st == (uint32_t)d.nst) { r.st = 0; r.ph ^= 1; }
}
// Lane 0 of the producer warp: rows [n0, n1) of W.
__device__ __forceinline__ void gemv_produce_rows(const uint16_t *W, int n0, int n1, int ldw, const GemvDims &d, GemvShared *sh, unsigned char *ring,
                                                  GemvCursor &r) {
  for (int n = n0; n < n1; n += d.tile_rows) {
    if (!sg_wait(sh, &sh->empty[r.st], r.ph)) break;
    const uint32_t bytes = (uint32_t)min(d.tile_rows, n1 - n) * (uint32_t)ldw * 2u;
    mbar_arrive_expect(&sh->full[r.st], bytes);
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                     smem_addr(ring + (size_t)r.st * d.stage_bytes)),
                 "l"(W + (size_t)n * ldw), "r"(bytes), "r"(smem_addr(&sh->full[r.st]))
                 : "memory");
    ++r.issued;
    gemv_next(r, d);
  }
}
// Lane 0 of the producer warp, after its last rows: copies in flight land before the block may end.
__device__ __forceinline__ void gemv_produce_end(const GemvDims &d, GemvShared *sh, const GemvCursor &r) {
  if (!*reinterpret_cast<volatile uint32_t *>(&sh->fail)) return;
  for (int i = 0; i < d.nst && (uint32_t)i < r.issued; ++i) {
    const uint32_t uses = (r.issued - (uint32_t)i + (uint32_t)d.nst - 1) / (uint32_t)d.nst;
    for (uint32_t s = 0; s < kSgSpin && !mbar_try(&sh->full[i], (uses - 1) & 1); ++s) {}
  }
}
// The producer warp's whole work; then it waits at the block's last barrier like everyone.
__device__ __forceinline__ void gemv_produce(const GemvShape &c, const GemvDims &d, GemvShared *sh, unsigned char *ring) {
  if ((threadIdx.x & 31) == 0) {
    const int n0 = blockIdx.x * c.rows_pb, n1 = min(c.N, n0 + c.rows_pb);
    GemvCursor r{0, 1, 0};
    gemv_produce_rows(c.W, n0, n1, c.ldw, d, sh, ring, r);
    gemv_produce_end(d, sh, r);
  }
  __syncwarp();
}
// `rows` rows against the vector in lo / hi: part[row][wpr] = factor * sums, added to what is there if `add`.
__device__ __forceinline__ void gemv_consume_rows(int rows, int ldw, const GemvDims &d, GemvShared *sh, const unsigned char *ring, const float *lo,
                                                  const float *hi, float *part, GemvCursor &cur, float factor = 1.0f, bool add = false) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pieces = ldw >> 3;
  const int mine = warp % d.wpr, r_step = kSgWarps / d.wpr;
  for (int n = 0; n < rows; n += d.tile_rows) {
    const int nr = min(d.tile_rows, rows - n);
    sg_wait(sh, &sh->full[cur.st], cur.ph);
    __syncwarp();
    const unsigned char *tile = ring + (size_t)cur.st * d.stage_bytes;
    for (int r = warp / d.wpr; r < nr; r += r_step) {
      const uint4 *row = reinterpret_cast<const uint4 *>(tile + (size_t)r * ldw * 2);
      float s0 = 0.0f, s1 = 0.0f;
      int i = mine * 32 + lane;
      const int step = 32 * d.wpr;
      for (; i + step < pieces; i += 2 * step) {
        s0 = dot8(row[i], *reinterpret_cast<const float4 *>(lo + 4 * i), *reinterpret_cast<const float4 *>(hi + 4 * i), s0);
        const int k = i + step;
        s1 = dot8(row[k], *reinterpret_cast<const float4 *>(lo + 4 * k), *reinterpret_cast<const float4 *>(hi + 4 * k), s1);
      }
      if (i < pieces) s0 = dot8(row[i], *reinterpret_cast<const float4 *>(lo + 4 * i), *reinterpret_cast<const float4 *>(hi + 4 * i), s0);
      s0 = warp_tree_sum(s0 + s1) * factor;
      if (lane == 0) {
        float *p = part + (n + r) * d.wpr + mine;
        *p = add ? *p + s0 : s0;
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&sh->empty[cur.st]);
    gemv_next(cur, d);
  }
}
__device__ __forceinline__ void gemv_consume(const GemvShape &c, const GemvDims &d, GemvShared *sh, const unsigned char *ring, const float *lo,
                                             const float *hi, float *part) {
  const int n0 = blockIdx.x * c.rows_pb, n1 = min(c.N, n0 + c.rows_pb);
  GemvCursor cur{0, 0, 0};
  gemv_consume_rows(n1 - n0, c.ldw, d, sh, ring, lo, hi, part, cur);
}
// After the block's last barrier: one thread per row.
__device__ __forceinline__ void gemv_store(const GemvShape &c, const GemvDims &d, const float *part) {
  const int n0 = blockIdx.x * c.rows_pb, n1 = min(c.N, n0 + c.rows_pb);
  for (int n = n0 + threadIdx.x; n < n1; n += kSgThreads) {
    float v = 0.0f;
    for (int i = 0; i < d.wpr; ++i) v += part[(n - n0) * d.wpr + i];
    c.Y[n] = apply_act(v + (c.Bias ? c.Bias[n] : 0.0f), c.act, c.cap);
  }
}
// shared memory: ring, vector halves, then `extra` floats, then the partial sums
__host__ __device__ inline uint32_t gemv_smem(int ldw, int rows_pb, int extra) {
  const GemvDims d = gemv_dims(ldw);
  return (uint32_t)(d.nst * d.stage_bytes) + 4u * (uint32_t)(ldw + extra + rows_pb * d.wpr);
}

extern __shared__ __align__(128) unsigned char sg_smem[];

}  // namespace ainfer
