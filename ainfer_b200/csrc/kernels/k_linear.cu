// Dense layers with bf16 weights W [N][ldw] (rows padded with zeros to a multiple of 8 values).
//
//   LinearRows        fp32 activations, fp32 sums on the CUDA cores (the 32-bit form)
//   StreamGemv        one fp32 row, weights streamed once: y = act(W x + bias)
//   HyperStreamGemv   the same, x made in the kernel from the residual streams: stream update of the
//                     previous sublayer, weighted read, RMS norm, optional token shift (every block
//                     makes the row for itself; block 0 stores the updated streams and the shift row)
// act: 0 none, 1 relu squared, 2 cap tanh(v / cap).
#include "hyper_core.cuh"
#include "weight_ring.cuh"

namespace ainfer {

enum { ACT_NONE = 0, ACT_RELU2 = 1, ACT_SOFTCAP = 2 };
__device__ __forceinline__ float apply_act(float v, int act, float cap) {
  if (act == ACT_RELU2) { v = v > 0.0f ? v : 0.0f; return v * v; }
  if (act == ACT_SOFTCAP) return cap * tanhf(v / cap);
  return v;
}

// ---------------------------------------------------------- LinearRows ---
struct LinearRowsArgs {
  const float *X;        // [rows][ldx]
  const uint16_t *W;     // [N][ldw]
  const float *Bias;     // [N] or null
  float *Y;              // [rows][ldy]
  int32_t rows, N, K, ldx, ldw, ldy, act;
  float cap;
};
constexpr int kLrTile = 64, kLrK = 16;
__global__ void __launch_bounds__(256) LinearRows(const LinearRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float xs[kLrK][kLrTile + 4], ws[kLrK][kLrTile + 4];
  const int nt = (a.N + kLrTile - 1) / kLrTile;
  const int n0 = (blockIdx.x % nt) * kLrTile, r0 = (blockIdx.x / nt) * kLrTile;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += kLrK) {
    for (int i = tid; i < kLrTile * kLrK; i += 256) {
      const int rr = i / kLrK, k = i % kLrK;
      const bool kin = k0 + k < a.K;
      xs[k][rr] = kin && r0 + rr < a.rows ? a.X[(size_t)(r0 + rr) * a.ldx + k0 + k] : 0.0f;
      ws[k][rr] = kin && n0 + rr < a.N ? bf16_to_f32(a.W[(size_t)(n0 + rr) * a.ldw + k0 + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kLrK; ++k) {
      float xv[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { xv[i] = xs[k][ty * 4 + i]; wv[i] = ws[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = r0 + ty * 4 + i;
    if (r >= a.rows) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < a.N) a.Y[(size_t)r * a.ldy + n] = apply_act(acc[i][j] + (a.Bias ? a.Bias[n] : 0.0f), a.act, a.cap);
    }
  }
}
#define F(f) AINFER_ARG(LinearRowsArgs, f)
AINFER_REGISTER(LinearRows, LinearRowsArgs, 256, 0, 0, nullptr, F(X), F(W), F(Bias), F(Y), F(rows), F(N), F(K), F(ldx), F(ldw), F(ldy),
                F(act), F(cap));
#undef F

// ---------------------------------------------------------- StreamGemv ---
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
// The producer warp's whole work; then it waits at the block's last barrier like everyone.
__device__ __forceinline__ void gemv_produce(const GemvShape &c, const GemvDims &d, GemvShared *sh, unsigned char *ring) {
  if ((threadIdx.x & 31) == 0) {
    const int n0 = blockIdx.x * c.rows_pb, n1 = min(c.N, n0 + c.rows_pb);
    uint32_t st = 0, ph = 1, issued = 0;
    for (int n = n0; n < n1; n += d.tile_rows) {
      if (!sg_wait(sh, &sh->empty[st], ph)) break;
      const uint32_t bytes = (uint32_t)min(d.tile_rows, n1 - n) * (uint32_t)c.ldw * 2u;
      mbar_arrive_expect(&sh->full[st], bytes);
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                       smem_addr(ring + (size_t)st * d.stage_bytes)),
                   "l"(c.W + (size_t)n * c.ldw), "r"(bytes), "r"(smem_addr(&sh->full[st]))
                   : "memory");
      ++issued;
      if (++st == (uint32_t)d.nst) { st = 0; ph ^= 1; }
    }
    if (*reinterpret_cast<volatile uint32_t *>(&sh->fail))   // copies in flight land before the block may end
      for (int i = 0; i < d.nst && (uint32_t)i < issued; ++i) {
        const uint32_t uses = (issued - (uint32_t)i + (uint32_t)d.nst - 1) / (uint32_t)d.nst;
        for (uint32_t s = 0; s < kSgSpin && !mbar_try(&sh->full[i], (uses - 1) & 1); ++s) {}
      }
  }
  __syncwarp();
}
__device__ __forceinline__ void gemv_consume(const GemvShape &c, const GemvDims &d, GemvShared *sh, const unsigned char *ring, const float *lo,
                                             const float *hi, float *part) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pieces = c.ldw >> 3;
  const int n0 = blockIdx.x * c.rows_pb, n1 = min(c.N, n0 + c.rows_pb), mine = warp % d.wpr, r_step = kSgWarps / d.wpr;
  uint32_t st = 0, ph = 0;
  for (int n = n0; n < n1; n += d.tile_rows) {
    const int nr = min(d.tile_rows, n1 - n);
    sg_wait(sh, &sh->full[st], ph);
    __syncwarp();
    const unsigned char *tile = ring + (size_t)st * d.stage_bytes;
    for (int r = warp / d.wpr; r < nr; r += r_step) {
      const uint4 *row = reinterpret_cast<const uint4 *>(tile + (size_t)r * c.ldw * 2);
      float s0 = 0.0f, s1 = 0.0f;
      int i = mine * 32 + lane;
      const int step = 32 * d.wpr;
      for (; i + step < pieces; i += 2 * step) {
        s0 = dot8(row[i], *reinterpret_cast<const float4 *>(lo + 4 * i), *reinterpret_cast<const float4 *>(hi + 4 * i), s0);
        const int k = i + step;
        s1 = dot8(row[k], *reinterpret_cast<const float4 *>(lo + 4 * k), *reinterpret_cast<const float4 *>(hi + 4 * k), s1);
      }
      if (i < pieces) s0 = dot8(row[i], *reinterpret_cast<const float4 *>(lo + 4 * i), *reinterpret_cast<const float4 *>(hi + 4 * i), s0);
      s0 = warp_tree_sum(s0 + s1);
      if (lane == 0) part[(n - n0 + r) * d.wpr + mine] = s0;
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&sh->empty[st]);
    if (++st == (uint32_t)d.nst) { st = 0; ph ^= 1; }
  }
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

struct StreamGemvArgs {
  const float *X;        // [K]
  const uint16_t *W;
  const float *Bias;     // [N] or null
  float *Y;              // [N]
  int32_t N, K, ldw, rows_pb, act;
  float cap;
};
extern __shared__ __align__(128) unsigned char sg_smem[];
__global__ void __launch_bounds__(kSgThreads, 4) StreamGemv(const StreamGemvArgs a) {
  __shared__ GemvShared sh;
  pdl_launch_dependents();
  const GemvDims d = gemv_dims(a.ldw);
  const GemvShape c{a.W, a.Bias, a.Y, a.N, a.ldw, a.rows_pb, a.act, a.cap};
  float *lo = reinterpret_cast<float *>(sg_smem + d.nst * d.stage_bytes), *hi = lo + a.ldw / 2, *part = hi + a.ldw / 2;
  gemv_init(&sh, d.nst);
  if (threadIdx.x >= kSgWarps * 32) {
    gemv_produce(c, d, &sh, sg_smem);
  } else {
    pdl_wait();
    for (int k = threadIdx.x; k < a.ldw; k += kSgWarps * 32) sg_put(lo, hi, k, k < a.K ? a.X[k] : 0.0f);
    asm volatile("bar.sync 1, 256;" ::: "memory");
    gemv_consume(c, d, &sh, sg_smem, lo, hi, part);
  }
  __syncthreads();
  gemv_store(c, d, part);
}
static uint32_t stream_gemv_smem(const void *args) {
  const StreamGemvArgs *a = (const StreamGemvArgs *)args;
  return gemv_smem(a->ldw, a->rows_pb, 0);
}
#define F(f) AINFER_ARG(StreamGemvArgs, f)
AINFER_REGISTER(StreamGemv, StreamGemvArgs, kSgThreads, 0, 0, stream_gemv_smem, F(X), F(W), F(Bias), F(Y), F(N), F(K), F(ldw), F(rows_pb),
                F(act), F(cap));
#undef F

struct HyperStreamGemvArgs {
  const float *Xin;        // [S][K] streams
  const float *Yp;         // [K] output of the sublayer whose update is pending; null: none
  const float *Mix, *Out;  // of that sublayer
  float *Xout;             // [S][K] (another buffer than Xin); null: not stored
  const float *In;         // [S]; null: plain sum
  const float *NormW;      // [K]
  const float *Shift;      // [K] or null
  float *State;            // [2][K] shift rows by position parity
  const int32_t *Ctrl;
  const uint16_t *W;
  const float *Bias;
  float *Y;
  int32_t S, N, K, ldw, rows_pb, act;
  float eps, cap;
};
__global__ void __launch_bounds__(kSgThreads, 4) HyperStreamGemv(const HyperStreamGemvArgs a) {
  __shared__ GemvShared sh;
  __shared__ StreamCoef coef;
  __shared__ float red[33];
  pdl_launch_dependents();
  const GemvDims d = gemv_dims(a.ldw);
  const GemvShape c{a.W, a.Bias, a.Y, a.N, a.ldw, a.rows_pb, a.act, a.cap};
  const int K = a.K, tid = threadIdx.x, nth = kSgWarps * 32;
  float *lo = reinterpret_cast<float *>(sg_smem + d.nst * d.stage_bytes), *hi = lo + a.ldw / 2, *us = hi + a.ldw / 2,
        *part = us + ((K + 3) & ~3);
  load_stream_coef(coef, a.Mix, a.Out, a.In, a.S);
  gemv_init(&sh, d.nst);
  if (tid >= nth) {
    gemv_produce(c, d, &sh, sg_smem);
  } else {
    const int lane = tid & 31, warp = tid >> 5;
    pdl_wait();
    float ss = stream_row_any(a.Xin, a.Yp, blockIdx.x == 0 ? a.Xout : nullptr, coef, a.S, K, a.Yp != nullptr, us, tid, nth);
    ss = warp_tree_sum(ss);
    if (lane == 0) red[warp] = ss;
    asm volatile("bar.sync 1, 256;" ::: "memory");   // also: every thread's u is visible
    ss = warp_tree_sum(lane < kSgWarps ? red[lane] : 0.0f);
    const float inv = 1.0f / sqrtf(ss / (float)K + a.eps);
    const int pos = a.Shift ? a.Ctrl[CTRL_POS] : 0;
    const float *prev = a.Shift ? a.State + (size_t)((pos - 1) & 1) * K : nullptr;
    float *next = a.Shift && blockIdx.x == 0 ? a.State + (size_t)(pos & 1) * K : nullptr;
    for (int k = tid; k < a.ldw; k += nth) {
      float v = 0.0f;
      if (k < K) {
        v = us[k] * inv * a.NormW[k];
        if (a.Shift) {
          const float pv = pos > 0 ? prev[k] : 0.0f;
          if (next) next[k] = v;
          v = fmaf(pv - v, a.Shift[k], v);
        }
      }
      sg_put(lo, hi, k, v);
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    gemv_consume(c, d, &sh, sg_smem, lo, hi, part);
  }
  __syncthreads();
  gemv_store(c, d, part);
}
static uint32_t hyper_gemv_smem(const void *args) {
  const HyperStreamGemvArgs *a = (const HyperStreamGemvArgs *)args;
  return gemv_smem(a->ldw, a->rows_pb, (a->K + 3) & ~3);
}
#define F(f) AINFER_ARG(HyperStreamGemvArgs, f)
AINFER_REGISTER(HyperStreamGemv, HyperStreamGemvArgs, kSgThreads, 0, 0, hyper_gemv_smem, F(Xin), F(Yp), F(Mix), F(Out), F(Xout), F(In),
                F(NormW), F(Shift), F(State), F(Ctrl), F(W), F(Bias), F(Y), F(S), F(N), F(K), F(ldw), F(rows_pb), F(act), F(eps), F(cap));
#undef F

// Copies [N][K] bf16 rows to rows of ld values, zero padded.
struct PackRowsBf16Args {
  uint16_t *Dst;
  const uint16_t *Src;
  int32_t N, K, ld;
};
__global__ void __launch_bounds__(256) PackRowsBf16(const PackRowsBf16Args a) {
  for (int n = blockIdx.x; n < a.N; n += gridDim.x)
    for (int k = threadIdx.x; k < a.ld; k += 256) a.Dst[(size_t)n * a.ld + k] = k < a.K ? a.Src[(size_t)n * a.K + k] : (uint16_t)0;
}
#define F(f) AINFER_ARG(PackRowsBf16Args, f)
AINFER_REGISTER(PackRowsBf16, PackRowsBf16Args, 256, 0, 0, nullptr, F(Dst), F(Src), F(N), F(K), F(ld));
#undef F

AINFER_EARLY_LAUNCH(LinearRows);
AINFER_EARLY_LAUNCH(StreamGemv);
AINFER_EARLY_LAUNCH(HyperStreamGemv);

}  // namespace ainfer
