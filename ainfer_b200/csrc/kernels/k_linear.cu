// Dense layers with bf16 weights W [N][ldw] (rows padded with zeros to a multiple of 8 values).
//
//   LinearRows        fp32 activations, fp32 sums on the CUDA cores (the 32-bit form)
//   StreamGemv        one fp32 row, weights streamed once: y = act(W x + bias)
//   HyperStreamGemv   the same, x made in the kernel from the residual streams: stream update of the
//                     previous sublayer, weighted read, RMS norm, optional token shift (every block
//                     makes the row for itself; block 0 stores the updated streams and the shift row)
// act: 0 none, 1 relu squared, 2 cap tanh(v / cap).
#include "hyper_core.cuh"

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
constexpr int kSgThreads = 512, kSgWarps = kSgThreads / 32;
constexpr int kSgPre = 2;   // 16-byte pieces of each of a warp's two rows fetched before the dependency wait

// The vector in shared memory, split so that a lane's eight values come from two conflict-free
// 16-byte reads: element k of piece k / 8 lies in half (k / 4) % 2 at (k / 8) * 4 + k % 4.
__device__ __forceinline__ void sg_put(float *lo, float *hi, int k, float v) { ((k & 4) ? hi : lo)[(k >> 3) * 4 + (k & 3)] = v; }
__host__ __device__ inline uint32_t sg_half(uint32_t ldw) { return ldw / 2; }

struct GemvShape {
  const uint16_t *W;
  const float *Bias;
  float *Y;
  int32_t N, ldw, wpr, act;   // wpr: warps that share a pair of rows (1, 2, 4 or 8)
  float cap;
};
__device__ __forceinline__ float dot8(const uint4 w, const float4 a, const float4 b, float s) {
  s = fmaf(u2f(w.x << 16), a.x, s); s = fmaf(u2f(w.x & 0xFFFF0000u), a.y, s);
  s = fmaf(u2f(w.y << 16), a.z, s); s = fmaf(u2f(w.y & 0xFFFF0000u), a.w, s);
  s = fmaf(u2f(w.z << 16), b.x, s); s = fmaf(u2f(w.z & 0xFFFF0000u), b.y, s);
  s = fmaf(u2f(w.w << 16), b.z, s); s = fmaf(u2f(w.w & 0xFFFF0000u), b.w, s);
  return s;
}
struct GemvFirst { uint4 w[2][kSgPre]; };
// This warp's first pair of rows and its first pieces of them.
__device__ __forceinline__ void gemv_prefetch(const GemvShape &c, GemvFirst &f) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pieces = c.ldw >> 3;
  const int pair = blockIdx.x * (kSgWarps / c.wpr) + warp / c.wpr, part = warp % c.wpr;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int n = min(2 * pair + i, c.N - 1);
    const uint4 *row = reinterpret_cast<const uint4 *>(c.W + (size_t)n * c.ldw);
#pragma unroll
    for (int j = 0; j < kSgPre; ++j) f.w[i][j] = __ldg(row + min(part * 32 + lane + 32 * c.wpr * j, pieces - 1));
  }
}
__device__ __forceinline__ void gemv_body(const GemvShape &c, const float *lo, const float *hi, float *part_sum, const GemvFirst &f) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pieces = c.ldw >> 3;
  const int gpb = kSgWarps / c.wpr, pairs = (c.N + 1) / 2, part = warp % c.wpr, step = 32 * c.wpr;
  bool first = true;
  for (int p0 = blockIdx.x * gpb; p0 < pairs; p0 += gridDim.x * gpb) {
    const int pair = p0 + warp / c.wpr;
    float s0 = 0.0f, s1 = 0.0f;
    if (pair < pairs) {
      const int n0 = 2 * pair, n1 = min(2 * pair + 1, c.N - 1);
      const uint4 *r0 = reinterpret_cast<const uint4 *>(c.W + (size_t)n0 * c.ldw), *r1 = reinterpret_cast<const uint4 *>(c.W + (size_t)n1 * c.ldw);
      int i = part * 32 + lane;
      if (first) {
#pragma unroll
        for (int j = 0; j < kSgPre; ++j) {
          if (i < pieces) {
            const float4 a = *reinterpret_cast<const float4 *>(lo + 4 * i), b = *reinterpret_cast<const float4 *>(hi + 4 * i);
            s0 = dot8(f.w[0][j], a, b, s0);
            s1 = dot8(f.w[1][j], a, b, s1);
          }
          i += step;
        }
      }
#pragma unroll 4
      for (; i < pieces; i += step) {
        const uint4 w0 = __ldg(r0 + i), w1 = __ldg(r1 + i);
        const float4 a = *reinterpret_cast<const float4 *>(lo + 4 * i), b = *reinterpret_cast<const float4 *>(hi + 4 * i);
        s0 = dot8(w0, a, b, s0);
        s1 = dot8(w1, a, b, s1);
      }
    }
    first = false;
    s0 = warp_tree_sum(s0);
    s1 = warp_tree_sum(s1);
    if (c.wpr > 1) {
      if (lane == 0) { part_sum[2 * warp] = s0; part_sum[2 * warp + 1] = s1; }
      __syncthreads();
      if (part == 0) {
        s0 = s1 = 0.0f;
        for (int i = 0; i < c.wpr; ++i) { s0 += part_sum[2 * (warp + i)]; s1 += part_sum[2 * (warp + i) + 1]; }
      }
      __syncthreads();
    }
    if (part == 0 && lane < 2 && pair < pairs) {
      const int n = 2 * pair + lane;
      if (n < c.N) c.Y[n] = apply_act((lane ? s1 : s0) + (c.Bias ? c.Bias[n] : 0.0f), c.act, c.cap);
    }
  }
}

struct StreamGemvArgs {
  const float *X;        // [K]
  const uint16_t *W;
  const float *Bias;     // [N] or null
  float *Y;              // [N]
  int32_t N, K, ldw, wpr, act;
  float cap;
};
__global__ void __launch_bounds__(kSgThreads, 2) StreamGemv(const StreamGemvArgs a) {
  extern __shared__ __align__(16) float sg_smem[];
  __shared__ float part_sum[2 * kSgWarps];
  pdl_launch_dependents();
  const GemvShape c{a.W, a.Bias, a.Y, a.N, a.ldw, a.wpr, a.act, a.cap};
  GemvFirst f;
  gemv_prefetch(c, f);
  pdl_wait();
  float *lo = sg_smem, *hi = sg_smem + sg_half((uint32_t)a.ldw);
  for (int k = threadIdx.x; k < a.ldw; k += kSgThreads) sg_put(lo, hi, k, k < a.K ? a.X[k] : 0.0f);
  __syncthreads();
  gemv_body(c, lo, hi, part_sum, f);
}
static uint32_t stream_gemv_smem(const void *args) { return 4u * (uint32_t)((const StreamGemvArgs *)args)->ldw; }
#define F(f) AINFER_ARG(StreamGemvArgs, f)
AINFER_REGISTER(StreamGemv, StreamGemvArgs, kSgThreads, 0, 0, stream_gemv_smem, F(X), F(W), F(Bias), F(Y), F(N), F(K), F(ldw), F(wpr), F(act),
                F(cap));
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
  int32_t S, N, K, ldw, wpr, act;
  float eps, cap;
};
__global__ void __launch_bounds__(kSgThreads, 2) HyperStreamGemv(const HyperStreamGemvArgs a) {
  extern __shared__ __align__(16) float hg_smem[];
  __shared__ float part_sum[2 * kSgWarps];
  __shared__ StreamCoef coef;
  __shared__ float red[33];
  pdl_launch_dependents();
  const GemvShape c{a.W, a.Bias, a.Y, a.N, a.ldw, a.wpr, a.act, a.cap};
  GemvFirst f;
  gemv_prefetch(c, f);
  load_stream_coef(coef, a.Mix, a.Out, a.In, a.S);
  pdl_wait();
  __syncthreads();
  const int K = a.K, tid = threadIdx.x;
  float *lo = hg_smem, *hi = lo + sg_half((uint32_t)a.ldw), *us = hi + sg_half((uint32_t)a.ldw);
  const float ss = stream_row_any(a.Xin, a.Yp, blockIdx.x == 0 ? a.Xout : nullptr, coef, a.S, K, a.Yp != nullptr, us);
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)K + a.eps);
  const int pos = a.Shift ? a.Ctrl[CTRL_POS] : 0;
  const float *prev = a.Shift ? a.State + (size_t)((pos - 1) & 1) * K : nullptr;
  float *next = a.Shift && blockIdx.x == 0 ? a.State + (size_t)(pos & 1) * K : nullptr;
  // the block_sum's barriers made every thread's u visible
  for (int k = tid; k < a.ldw; k += kSgThreads) {
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
  __syncthreads();
  gemv_body(c, lo, hi, part_sum, f);
}
static uint32_t hyper_gemv_smem(const void *args) {
  const HyperStreamGemvArgs *a = (const HyperStreamGemvArgs *)args;
  return 4u * ((uint32_t)a->ldw + (uint32_t)((a->K + 3) & ~3));
}
#define F(f) AINFER_ARG(HyperStreamGemvArgs, f)
AINFER_REGISTER(HyperStreamGemv, HyperStreamGemvArgs, kSgThreads, 0, 0, hyper_gemv_smem, F(Xin), F(Yp), F(Mix), F(Out), F(Xout), F(In),
                F(NormW), F(Shift), F(State), F(Ctrl), F(W), F(Bias), F(Y), F(S), F(N), F(K), F(ldw), F(wpr), F(act), F(eps), F(cap));
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
