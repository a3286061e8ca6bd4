// Dense layers with bf16 weights W [N][ldw] (rows padded with zeros to a multiple of 8 values).
//
//   LinearRows        fp32 activations, fp32 sums on the CUDA cores (the 32-bit form)
//   StreamGemv        one fp32 row, weights streamed once: y = act(W x + bias)
//   HyperStreamGemv   the same, x made in the kernel from the residual streams: stream update of the
//                     previous sublayer, weighted read, RMS norm, optional token shift (every block
//                     makes the row for itself; block 0 stores the updated streams and the shift row)
// act: 0 none, 1 relu squared, 2 cap tanh(v / cap).
#include "hyper_core.cuh"
#include "stream_gemv.cuh"

namespace ainfer {

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
struct StreamGemvArgs {
  const float *X;        // [K]
  const uint16_t *W;
  const float *Bias;     // [N] or null
  float *Y;              // [N]
  int32_t N, K, ldw, rows_pb, act;
  float cap;
};
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
