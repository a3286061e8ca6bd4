// minGRU: s' = (1 - z) s + z c with z = logistic(.), c = u + 1/2 where u >= 0 and logistic(u) where
// u < 0, read through silu(g). z, u and g are projections of the current token, so a run of tokens is a
// first-order linear recurrence per channel: chunks of rows are folded to one (decay, gain) pair each,
// every chunk folds the pairs before it to find its start, and then walks its rows.
//
//   U      [rows][3 K]: z (before the logistic), u, g; biases included
//   State  [seq][2][K] fp32, position p in slot p & 1: a step reads the slot it does not write
//
//   MinGruChunkF32/B16      the pair of every chunk, and the state before the pass
//   MinGruScanF32/B16       the rows' outputs s silu(g), and the state after the pass
//   MinGruStepRowsF32/B16   one step of every sequence of a batch
//   MinGruStreamGemv        one step of one sequence in the prologue of the output projection
#include "row_types.cuh"
#include "stream_gemv.cuh"

namespace ainfer {

constexpr int kMgRows = 32, kMgBatch = 8;   // rows of a chunk, rows whose loads are in flight together
struct MinGruGate { float keep, add; };
// The logistic function in 32 bits; T = uint16_t (rows that leave in bf16): by approximate instructions of a
// few ulp.
template <typename T>
__device__ __forceinline__ float gate_logistic(float v) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.0f, 1.0f + __expf(-v));
  else return logistic(v);
}
template <typename T>
__device__ __forceinline__ MinGruGate mingru_gate(float zp, float u) {
  const float z = gate_logistic<T>(zp), c = u >= 0.0f ? u + 0.5f : gate_logistic<T>(u);
  return MinGruGate{1.0f - z, z * c};
}
template <typename T>
__device__ __forceinline__ float mingru_out(float s, float g) { return s * (g * gate_logistic<T>(g)); }

struct MinGruChunkArgs {
  const float *U;          // [rows][3 K]
  const float *State;      // [2][K] of the pass's sequence
  const int32_t *Ctrl;     // [rows][4]
  float *Pair;             // [1 + chunks][2][K]: the state before the pass (second value), then decay and gain
  int32_t rows, K;
};
template <typename T>
__device__ __forceinline__ void mingru_chunk_body(const MinGruChunkArgs &a) {
  const int cb = (a.K + 255) / 256, k = (blockIdx.x % cb) * 256 + threadIdx.x, c = blockIdx.x / cb;
  if (k >= a.K) return;
  const int r0 = c * kMgRows, n = min(kMgRows, a.rows - r0);
  if (c == 0) {
    const int pos = a.Ctrl[CTRL_POS];
    a.Pair[a.K + k] = pos > 0 ? a.State[(size_t)((pos - 1) & 1) * a.K + k] : 0.0f;
  }
  const float *u = a.U + (size_t)r0 * 3 * a.K + k;
  const size_t step = (size_t)3 * a.K;
  float A = 1.0f, B = 0.0f;
  for (int r = 0; r < n; r += kMgBatch) {
    float z[kMgBatch], x[kMgBatch];
#pragma unroll
    for (int i = 0; i < kMgBatch; ++i) {   // past the end: the last row again, not used
      const float *p = u + (size_t)min(r + i, n - 1) * step;
      z[i] = p[0];
      x[i] = p[a.K];
    }
#pragma unroll
    for (int i = 0; i < kMgBatch; ++i)
      if (r + i < n) {
        const MinGruGate g = mingru_gate<T>(z[i], x[i]);
        A = A * g.keep;
        B = fmaf(B, g.keep, g.add);
      }
  }
  float *p = a.Pair + (size_t)(c + 1) * 2 * a.K + k;
  p[0] = A;
  p[a.K] = B;
}
__global__ void __launch_bounds__(256) MinGruChunkF32(const MinGruChunkArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  mingru_chunk_body<float>(a);
}
__global__ void __launch_bounds__(256) MinGruChunkB16(const MinGruChunkArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  mingru_chunk_body<uint16_t>(a);
}
#define F(f) AINFER_ARG(MinGruChunkArgs, f)
AINFER_REGISTER(MinGruChunkF32, MinGruChunkArgs, 256, 0, 0, nullptr, F(U), F(State), F(Ctrl), F(Pair), F(rows), F(K));
AINFER_REGISTER(MinGruChunkB16, MinGruChunkArgs, 256, 0, 0, nullptr, F(U), F(State), F(Ctrl), F(Pair), F(rows), F(K));
#undef F

struct MinGruScanArgs {
  const float *U, *Pair;
  float *State;
  const int32_t *Ctrl;
  void *A;                 // [rows][lda]
  int32_t rows, K, lda;
};
template <typename T>
__device__ __forceinline__ void mingru_scan_body(const MinGruScanArgs &a) {
  const int cb = (a.K + 255) / 256, k = (blockIdx.x % cb) * 256 + threadIdx.x, c = blockIdx.x / cb;
  if (k >= a.K) return;
  const int r0 = c * kMgRows, n = min(kMgRows, a.rows - r0);
  float s = a.Pair[a.K + k];
  for (int j = 1; j <= c; j += kMgBatch) {
    float A[kMgBatch], B[kMgBatch];
#pragma unroll
    for (int i = 0; i < kMgBatch; ++i) {
      const float *p = a.Pair + (size_t)min(j + i, c) * 2 * a.K + k;
      A[i] = p[0];
      B[i] = p[a.K];
    }
#pragma unroll
    for (int i = 0; i < kMgBatch; ++i)
      if (j + i <= c) s = fmaf(s, A[i], B[i]);
  }
  const float *u = a.U + (size_t)r0 * 3 * a.K + k;
  const size_t step = (size_t)3 * a.K;
  T *o = reinterpret_cast<T *>(a.A) + (size_t)r0 * a.lda + k;
  for (int r = 0; r < n; r += kMgBatch) {
    float z[kMgBatch], x[kMgBatch], g[kMgBatch];
#pragma unroll
    for (int i = 0; i < kMgBatch; ++i) {
      const float *p = u + (size_t)min(r + i, n - 1) * step;
      z[i] = p[0];
      x[i] = p[a.K];
      g[i] = p[2 * a.K];
    }
#pragma unroll
    for (int i = 0; i < kMgBatch; ++i)
      if (r + i < n) {
        const MinGruGate q = mingru_gate<T>(z[i], x[i]);
        s = fmaf(s, q.keep, q.add);
        st_val(o + (size_t)(r + i) * a.lda, mingru_out<T>(s, g[i]));
      }
  }
  if (r0 + n == a.rows) a.State[(size_t)(a.Ctrl[4 * (a.rows - 1) + CTRL_POS] & 1) * a.K + k] = s;
}
__global__ void __launch_bounds__(256) MinGruScanF32(const MinGruScanArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  mingru_scan_body<float>(a);
}
__global__ void __launch_bounds__(256) MinGruScanB16(const MinGruScanArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  mingru_scan_body<uint16_t>(a);
}
#define F(f) AINFER_ARG(MinGruScanArgs, f)
AINFER_REGISTER(MinGruScanF32, MinGruScanArgs, 256, 0, 0, nullptr, F(U), F(Pair), F(State), F(Ctrl), F(A), F(rows), F(K), F(lda));
AINFER_REGISTER(MinGruScanB16, MinGruScanArgs, 256, 0, 0, nullptr, F(U), F(Pair), F(State), F(Ctrl), F(A), F(rows), F(K), F(lda));
#undef F

struct MinGruStepRowsArgs {
  const float *U;          // [seq][3 K]
  float *State;            // [seq][2][K]
  const int32_t *Ctrl;     // [seq][4]
  void *A;                 // [seq][lda]
  int32_t nseq, K, lda;
};
template <typename T>
__device__ __forceinline__ void mingru_step_rows_body(const MinGruStepRowsArgs &a) {
  const int cb = (a.K + 255) / 256, k = (blockIdx.x % cb) * 256 + threadIdx.x, q = blockIdx.x / cb;
  if (k >= a.K || q >= a.nseq) return;
  const int pos = a.Ctrl[4 * q + CTRL_POS];
  float *st = a.State + (size_t)q * 2 * a.K;
  const float *u = a.U + (size_t)q * 3 * a.K + k;
  const MinGruGate g = mingru_gate<T>(u[0], u[a.K]);
  const float s = fmaf(pos > 0 ? st[(size_t)((pos - 1) & 1) * a.K + k] : 0.0f, g.keep, g.add);
  st[(size_t)(pos & 1) * a.K + k] = s;
  st_val(reinterpret_cast<T *>(a.A) + (size_t)q * a.lda + k, mingru_out<T>(s, u[2 * a.K]));
}
__global__ void __launch_bounds__(256) MinGruStepRowsF32(const MinGruStepRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  mingru_step_rows_body<float>(a);
}
__global__ void __launch_bounds__(256) MinGruStepRowsB16(const MinGruStepRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  mingru_step_rows_body<uint16_t>(a);
}
#define F(f) AINFER_ARG(MinGruStepRowsArgs, f)
AINFER_REGISTER(MinGruStepRowsF32, MinGruStepRowsArgs, 256, 0, 0, nullptr, F(U), F(State), F(Ctrl), F(A), F(nseq), F(K), F(lda));
AINFER_REGISTER(MinGruStepRowsB16, MinGruStepRowsArgs, 256, 0, 0, nullptr, F(U), F(State), F(Ctrl), F(A), F(nseq), F(K), F(lda));
#undef F

struct MinGruStreamGemvArgs {
  const float *U;          // [3 K]
  float *State;            // [2][K]
  const int32_t *Ctrl;
  const uint16_t *W;       // [N][ldw]
  float *Y;                // [N]
  int32_t N, K, ldw, rows_pb;
};
__global__ void __launch_bounds__(kSgThreads, 3) MinGruStreamGemv(const MinGruStreamGemvArgs a) {
  __shared__ GemvShared sh;
  pdl_launch_dependents();
  const GemvDims d = gemv_dims(a.ldw);
  const GemvShape c{a.W, nullptr, a.Y, a.N, a.ldw, a.rows_pb, ACT_NONE, 0.0f};
  float *lo = reinterpret_cast<float *>(sg_smem + d.nst * d.stage_bytes), *hi = lo + a.ldw / 2, *part = hi + a.ldw / 2;
  gemv_init(&sh, d.nst);
  if (threadIdx.x >= kSgWarps * 32) {
    gemv_produce(c, d, &sh, sg_smem);
  } else {
    pdl_wait();
    const int pos = a.Ctrl[CTRL_POS];
    const float *prev = a.State + (size_t)((pos - 1) & 1) * a.K;
    float *next = blockIdx.x == 0 ? a.State + (size_t)(pos & 1) * a.K : nullptr;
    constexpr int Q = 8, nth = kSgWarps * 32;   // elements of a thread whose loads are in flight together
    for (int k0 = threadIdx.x; k0 < a.ldw; k0 += nth * Q) {
      float z[Q], x[Q], g[Q], p[Q];
#pragma unroll
      for (int i = 0; i < Q; ++i) {
        const int k = min(k0 + i * nth, a.K - 1);
        z[i] = a.U[k];
        x[i] = a.U[a.K + k];
        g[i] = a.U[2 * a.K + k];
        p[i] = pos > 0 ? prev[k] : 0.0f;
      }
#pragma unroll
      for (int i = 0; i < Q; ++i) {
        const int k = k0 + i * nth;
        if (k >= a.ldw) continue;
        const MinGruGate q = mingru_gate<float>(z[i], x[i]);
        const float s = fmaf(p[i], q.keep, q.add);
        if (next && k < a.K) next[k] = s;
        sg_put(lo, hi, k, k < a.K ? mingru_out<float>(s, g[i]) : 0.0f);
      }
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    gemv_consume(c, d, &sh, sg_smem, lo, hi, part);
  }
  __syncthreads();
  gemv_store(c, d, part);
}
static uint32_t mingru_gemv_smem(const void *args) {
  const MinGruStreamGemvArgs *a = (const MinGruStreamGemvArgs *)args;
  return gemv_smem(a->ldw, a->rows_pb, 0);
}
#define F(f) AINFER_ARG(MinGruStreamGemvArgs, f)
AINFER_REGISTER(MinGruStreamGemv, MinGruStreamGemvArgs, kSgThreads, 0, 0, mingru_gemv_smem, F(U), F(State), F(Ctrl), F(W), F(Y), F(N), F(K),
                F(ldw), F(rows_pb));
#undef F

AINFER_EARLY_LAUNCH(MinGruChunkF32);
AINFER_EARLY_LAUNCH(MinGruChunkB16);
AINFER_EARLY_LAUNCH(MinGruScanF32);
AINFER_EARLY_LAUNCH(MinGruScanB16);
AINFER_EARLY_LAUNCH(MinGruStepRowsF32);
AINFER_EARLY_LAUNCH(MinGruStepRowsB16);
AINFER_EARLY_LAUNCH(MinGruStreamGemv);

}  // namespace ainfer
