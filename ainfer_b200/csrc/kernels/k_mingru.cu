// minGRU: s' = (1 - z) s + z c with z = logistic(.), c = u + 1/2 where u >= 0 and logistic(u) where
// u < 0, read through silu(g). z, u and g are projections of the current token, so a run of tokens is a
// first-order linear recurrence per channel: chunks of rows are folded to one (decay, gain) pair each,
// every chunk folds the pairs before it to find its start, and then walks its rows.
//
//   U      [rows][3 K]: z (before the logistic), u, g; biases included
//   State  [seq][2][K] fp32, position p in slot p & 1: a step reads the slot it does not write
//
//   MinGruChunk             the pair of every chunk, and the state before the pass
//   MinGruScanF32/B16       the rows' outputs s silu(g), and the state after the pass
//   MinGruStepRowsF32/B16   one step of every sequence of a batch
//   MinGruStreamGemv        one step of one sequence in the prologue of the output projection
#include "row_types.cuh"
#include "stream_gemv.cuh"

namespace ainfer {

constexpr int kMgRows = 32;   // rows of a chunk
struct MinGruGate { float keep, add; };
__device__ __forceinline__ MinGruGate mingru_gate(float zp, float u) {
  const float z = logistic(zp), c = u >= 0.0f ? u + 0.5f : logistic(u);
  return MinGruGate{1.0f - z, z * c};
}
__device__ __forceinline__ float mingru_out(float s, float g) { return s * (g / (1.0f + expf(-g))); }

struct MinGruChunkArgs {
  const float *U;          // [rows][3 K]
  const float *State;      // [2][K] of the pass's sequence
  const int32_t *Ctrl;     // [rows][4]
  float *Pair;             // [1 + chunks][2][K]: the state before the pass (second value), then decay and gain
  int32_t rows, K;
};
__global__ void __launch_bounds__(256) MinGruChunk(const MinGruChunkArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int cb = (a.K + 255) / 256, k = (blockIdx.x % cb) * 256 + threadIdx.x, c = blockIdx.x / cb;
  if (k >= a.K) return;
  const int r0 = c * kMgRows, r1 = min(a.rows, r0 + kMgRows);
  if (c == 0) {
    const int pos = a.Ctrl[CTRL_POS];
    a.Pair[a.K + k] = pos > 0 ? a.State[(size_t)((pos - 1) & 1) * a.K + k] : 0.0f;
  }
  float A = 1.0f, B = 0.0f;
#pragma unroll 8
  for (int r = r0; r < r1; ++r) {
    const float *u = a.U + (size_t)r * 3 * a.K + k;
    const MinGruGate g = mingru_gate(u[0], u[a.K]);
    A = A * g.keep;
    B = fmaf(B, g.keep, g.add);
  }
  float *p = a.Pair + (size_t)(c + 1) * 2 * a.K + k;
  p[0] = A;
  p[a.K] = B;
}
#define F(f) AINFER_ARG(MinGruChunkArgs, f)
AINFER_REGISTER(MinGruChunk, MinGruChunkArgs, 256, 0, 0, nullptr, F(U), F(State), F(Ctrl), F(Pair), F(rows), F(K));
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
  const int r0 = c * kMgRows, r1 = min(a.rows, r0 + kMgRows);
  float s = a.Pair[a.K + k];
#pragma unroll 8
  for (int j = 1; j <= c; ++j) {
    const float *p = a.Pair + (size_t)j * 2 * a.K + k;
    s = fmaf(s, p[0], p[a.K]);
  }
#pragma unroll 8
  for (int r = r0; r < r1; ++r) {
    const float *u = a.U + (size_t)r * 3 * a.K + k;
    const MinGruGate g = mingru_gate(u[0], u[a.K]);
    s = fmaf(s, g.keep, g.add);
    st_val(reinterpret_cast<T *>(a.A) + (size_t)r * a.lda + k, mingru_out(s, u[2 * a.K]));
  }
  if (r1 == a.rows) a.State[(size_t)(a.Ctrl[4 * (a.rows - 1) + CTRL_POS] & 1) * a.K + k] = s;
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

// Element k of one step; next may be null (another block stores it).
__device__ __forceinline__ float mingru_step(const float *u, const float *prev, float *next, int K, int k) {
  const MinGruGate g = mingru_gate(u[k], u[K + k]);
  const float s = fmaf(prev ? prev[k] : 0.0f, g.keep, g.add);
  if (next) next[k] = s;
  return mingru_out(s, u[2 * K + k]);
}

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
  const float y = mingru_step(a.U + (size_t)q * 3 * a.K, pos > 0 ? st + (size_t)((pos - 1) & 1) * a.K : nullptr, st + (size_t)(pos & 1) * a.K, a.K, k);
  st_val(reinterpret_cast<T *>(a.A) + (size_t)q * a.lda + k, y);
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
__global__ void __launch_bounds__(kSgThreads, 4) MinGruStreamGemv(const MinGruStreamGemvArgs a) {
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
    const float *prev = pos > 0 ? a.State + (size_t)((pos - 1) & 1) * a.K : nullptr;
    float *next = blockIdx.x == 0 ? a.State + (size_t)(pos & 1) * a.K : nullptr;
#pragma unroll 4
    for (int k = threadIdx.x; k < a.ldw; k += kSgWarps * 32) sg_put(lo, hi, k, k < a.K ? mingru_step(a.U, prev, next, a.K, k) : 0.0f);
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

AINFER_EARLY_LAUNCH(MinGruChunk);
AINFER_EARLY_LAUNCH(MinGruScanF32);
AINFER_EARLY_LAUNCH(MinGruScanB16);
AINFER_EARLY_LAUNCH(MinGruStepRowsF32);
AINFER_EARLY_LAUNCH(MinGruStepRowsB16);
AINFER_EARLY_LAUNCH(MinGruStreamGemv);

}  // namespace ainfer
