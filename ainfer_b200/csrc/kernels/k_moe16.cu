// Mixture of experts with bf16 weights: softmax router whose choice is corrected per expert while the
// weights are not, experts without gates (up, activation, down), and identity experts, which pass their
// input. The router's outputs [E, E + I) are the identities.
//
// Rows (prompt passes, batches): RouterTopRows chooses, MoePlanRows sorts the chosen (row, expert)
// pairs by expert and cuts every expert's rows into tiles, GatherRows brings the inputs into that
// order, two grouped products (LinearTcGrouped in k_linear_tc.cu, LinearRowsGrouped here) leave the
// experts' outputs there, and the consumer of the outputs adds each row's up by place and weight.
// Decode step: ExpertUpStreamGemv chooses for itself in every block and streams the chosen experts'
// rows only; ExpertDownStreamGemv adds the experts' outputs in rank order.
#include "row_types.cuh"
#include "stream_gemv.cuh"

namespace ainfer {

constexpr int kMxMaxExperts = 1024, kMxMaxTop = 32;   // router outputs, chosen ones

// One warp: softmax of lg[0..E), then the `top` largest of softmax + corr (lowest index first among
// equals). sc and ch: E floats of scratch each, of this warp alone. Lane s < top returns the s-th choice.
__device__ __forceinline__ void router_choose(const float *lg, const float *corr, int E, int top, float *sc, float *ch, int &sel, float &w) {
  const int lane = threadIdx.x & 31;
  float mx = -INFINITY;
  for (int e = lane; e < E; e += 32) mx = fmaxf(mx, lg[e]);
  mx = warp_max(mx);
  float sum = 0.0f;
  for (int e = lane; e < E; e += 32) {
    const float v = expf(lg[e] - mx);
    sc[e] = v;
    sum += v;
  }
  sum = warp_tree_sum(sum);
  float best = -INFINITY;   // this lane's best candidate
  int at = INT32_MAX;
  for (int e = lane; e < E; e += 32) {
    const float s = sc[e] / sum, c = s + corr[e];
    sc[e] = s;
    ch[e] = c;
    if (c > best) { best = c; at = e; }
  }
  sel = 0;
  w = 0.0f;
  for (int s = 0; s < top; ++s) {
    const float m = warp_max(best);
    const int e = __reduce_min_sync(kFull, best == m ? at : INT32_MAX);
    if (e >= E) break;                                  // scores that are not numbers: nothing to choose
    if (lane == s) sel = e;
    const float we = __shfl_sync(kFull, (e & 31) == lane ? sc[e] : 0.0f, e & 31);
    if (lane == s) w = we;
    if ((e & 31) == lane) {                             // the owner looks for its next best
      ch[e] = -INFINITY;
      best = -INFINITY;
      at = INT32_MAX;
      for (int j = lane; j < E; j += 32)
        if (ch[j] > best) { best = ch[j]; at = j; }
    }
  }
}

// ------------------------------------------------------- RouterTopRows ---
struct RouterTopRowsArgs {
  const float *Logits;     // [rows][E]
  const float *Corr;       // [E]
  int32_t *Sel;            // [rows][top]
  float *SelW;             // [rows][top]
  int32_t rows, E, top;
};
constexpr int kRtWarps = 4;
__global__ void __launch_bounds__(kRtWarps * 32) RouterTopRows(const RouterTopRowsArgs a) {
  extern __shared__ __align__(16) float rt_smem[];   // [warps][2][E]
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = blockIdx.x * kRtWarps + warp;
  if (r >= a.rows) return;
  float *sc = rt_smem + (size_t)warp * 2 * a.E;
  int sel;
  float w;
  router_choose(a.Logits + (size_t)r * a.E, a.Corr, a.E, a.top, sc, sc + a.E, sel, w);
  if (lane < a.top) {
    a.Sel[(size_t)r * a.top + lane] = sel;
    a.SelW[(size_t)r * a.top + lane] = w;
  }
}
static uint32_t router_top_smem(const void *args) { return (uint32_t)(kRtWarps * 2 * 4) * (uint32_t)((const RouterTopRowsArgs *)args)->E; }
#define F(f) AINFER_ARG(RouterTopRowsArgs, f)
AINFER_REGISTER(RouterTopRows, RouterTopRowsArgs, kRtWarps * 32, kRtWarps, 0, router_top_smem, F(Logits), F(Corr), F(Sel), F(SelW), F(rows), F(E),
                F(top));
#undef F

// --------------------------------------------------------- MoePlanRows ---
// One block. Places of an expert's rows are consecutive; the order of rows within an expert is free (a
// row's result does not depend on its place).
struct MoePlanRowsArgs {
  const int32_t *Sel;      // [rows][top]
  int32_t *Place;          // [rows][top] place, -1: identity
  int32_t *RowOf;          // [places] row
  int4 *Tiles;             // (expert, first place, places, 0)
  int32_t *Count;          // [2] tiles, places
  int32_t rows, top, E, nt;   // E: experts with weights; nt: rows of a tile
};
constexpr int kMpThreads = 1024;
__global__ void __launch_bounds__(kMpThreads) MoePlanRows(const MoePlanRowsArgs a) {
  __shared__ int count[kMxMaxExperts], next[kMxMaxExperts], wsum[2][32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = a.rows * a.top;
  count[tid] = 0;
  __syncthreads();
  for (int i = tid; i < n; i += kMpThreads) {
    const int e = a.Sel[i];
    if (e < a.E) atomicAdd(&count[e], 1);
  }
  __syncthreads();
  // running sums of places and tiles over the experts (one expert per thread)
  const int c = tid < a.E ? count[tid] : 0, t = (c + a.nt - 1) / a.nt;
  int pc = c, pt = t;
#pragma unroll
  for (int off = 1; off < 32; off <<= 1) {
    const int x = __shfl_up_sync(kFull, pc, off), y = __shfl_up_sync(kFull, pt, off);
    if (lane >= off) { pc += x; pt += y; }
  }
  if (lane == 31) { wsum[0][warp] = pc; wsum[1][warp] = pt; }
  __syncthreads();
  if (warp == 0) {
    int x = wsum[0][lane], y = wsum[1][lane];
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const int u = __shfl_up_sync(kFull, x, off), v = __shfl_up_sync(kFull, y, off);
      if (lane >= off) { x += u; y += v; }
    }
    wsum[0][lane] = x;
    wsum[1][lane] = y;
  }
  __syncthreads();
  if (warp > 0) { pc += wsum[0][warp - 1]; pt += wsum[1][warp - 1]; }
  const int p0 = pc - c, t0 = pt - t;
  next[tid] = p0;
  for (int i = 0; i < t; ++i) a.Tiles[t0 + i] = make_int4(tid, p0 + i * a.nt, min(a.nt, c - i * a.nt), 0);
  if (tid == kMpThreads - 1) { a.Count[0] = pt; a.Count[1] = pc; }
  __syncthreads();
  for (int i = tid; i < n; i += kMpThreads) {
    const int e = a.Sel[i];
    int p = -1;
    if (e < a.E) {
      p = atomicAdd(&next[e], 1);
      a.RowOf[p] = i / a.top;
    }
    a.Place[i] = p;
  }
}
#define F(f) AINFER_ARG(MoePlanRowsArgs, f)
AINFER_REGISTER(MoePlanRows, MoePlanRowsArgs, kMpThreads, 0, 0, nullptr, F(Sel), F(Place), F(RowOf), F(Tiles), F(Count), F(rows), F(top), F(E),
                F(nt));
#undef F

// ---------------------------------------------------------- GatherRows ---
// Dst[p] = Src[RowOf[p]] for p < Count[1]; rows of `bytes` (a multiple of 4), strides in bytes.
struct GatherRowsArgs {
  void *Dst;
  const void *Src;
  const int32_t *RowOf, *Count;
  int64_t src_stride, dst_stride;
  int32_t bytes;
};
__global__ void __launch_bounds__(128) GatherRows(const GatherRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int n = a.Count[1];
  const bool wide = ((a.bytes | a.src_stride | a.dst_stride) & 15) == 0;
  for (int p = blockIdx.x; p < n; p += gridDim.x) {
    const char *s = reinterpret_cast<const char *>(a.Src) + (size_t)a.RowOf[p] * a.src_stride;
    char *d = reinterpret_cast<char *>(a.Dst) + (size_t)p * a.dst_stride;
    if (wide) {
#pragma unroll 4
      for (int i = threadIdx.x; i < a.bytes / 16; i += 128) reinterpret_cast<uint4 *>(d)[i] = reinterpret_cast<const uint4 *>(s)[i];
    } else {
      for (int i = threadIdx.x; i < a.bytes / 4; i += 128) reinterpret_cast<uint32_t *>(d)[i] = reinterpret_cast<const uint32_t *>(s)[i];
    }
  }
}
#define F(f) AINFER_ARG(GatherRowsArgs, f)
AINFER_REGISTER(GatherRows, GatherRowsArgs, 128, 0, 0, nullptr, F(Dst), F(Src), F(RowOf), F(Count), F(src_stride), F(dst_stride), F(bytes));
#undef F

// --------------------------------------------------- LinearRowsGrouped ---
// The 32-bit form of the grouped product: tiles of up to 64 rows of one expert, W [E][N][ldw].
struct LinearRowsGroupedArgs {
  const float *X;          // [places][ldx]
  const uint16_t *W;
  float *Y;                // [places][ldy]
  const int4 *Tiles;
  const int32_t *Count;
  int32_t N, K, ldx, ldw, ldy, act;
};
constexpr int kLgTile = 64, kLgK = 16;
__global__ void __launch_bounds__(256) LinearRowsGrouped(const LinearRowsGroupedArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float xs[kLgK][kLgTile + 4], ws[kLgK][kLgTile + 4];
  const int n_tiles = (a.N + kLgTile - 1) / kLgTile, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int units = a.Count[0] * n_tiles;
  for (int u = blockIdx.x; u < units; u += gridDim.x) {
    const int4 t = a.Tiles[u / n_tiles];
    const int n0 = (u % n_tiles) * kLgTile;
    const uint16_t *W = a.W + (size_t)t.x * a.N * a.ldw;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.K; k0 += kLgK) {
      for (int i = tid; i < kLgTile * kLgK; i += 256) {
        const int rr = i / kLgK, k = i % kLgK;
        const bool kin = k0 + k < a.K;
        xs[k][rr] = kin && rr < t.z ? a.X[(size_t)(t.y + rr) * a.ldx + k0 + k] : 0.0f;
        ws[k][rr] = kin && n0 + rr < a.N ? bf16_to_f32(W[(size_t)(n0 + rr) * a.ldw + k0 + k]) : 0.0f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < kLgK; ++k) {
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
      const int r = ty * 4 + i;
      if (r >= t.z) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + tx * 4 + j;
        if (n < a.N) a.Y[(size_t)(t.y + r) * a.ldy + n] = apply_act(acc[i][j], a.act, 0.0f);
      }
    }
  }
}
#define F(f) AINFER_ARG(LinearRowsGroupedArgs, f)
AINFER_REGISTER(LinearRowsGrouped, LinearRowsGroupedArgs, 256, 0, 0, nullptr, F(X), F(W), F(Y), F(Tiles), F(Count), F(N), F(K), F(ldx), F(ldw),
                F(ldy), F(act));
#undef F

// -------------------------------------------------- ExpertUpStreamGemv ---
// grid = top x blocks per expert. Block 0 leaves the choice for the down product.
struct ExpertUpStreamGemvArgs {
  const float *Logits;     // [EI]
  const float *Corr;       // [EI]
  const float *X;          // [K]
  const uint16_t *W;       // [E][N][ldw]
  float *Y;                // [top][N]
  int32_t *Sel;            // [top]
  float *SelW;             // [top]
  int32_t E, EI, top, N, K, ldw, rows_pb, act;
};
__global__ void __launch_bounds__(kSgThreads, 3) ExpertUpStreamGemv(const ExpertUpStreamGemvArgs a) {
  __shared__ GemvShared sh;
  __shared__ int s_sel;
  pdl_launch_dependents();
  const GemvDims d = gemv_dims(a.ldw);
  const int per = gridDim.x / a.top, slot = blockIdx.x / per, n0 = (blockIdx.x % per) * a.rows_pb, n1 = min(a.N, n0 + a.rows_pb);
  const int tid = threadIdx.x, nth = kSgWarps * 32;
  float *lo = reinterpret_cast<float *>(sg_smem + d.nst * d.stage_bytes), *hi = lo + a.ldw / 2, *sc = hi + a.ldw / 2, *part = sc + 2 * a.EI;
  gemv_init(&sh, d.nst);
  pdl_wait();
  if (tid >= nth) {   // the producer's warp chooses while the others bring the vector
    int sel;
    float w;
    router_choose(a.Logits, a.Corr, a.EI, a.top, sc, sc + a.EI, sel, w);
    const int lane = tid & 31;
    if (blockIdx.x == 0 && lane < a.top) { a.Sel[lane] = sel; a.SelW[lane] = w; }
    const int mine = __shfl_sync(kFull, sel, slot);
    if (lane == 0) s_sel = mine;
    __syncwarp();
    asm volatile("bar.arrive 2, 288;" ::: "memory");
    if (lane == 0 && mine < a.E) {
      GemvCursor r{0, 1, 0};
      gemv_produce_rows(a.W + (size_t)mine * a.N * a.ldw, n0, n1, a.ldw, d, &sh, sg_smem, r);
      gemv_produce_end(d, &sh, r);
    }
    __syncwarp();
  } else {
    static_assert(kSgThreads == 288, "barrier 2 counts producer and consumers");
    for (int k = tid; k < a.ldw; k += nth) sg_put(lo, hi, k, k < a.K ? a.X[k] : 0.0f);
    asm volatile("bar.sync 2, 288;" ::: "memory");   // the choice is known, the vector complete
    if (s_sel < a.E) {
      GemvCursor cur{0, 0, 0};
      gemv_consume_rows(n1 - n0, a.ldw, d, &sh, sg_smem, lo, hi, part, cur);
    }
  }
  __syncthreads();
  if (s_sel >= a.E) return;
  for (int n = n0 + tid; n < n1; n += kSgThreads) {
    float v = 0.0f;
    for (int i = 0; i < d.wpr; ++i) v += part[(n - n0) * d.wpr + i];
    a.Y[(size_t)slot * a.N + n] = apply_act(v, a.act, 0.0f);
  }
}
static uint32_t expert_up_smem(const void *args) {
  const ExpertUpStreamGemvArgs *a = (const ExpertUpStreamGemvArgs *)args;
  return gemv_smem(a->ldw, a->rows_pb, 2 * a->EI);
}
#define F(f) AINFER_ARG(ExpertUpStreamGemvArgs, f)
AINFER_REGISTER(ExpertUpStreamGemv, ExpertUpStreamGemvArgs, kSgThreads, 0, 0, expert_up_smem, F(Logits), F(Corr), F(X), F(W), F(Y), F(Sel), F(SelW),
                F(E), F(EI), F(top), F(N), F(K), F(ldw), F(rows_pb), F(act));
#undef F

// ------------------------------------------------ ExpertDownStreamGemv ---
struct ExpertDownStreamGemvArgs {
  const float *A;          // [top][K]
  const float *X;          // [N] input of the mixture (identities)
  const int32_t *Sel;
  const float *SelW;
  const uint16_t *W;       // [E][N][ldw]
  float *Y;                // [N]
  int32_t E, top, N, K, ldw, rows_pb;
};
__global__ void __launch_bounds__(kSgThreads, 3) ExpertDownStreamGemv(const ExpertDownStreamGemvArgs a) {
  __shared__ GemvShared sh;
  pdl_launch_dependents();
  const GemvDims d = gemv_dims(a.ldw);
  const int n0 = blockIdx.x * a.rows_pb, n1 = min(a.N, n0 + a.rows_pb), tid = threadIdx.x, nth = kSgWarps * 32;
  float *vec = reinterpret_cast<float *>(sg_smem + d.nst * d.stage_bytes), *part = vec + (size_t)a.top * a.ldw;
  gemv_init(&sh, d.nst);
  pdl_wait();
  if (tid >= nth) {
    if ((tid & 31) == 0) {
      GemvCursor r{0, 1, 0};
      for (int s = 0; s < a.top; ++s) {
        const int e = a.Sel[s];
        if (e < a.E) gemv_produce_rows(a.W + (size_t)e * a.N * a.ldw, n0, n1, a.ldw, d, &sh, sg_smem, r);
      }
      gemv_produce_end(d, &sh, r);
    }
    __syncwarp();
  } else {
    for (int s = 0; s < a.top; ++s) {
      float *lo = vec + (size_t)s * a.ldw, *hi = lo + a.ldw / 2;
      if (a.Sel[s] < a.E)
        for (int k = tid; k < a.ldw; k += nth) sg_put(lo, hi, k, k < a.K ? a.A[(size_t)s * a.K + k] : 0.0f);
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    GemvCursor cur{0, 0, 0};
    bool any = false;
    for (int s = 0; s < a.top; ++s) {
      if (a.Sel[s] >= a.E) continue;
      const float *lo = vec + (size_t)s * a.ldw, *hi = lo + a.ldw / 2;
      gemv_consume_rows(n1 - n0, a.ldw, d, &sh, sg_smem, lo, hi, part, cur, a.SelW[s], any);
      any = true;
    }
  }
  __syncthreads();
  bool any = false;
  float wx = 0.0f;
  for (int s = 0; s < a.top; ++s) {
    if (a.Sel[s] < a.E) any = true;
    else wx += a.SelW[s];
  }
  for (int n = n0 + tid; n < n1; n += kSgThreads) {
    float v = 0.0f;
    if (any)
      for (int i = 0; i < d.wpr; ++i) v += part[(n - n0) * d.wpr + i];
    a.Y[n] = fmaf(wx, a.X[n], v);
  }
}
static uint32_t expert_down_smem(const void *args) {
  const ExpertDownStreamGemvArgs *a = (const ExpertDownStreamGemvArgs *)args;
  return gemv_smem(a->ldw, a->rows_pb, (a->top - 1) * a->ldw);
}
#define F(f) AINFER_ARG(ExpertDownStreamGemvArgs, f)
AINFER_REGISTER(ExpertDownStreamGemv, ExpertDownStreamGemvArgs, kSgThreads, 0, 0, expert_down_smem, F(A), F(X), F(Sel), F(SelW), F(W), F(Y), F(E),
                F(top), F(N), F(K), F(ldw), F(rows_pb));
#undef F

AINFER_EARLY_LAUNCH(RouterTopRows);
AINFER_EARLY_LAUNCH(MoePlanRows);
AINFER_EARLY_LAUNCH(GatherRows);
AINFER_EARLY_LAUNCH(LinearRowsGrouped);
AINFER_EARLY_LAUNCH(ExpertUpStreamGemv);
AINFER_EARLY_LAUNCH(ExpertDownStreamGemv);

}  // namespace ainfer
