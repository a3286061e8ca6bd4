// Short causal convolution and chunk-local attention whose keys are also its values.
//
//   u      projections of q and k, [rows][C], C = (H + G) D channels (q first), bias included
//   y_t    = sum_j w[c][j] u_(t - taps + 1 + j), u = 0 before the sequence's start
//   score  = (q . k) scale temp_h - LB_h[i - j]      LB_h[d] = r1_h ln(1 + r2_h d), a table
//   row i sees the keys j <= i of its own chunk of positions: j >= i - i % chunk
//   out    = softmax(score) over the keys, times the same keys
//
// The cache of a sequence is a ring of `cap` positions, position p in slot p % cap, one row of G D
// values per slot. A chunk's keys are never needed once the chunk is over, so cap = chunk + (rows a
// pass may hold) positions are enough whatever the context; only keys are stored.
//
// Scores, weights, sums and the convolution are fp32; the cache holds fp32 or bf16.
#include "hyper_core.cuh"

namespace ainfer {

// ------------------------------------------------------- ShortConvRows ---
struct ShortConvRowsArgs {
  const float *U;          // [rows][ldu] projections (q channels, then k channels)
  const float *CW;         // [taps][C]
  const float *State;      // [seq][taps][C]: position p in slot p % taps
  float *Pend;             // [seq][taps][C]: the pass's last taps - 1 positions
  const int32_t *Ctrl, *Seq, *First;
  void *Q;                 // [rows][Qc]
  void *Kc;                // sequence s at + s * kv_stride elements: [cap][C - Qc]
  int64_t kv_stride;
  int32_t rows, C, Qc, taps, cap, ldu, per;   // per: rows of a block
};
// Four channels per thread, TAPS known, the last TAPS - 1 projections in registers.
template <typename T, int TAPS>
__device__ __forceinline__ void short_conv4_body(const ShortConvRowsArgs &a) {
  const int cb = (a.C + 1023) / 1024;
  const int c = ((blockIdx.x % cb) * 256 + threadIdx.x) * 4, r0 = blockIdx.x / cb * a.per;
  if (c >= a.C) return;
  const int r1 = min(a.rows, r0 + a.per), Kn = a.C - a.Qc;
  auto ld4 = [](const float *p) { return *reinterpret_cast<const float4 *>(p); };
  float4 w[TAPS], win[TAPS];   // win[j]: the projection that tap j meets
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = ld4(a.CW + (size_t)j * a.C + c);
  int first = -1;
  for (int r = r0; r < r1; ++r) {
    const int pos = a.Ctrl[4 * r + CTRL_POS], seq = a.Seq[r], f = a.First[r];
    if (f != first) {   // (re)load the history before row r
      first = f;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) {
        const int back = TAPS - 1 - j, p = pos - back;
        win[j + 1] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (r - back >= f) win[j + 1] = ld4(a.U + (size_t)(r - back) * a.ldu + c);
        else if (p >= 0) win[j + 1] = ld4(a.State + ((size_t)seq * TAPS + p % TAPS) * a.C + c);
      }
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) win[j] = win[j + 1];
    win[TAPS - 1] = ld4(a.U + (size_t)r * a.ldu + c);
    float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      y.x = fmaf(w[j].x, win[j].x, y.x); y.y = fmaf(w[j].y, win[j].y, y.y);
      y.z = fmaf(w[j].z, win[j].z, y.z); y.w = fmaf(w[j].w, win[j].w, y.w);
    }
    if (TAPS > 1 && (r + TAPS - 1 >= a.rows || a.First[r + TAPS - 1] != f))   // among the sequence's last TAPS - 1 rows
      *reinterpret_cast<float4 *>(a.Pend + ((size_t)seq * TAPS + pos % TAPS) * a.C + c) = win[TAPS - 1];
    if (c < a.Qc) st_val4(reinterpret_cast<T *>(a.Q) + (size_t)r * a.Qc + c, y);
    else st_val4(reinterpret_cast<T *>(a.Kc) + (size_t)seq * a.kv_stride + (size_t)(pos % a.cap) * Kn + (c - a.Qc), y);
  }
}
// grid = ceil(rows / per) x ceil(C / 1024) with whole quads of channels and 2..4 taps, else x ceil(C / 256)
template <typename T>
__device__ __forceinline__ void short_conv_body(const ShortConvRowsArgs &a) {
  if ((a.C & 3) == 0 && (a.Qc & 3) == 0 && (a.ldu & 3) == 0 && a.taps >= 2 && a.taps <= 4) {
    if (a.taps == 4) short_conv4_body<T, 4>(a);
    else if (a.taps == 3) short_conv4_body<T, 3>(a);
    else short_conv4_body<T, 2>(a);
    return;
  }
  const int cb = (a.C + 255) / 256;
  const int c = (blockIdx.x % cb) * 256 + threadIdx.x, r0 = blockIdx.x / cb * a.per;
  if (c >= a.C) return;
  const int r1 = min(a.rows, r0 + a.per), taps = a.taps, Kn = a.C - a.Qc;
  for (int r = r0; r < r1; ++r) {
    const int pos = a.Ctrl[4 * r + CTRL_POS], seq = a.Seq[r], first = a.First[r];
    const float *st = a.State + (size_t)seq * taps * a.C + c;
    float y = 0.0f, cur = 0.0f;
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j, p = pos - back;
      if (p < 0) continue;
      const float u = r - back >= first ? a.U[(size_t)(r - back) * a.ldu + c] : st[(size_t)(p % taps) * a.C];
      y = fmaf(a.CW[(size_t)j * a.C + c], u, y);
      cur = u;
    }
    // the sequence's last row of this pass is at r + e: keep the last taps - 1 projections
    bool tail = false;
    for (int e = 0; e < taps - 1 && !tail; ++e)
      tail = r + e + 1 == a.rows ? true : (a.First[r + e + 1] != first);
    if (tail && taps > 1) a.Pend[((size_t)seq * taps + pos % taps) * a.C + c] = cur;
    if (c < a.Qc) st_val(reinterpret_cast<T *>(a.Q) + (size_t)r * a.Qc + c, y);
    else st_val(reinterpret_cast<T *>(a.Kc) + (size_t)seq * a.kv_stride + (size_t)(pos % a.cap) * Kn + (c - a.Qc), y);
  }
}
__global__ void __launch_bounds__(256) ShortConvRowsF32(const ShortConvRowsArgs a) { short_conv_body<float>(a); }
__global__ void __launch_bounds__(256) ShortConvRowsB16(const ShortConvRowsArgs a) { short_conv_body<uint16_t>(a); }
#define F(f) AINFER_ARG(ShortConvRowsArgs, f)
#define CONV_FIELDS                                                                                                                \
  F(U), F(CW), F(State), F(Pend), F(Ctrl), F(Seq), F(First), F(Q), F(Kc), F(kv_stride), F(rows), F(C), F(Qc), F(taps), F(cap), \
      F(ldu), F(per)
AINFER_REGISTER(ShortConvRowsF32, ShortConvRowsArgs, 256, 0, 0, nullptr, CONV_FIELDS);
AINFER_REGISTER(ShortConvRowsB16, ShortConvRowsArgs, 256, 0, 0, nullptr, CONV_FIELDS);
#undef F

// ------------------------------------------------------- ChunkAttnRows ---
// Rows of ONE sequence at consecutive positions, their keys already in the cache. A block takes 16
// rows of one query head; keys come in tiles of 32 through shared memory; a warp owns four rows, a
// lane one key of the tile for the scores and the value columns lane, lane + 32, ... for the sums.
struct ChunkAttnRowsArgs {
  const void *Q;           // [rows][H D]
  const void *Kc;          // [cap][G D]
  const float *LB;         // [H][lb_len]
  const float *Temp;       // [H]
  const int32_t *Ctrl;     // [rows][4]
  void *O;                 // [rows][ldo]
  int32_t rows, H, G, D, cap, chunk, lb_len, ldo;
  float scale;
};
constexpr int kCaRows = 16, kCaKeys = 32, kCaMaxD = 512;
template <typename T>
__device__ __forceinline__ void chunk_attn_rows_body(const ChunkAttnRowsArgs &a) {
  extern __shared__ __align__(16) float ca_smem[];   // q [16][D], k [32][D + 1]
  const int D = a.D, h = blockIdx.x % a.H, r0 = blockIdx.x / a.H * kCaRows, g = h / (a.H / a.G);
  float *qs = ca_smem, *ks = ca_smem + kCaRows * D;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nr = min(kCaRows, a.rows - r0), KW = a.G * D;
  const T *Q = reinterpret_cast<const T *>(a.Q), *K = reinterpret_cast<const T *>(a.Kc) + (size_t)g * D;
  for (int i = tid; i < kCaRows * D; i += 128) {
    const int rr = i / D, d = i - rr * D;
    qs[i] = rr < nr ? ld_val(Q + (size_t)(r0 + rr) * a.H * D + (size_t)h * D + d) : 0.0f;
  }
  const int pos0 = a.Ctrl[4 * r0 + CTRL_POS];
  const float mul = a.scale, temp = a.Temp[h];
  const float *lb = a.LB + (size_t)h * a.lb_len;
  float m[4], l[4], acc[4][kCaMaxD / 32];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    m[i] = -INFINITY; l[i] = 0.0f;
#pragma unroll
    for (int x = 0; x < kCaMaxD / 32; ++x) acc[i][x] = 0.0f;
  }
  const int lo = pos0 - pos0 % a.chunk, hi = pos0 + nr - 1;   // the first row's chunk start is the lowest key of the tile
  for (int k0 = lo; k0 <= hi; k0 += kCaKeys) {
    __syncthreads();
    for (int i = tid; i < kCaKeys * D; i += 128) {
      const int kk = i / D, d = i - kk * D, p = k0 + kk;
      ks[kk * (D + 1) + d] = p <= hi ? ld_val(K + (size_t)(p % a.cap) * KW + d) : 0.0f;
    }
    __syncthreads();
    const int kp = k0 + lane;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int rr = warp * 4 + i, p = pos0 + rr;
      if (rr >= nr) continue;
      const bool see = kp <= p && kp >= p - p % a.chunk;
      float s = -INFINITY;
      if (see) {
        float dot = 0.0f;
        const float *q = qs + rr * D, *k = ks + lane * (D + 1);
        for (int d = 0; d < D; ++d) dot = fmaf(q[d], k[d], dot);
        s = dot * mul * temp - lb[p - kp];
      }
      const float mx = fmaxf(m[i], warp_max(s));
      if (mx == -INFINITY) continue;   // nothing visible yet (uniform over the warp)
      const float corr = expf(m[i] - mx), w = see ? expf(s - mx) : 0.0f;
      m[i] = mx;
      l[i] = fmaf(l[i], corr, warp_tree_sum(w));
#pragma unroll
      for (int x = 0; x < kCaMaxD / 32; ++x)
        if (x * 32 < D) acc[i][x] *= corr;
      for (int j = 0; j < kCaKeys; ++j) {
        const float wj = __shfl_sync(kFull, w, j);
#pragma unroll
        for (int x = 0; x < kCaMaxD / 32; ++x)
          if (x * 32 < D) {
            const int d = x * 32 + lane;
            if (d < D) acc[i][x] = fmaf(wj, ks[j * (D + 1) + d], acc[i][x]);
          }
      }
    }
  }
  T *O = reinterpret_cast<T *>(a.O);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int rr = warp * 4 + i;
    if (rr >= nr) continue;
#pragma unroll
    for (int x = 0; x < kCaMaxD / 32; ++x) {
      const int d = x * 32 + lane;
      if (d < D) st_val(O + (size_t)(r0 + rr) * a.ldo + (size_t)h * D + d, acc[i][x] / l[i]);
    }
  }
}
__global__ void __launch_bounds__(128) ChunkAttnRowsF32(const ChunkAttnRowsArgs a) { chunk_attn_rows_body<float>(a); }
__global__ void __launch_bounds__(128) ChunkAttnRowsB16(const ChunkAttnRowsArgs a) { chunk_attn_rows_body<uint16_t>(a); }
static uint32_t chunk_attn_rows_smem(const void *args) {
  const int D = ((const ChunkAttnRowsArgs *)args)->D;
  return 4u * (uint32_t)(kCaRows * D + kCaKeys * (D + 1));
}
#define F(f) AINFER_ARG(ChunkAttnRowsArgs, f)
#define CAR_FIELDS F(Q), F(Kc), F(LB), F(Temp), F(Ctrl), F(O), F(rows), F(H), F(G), F(D), F(cap), F(chunk), F(lb_len), F(ldo), F(scale)
AINFER_REGISTER(ChunkAttnRowsF32, ChunkAttnRowsArgs, 128, 0, 0, chunk_attn_rows_smem, CAR_FIELDS);
AINFER_REGISTER(ChunkAttnRowsB16, ChunkAttnRowsArgs, 128, 0, 0, chunk_attn_rows_smem, CAR_FIELDS);
#undef F

// ------------------------------------------------------- ChunkAttnStep ---
// One decode step of every sequence: convolution, append, and attention over the sequence's current
// chunk in one launch. Blocks: sequence x key head x split. A split takes a contiguous share of the
// chunk's keys; the last block of a (sequence, key head) to finish merges the splits in their order.
// The convolution history is a ring over positions in which a step writes the one slot it does not
// read, so the blocks of a sequence need no order among themselves.
struct ChunkAttnStepArgs {
  const float *U;          // [seq][ldu]
  const float *CW;         // [taps][C]
  float *State;            // [seq][taps][C]
  const int32_t *Ctrl;     // [seq][4]
  void *Kc;
  int64_t kv_stride;
  const float *LB;         // [H][lb_len]
  const float *Temp;       // [H]
  float *Part;             // [seq][G][splits][HG (D + 2)]: per head m, l, then the D sums
  uint32_t *Count;         // [seq][G], zero between launches
  void *O;                 // [seq][ldo]
  int32_t nseq, H, G, D, taps, cap, chunk, lb_len, splits, ldu, ldo, out16;   // out16: O holds bf16
  float scale;
};
constexpr int kCsKeys = 64, kCsThreads = 256;
// floats of shared memory: q [HG][D], new key [D], key tile [64][D + 1], scores [HG][64], head state
// [HG] x 3 (maximum, correction, sum), sums [HG][D]
__host__ __device__ inline uint32_t chunk_step_floats(int HG, int D) {
  return (uint32_t)(2 * HG * D + D + kCsKeys * (D + 1) + HG * kCsKeys + 3 * HG);
}
template <typename T>
__device__ __forceinline__ void chunk_attn_step_body(const ChunkAttnStepArgs &a) {
  extern __shared__ __align__(16) float cs_smem[];
  __shared__ int s_last;
  const int D = a.D, HG = a.H / a.G, C = (a.H + a.G) * D, Qc = a.H * D, KW = a.G * D;
  const int split = blockIdx.x % a.splits, g = blockIdx.x / a.splits % a.G, seq = blockIdx.x / (a.splits * a.G);
  if (seq >= a.nseq) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *qs = cs_smem, *kn = qs + HG * D, *ks = kn + D, *sc = ks + kCsKeys * (D + 1), *hm = sc + HG * kCsKeys, *hc = hm + HG, *hl = hc + HG,
        *acc = hl + HG;
  const int pos = a.Ctrl[4 * seq + CTRL_POS];
  const int lo = pos - pos % a.chunk, count = pos - lo + 1;
  const int per = max(kCsKeys, (count + a.splits - 1) / a.splits), active = (count + per - 1) / per;
  if (split >= active) return;
  const int k_lo = lo + split * per, k_hi = min(pos, k_lo + per - 1);
  float *st = a.State + (size_t)seq * a.taps * C;
  const float *u0 = a.U + (size_t)seq * a.ldu;
  T *K = reinterpret_cast<T *>(a.Kc) + (size_t)seq * a.kv_stride + (size_t)g * D;
  // ---- convolution of this key head's channels ----
  for (int i = tid; i < (HG + 1) * D; i += kCsThreads) {
    const bool isk = i >= HG * D;
    const int c = isk ? Qc + g * D + (i - HG * D) : g * HG * D + i;
    float y = 0.0f;
    for (int j = 0; j < a.taps - 1; ++j) {
      const int p = pos - (a.taps - 1 - j);
      if (p >= 0) y = fmaf(a.CW[(size_t)j * C + c], st[(size_t)(p % a.taps) * C + c], y);
    }
    const float u = u0[c];
    y = fmaf(a.CW[(size_t)(a.taps - 1) * C + c], u, y);
    if (split == 0) st[(size_t)(pos % a.taps) * C + c] = u;
    if (isk) {
      T t;
      st_val(&t, y);
      kn[i - HG * D] = ld_val(&t);
      if (k_hi == pos) K[(size_t)(pos % a.cap) * KW + (i - HG * D)] = t;
    } else {
      qs[i] = y;
    }
  }
  for (int i = tid; i < HG * D; i += kCsThreads) acc[i] = 0.0f;
  for (int i = tid; i < HG; i += kCsThreads) { hm[i] = -INFINITY; hl[i] = 0.0f; }
  __syncthreads();
  for (int t0 = k_lo; t0 <= k_hi; t0 += kCsKeys) {
    const int nk = min(kCsKeys, k_hi - t0 + 1);
    if ((D & 7) == 0 && sizeof(T) == 2) {
      const int pr = D >> 3;
      for (int i = tid; i < nk * pr; i += kCsThreads) {
        const int kk = i / pr, d = (i - kk * pr) * 8, p = t0 + kk;
        if (p != pos) {
          const uint4 v = *reinterpret_cast<const uint4 *>(K + (size_t)(p % a.cap) * KW + d);
          float *o = ks + kk * (D + 1) + d;
          o[0] = u2f(v.x << 16); o[1] = u2f(v.x & 0xFFFF0000u); o[2] = u2f(v.y << 16); o[3] = u2f(v.y & 0xFFFF0000u);
          o[4] = u2f(v.z << 16); o[5] = u2f(v.z & 0xFFFF0000u); o[6] = u2f(v.w << 16); o[7] = u2f(v.w & 0xFFFF0000u);
        } else {
          for (int x = 0; x < 8; ++x) ks[kk * (D + 1) + d + x] = kn[d + x];
        }
      }
    } else {
      for (int i = tid; i < nk * D; i += kCsThreads) {
        const int kk = i / D, d = i - kk * D, p = t0 + kk;
        ks[kk * (D + 1) + d] = p != pos ? ld_val(K + (size_t)(p % a.cap) * KW + d) : kn[d];
      }
    }
    __syncthreads();
    {
      const int kk = tid & (kCsKeys - 1);
      for (int hh = tid / kCsKeys; hh < HG; hh += kCsThreads / kCsKeys) {
        float s = -INFINITY;
        if (kk < nk) {
          const float *q = qs + hh * D, *k = ks + kk * (D + 1);
          float d0 = 0.0f, d1 = 0.0f;
          int d = 0;
          for (; d + 1 < D; d += 2) { d0 = fmaf(q[d], k[d], d0); d1 = fmaf(q[d + 1], k[d + 1], d1); }
          if (d < D) d0 = fmaf(q[d], k[d], d0);
          const int h = g * HG + hh;
          s = (d0 + d1) * a.scale * a.Temp[h] - a.LB[(size_t)h * a.lb_len + (pos - t0 - kk)];
        }
        sc[hh * kCsKeys + kk] = s;
      }
    }
    __syncthreads();
    for (int hh = warp; hh < HG; hh += kCsThreads / 32) {
      const float s0 = sc[hh * kCsKeys + lane], s1 = sc[hh * kCsKeys + 32 + lane];
      const float mx = fmaxf(hm[hh], warp_max(fmaxf(s0, s1)));
      const float w0 = lane < nk ? expf(s0 - mx) : 0.0f, w1 = lane + 32 < nk ? expf(s1 - mx) : 0.0f;
      const float sum = warp_tree_sum(w0 + w1);
      sc[hh * kCsKeys + lane] = w0;
      sc[hh * kCsKeys + 32 + lane] = w1;
      __syncwarp();
      if (lane == 0) {
        const float corr = expf(hm[hh] - mx);
        hc[hh] = corr;
        hl[hh] = fmaf(hl[hh], corr, sum);
        hm[hh] = mx;
      }
    }
    __syncthreads();
    for (int i = tid; i < HG * D; i += kCsThreads) {
      const int hh = i / D, d = i - hh * D;
      float v = acc[i] * hc[hh];
      const float *w = sc + hh * kCsKeys;
      for (int kk = 0; kk < nk; ++kk) v = fmaf(w[kk], ks[kk * (D + 1) + d], v);
      acc[i] = v;
    }
    __syncthreads();
  }
  auto put = [&](int h, int d, float v) {
    const size_t o = (size_t)seq * a.ldo + (size_t)h * D + d;
    if (a.out16) reinterpret_cast<uint16_t *>(a.O)[o] = f32_to_bf16(v);
    else reinterpret_cast<float *>(a.O)[o] = v;
  };
  if (active == 1) {
    for (int i = tid; i < HG * D; i += kCsThreads) put(g * HG + i / D, i % D, acc[i] / hl[i / D]);
    return;
  }
  const int per_head = D + 2;
  float *base = a.Part + ((size_t)seq * a.G + g) * a.splits * HG * per_head;
  float *mine = base + (size_t)split * HG * per_head;
  for (int i = tid; i < HG * D; i += kCsThreads) __stcg(mine + (size_t)(i / D) * per_head + 2 + i % D, acc[i]);
  for (int i = tid; i < HG; i += kCsThreads) { __stcg(mine + (size_t)i * per_head, hm[i]); __stcg(mine + (size_t)i * per_head + 1, hl[i]); }
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    const uint32_t n = atomicAdd(a.Count + (size_t)seq * a.G + g, 1u);
    s_last = n + 1 == (uint32_t)active;
    if (s_last) a.Count[(size_t)seq * a.G + g] = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  for (int hh = tid; hh < HG; hh += kCsThreads) {
    float mx = -INFINITY;
    for (int s = 0; s < active; ++s) mx = fmaxf(mx, __ldcg(base + ((size_t)s * HG + hh) * per_head));
    float l = 0.0f;
    for (int s = 0; s < active; ++s) {
      const float *p = base + ((size_t)s * HG + hh) * per_head;
      l = fmaf(__ldcg(p + 1), expf(__ldcg(p) - mx), l);
    }
    hm[hh] = mx; hl[hh] = l;
  }
  __syncthreads();
  for (int i = tid; i < HG * D; i += kCsThreads) {
    const int hh = i / D, d = i - hh * D;
    float v = 0.0f;
    for (int s = 0; s < active; ++s) {
      const float *p = base + ((size_t)s * HG + hh) * per_head;
      v = fmaf(__ldcg(p + 2 + d), expf(__ldcg(p) - hm[hh]), v);
    }
    put(g * HG + hh, d, v / hl[hh]);
  }
}
__global__ void __launch_bounds__(kCsThreads) ChunkAttnStepF32(const ChunkAttnStepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  chunk_attn_step_body<float>(a);
}
__global__ void __launch_bounds__(kCsThreads) ChunkAttnStepB16(const ChunkAttnStepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  chunk_attn_step_body<uint16_t>(a);
}
static uint32_t chunk_step_smem(const void *args) {
  const ChunkAttnStepArgs *a = (const ChunkAttnStepArgs *)args;
  return 4u * chunk_step_floats(a->H / a->G, a->D);
}
#define F(f) AINFER_ARG(ChunkAttnStepArgs, f)
#define CAS_FIELDS                                                                                                              \
  F(U), F(CW), F(State), F(Ctrl), F(Kc), F(kv_stride), F(LB), F(Temp), F(Part), F(Count), F(O), F(nseq), F(H), F(G), F(D), F(taps), \
      F(cap), F(chunk), F(lb_len), F(splits), F(ldu), F(ldo), F(out16), F(scale)
AINFER_REGISTER(ChunkAttnStepF32, ChunkAttnStepArgs, kCsThreads, 0, 0, chunk_step_smem, CAS_FIELDS);
AINFER_REGISTER(ChunkAttnStepB16, ChunkAttnStepArgs, kCsThreads, 0, 0, chunk_step_smem, CAS_FIELDS);
#undef F

AINFER_EARLY_LAUNCH(ChunkAttnStepF32);
AINFER_EARLY_LAUNCH(ChunkAttnStepB16);

// LB[h][d] = r1_h ln(1 + r2_h d), evaluated in double and rounded once.
struct LogDistanceTableArgs {
  float *LB;               // [H][len]
  const float *R1, *R2;    // [H]
  int32_t H, len;
};
__global__ void __launch_bounds__(256) LogDistanceTable(const LogDistanceTableArgs a) {
  const size_t n = (size_t)a.H * a.len;
  for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (size_t)gridDim.x * 256) {
    const int h = (int)(i / a.len), d = (int)(i % a.len);
    a.LB[i] = (float)((double)a.R1[h] * log1p((double)a.R2[h] * (double)d));
  }
}
#define F(f) AINFER_ARG(LogDistanceTableArgs, f)
AINFER_REGISTER(LogDistanceTable, LogDistanceTableArgs, 256, 0, 0, nullptr, F(LB), F(R1), F(R2), F(H), F(len));
#undef F

}  // namespace ainfer
