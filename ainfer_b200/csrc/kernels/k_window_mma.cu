// Windowed attention with pooled blocks and sinks (window_attn.cuh) in bf16 on the tensor cores, for key
// and value sizes that are multiples of 8 up to 256. Block means and tokens are walked as one run of
// tiles of 64 keys, means first. Scores, caps, maxima, weights and sums are fp32; the weights are
// rounded to bf16 for the second product only.
//
//   WindowAttnMma       rows of one sequence: a block takes 64 rows of one query head, a warp 16 rows
//   WindowAttnStepMma   a decode step of every sequence (up to 16 query heads per key head): the heads
//                       are the 16 rows of the products, a warp takes 16 keys of every tile of 64
#include "attn_mma.cuh"
#include "window_attn.cuh"

namespace ainfer {

__device__ __forceinline__ float fast_rcp(float x) {   // one instruction, 1 ulp
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float fast_logistic(float v) { return fast_rcp(1.0f + fast_exp2(-v * kLog2e)); }
// A product q . k to a score in powers of two: scale, and cap tanh(. / cap) as cap - 2 cap / (1 + e^(2 . / cap)).
// bounded: a cap so low that weights relative to it, 2^(score - cap), cannot underflow.
constexpr float kUnseen = -3.0e38f;   // in the place of a product whose key the row does not see
struct ScoreMap {
  float mul, c, c2;   // c2 = 0: no cap
  bool bounded;
  __device__ __forceinline__ ScoreMap(float scale, float cap)
      : mul(cap > 0.0f ? 2.0f * scale / cap * kLog2e : scale * kLog2e), c(cap * kLog2e), c2(cap > 0.0f ? -2.0f * cap * kLog2e : 0.0f),
        bounded(cap > 0.0f && 2.0f * cap * kLog2e < 100.0f) {}
  __device__ __forceinline__ float below(float s) const { return c2 * fast_rcp(1.0f + fast_exp2(s * mul)); }   // score - cap
  __device__ __forceinline__ float operator()(float s) const { return c2 != 0.0f ? below(s) + c : s * mul; }
};

// ------------------------------------------------------ WindowAttnMma ---
struct WindowAttnMmaArgs {
  const uint16_t *Q;         // [rows][H D]
  const uint16_t *Kc, *Vc;   // [cap][G D], [cap][G E], cap a multiple of 64
  const uint16_t *Pk, *Pv;   // [blocks rounded up to 64][G D], [..][G E]; null: no blocks
  const float *Sink;         // [H] or null
  const float *Gate;         // [rows][ldg] or null
  const int32_t *Ctrl;       // [rows][4]
  uint16_t *O;               // [rows][ldo]
  int32_t rows, H, G, D, E, cap, window, pool, ldg, ldo;
  float scale, softcap;
};
constexpr int kWmRows = 64;
template <int DP>
__device__ __forceinline__ void window_attn_mma_body(const WindowAttnMmaArgs &a) {
  extern __shared__ __align__(128) unsigned char wm_raw[];
  constexpr int LD = DP + 8;
  uint16_t *Qs = reinterpret_cast<uint16_t *>(wm_raw);                // [64][LD]
  const uint32_t qa = cm_smem(Qs), ka = qa + kWmRows * LD * 2, va = ka + 2 * kCmKeys * LD * 2;   // keys [2][64][LD], values [64][LD]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int tiles = (a.rows + kWmRows - 1) / kWmRows;
  const int h = blockIdx.x % a.H, r0 = (tiles - 1 - blockIdx.x / a.H) * kWmRows, g = h / (a.H / a.G);   // long rows first
  const int nr = min(kWmRows, a.rows - r0), KW = a.G * a.D, VW = a.G * a.E;
  {
    constexpr int P = DP / 8;
    for (int i = tid; i < kWmRows * P; i += 128) {
      const int r = i / P, c = i % P;
      const bool in = r < nr && c * 8 < a.D;
      cpa16(qa + (uint32_t)(r * LD + c * 8) * 2, a.Q + (in ? ((size_t)(r0 + r) * a.H + h) * a.D + c * 8 : 0), in);
    }
  }
  const int p0 = a.Ctrl[4 * r0 + CTRL_POS], p1 = p0 + nr - 1;
  const int nb0 = a.Pk ? blocks_seen(p0, a.window, a.pool) : 0, nb1 = a.Pk ? blocks_seen(p1, a.window, a.pool) : 0;
  const int lo0 = max(0, p0 - a.window + 1), kb0 = lo0 / kCmKeys * kCmKeys;
  const int nbt = (nb1 + kCmKeys - 1) / kCmKeys, nt = nbt + (p1 - kb0) / kCmKeys + 1;
  const uint16_t *K = a.Kc + (size_t)g * a.D, *V = a.Vc + (size_t)g * a.E, *PK = a.Pk + (size_t)g * a.D, *PV = a.Pv + (size_t)g * a.E;
  auto fetch = [&](int t, bool vals) {   // one commit group: the keys or the values of tile t
    const bool pooled = t < nbt;
    const int at = pooled ? t * kCmKeys : (kb0 + (t - nbt) * kCmKeys) % a.cap;
    if (vals) load_keys<DP, 128>(va, pooled ? PV : V, at, VW, a.E);
    else load_keys<DP, 128>(ka + (uint32_t)((t & 1) * kCmKeys * LD) * 2, pooled ? PK : K, at, KW, a.D);
    cpa_commit();
  };
  fetch(0, false);
  const ScoreMap map(a.scale, a.softcap);
  float o[DP / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
  for (int d = 0; d < DP / 8; ++d)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[d][i] = 0.0f;
  const uint32_t qw = qa + (uint32_t)((warp * 16 + (lane & 15)) * LD + (lane >> 4) * 8) * 2;
  const int rw = warp * 16 + (lane >> 2);                 // this thread's rows rw and rw + 8
  for (int t = 0; t < nt; ++t) {
    cpa_wait<0>();
    __syncthreads();   // the keys are there; every warp is done with the values before and the keys two tiles ago
    fetch(t, true);
    const bool more = t + 1 < nt;
    if (more) fetch(t + 1, false);
    float s[kCmKeys / 8][4];
    scores_smem<DP, kCmKeys>(s, qw, ka + (uint32_t)((t & 1) * kCmKeys * LD) * 2, lane);
    const bool pooled = t < nbt;
    const int k0 = pooled ? t * kCmKeys : kb0 + (t - nbt) * kCmKeys;
    const bool whole = pooled ? k0 + kCmKeys <= nb0 : k0 + kCmKeys - 1 <= p0 && k0 > p1 - a.window;   // every row sees every key of the tile
    if (!whole) {
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int p = p0 + rw + 8 * x;
        const int first = pooled ? 0 : p - a.window + 1, last = pooled ? blocks_seen(p, a.window, a.pool) - 1 : p;   // the keys this row sees
#pragma unroll
        for (int n = 0; n < kCmKeys / 8; ++n)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int key = k0 + n * 8 + (lane & 3) * 2 + e;
            if (key < first || key > last) s[n][2 * x + e] = kUnseen;
          }
      }
    }
    float sum[2] = {0.0f, 0.0f};
    if (map.bounded) {   // weights relative to the cap itself: no maximum to follow
#pragma unroll
      for (int n = 0; n < kCmKeys / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float w = fast_exp2(map.below(s[n][i]));
          s[n][i] = whole || s[n][i] != kUnseen ? w : 0.0f;
          sum[i >> 1] += s[n][i];
        }
      l[0] += sum[0];
      l[1] += sum[1];
    } else {
      float mx[2] = {m[0], m[1]};
#pragma unroll
      for (int n = 0; n < kCmKeys / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float v = map(s[n][i]);
          s[n][i] = whole || s[n][i] != kUnseen ? v : -INFINITY;
          mx[i >> 1] = fmaxf(mx[i >> 1], s[n][i]);
        }
      float corr[2], base[2];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        mx[x] = quad_max(mx[x]);
        base[x] = mx[x] == -INFINITY ? 0.0f : mx[x];
        corr[x] = fast_exp2(m[x] - base[x]);
        m[x] = mx[x];
      }
#pragma unroll
      for (int n = 0; n < kCmKeys / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          s[n][i] = fast_exp2(s[n][i] - base[i >> 1]);
          sum[i >> 1] += s[n][i];
        }
#pragma unroll
      for (int x = 0; x < 2; ++x) l[x] = fmaf(l[x], corr[x], sum[x]);
      if (__any_sync(kFull, corr[0] != 1.0f || corr[1] != 1.0f)) {   // some row's maximum moved
#pragma unroll
        for (int d = 0; d < DP / 8; ++d)
#pragma unroll
          for (int i = 0; i < 4; ++i) o[d][i] *= corr[i >> 1];
      }
    }
    if (more) cpa_wait<1>(); else cpa_wait<0>();
    __syncthreads();   // the values are there
    values<DP, kCmKeys>(o, s, va, lane);
  }
  if (map.bounded) m[0] = m[1] = map.c;
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    float den = quad_sum(l[x]);
    if (a.Sink) den += fast_exp2(a.Sink[h] * kLog2e - m[x]);
    l[x] = 1.0f / den;
  }
#pragma unroll
  for (int d = 0; d < DP / 8; ++d)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = rw + 8 * x, c = d * 8 + (lane & 3) * 2;
      if (r >= nr || c >= a.E) continue;
      float v0 = o[d][2 * x] * l[x], v1 = o[d][2 * x + 1] * l[x];
      if (a.Gate) {
        const float *gp = a.Gate + (size_t)(r0 + r) * a.ldg + (size_t)h * a.E + c;
        v0 *= fast_logistic(gp[0]);
        v1 *= fast_logistic(gp[1]);
      }
      *reinterpret_cast<uint32_t *>(a.O + (size_t)(r0 + r) * a.ldo + (size_t)h * a.E + c) = pack2(v0, v1);
    }
}
#define WINDOW_MMA(DP, BLOCKS)                                                                                      \
  __global__ void __launch_bounds__(128, BLOCKS) WindowAttnMma##DP(const __grid_constant__ WindowAttnMmaArgs a) {   \
    pdl_launch_dependents();                                                                                        \
    pdl_wait();                                                                                                     \
    window_attn_mma_body<DP>(a);                                                                                    \
  }                                                                                                                 \
  static uint32_t window_mma_smem##DP(const void *) { return (kWmRows + 3 * kCmKeys) * (DP + 8) * 2; }
WINDOW_MMA(32, 4)
WINDOW_MMA(64, 4)
WINDOW_MMA(96, 3)
WINDOW_MMA(128, 3)
WINDOW_MMA(192, 2)
WINDOW_MMA(256, 1)
#define F(f) AINFER_ARG(WindowAttnMmaArgs, f)
#define WM_FIELDS                                                                                                                              \
  F(Q), F(Kc), F(Vc), F(Pk), F(Pv), F(Sink), F(Gate), F(Ctrl), F(O), F(rows), F(H), F(G), F(D), F(E), F(cap), F(window), F(pool), F(ldg), \
      F(ldo), F(scale), F(softcap)
#define WM_REGISTER(DP) AINFER_REGISTER(WindowAttnMma##DP, WindowAttnMmaArgs, 128, 0, 0, window_mma_smem##DP, WM_FIELDS); AINFER_EARLY_LAUNCH(WindowAttnMma##DP)
WM_REGISTER(32);
WM_REGISTER(64);
WM_REGISTER(96);
WM_REGISTER(128);
WM_REGISTER(192);
WM_REGISTER(256);
#undef F

// -------------------------------------------------- WindowAttnStepMma ---
// Blocks: sequence x key head x (splits + 1); the extra block appends and averages (see WindowAttnStep).
struct WindowAttnStepMmaArgs {
  const float *U;          // [seq][ldu]: q at 0, k at koff, v at voff, output gate at goff
  const float *QN, *KN;    // [D] or null
  const float2 *Rot;       // [position][rd / 2]
  const int32_t *Ctrl;     // [seq][4]
  uint16_t *Kc, *Vc, *Pk, *Pv;
  int64_t k_stride, v_stride, pk_stride, pv_stride;
  const float *Sink;       // [H] or null
  float *Part;             // [seq][G] blocks of splits HG (E + 4) floats
  uint32_t *Count;         // [seq][G], zero between launches
  void *O;                 // [seq][ldo]
  int32_t nseq, H, G, D, E, rd, cap, window, pool, koff, voff, goff;
  int32_t own_pool, splits, ldu, ldo, out16;   // splits <= 16
  float scale, softcap, eps;
};
constexpr int kWsStages = 2, kWsMaxSplits = 16;
template <int DP>
__device__ __forceinline__ void window_step_mma_body(const WindowAttnStepMmaArgs &a) {
  extern __shared__ __align__(128) unsigned char sm_raw[];
  __shared__ float wm[4][16], wl[4][16];
  __shared__ int s_last;
  constexpr int LD = DP + 8;
  uint16_t *Qs = reinterpret_cast<uint16_t *>(sm_raw);                // [16][LD]
  uint16_t *kn = Qs + 16 * LD, *vn = kn + LD;                         // the new key and value [DP]
  uint16_t *Ks = vn + LD, *Vs = Ks + kWsStages * kCmKeys * LD;        // [stages][64][LD] each
  const int D = a.D, E = a.E, HG = a.H / a.G, KW = a.G * D, VW = a.G * E;
  const int per_seq = a.splits + 1, split = blockIdx.x % per_seq, g = blockIdx.x / per_seq % a.G, seq = blockIdx.x / (per_seq * a.G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos = a.Ctrl[4 * seq + CTRL_POS];
  const float *u = a.U + (size_t)seq * a.ldu;
  const float2 *rot = a.Rot + (size_t)pos * (a.rd >> 1);
  uint16_t *K = a.Kc + (size_t)seq * a.k_stride + (size_t)g * D, *V = a.Vc + (size_t)seq * a.v_stride + (size_t)g * E;
  uint16_t *PK = a.Pk + (size_t)seq * a.pk_stride + (size_t)g * D, *PV = a.Pv + (size_t)seq * a.pv_stride + (size_t)g * E;
  const bool fresh = a.koff >= 0;
  auto new_key = [&]() {   // warp 2: the key, warp 3: the value
    if (!fresh) return;
    if (warp == 2) head_norm_turn(u + a.koff + (size_t)g * D, D, a.KN, a.eps, rot, a.rd, [&](int d, float x, float y, bool both) { st_pair(kn + d, x, y, both); });
    if (warp == 3)
      for (int d = lane; d < E; d += 32) vn[d] = f32_to_bf16(u[a.voff + (size_t)g * E + d]);
  };
  if (split == a.splits) {
    const bool done = a.own_pool && a.pool > 0 && (pos + 1) % a.pool == 0;
    if (!fresh && !done) return;
    new_key();
    __syncthreads();
    for (int i = tid; i < D + E; i += 128) {
      const bool isv = i >= D;
      const int x = isv ? i - D : i, w = isv ? VW : KW;
      uint16_t *ring = (isv ? V : K) + x;
      const uint16_t mine = fresh ? (isv ? vn[x] : kn[x]) : ring[(size_t)(pos % a.cap) * w];
      if (fresh) ring[(size_t)(pos % a.cap) * w] = mine;
      if (done) {
        float s = 0.0f;
        int at = (pos - a.pool + 1) % a.cap;
#pragma unroll 8
        for (int j = 1; j < a.pool; ++j) {
          s += bf16_to_f32(ring[(size_t)at * w]);
          if (++at == a.cap) at = 0;
        }
        (isv ? PV : PK)[(size_t)(pos / a.pool) * w + x] = f32_to_bf16((s + bf16_to_f32(mine)) / (float)a.pool);
      }
    }
    return;
  }
  const int lo = max(0, pos - a.window + 1), nb = a.Pk ? blocks_seen(pos, a.window, a.pool) : 0;
  const int nbt = (nb + kCmKeys - 1) / kCmKeys, tok0 = lo / kCmKeys, nt = nbt + pos / kCmKeys - tok0 + 1;   // tiles: means, then tokens
  const int per = (nt + a.splits - 1) / a.splits, active = (nt + per - 1) / per;
  if (split >= active) return;
  const int t0 = split * per, t1 = min(nt, t0 + per);
  const uint32_t ka = cm_smem(Ks), va = cm_smem(Vs);
  auto fetch = [&](int t) {
    if (t < t1) {
      const uint32_t o = (uint32_t)(((t - t0) % kWsStages) * kCmKeys * LD) * 2;
      const bool pooled = t < nbt;
      const int at = pooled ? t * kCmKeys : (tok0 + t - nbt) * kCmKeys % a.cap;
      load_keys<DP, 128>(ka + o, pooled ? PK : K, at, KW, D);
      load_keys<DP, 128>(va + o, pooled ? PV : V, at, VW, E);
    }
    cpa_commit();
  };
  for (int i = 0; i < kWsStages - 1; ++i) fetch(t0 + i);
  for (int i = tid; i < 16 * LD; i += 128) Qs[i] = 0;
  __syncthreads();
  for (int hh = warp; hh < HG; hh += 4)
    head_norm_turn(u + (size_t)(g * HG + hh) * D, D, a.QN, a.eps, rot, a.rd, [&](int d, float x, float y, bool both) { st_pair(Qs + hh * LD + d, x, y, both); });
  new_key();
  __syncthreads();
  uint32_t q[DP / 16][4];
#pragma unroll
  for (int kk = 0; kk < DP / 16; ++kk) ldm4(q[kk], cm_smem(Qs) + (uint32_t)((lane & 15) * LD + kk * 16 + (lane >> 4) * 8) * 2);
  const ScoreMap map(a.scale, a.softcap);
  float o[DP / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
  for (int d = 0; d < DP / 8; ++d)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[d][i] = 0.0f;
  for (int t = t0; t < t1; ++t) {
    const bool pooled = t < nbt;
    const int k0 = (pooled ? t : tok0 + t - nbt) * kCmKeys + warp * 16, stage = (t - t0) % kWsStages;
    cpa_wait<kWsStages - 2>();
    __syncthreads();
    if (fresh && t == nt - 1) {   // the step's own key and value into the tile
      const int row = (stage * kCmKeys + pos % kCmKeys) * LD;
      for (int i = tid; i < D; i += 128) Ks[row + i] = kn[i];
      for (int i = tid; i < E; i += 128) Vs[row + i] = vn[i];
      __syncthreads();
    }
    fetch(t + kWsStages - 1);
    const uint32_t off = (uint32_t)((stage * kCmKeys + warp * 16) * LD) * 2;
    float s[2][4];
    scores<DP, 16>(s, q, ka + off, lane);
    const int first = pooled ? 0 : lo, last = pooled ? nb - 1 : pos;
    float mx[2] = {m[0], m[1]};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int key = k0 + n * 8 + (lane & 3) * 2 + (i & 1);
        s[n][i] = key < first || key > last ? -INFINITY : map(s[n][i]);
        mx[i >> 1] = fmaxf(mx[i >> 1], s[n][i]);
      }
    float corr[2], sum[2] = {0.0f, 0.0f}, base[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      mx[x] = quad_max(mx[x]);
      base[x] = mx[x] == -INFINITY ? 0.0f : mx[x];
      corr[x] = fast_exp2(m[x] - base[x]);
      m[x] = mx[x];
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        s[n][i] = fast_exp2(s[n][i] - base[i >> 1]);
        sum[i >> 1] += s[n][i];
      }
#pragma unroll
    for (int x = 0; x < 2; ++x) l[x] = fmaf(l[x], corr[x], sum[x]);
#pragma unroll
    for (int d = 0; d < DP / 8; ++d)
#pragma unroll
      for (int i = 0; i < 4; ++i) o[d][i] *= corr[i >> 1];
    values<DP, 16>(o, s, va + off, lane);
  }
  cpa_wait<0>();
  // ---- the four warps' shares of this block ----
  float *os = reinterpret_cast<float *>(Ks);   // [4][16][DP], in the tiles' place
  __syncthreads();
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int r = (lane >> 2) + 8 * x;
    l[x] = quad_sum(l[x]);
    if ((lane & 3) == 0) { wm[warp][r] = m[x]; wl[warp][r] = l[x]; }
    if (r < HG)
#pragma unroll
      for (int d = 0; d < DP / 8; ++d) *reinterpret_cast<float2 *>(os + (warp * 16 + r) * DP + d * 8 + (lane & 3) * 2) = make_float2(o[d][2 * x], o[d][2 * x + 1]);
  }
  __syncthreads();
  auto put = [&](int hh, int d, float v) {
    const int c = (g * HG + hh) * E + d;
    if (a.goff >= 0) v *= fast_logistic(u[a.goff + c]);
    const size_t at = (size_t)seq * a.ldo + c;
    if (a.out16) reinterpret_cast<uint16_t *>(a.O)[at] = f32_to_bf16(v);
    else reinterpret_cast<float *>(a.O)[at] = v;
  };
  auto sink = [&](int hh, float M) { return a.Sink ? fast_exp2(a.Sink[g * HG + hh] * kLog2e - M) : 0.0f; };
  // partials of a (sequence, key head): sums [splits][HG][E], then (maximum, sum) [splits][HG][2]
  float *base_p = a.Part + ((size_t)seq * a.G + g) * a.splits * HG * (E + 4);   // E + 4 keeps 16-byte alignment
  float *base_m = base_p + (size_t)a.splits * HG * E;
  for (int i = tid; i < HG * E; i += 128) {
    const int hh = i / E, d = i - hh * E;
    const float M = fmaxf(fmaxf(wm[0][hh], wm[1][hh]), fmaxf(wm[2][hh], wm[3][hh]));
    float v = 0.0f, L = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = fast_exp2(wm[w][hh] - M);
      v = fmaf(os[(w * 16 + hh) * DP + d], f, v);
      L = fmaf(wl[w][hh], f, L);
    }
    if (active == 1) {
      put(hh, d, v / (L + sink(hh, M)));
    } else {
      __stcg(base_p + (size_t)split * HG * E + i, v);
      if (d == 0) __stcg(reinterpret_cast<float2 *>(base_m) + split * HG + hh, make_float2(M, L));
    }
  }
  if (active == 1) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    const uint32_t c = atomicAdd(a.Count + (size_t)seq * a.G + g, 1u);
    s_last = c + 1 == (uint32_t)active;
    if (s_last) a.Count[(size_t)seq * a.G + g] = 0;
  }
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  // every split's factor exp2(m_s - M) / L, then the sums with the loads of all splits in flight
  float *fac = os;   // [HG][kWsMaxSplits]
  for (int hh = warp; hh < HG; hh += 4) {
    const float2 ml = lane < active ? __ldcg(reinterpret_cast<const float2 *>(base_m) + lane * HG + hh) : make_float2(-INFINITY, 0.0f);
    const float M = warp_max(ml.x), f = fast_exp2(ml.x - M), L = warp_tree_sum(ml.y * f) + sink(hh, M);
    if (lane < kWsMaxSplits) fac[hh * kWsMaxSplits + lane] = lane < active ? f / L : 0.0f;
  }
  __syncthreads();
  for (int i = tid * 4; i < HG * E; i += 512) {
    const int hh = i / E;
    const float *p = base_p + i, *f = fac + hh * kWsMaxSplits;
    float4 x[kWsMaxSplits], v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int s = 0; s < kWsMaxSplits; ++s) x[s] = __ldcg(reinterpret_cast<const float4 *>(p + (size_t)min(s, active - 1) * HG * E));
#pragma unroll
    for (int s = 0; s < kWsMaxSplits; ++s) {
      const float w = f[s];
      v.x = fmaf(x[s].x, w, v.x); v.y = fmaf(x[s].y, w, v.y); v.z = fmaf(x[s].z, w, v.z); v.w = fmaf(x[s].w, w, v.w);
    }
    put(hh, i % E, v.x); put(hh, i % E + 1, v.y); put(hh, i % E + 2, v.z); put(hh, i % E + 3, v.w);
  }
}
#define WINDOW_STEP(DP)                                                                                              \
  __global__ void __launch_bounds__(128) WindowAttnStepMma##DP(const __grid_constant__ WindowAttnStepMmaArgs a) {    \
    pdl_launch_dependents();                                                                                         \
    pdl_wait();                                                                                                      \
    window_step_mma_body<DP>(a);                                                                                     \
  }                                                                                                                  \
  static uint32_t window_step_smem##DP(const void *) { return (16 + 2 + 2 * kWsStages * kCmKeys) * (DP + 8) * 2; }   \
  static_assert(2 * kWsStages * kCmKeys * (DP + 8) * 2 >= 4 * 16 * DP * 4 && 16 * kWsMaxSplits <= 4 * 16 * DP, "merge buffers lie in the tiles' place");
WINDOW_STEP(32)
WINDOW_STEP(64)
WINDOW_STEP(96)
WINDOW_STEP(128)
WINDOW_STEP(192)
WINDOW_STEP(256)
#define F(f) AINFER_ARG(WindowAttnStepMmaArgs, f)
#define WS_FIELDS                                                                                                                           \
  F(U), F(QN), F(KN), F(Rot), F(Ctrl), F(Kc), F(Vc), F(Pk), F(Pv), F(k_stride), F(v_stride), F(pk_stride), F(pv_stride), F(Sink), F(Part), \
      F(Count), F(O), F(nseq), F(H), F(G), F(D), F(E), F(rd), F(cap), F(window), F(pool), F(koff), F(voff), F(goff), F(own_pool), F(splits), \
      F(ldu), F(ldo), F(out16), F(scale), F(softcap), F(eps)
#define WS_REGISTER(DP) \
  AINFER_REGISTER(WindowAttnStepMma##DP, WindowAttnStepMmaArgs, 128, 0, 0, window_step_smem##DP, WS_FIELDS); AINFER_EARLY_LAUNCH(WindowAttnStepMma##DP)
WS_REGISTER(32);
WS_REGISTER(64);
WS_REGISTER(96);
WS_REGISTER(128);
WS_REGISTER(192);
WS_REGISTER(256);
#undef F

}  // namespace ainfer
