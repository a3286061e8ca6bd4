// Chunk-local shared-key attention (see k_chunk_attn.cu) in bf16 on the tensor cores, for head sizes
// that are multiples of 8 up to 256. One tile of keys in shared memory serves both products: read
// plainly it is the B operand of q . k, read transposed it is the B operand of weights . values.
// Scores, the distance penalty, maxima, weights and sums are fp32; the weights are rounded to bf16
// for the second product only.
//
//   ChunkAttnMma       rows of one sequence: a block takes 64 rows of one query head, a warp 16 rows
//   ChunkAttnStepMma   a decode step of every sequence (up to 16 query heads per key head): the heads
//                      are the 16 rows of the products, a warp takes 16 keys of every tile of 64
#include "attn_mma.cuh"
#include "hyper_core.cuh"

namespace ainfer {

// ------------------------------------------------------- ChunkAttnMma ---
struct ChunkAttnMmaArgs {
  const uint16_t *Q;       // [rows][H D]
  const uint16_t *Kc;      // [cap][G D], cap a multiple of 64
  const float *LB;         // [H][lb_len]
  const float *Temp;       // [H]
  const int32_t *Ctrl;     // [rows][4]
  uint16_t *O;             // [rows][ldo]
  int32_t rows, H, G, D, cap, chunk, lb_len, ldo;
  float scale;
};
constexpr int kCmRows = 64;
template <int DP>
__device__ __forceinline__ void chunk_attn_mma_body(const ChunkAttnMmaArgs &a) {
  extern __shared__ __align__(128) unsigned char cm_raw[];
  constexpr int LD = DP + 8;
  uint16_t *Qs = reinterpret_cast<uint16_t *>(cm_raw);
  uint16_t *Ks = Qs + kCmRows * LD;                                   // [2][64][LD]
  float *lbw = reinterpret_cast<float *>(Ks + 2 * kCmKeys * LD);      // [2][128] penalty by row - key + 63
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int tiles = (a.rows + kCmRows - 1) / kCmRows;
  const int h = blockIdx.x % a.H, r0 = (tiles - 1 - blockIdx.x / a.H) * kCmRows, g = h / (a.H / a.G);   // long rows first
  const int nr = min(kCmRows, a.rows - r0), KW = a.G * a.D;
  const uint32_t qa = cm_smem(Qs), ka = cm_smem(Ks);
  {
    constexpr int P = DP / 8;
    for (int i = tid; i < kCmRows * P; i += 128) {
      const int r = i / P, c = i % P;
      const bool in = r < nr && c * 8 < a.D;
      cpa16(qa + (uint32_t)(r * LD + c * 8) * 2, a.Q + (in ? (size_t)(r0 + r) * a.H * a.D + (size_t)h * a.D + c * 8 : 0), in);
    }
  }
  const int p0 = a.Ctrl[4 * r0 + CTRL_POS], p1 = p0 + nr - 1;
  const int lo = p0 - p0 % a.chunk, kb0 = lo / kCmKeys * kCmKeys;
  const uint16_t *K = a.Kc + (size_t)g * a.D;
  const float *lb = a.LB + (size_t)h * a.lb_len;
  // keys of a tile by asynchronous copies; its penalties (entry tid: distance p0 - k0 - 63 + tid, 127 used) wait
  // in a register until the tile before is done
  int slot = kb0 % a.cap;
  float pen = 0.0f;
  auto fetch = [&](int k0, int b) {
    pen = __ldg(lb + min(max(p0 - k0 - 63 + tid, 0), a.lb_len - 1));
    load_keys<DP, 128>(ka + (uint32_t)(b * kCmKeys * LD) * 2, K, slot, KW, a.D);
    cpa_commit();
    slot += kCmKeys;
    if (slot == a.cap) slot = 0;
  };
  fetch(kb0, 0);
  lbw[tid] = pen * kLog2e;
  const float mul = a.scale * a.Temp[h] * kLog2e;
  float o[DP / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
  for (int d = 0; d < DP / 8; ++d)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[d][i] = 0.0f;
  const uint32_t qw = qa + (uint32_t)((warp * 16 + (lane & 15)) * LD + (lane >> 4) * 8) * 2;
  const int rw = warp * 16 + (lane >> 2);                 // this thread's rows rw and rw + 8
  const int pr[2] = {p0 + rw, p0 + rw + 8};
  const int cs[2] = {pr[0] - pr[0] % a.chunk, pr[1] - pr[1] % a.chunk};
  const int cs_last = p1 - p1 % a.chunk;
  int b = 0;
  for (int k0 = kb0; k0 <= p1; k0 += kCmKeys) {
    const bool more = k0 + kCmKeys <= p1;
    if (more) fetch(k0 + kCmKeys, b ^ 1);
    if (more) cpa_wait<1>(); else cpa_wait<0>();
    __syncthreads();
    float s[kCmKeys / 8][4];
    const uint32_t kt = ka + (uint32_t)(b * kCmKeys * LD) * 2;
    scores_smem<DP, kCmKeys>(s, qw, kt, lane);
    const bool whole = k0 + kCmKeys - 1 <= p0 && k0 >= cs_last;   // every row sees every key of the tile
    const float *lw = lbw + b * 128;
    float mx[2] = {m[0], m[1]};
    const float *lr = lw + rw + 63 - (lane & 3) * 2;   // entry of (row, key): + 8 per row half, - key
    if (whole) {
#pragma unroll
      for (int n = 0; n < kCmKeys / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          s[n][i] = fmaf(s[n][i], mul, -lr[8 * (i >> 1) - n * 8 - (i & 1)]);
          mx[i >> 1] = fmaxf(mx[i >> 1], s[n][i]);
        }
    } else {
#pragma unroll
      for (int n = 0; n < kCmKeys / 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int x = i >> 1, key = k0 + n * 8 + (lane & 3) * 2 + (i & 1);
          const float v = fmaf(s[n][i], mul, -lr[8 * x - n * 8 - (i & 1)]);
          s[n][i] = key > pr[x] || key < cs[x] ? -INFINITY : v;
          mx[x] = fmaxf(mx[x], s[n][i]);
        }
    }
    float corr[2], base[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      mx[x] = quad_max(mx[x]);
      base[x] = mx[x] == -INFINITY ? 0.0f : mx[x];
      corr[x] = fast_exp2(m[x] - base[x]);
      m[x] = mx[x];
    }
    float sum[2] = {0.0f, 0.0f};
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
    values<DP, kCmKeys>(o, s, kt, lane);
    if (more) lbw[(b ^ 1) * 128 + tid] = pen * kLog2e;
    __syncthreads();
    b ^= 1;
  }
#pragma unroll
  for (int x = 0; x < 2; ++x) l[x] = 1.0f / quad_sum(l[x]);
#pragma unroll
  for (int d = 0; d < DP / 8; ++d)
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = rw + 8 * x, c = d * 8 + (lane & 3) * 2;
      if (r < nr && c < a.D) *reinterpret_cast<uint32_t *>(a.O + (size_t)(r0 + r) * a.ldo + (size_t)h * a.D + c) = pack2(o[d][2 * x] * l[x], o[d][2 * x + 1] * l[x]);
    }
}
__host__ __device__ inline int cm_pad(int D) { return D <= 32 ? 32 : D <= 64 ? 64 : D <= 96 ? 96 : D <= 128 ? 128 : D <= 192 ? 192 : 256; }
#define CHUNK_MMA(DP, BLOCKS)                                                                             \
  __global__ void __launch_bounds__(128, BLOCKS) ChunkAttnMma##DP(const __grid_constant__ ChunkAttnMmaArgs a) { \
    pdl_launch_dependents();                                                                              \
    pdl_wait();                                                                                           \
    chunk_attn_mma_body<DP>(a);                                                                           \
  }                                                                                                       \
  static uint32_t chunk_mma_smem##DP(const void *) { return (kCmRows + 2 * kCmKeys) * (DP + 8) * 2 + 2 * 128 * 4; }
CHUNK_MMA(32, 4)
CHUNK_MMA(64, 4)
CHUNK_MMA(96, 3)
CHUNK_MMA(128, 3)
CHUNK_MMA(192, 2)
CHUNK_MMA(256, 2)
#define F(f) AINFER_ARG(ChunkAttnMmaArgs, f)
#define CM_FIELDS F(Q), F(Kc), F(LB), F(Temp), F(Ctrl), F(O), F(rows), F(H), F(G), F(D), F(cap), F(chunk), F(lb_len), F(ldo), F(scale)
#define CM_REGISTER(DP) AINFER_REGISTER(ChunkAttnMma##DP, ChunkAttnMmaArgs, 128, 0, 0, chunk_mma_smem##DP, CM_FIELDS); AINFER_EARLY_LAUNCH(ChunkAttnMma##DP)
CM_REGISTER(32);
CM_REGISTER(64);
CM_REGISTER(96);
CM_REGISTER(128);
CM_REGISTER(192);
CM_REGISTER(256);
#undef F

// --------------------------------------------------- ChunkAttnStepMma ---
struct ChunkAttnStepMmaArgs {
  const float *U;          // [seq][ldu]
  const float *CW;         // [taps][C]
  float *State;            // [seq][taps][C]
  const int32_t *Ctrl;     // [seq][4]
  uint16_t *Kc;
  int64_t kv_stride;
  const float *LB;         // [H][lb_len]
  const float *Temp;       // [H]
  float *Part;             // [seq][G] blocks of splits HG (D + 4) floats
  uint32_t *Count;         // [seq][G], zero between launches
  void *O;                 // [seq][ldo]
  int32_t nseq, H, G, D, taps, cap, chunk, lb_len, splits, ldu, ldo, out16;   // splits <= 16, ldu a multiple of 4
  float scale;
};
constexpr int kSmStages = 3, kSmMaxSplits = 16;   // at most 16 splits
template <int DP>
__device__ __forceinline__ void chunk_step_mma_body(const ChunkAttnStepMmaArgs &a) {
  extern __shared__ __align__(128) unsigned char sm_raw[];
  __shared__ float wm[4][16], wl[4][16];
  __shared__ int s_last;
  constexpr int LD = DP + 8;
  uint16_t *Qs = reinterpret_cast<uint16_t *>(sm_raw);                // [16][LD]
  uint16_t *kn = Qs + 16 * LD;                                        // the new key [DP]
  uint16_t *Ks = kn + LD;                                             // [stages][64][LD]
  const int D = a.D, HG = a.H / a.G, C = (a.H + a.G) * D, Qc = a.H * D, KW = a.G * D;
  const int split = blockIdx.x % a.splits, g = blockIdx.x / a.splits % a.G, seq = blockIdx.x / (a.splits * a.G);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos = a.Ctrl[4 * seq + CTRL_POS], lo = pos - pos % a.chunk;
  const int t_lo = lo / kCmKeys, t_hi = pos / kCmKeys, nt = t_hi - t_lo + 1;
  const int per = (nt + a.splits - 1) / a.splits, active = (nt + per - 1) / per;
  if (split >= active) return;
  const int t0 = t_lo + split * per, t1 = min(t_hi, t0 + per - 1);
  uint16_t *K = a.Kc + (size_t)seq * a.kv_stride + (size_t)g * D;
  const uint32_t ka = cm_smem(Ks);
  auto fetch = [&](int t) {
    if (t <= t1) load_keys<DP, 128>(ka + (uint32_t)(((t - t0) % kSmStages) * kCmKeys * LD) * 2, K, t * kCmKeys % a.cap, KW, D);
    cpa_commit();
  };
  for (int i = 0; i < kSmStages - 1; ++i) fetch(t0 + i);
  // ---- convolution of this key head's channels (its query heads, then the key) ----
  for (int i = tid; i < 16 * LD; i += 128) Qs[i] = 0;
  __syncthreads();
  float *st = a.State + (size_t)seq * a.taps * C;
  const float *u0 = a.U + (size_t)seq * a.ldu;
  const int slot = pos % a.taps;
  for (int i = tid * 4; i < (HG + 1) * D; i += 512) {
    const bool isk = i >= HG * D;
    const int c = isk ? Qc + g * D + (i - HG * D) : g * HG * D + i;
    const float4 u = *reinterpret_cast<const float4 *>(u0 + c);
    const float4 wl4 = __ldg(reinterpret_cast<const float4 *>(a.CW + (size_t)(a.taps - 1) * C + c));
    float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 4
    for (int j = 0; j < a.taps - 1; ++j) {
      const int back = a.taps - 1 - j, s = slot - back < 0 ? slot - back + a.taps : slot - back;
      const float4 w = __ldg(reinterpret_cast<const float4 *>(a.CW + (size_t)j * C + c));
      float4 v = *reinterpret_cast<const float4 *>(st + (size_t)s * C + c);
      if (pos < back) v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      y.x = fmaf(w.x, v.x, y.x); y.y = fmaf(w.y, v.y, y.y); y.z = fmaf(w.z, v.z, y.z); y.w = fmaf(w.w, v.w, y.w);
    }
    y.x = fmaf(wl4.x, u.x, y.x); y.y = fmaf(wl4.y, u.y, y.y); y.z = fmaf(wl4.z, u.z, y.z); y.w = fmaf(wl4.w, u.w, y.w);
    if (split == 0) *reinterpret_cast<float4 *>(st + (size_t)slot * C + c) = u;
    const uint2 v = make_uint2(pack2(y.x, y.y), pack2(y.z, y.w));
    *reinterpret_cast<uint2 *>(isk ? kn + (i - HG * D) : Qs + (i / D) * LD + i % D) = v;
  }
  __syncthreads();
  uint32_t q[DP / 16][4];
#pragma unroll
  for (int kk = 0; kk < DP / 16; ++kk) ldm4(q[kk], cm_smem(Qs) + (uint32_t)((lane & 15) * LD + kk * 16 + (lane >> 4) * 8) * 2);
  float o[DP / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f}, mul[2];
  const float *lb[2];
#pragma unroll
  for (int d = 0; d < DP / 8; ++d)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[d][i] = 0.0f;
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int h = g * HG + min((lane >> 2) + 8 * x, HG - 1);   // rows past the head count repeat the last head
    mul[x] = a.scale * a.Temp[h] * kLog2e;
    lb[x] = a.LB + (size_t)h * a.lb_len;
  }
  for (int t = t0; t <= t1; ++t) {
    const int k0 = t * kCmKeys + warp * 16;
    float pen[2][2][2];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) pen[x][n][e] = __ldg(lb[x] + min(max(pos - (k0 + n * 8 + (lane & 3) * 2 + e), 0), a.lb_len - 1));
    cpa_wait<kSmStages - 2>();
    __syncthreads();
    if (t == t_hi) {   // the step's own key: into the tile and the cache
      uint16_t *row = Ks + ((t - t0) % kSmStages) * kCmKeys * LD + (pos % kCmKeys) * LD;
      for (int i = tid; i < D; i += 128) {
        row[i] = kn[i];
        K[(size_t)(pos % a.cap) * KW + i] = kn[i];
      }
      __syncthreads();
    }
    fetch(t + kSmStages - 1);
    const uint32_t kt = ka + (uint32_t)((((t - t0) % kSmStages) * kCmKeys + warp * 16) * LD) * 2;
    float s[2][4];
    scores<DP, 16>(s, q, kt, lane);
    float mx[2] = {m[0], m[1]};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int x = i >> 1, key = k0 + n * 8 + (lane & 3) * 2 + (i & 1);
        float v = fmaf(s[n][i], mul[x], -pen[x][n][i & 1] * kLog2e);
        if (key > pos || key < lo) v = -INFINITY;
        s[n][i] = v;
        mx[x] = fmaxf(mx[x], v);
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
    values<DP, 16>(o, s, kt, lane);
  }
  cpa_wait<0>();
  // ---- the four warps' shares of this block ----
  float *os = reinterpret_cast<float *>(Ks);   // [4][16][DP], in the key tiles' place
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
  auto put = [&](int h, int d, float v) {
    const size_t at = (size_t)seq * a.ldo + (size_t)h * D + d;
    if (a.out16) reinterpret_cast<uint16_t *>(a.O)[at] = f32_to_bf16(v);
    else reinterpret_cast<float *>(a.O)[at] = v;
  };
  // partials of a (sequence, key head): sums [splits][HG][D], then (maximum, sum) [splits][HG][2]
  float *base_p = a.Part + ((size_t)seq * a.G + g) * a.splits * HG * (D + 4);   // D + 4 keeps 16-byte alignment
  float *base_m = base_p + (size_t)a.splits * HG * D;
  for (int i = tid; i < HG * D; i += 128) {
    const int hh = i / D, d = i - hh * D;
    const float M = fmaxf(fmaxf(wm[0][hh], wm[1][hh]), fmaxf(wm[2][hh], wm[3][hh]));
    float v = 0.0f, L = 0.0f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = fast_exp2(wm[w][hh] - M);
      v = fmaf(os[(w * 16 + hh) * DP + d], f, v);
      L = fmaf(wl[w][hh], f, L);
    }
    if (active == 1) {
      put(g * HG + hh, d, v / L);
    } else {
      __stcg(base_p + (size_t)split * HG * D + i, v);
      if (d == 0) __stcg(reinterpret_cast<float2 *>(base_m) + split * HG + hh, make_float2(M, L));
    }
  }
  if (active == 1) return;
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
  // every split's factor exp2(m_s - M) / L, then the sums with the loads of all splits in flight
  float *fac = os;   // [HG][kSmMaxSplits]
  for (int hh = warp; hh < HG; hh += 4) {
    const float2 ml = lane < active ? __ldcg(reinterpret_cast<const float2 *>(base_m) + lane * HG + hh) : make_float2(-INFINITY, 0.0f);
    const float M = warp_max(ml.x), f = fast_exp2(ml.x - M), L = warp_tree_sum(ml.y * f);
    if (lane < kSmMaxSplits) fac[hh * kSmMaxSplits + lane] = lane < active ? f / L : 0.0f;
  }
  __syncthreads();
  for (int i = tid * 4; i < HG * D; i += 512) {
    const int hh = i / D;
    const float *p = base_p + i, *f = fac + hh * kSmMaxSplits;
    float4 x[kSmMaxSplits], v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
    for (int s = 0; s < kSmMaxSplits; ++s) x[s] = __ldcg(reinterpret_cast<const float4 *>(p + (size_t)min(s, active - 1) * HG * D));
#pragma unroll
    for (int s = 0; s < kSmMaxSplits; ++s) {
      const float w = f[s];
      v.x = fmaf(x[s].x, w, v.x); v.y = fmaf(x[s].y, w, v.y); v.z = fmaf(x[s].z, w, v.z); v.w = fmaf(x[s].w, w, v.w);
    }
    put(g * HG + hh, i % D, v.x); put(g * HG + hh, i % D + 1, v.y); put(g * HG + hh, i % D + 2, v.z); put(g * HG + hh, i % D + 3, v.w);
  }
}
#define CHUNK_STEP(DP)                                                                                                  \
  __global__ void __launch_bounds__(128) ChunkAttnStepMma##DP(const __grid_constant__ ChunkAttnStepMmaArgs a) {         \
    pdl_launch_dependents();                                                                                            \
    pdl_wait();                                                                                                         \
    chunk_step_mma_body<DP>(a);                                                                                         \
  }                                                                                                                     \
  static uint32_t chunk_step_smem##DP(const void *) {                                                                   \
    return (16 + 1 + kSmStages * kCmKeys) * (DP + 8) * 2;                                                               \
  }                                                                                                                     \
  static_assert(kSmStages * kCmKeys * (DP + 8) * 2 >= 4 * 16 * DP * 4 && 16 * kSmMaxSplits <= 4 * 16 * DP, "merge buffers lie in the key tiles' place");
CHUNK_STEP(32)
CHUNK_STEP(64)
CHUNK_STEP(96)
CHUNK_STEP(128)
CHUNK_STEP(192)
CHUNK_STEP(256)
#define F(f) AINFER_ARG(ChunkAttnStepMmaArgs, f)
#define CS_FIELDS                                                                                                                  \
  F(U), F(CW), F(State), F(Ctrl), F(Kc), F(kv_stride), F(LB), F(Temp), F(Part), F(Count), F(O), F(nseq), F(H), F(G), F(D), F(taps), \
      F(cap), F(chunk), F(lb_len), F(splits), F(ldu), F(ldo), F(out16), F(scale)
#define CS_REGISTER(DP) \
  AINFER_REGISTER(ChunkAttnStepMma##DP, ChunkAttnStepMmaArgs, 128, 0, 0, chunk_step_smem##DP, CS_FIELDS); AINFER_EARLY_LAUNCH(ChunkAttnStepMma##DP)
CS_REGISTER(32);
CS_REGISTER(64);
CS_REGISTER(96);
CS_REGISTER(128);
CS_REGISTER(192);
CS_REGISTER(256);
#undef F

}  // namespace ainfer
