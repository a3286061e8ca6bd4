// Windowed attention with pooled blocks and sinks (window_attn.cuh): rotary tables, head norm + rotation
// + append, block means, and the CUDA-core forms of the attention itself (fp32, and bf16 caches whose
// head sizes the tensor-core forms in k_window_mma.cu do not take).
#include "window_attn.cuh"

namespace ainfer {

// --------------------------------------------------------- RotaryTable ---
// T[p][i] = (cos, sin)(p F[i]), evaluated in double and rounded once.
struct RotaryTableArgs {
  float2 *T;
  const double *F;         // [pairs] angle per position
  int32_t positions, pairs;
};
__global__ void __launch_bounds__(256) RotaryTable(const RotaryTableArgs a) {
  const size_t n = (size_t)a.positions * a.pairs;
  for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (size_t)gridDim.x * 256) {
    double s, c;
    sincos((double)(i / a.pairs) * a.F[i % a.pairs], &s, &c);
    a.T[i] = make_float2((float)c, (float)s);
  }
}
#define F(f) AINFER_ARG(RotaryTableArgs, f)
AINFER_REGISTER(RotaryTable, RotaryTableArgs, 256, 0, 0, nullptr, F(T), F(F), F(positions), F(pairs));
#undef F

// ------------------------------------------------------------- QkvRows ---
// Rows of ONE sequence: projections U (q heads; with koff >= 0 also k and v heads) -> Q [rows][H D], and
// the keys and values into the ring. One warp per (row, head).
struct QkvRowsArgs {
  const float *U;          // [rows][ldu]: q at 0, k at koff, v at voff
  const float *QN, *KN;    // [D] norm weights; null: no norm
  const float2 *Rot;       // [position][rd / 2]; null when rd = 0
  const int32_t *Ctrl;
  void *Q, *Kc, *Vc;       // Kc [cap][G D], Vc [cap][G E]
  int32_t rows, H, G, D, E, rd, cap, ldu, koff, voff;   // koff < 0: no keys and values
  float eps;
};
template <typename T>
__device__ __forceinline__ void qkv_rows_body(const QkvRowsArgs &a) {
  const int units = a.H + (a.koff >= 0 ? 2 * a.G : 0), i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int r = i / units, u = i - r * units;
  if (r >= a.rows) return;
  const int pos = a.Ctrl[4 * r + CTRL_POS];
  const float *src = a.U + (size_t)r * a.ldu;
  const float2 *rot = a.Rot + (size_t)pos * (a.rd >> 1);
  if (u < a.H) {
    T *q = reinterpret_cast<T *>(a.Q) + ((size_t)r * a.H + u) * a.D;
    head_norm_turn(src + (size_t)u * a.D, a.D, a.QN, a.eps, rot, a.rd, [&](int d, float x, float y, bool both) { st_pair(q + d, x, y, both); });
  } else if (u < a.H + a.G) {
    const int g = u - a.H;
    T *k = reinterpret_cast<T *>(a.Kc) + ((size_t)(pos % a.cap) * a.G + g) * a.D;
    head_norm_turn(src + a.koff + (size_t)g * a.D, a.D, a.KN, a.eps, rot, a.rd, [&](int d, float x, float y, bool both) { st_pair(k + d, x, y, both); });
  } else {
    const int g = u - a.H - a.G;
    T *v = reinterpret_cast<T *>(a.Vc) + ((size_t)(pos % a.cap) * a.G + g) * a.E;
    const float *s = src + a.voff + (size_t)g * a.E;
    const bool wide = (reinterpret_cast<unsigned long long>(s) & 7) == 0;
#pragma unroll 4
    for (int d = lane * 2; d < a.E; d += 64) {
      const bool both = d + 1 < a.E;
      const float2 t = both && wide ? *reinterpret_cast<const float2 *>(s + d) : make_float2(s[d], both ? s[d + 1] : 0.0f);
      st_pair(v + d, t.x, t.y, both);
    }
  }
}
__global__ void __launch_bounds__(256) QkvRowsF32(const QkvRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  qkv_rows_body<float>(a);
}
__global__ void __launch_bounds__(256) QkvRowsB16(const QkvRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  qkv_rows_body<uint16_t>(a);
}
#define F(f) AINFER_ARG(QkvRowsArgs, f)
#define QKV_FIELDS                                                                                                                         \
  F(U), F(QN), F(KN), F(Rot), F(Ctrl), F(Q), F(Kc), F(Vc), F(rows), F(H), F(G), F(D), F(E), F(rd), F(cap), F(ldu), F(koff), F(voff), F(eps)
AINFER_REGISTER(QkvRowsF32, QkvRowsArgs, 256, 0, 0, nullptr, QKV_FIELDS);
AINFER_REGISTER(QkvRowsB16, QkvRowsArgs, 256, 0, 0, nullptr, QKV_FIELDS);
#undef F

// ------------------------------------------------------------ PoolRows ---
// Means of the blocks whose last position lies among the pass's rows [p0, p0 + rows). One group of the
// grid per block and 256 channels of the keys, then of the values: grid = (rows / pool + 1) x channel groups.
struct PoolRowsArgs {
  const void *Kc, *Vc;     // [cap][KW], [cap][VW]
  void *Pk, *Pv;           // [blocks][KW], [blocks][VW]
  const int32_t *Ctrl;
  int32_t rows, KW, VW, cap, pool;
};
template <typename T>
__device__ __forceinline__ void pool_rows_body(const PoolRowsArgs &a) {
  const int cg = (a.KW + a.VW + 255) / 256, c = (blockIdx.x % cg) * 256 + threadIdx.x;
  const int p0 = a.Ctrl[CTRL_POS], b = p0 / a.pool + blockIdx.x / cg;
  if (c >= a.KW + a.VW || (b + 1) * a.pool > p0 + a.rows) return;
  const bool isv = c >= a.KW;
  const int w = isv ? a.VW : a.KW, x = isv ? c - a.KW : c;
  const T *src = reinterpret_cast<const T *>(isv ? a.Vc : a.Kc) + x;
  float s = 0.0f;
  int slot = b * a.pool % a.cap;
#pragma unroll 4
  for (int i = 0; i < a.pool; ++i) {
    s += ld_val(src + (size_t)slot * w);
    if (++slot == a.cap) slot = 0;
  }
  st_val(reinterpret_cast<T *>(isv ? a.Pv : a.Pk) + (size_t)b * w + x, s / (float)a.pool);
}
__global__ void __launch_bounds__(256) PoolRowsF32(const PoolRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  pool_rows_body<float>(a);
}
__global__ void __launch_bounds__(256) PoolRowsB16(const PoolRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  pool_rows_body<uint16_t>(a);
}
#define F(f) AINFER_ARG(PoolRowsArgs, f)
#define POOL_FIELDS F(Kc), F(Vc), F(Pk), F(Pv), F(Ctrl), F(rows), F(KW), F(VW), F(cap), F(pool)
AINFER_REGISTER(PoolRowsF32, PoolRowsArgs, 256, 0, 0, nullptr, POOL_FIELDS);
AINFER_REGISTER(PoolRowsB16, PoolRowsArgs, 256, 0, 0, nullptr, POOL_FIELDS);
#undef F

// ------------------------------------------------------ WindowAttnRows ---
// Rows of ONE sequence, their keys and values already in the cache. A block takes 16 rows of one query
// head; keys come in tiles of 32 through shared memory (blocks first, then tokens); a warp owns four
// rows, a lane one key of the tile for the scores and the value columns lane, lane + 32, ... for the sums.
struct WindowAttnArgs {
  const void *Q;           // [rows][H D]
  const void *Kc, *Vc;     // [cap][G D], [cap][G E]
  const void *Pk, *Pv;     // [blocks][G D], [blocks][G E]; null: no blocks
  const float *Sink;       // [H] or null
  const float *Gate;       // [rows][ldg] or null: the output times logistic(gate), H E values per row
  const int32_t *Ctrl;     // [rows][4]
  void *O;                 // [rows][ldo]
  int32_t rows, H, G, D, E, cap, window, pool, ldg, ldo;
  float scale, softcap;
};
constexpr int kWaRows = 16, kWaKeys = 32, kWaMaxD = 512;
template <typename T>
__device__ __forceinline__ void window_attn_rows_body(const WindowAttnArgs &a) {
  extern __shared__ __align__(16) float wa_smem[];   // q [16][D], k [32][D + 1], v [32][E]
  const int D = a.D, E = a.E, h = blockIdx.x % a.H, r0 = blockIdx.x / a.H * kWaRows, g = h / (a.H / a.G);
  float *qs = wa_smem, *ks = qs + kWaRows * D, *vs = ks + kWaKeys * (D + 1);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nr = min(kWaRows, a.rows - r0);
  const T *Q = reinterpret_cast<const T *>(a.Q);
  for (int i = tid; i < kWaRows * D; i += 128) {
    const int rr = i / D, d = i - rr * D;
    qs[i] = rr < nr ? ld_val(Q + ((size_t)(r0 + rr) * a.H + h) * D + d) : 0.0f;
  }
  const int pos0 = a.Ctrl[4 * r0 + CTRL_POS], last = pos0 + nr - 1;
  float m[4], l[4], acc[4][kWaMaxD / 32];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    m[i] = -INFINITY; l[i] = 0.0f;
#pragma unroll
    for (int x = 0; x < kWaMaxD / 32; ++x) acc[i][x] = 0.0f;
  }
  // keys [k0, hi) of an array of rows (index % mod), row (position p) sees [lo(p), up(p)]
  auto walk = [&](const T *K, const T *V, int k0, int hi, int mod, auto lo, auto up) {
    for (; k0 < hi; k0 += kWaKeys) {
      __syncthreads();
      for (int i = tid; i < kWaKeys * D; i += 128) {
        const int kk = i / D, d = i - kk * D, p = k0 + kk;
        ks[kk * (D + 1) + d] = p < hi ? ld_val(K + ((size_t)(p % mod) * a.G + g) * D + d) : 0.0f;
      }
      for (int i = tid; i < kWaKeys * E; i += 128) {
        const int kk = i / E, d = i - kk * E, p = k0 + kk;
        vs[kk * E + d] = p < hi ? ld_val(V + ((size_t)(p % mod) * a.G + g) * E + d) : 0.0f;
      }
      __syncthreads();
      const int kp = k0 + lane;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int rr = warp * 4 + i, p = pos0 + rr;
        if (rr >= nr) continue;
        const bool see = kp < hi && kp >= lo(p) && kp <= up(p);
        float s = -INFINITY;
        if (see) {
          float dot = 0.0f;
          const float *q = qs + rr * D, *k = ks + lane * (D + 1);
          for (int d = 0; d < D; ++d) dot = fmaf(q[d], k[d], dot);
          s = cap_score(dot * a.scale, a.softcap);
        }
        const float mx = fmaxf(m[i], warp_max(s));
        if (mx == -INFINITY) continue;   // nothing visible yet (uniform over the warp)
        const float corr = expf(m[i] - mx), w = see ? expf(s - mx) : 0.0f;
        m[i] = mx;
        l[i] = fmaf(l[i], corr, warp_tree_sum(w));
#pragma unroll
        for (int x = 0; x < kWaMaxD / 32; ++x)
          if (x * 32 < E) acc[i][x] *= corr;
        for (int j = 0; j < kWaKeys; ++j) {
          const float wj = __shfl_sync(kFull, w, j);
#pragma unroll
          for (int x = 0; x < kWaMaxD / 32; ++x)
            if (x * 32 < E) {
              const int d = x * 32 + lane;
              if (d < E) acc[i][x] = fmaf(wj, vs[j * E + d], acc[i][x]);
            }
        }
      }
    }
  };
  const int nb = a.Pk ? blocks_seen(last, a.window, a.pool) : 0;
  if (nb > 0)
    walk(reinterpret_cast<const T *>(a.Pk), reinterpret_cast<const T *>(a.Pv), 0, nb, INT32_MAX, [](int) { return 0; },
         [&](int p) { return blocks_seen(p, a.window, a.pool) - 1; });
  walk(reinterpret_cast<const T *>(a.Kc), reinterpret_cast<const T *>(a.Vc), max(0, pos0 - a.window + 1), last + 1, a.cap,
       [&](int p) { return p - a.window + 1; }, [](int p) { return p; });
  T *O = reinterpret_cast<T *>(a.O);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int rr = warp * 4 + i;
    if (rr >= nr) continue;
    float den = l[i];
    if (a.Sink) den += expf(a.Sink[h] - m[i]);
#pragma unroll
    for (int x = 0; x < kWaMaxD / 32; ++x) {
      const int d = x * 32 + lane;
      if (d < E) {
        float v = acc[i][x] / den;
        if (a.Gate) v = v * logistic(a.Gate[(size_t)(r0 + rr) * a.ldg + (size_t)h * E + d]);
        st_val(O + (size_t)(r0 + rr) * a.ldo + (size_t)h * E + d, v);
      }
    }
  }
}
__global__ void __launch_bounds__(128) WindowAttnRowsF32(const WindowAttnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  window_attn_rows_body<float>(a);
}
__global__ void __launch_bounds__(128) WindowAttnRowsB16(const WindowAttnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  window_attn_rows_body<uint16_t>(a);
}
static uint32_t window_attn_rows_smem(const void *args) {
  const WindowAttnArgs *a = (const WindowAttnArgs *)args;
  return 4u * (uint32_t)(kWaRows * a->D + kWaKeys * (a->D + 1) + kWaKeys * a->E);
}
#define F(f) AINFER_ARG(WindowAttnArgs, f)
#define WAR_FIELDS                                                                                                                             \
  F(Q), F(Kc), F(Vc), F(Pk), F(Pv), F(Sink), F(Gate), F(Ctrl), F(O), F(rows), F(H), F(G), F(D), F(E), F(cap), F(window), F(pool), F(ldg), \
      F(ldo), F(scale), F(softcap)
AINFER_REGISTER(WindowAttnRowsF32, WindowAttnArgs, 128, 0, 0, window_attn_rows_smem, WAR_FIELDS);
AINFER_REGISTER(WindowAttnRowsB16, WindowAttnArgs, 128, 0, 0, window_attn_rows_smem, WAR_FIELDS);
#undef F

// ------------------------------------------------------ WindowAttnStep ---
// One decode step of every sequence: head norm, rotation, append, block means, attention and output gate
// in one launch. Blocks: sequence x key head x (splits + 1). A split takes a contiguous share of the
// visible blocks and tokens; the last one of a (sequence, key head) to finish merges them in their
// order. The extra block appends the step's key and value and averages a block that they complete:
// nobody reads either in this step (the splits make the step's own key for themselves).
struct WindowAttnStepArgs {
  const float *U;          // [seq][ldu]: q at 0, k at koff, v at voff, output gate at goff
  const float *QN, *KN;    // [D] or null
  const float2 *Rot;       // [position][rd / 2]
  const int32_t *Ctrl;     // [seq][4]
  void *Kc, *Vc, *Pk, *Pv;
  int64_t k_stride, v_stride, pk_stride, pv_stride;   // elements between sequences
  const float *Sink;       // [H] or null
  float *Part;             // [seq][G][splits][HG (E + 4)]
  uint32_t *Count;         // [seq][G], zero between launches
  void *O;                 // [seq][ldo]
  int32_t nseq, H, G, D, E, rd, cap, window, pool, koff, voff, goff;   // koff < 0: key and value are in the ring; goff < 0: no gate
  int32_t own_pool, splits, ldu, ldo, out16;   // own_pool: this launch averages; out16: O holds bf16
  float scale, softcap, eps;
};
constexpr int kWsKeys = 64, kWsThreads = 256;
// floats of shared memory: q [HG][D], new key [D] and value [E], tiles [64][D + 1] and [64][E], scores
// [HG][64], head state [HG] x 3, sums [HG][E]
__host__ __device__ inline uint32_t window_step_floats(int HG, int D, int E) {
  return (uint32_t)(HG * (D + E) + D + E + kWsKeys * (D + 1 + E) + HG * kWsKeys + 3 * HG);
}
template <typename T>
__device__ __forceinline__ float as_stored(float v) {
  T t;
  st_val(&t, v);
  return ld_val(&t);
}
template <typename T>
__device__ __forceinline__ void window_attn_step_body(const WindowAttnStepArgs &a) {
  extern __shared__ __align__(16) float ws_smem[];
  __shared__ int s_last;
  const int D = a.D, E = a.E, HG = a.H / a.G, KW = a.G * D, VW = a.G * E;
  const int per_seq = a.splits + 1, split = blockIdx.x % per_seq, g = blockIdx.x / per_seq % a.G, seq = blockIdx.x / (per_seq * a.G);
  if (seq >= a.nseq) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *qs = ws_smem, *kn = qs + HG * D, *vn = kn + D, *ks = vn + E, *vs = ks + kWsKeys * (D + 1), *sc = vs + kWsKeys * E, *hm = sc + HG * kWsKeys,
        *hc = hm + HG, *hl = hc + HG, *acc = hl + HG;
  const int pos = a.Ctrl[4 * seq + CTRL_POS];
  const float *u = a.U + (size_t)seq * a.ldu;
  const float2 *rot = a.Rot + (size_t)pos * (a.rd >> 1);
  T *K = reinterpret_cast<T *>(a.Kc) + (size_t)seq * a.k_stride + (size_t)g * D, *V = reinterpret_cast<T *>(a.Vc) + (size_t)seq * a.v_stride + (size_t)g * E;
  T *Pk = reinterpret_cast<T *>(a.Pk) + (size_t)seq * a.pk_stride + (size_t)g * D, *Pv = reinterpret_cast<T *>(a.Pv) + (size_t)seq * a.pv_stride + (size_t)g * E;
  const bool fresh = a.koff >= 0;
  auto new_key = [&]() {   // warp 0: the key, warp 1: the value, as the cache holds them
    if (!fresh) return;
    if (warp == 0) head_norm_turn(u + a.koff + (size_t)g * D, D, a.KN, a.eps, rot, a.rd, [&](int d, float x, float y, bool both) { kn[d] = as_stored<T>(x); if (both) kn[d + 1] = as_stored<T>(y); });
    if (warp == 1)
      for (int d = lane; d < E; d += 32) vn[d] = as_stored<T>(u[a.voff + (size_t)g * E + d]);
  };
  if (split == a.splits) {
    const bool done = a.own_pool && a.pool > 0 && (pos + 1) % a.pool == 0;
    if (!fresh && !done) return;
    new_key();
    __syncthreads();
    for (int i = tid; i < D + E; i += kWsThreads) {
      const bool isv = i >= D;
      const int x = isv ? i - D : i, w = isv ? VW : KW;
      T *ring = (isv ? V : K) + x;
      if (fresh) st_val(ring + (size_t)(pos % a.cap) * w, isv ? vn[x] : kn[x]);
      if (done) {
        float s = 0.0f;
#pragma unroll 4
        for (int p = pos - a.pool + 1; p < pos; ++p) s += ld_val(ring + (size_t)(p % a.cap) * w);
        s += fresh ? (isv ? vn[x] : kn[x]) : ld_val(ring + (size_t)(pos % a.cap) * w);
        st_val((isv ? Pv : Pk) + (size_t)(pos / a.pool) * w + x, s / (float)a.pool);
      }
    }
    return;
  }
  const int lo = max(0, pos - a.window + 1), nb = a.Pk ? blocks_seen(pos, a.window, a.pool) : 0, n = nb + pos - lo + 1;
  const int per = max(kWsKeys, (n + a.splits - 1) / a.splits), active = (n + per - 1) / per;
  if (split >= active) return;
  const int j_lo = split * per, j_hi = min(n, j_lo + per);   // blocks 0..nb-1, then tokens lo..pos
  for (int hh = warp; hh < HG; hh += kWsThreads / 32)
    head_norm_turn(u + (size_t)(g * HG + hh) * D, D, a.QN, a.eps, rot, a.rd, [&](int d, float x, float y, bool both) { qs[hh * D + d] = x; if (both) qs[hh * D + d + 1] = y; });
  new_key();
  for (int i = tid; i < HG * E; i += kWsThreads) acc[i] = 0.0f;
  for (int i = tid; i < HG; i += kWsThreads) { hm[i] = -INFINITY; hl[i] = 0.0f; }
  __syncthreads();
  for (int t0 = j_lo; t0 < j_hi; t0 += kWsKeys) {
    const int nk = min(kWsKeys, j_hi - t0);
    for (int i = tid; i < nk * D; i += kWsThreads) {
      const int kk = i / D, d = i - kk * D, j = t0 + kk, p = lo + j - nb;
      ks[kk * (D + 1) + d] = j < nb ? ld_val(Pk + (size_t)j * KW + d) : fresh && p == pos ? kn[d] : ld_val(K + (size_t)(p % a.cap) * KW + d);
    }
    for (int i = tid; i < nk * E; i += kWsThreads) {
      const int kk = i / E, d = i - kk * E, j = t0 + kk, p = lo + j - nb;
      vs[kk * E + d] = j < nb ? ld_val(Pv + (size_t)j * VW + d) : fresh && p == pos ? vn[d] : ld_val(V + (size_t)(p % a.cap) * VW + d);
    }
    __syncthreads();
    {
      const int kk = tid & (kWsKeys - 1);
      for (int hh = tid / kWsKeys; hh < HG; hh += kWsThreads / kWsKeys) {
        float s = -INFINITY;
        if (kk < nk) {
          const float *q = qs + hh * D, *k = ks + kk * (D + 1);
          float d0 = 0.0f, d1 = 0.0f;
          int d = 0;
          for (; d + 1 < D; d += 2) { d0 = fmaf(q[d], k[d], d0); d1 = fmaf(q[d + 1], k[d + 1], d1); }
          if (d < D) d0 = fmaf(q[d], k[d], d0);
          s = cap_score((d0 + d1) * a.scale, a.softcap);
        }
        sc[hh * kWsKeys + kk] = s;
      }
    }
    __syncthreads();
    for (int hh = warp; hh < HG; hh += kWsThreads / 32) {
      const float s0 = sc[hh * kWsKeys + lane], s1 = sc[hh * kWsKeys + 32 + lane];
      const float mx = fmaxf(hm[hh], warp_max(fmaxf(s0, s1)));
      const float w0 = lane < nk ? expf(s0 - mx) : 0.0f, w1 = lane + 32 < nk ? expf(s1 - mx) : 0.0f;
      const float sum = warp_tree_sum(w0 + w1);
      sc[hh * kWsKeys + lane] = w0;
      sc[hh * kWsKeys + 32 + lane] = w1;
      __syncwarp();
      if (lane == 0) {
        const float corr = expf(hm[hh] - mx);
        hc[hh] = corr;
        hl[hh] = fmaf(hl[hh], corr, sum);
        hm[hh] = mx;
      }
    }
    __syncthreads();
    for (int i = tid; i < HG * E; i += kWsThreads) {
      const int hh = i / E, d = i - hh * E;
      float v = acc[i] * hc[hh];
      const float *w = sc + hh * kWsKeys;
      for (int kk = 0; kk < nk; ++kk) v = fmaf(w[kk], vs[kk * E + d], v);
      acc[i] = v;
    }
    __syncthreads();
  }
  auto put = [&](int hh, int d, float v, float m, float l) {   // sum, maximum and weight sum of a head
    const int c = (g * HG + hh) * E + d;
    if (a.Sink) l += expf(a.Sink[g * HG + hh] - m);
    v = v / l;
    if (a.goff >= 0) v = v * logistic(u[a.goff + c]);
    const size_t o = (size_t)seq * a.ldo + c;
    if (a.out16) reinterpret_cast<uint16_t *>(a.O)[o] = f32_to_bf16(v);
    else reinterpret_cast<float *>(a.O)[o] = v;
  };
  if (active == 1) {
    for (int i = tid; i < HG * E; i += kWsThreads) put(i / E, i % E, acc[i], hm[i / E], hl[i / E]);
    return;
  }
  const int per_head = E + 2;
  float *base = a.Part + ((size_t)seq * a.G + g) * a.splits * HG * (E + 4);
  float *mine = base + (size_t)split * HG * per_head;
  for (int i = tid; i < HG * E; i += kWsThreads) __stcg(mine + (size_t)(i / E) * per_head + 2 + i % E, acc[i]);
  for (int i = tid; i < HG; i += kWsThreads) { __stcg(mine + (size_t)i * per_head, hm[i]); __stcg(mine + (size_t)i * per_head + 1, hl[i]); }
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
  for (int hh = tid; hh < HG; hh += kWsThreads) {
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
  for (int i = tid; i < HG * E; i += kWsThreads) {
    const int hh = i / E, d = i - hh * E;
    float v = 0.0f;
    for (int s = 0; s < active; ++s) {
      const float *p = base + ((size_t)s * HG + hh) * per_head;
      v = fmaf(__ldcg(p + 2 + d), expf(__ldcg(p) - hm[hh]), v);
    }
    put(hh, d, v, hm[hh], hl[hh]);
  }
}
__global__ void __launch_bounds__(kWsThreads) WindowAttnStepF32(const WindowAttnStepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  window_attn_step_body<float>(a);
}
__global__ void __launch_bounds__(kWsThreads) WindowAttnStepB16(const WindowAttnStepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  window_attn_step_body<uint16_t>(a);
}
static uint32_t window_step_smem(const void *args) {
  const WindowAttnStepArgs *a = (const WindowAttnStepArgs *)args;
  return 4u * window_step_floats(a->H / a->G, a->D, a->E);
}
#define F(f) AINFER_ARG(WindowAttnStepArgs, f)
#define WAS_FIELDS                                                                                                                           \
  F(U), F(QN), F(KN), F(Rot), F(Ctrl), F(Kc), F(Vc), F(Pk), F(Pv), F(k_stride), F(v_stride), F(pk_stride), F(pv_stride), F(Sink), F(Part), \
      F(Count), F(O), F(nseq), F(H), F(G), F(D), F(E), F(rd), F(cap), F(window), F(pool), F(koff), F(voff), F(goff), F(own_pool), F(splits), \
      F(ldu), F(ldo), F(out16), F(scale), F(softcap), F(eps)
AINFER_REGISTER(WindowAttnStepF32, WindowAttnStepArgs, kWsThreads, 0, 0, window_step_smem, WAS_FIELDS);
AINFER_REGISTER(WindowAttnStepB16, WindowAttnStepArgs, kWsThreads, 0, 0, window_step_smem, WAS_FIELDS);
#undef F

AINFER_EARLY_LAUNCH(QkvRowsF32);
AINFER_EARLY_LAUNCH(QkvRowsB16);
AINFER_EARLY_LAUNCH(PoolRowsF32);
AINFER_EARLY_LAUNCH(PoolRowsB16);
AINFER_EARLY_LAUNCH(WindowAttnRowsF32);
AINFER_EARLY_LAUNCH(WindowAttnRowsB16);
AINFER_EARLY_LAUNCH(WindowAttnStepF32);
AINFER_EARLY_LAUNCH(WindowAttnStepB16);

}  // namespace ainfer
