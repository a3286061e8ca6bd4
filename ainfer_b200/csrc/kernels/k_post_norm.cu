// Layers that normalise a sublayer's output instead of its input: x <- x + norm(y) * gain, the next
// sublayer reads x itself. The residual x is fp32.
//
//   PostNormRowsF32/B16   rows: x update, and x (or its norm under a second gain) for the next product;
//                         y is one row per row, or the weighted sum of the rows a mixture's chosen
//                         experts left (a negative place: the identity, y = x)
//   PostNormStreamGemv    decode step: the same in the prologue of a GEMV; every block makes the row for
//                         itself, block 0 stores it
//   PolyNormRowsF32/B16   act = a n(z) + b n(z^2) + c n(z^3) + e, n = division by the row's root mean
//                         square, for rows
//   PolyStreamGemv        decode step: the same in the prologue of a GEMV
#include "row_types.cuh"
#include "stream_gemv.cuh"

namespace ainfer {

// -------------------------------------------------------- PostNormRows ---
struct PostNormRowsArgs {
  const float *X;          // [rows][W]
  const void *Y;           // [rows][W] fp32, or the experts' rows [...][W] in the type of H; null: no update
  const float *G;          // [W] gain of y's norm
  float *Xout;             // [rows][W]; null: not stored
  const int32_t *Place;    // [rows][top] row of Y, < 0: identity
  const float *PlaceW;     // [rows][top]
  const float *FinalG;     // [W] gain of a norm of the updated x; null: H = x
  const int32_t *Idx;      // input row of output row r (then Xout is null); null: r
  void *H;                 // [rows][ldh] output; null: none
  int32_t W, rows, top, ldh;   // top 0: Y has one row per row
  float eps;
};
constexpr int kPnMaxTop = 32;
template <typename T, int V>
__device__ __forceinline__ void post_norm_row(const PostNormRowsArgs &a, float *ys, float *red, const int *place, const float *pw) {
  const int W = a.W, tid = threadIdx.x, out = blockIdx.x, r = a.Idx ? a.Idx[out] : out;
  const float *x = a.X + (size_t)r * W;
  T *h = a.H ? reinterpret_cast<T *>(a.H) + (size_t)out * a.ldh : nullptr;
  auto load = [&](const auto *p, float (&v)[V]) {
    if constexpr (V == 4) { const float4 t = ld_val4(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
    else v[0] = ld_val(p);
  };
  float ss = 0.0f;
  if (a.Y) {
    for (int w = tid * V; w < W; w += 256 * V) {
      float y[V];
      if (a.top == 0) {
        load(reinterpret_cast<const float *>(a.Y) + (size_t)r * W + w, y);
      } else {
        float t[V];
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = 0.0f;
        for (int s = 0; s < a.top; ++s) {
          if (place[s] >= 0) load(reinterpret_cast<const T *>(a.Y) + (size_t)place[s] * W + w, t);
          else load(x + w, t);
#pragma unroll
          for (int i = 0; i < V; ++i) y[i] = fmaf(pw[s], t[i], y[i]);
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) { ys[w + i] = y[i]; ss = fmaf(y[i], y[i], ss); }
    }
    ss = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
  }
  const float inv = ss;
  float s2 = 0.0f;
  for (int w = tid * V; w < W; w += 256 * V) {   // every thread meets the elements it wrote
    float v[V], g[V];
    load(x + w, v);
    if (a.Y) {
      load(a.G + w, g);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = fmaf(ys[w + i] * inv, g[i], v[i]);
    }
    if (a.Xout) {
      float *o = a.Xout + (size_t)r * W + w;
      if constexpr (V == 4) st_val4(o, make_float4(v[0], v[1], v[2], v[3]));
      else *o = v[0];
    }
    if (a.FinalG) {
#pragma unroll
      for (int i = 0; i < V; ++i) { ys[w + i] = v[i]; s2 = fmaf(v[i], v[i], s2); }
    } else if (h) {
      if constexpr (V == 4) {
        if ((a.ldh & 3) == 0) { st_val4(h + w, make_float4(v[0], v[1], v[2], v[3])); continue; }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) st_val(h + w + i, v[i]);
    }
  }
  if (!a.FinalG || !h) return;
  const float inv2 = 1.0f / sqrtf(block_sum(s2, red) / (float)W + a.eps);
  for (int w = tid * V; w < W; w += 256 * V) {
    float g[V];
    load(a.FinalG + w, g);
#pragma unroll
    for (int i = 0; i < V; ++i) st_val(h + w + i, ys[w + i] * inv2 * g[i]);
  }
}
template <typename T>
__device__ __forceinline__ void post_norm_rows_body(const PostNormRowsArgs &a) {
  extern __shared__ __align__(16) float pn_smem[];   // [W]
  __shared__ float red[33], pw[kPnMaxTop];
  __shared__ int place[kPnMaxTop];
  pdl_wait();
  if (a.top > 0) {
    const int r = a.Idx ? a.Idx[blockIdx.x] : blockIdx.x;
    if (threadIdx.x < a.top) {
      place[threadIdx.x] = a.Place[(size_t)r * a.top + threadIdx.x];
      pw[threadIdx.x] = a.PlaceW[(size_t)r * a.top + threadIdx.x];
    }
    __syncthreads();
  }
  if ((a.W & 3) == 0) post_norm_row<T, 4>(a, pn_smem, red, place, pw);
  else post_norm_row<T, 1>(a, pn_smem, red, place, pw);
}
__global__ void __launch_bounds__(256) PostNormRowsF32(const PostNormRowsArgs a) {
  pdl_launch_dependents();
  post_norm_rows_body<float>(a);
}
__global__ void __launch_bounds__(256) PostNormRowsB16(const PostNormRowsArgs a) {
  pdl_launch_dependents();
  post_norm_rows_body<uint16_t>(a);
}
static uint32_t post_norm_rows_smem(const void *args) { return 4u * (uint32_t)((((const PostNormRowsArgs *)args)->W + 3) & ~3); }
#define F(f) AINFER_ARG(PostNormRowsArgs, f)
#define PN_FIELDS \
  F(X), F(Y), F(G), F(Xout), F(Place), F(PlaceW), F(FinalG), F(Idx), F(H), F(W), F(rows), F(top), F(ldh), F(eps)
AINFER_REGISTER(PostNormRowsF32, PostNormRowsArgs, 256, 1, 0, post_norm_rows_smem, PN_FIELDS);
AINFER_REGISTER(PostNormRowsB16, PostNormRowsArgs, 256, 1, 0, post_norm_rows_smem, PN_FIELDS);
#undef F

// -------------------------------------------------- PostNormStreamGemv ---
struct PostNormStreamGemvArgs {
  const float *X;          // [K]
  const float *Yp;         // [K] output of the sublayer whose norm is pending; null: none
  const float *G;          // [K] its gain
  float *Xout;             // [K] (another buffer than X); null: not stored
  const float *FinalG;     // [K] gain of a norm of the updated x; null: the product takes x
  const uint16_t *W;
  const float *Bias;       // [N] or null
  float *Y;                // [N]
  int32_t N, K, ldw, rows_pb, act;
  float eps, cap;
};
// Sum over the 8 consumer warps; every one of their threads gets it. red: 8 floats per use.
__device__ __forceinline__ float consumers_sum(float v, float *red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  v = warp_tree_sum(v);
  if (lane == 0) red[warp] = v;
  asm volatile("bar.sync 1, 256;" ::: "memory");
  return warp_tree_sum(lane < kSgWarps ? red[lane] : 0.0f);
}
__device__ __forceinline__ float sum_sq(const float4 v, float s) { return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, fmaf(v.x, v.x, s)))); }
__global__ void __launch_bounds__(kSgThreads, 3) PostNormStreamGemv(const PostNormStreamGemvArgs a) {
  __shared__ GemvShared sh;
  __shared__ float red[2][8];
  pdl_launch_dependents();
  const GemvDims d = gemv_dims(a.ldw);
  const GemvShape c{a.W, a.Bias, a.Y, a.N, a.ldw, a.rows_pb, a.act, a.cap};
  const int K = a.K, tid = threadIdx.x, nth = kSgWarps * 32;
  float *lo = reinterpret_cast<float *>(sg_smem + d.nst * d.stage_bytes), *hi = lo + a.ldw / 2, *part = hi + a.ldw / 2;
  gemv_init(&sh, d.nst);
  if (tid >= nth) {
    gemv_produce(c, d, &sh, sg_smem);
  } else {
    float *out = blockIdx.x == 0 ? a.Xout : nullptr;
    constexpr int Q = 4;   // quads of a thread that stay in registers
    float s2 = 0.0f;
    if ((K & 3) == 0 && K <= nth * 4 * Q) {
      float4 g[Q], x[Q], y[Q];
#pragma unroll
      for (int q = 0; q < Q; ++q) {   // the gain is a weight: it does not depend on the predecessor
        const int k = (q * nth + tid) * 4;
        g[q] = a.Yp && k < K ? ld_val4(a.G + k) : make_float4(0, 0, 0, 0);
      }
      pdl_wait();
      float ss = 0.0f;
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const int k = (q * nth + tid) * 4;
        x[q] = k < K ? ld_val4(a.X + k) : make_float4(0, 0, 0, 0);
        y[q] = a.Yp && k < K ? ld_val4(a.Yp + k) : make_float4(0, 0, 0, 0);
      }
#pragma unroll
      for (int q = 0; q < Q; ++q) ss = sum_sq(y[q], ss);
      const float inv = a.Yp ? 1.0f / sqrtf(consumers_sum(ss, red[0]) / (float)K + a.eps) : 0.0f;
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const int k = (q * nth + tid) * 4;
        if (a.Yp) {
          x[q].x = fmaf(y[q].x * inv, g[q].x, x[q].x); x[q].y = fmaf(y[q].y * inv, g[q].y, x[q].y);
          x[q].z = fmaf(y[q].z * inv, g[q].z, x[q].z); x[q].w = fmaf(y[q].w * inv, g[q].w, x[q].w);
        }
        if (out && k < K) st_val4(out + k, x[q]);
        s2 = sum_sq(x[q], s2);
      }
      if (a.FinalG) {
        const float i2 = 1.0f / sqrtf(consumers_sum(s2, red[1]) / (float)K + a.eps);
#pragma unroll
        for (int q = 0; q < Q; ++q) {
          const int k = (q * nth + tid) * 4;
          const float4 f = k < K ? ld_val4(a.FinalG + k) : make_float4(0, 0, 0, 0);
          x[q].x *= i2 * f.x; x[q].y *= i2 * f.y; x[q].z *= i2 * f.z; x[q].w *= i2 * f.w;
        }
      }
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const int k = (q * nth + tid) * 4;
        if (k < a.ldw) st_val4(((k & 4) ? hi : lo) + (k >> 3) * 4, x[q]);
      }
    } else {
      pdl_wait();
      float ss = 0.0f, inv = 0.0f;
      if (a.Yp) {
        for (int k = tid; k < K; k += nth) ss = fmaf(a.Yp[k], a.Yp[k], ss);
        inv = 1.0f / sqrtf(consumers_sum(ss, red[0]) / (float)K + a.eps);
      }
      auto value = [&](int k) { return a.Yp ? fmaf(a.Yp[k] * inv, a.G[k], a.X[k]) : a.X[k]; };
      float i2 = 1.0f;
      if (a.FinalG) {
        for (int k = tid; k < K; k += nth) { const float v = value(k); s2 = fmaf(v, v, s2); }
        i2 = 1.0f / sqrtf(consumers_sum(s2, red[1]) / (float)K + a.eps);
      }
      for (int k = tid; k < a.ldw; k += nth) {
        float v = 0.0f;
        if (k < K) {
          v = value(k);
          if (out) out[k] = v;
          if (a.FinalG) v = v * (i2 * a.FinalG[k]);
        }
        sg_put(lo, hi, k, v);
      }
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    gemv_consume(c, d, &sh, sg_smem, lo, hi, part);
  }
  __syncthreads();
  gemv_store(c, d, part);
}
static uint32_t post_norm_gemv_smem(const void *args) {
  const PostNormStreamGemvArgs *a = (const PostNormStreamGemvArgs *)args;
  return gemv_smem(a->ldw, a->rows_pb, 0);
}
#define F(f) AINFER_ARG(PostNormStreamGemvArgs, f)
AINFER_REGISTER(PostNormStreamGemv, PostNormStreamGemvArgs, kSgThreads, 0, 0, post_norm_gemv_smem, F(X), F(Yp), F(G), F(Xout), F(FinalG), F(W),
                F(Bias), F(Y), F(N), F(K), F(ldw), F(rows_pb), F(act), F(eps), F(cap));
#undef F

// ------------------------------------------------------------ PolyNorm ---
// act = z (k1 + z (k2 + z k3)) + e with k_p = coefficient / sqrt(mean z^2p + eps)
struct PolySums { float s1, s2, s3; };
__device__ __forceinline__ void poly_add(PolySums &s, float z) {
  const float z2 = z * z;
  s.s1 = s.s1 + z2;
  s.s2 = fmaf(z2, z2, s.s2);
  s.s3 = fmaf(z2 * z2, z2, s.s3);
}
__device__ __forceinline__ float poly_value(float z, float k1, float k2, float k3, float e) { return fmaf(z, fmaf(z, fmaf(z, k3, k2), k1), e); }

struct PolyNormRowsArgs {
  const void *Z;           // [rows][ldz]
  const float *Coef;       // a, b, c, e
  void *A;                 // [rows][lda]
  int32_t F, ldz, lda;
  float eps;
};
template <typename T>
__device__ __forceinline__ void poly_norm_rows_body(const PolyNormRowsArgs &a) {
  __shared__ float red[33];
  pdl_wait();
  const T *z = reinterpret_cast<const T *>(a.Z) + (size_t)blockIdx.x * a.ldz;
  T *o = reinterpret_cast<T *>(a.A) + (size_t)blockIdx.x * a.lda;
  const int F = a.F, tid = threadIdx.x;
  const bool vec = (F & 3) == 0 && (a.ldz & 3) == 0 && (a.lda & 3) == 0;
  constexpr int Q = 8;       // quads of a thread that stay in registers
  float4 keep[Q];
  PolySums s{0.0f, 0.0f, 0.0f};
  auto add4 = [&](const float4 v) { poly_add(s, v.x); poly_add(s, v.y); poly_add(s, v.z); poly_add(s, v.w); };
  if (vec) {
#pragma unroll
    for (int q = 0; q < Q; ++q) {
      const int f = (q * 256 + tid) * 4;
      keep[q] = f < F ? ld_val4(z + f) : make_float4(0, 0, 0, 0);
    }
#pragma unroll
    for (int q = 0; q < Q; ++q) add4(keep[q]);
    for (int f = (Q * 256 + tid) * 4; f < F; f += 1024) add4(ld_val4(z + f));
  } else {
    for (int f = tid; f < F; f += 256) poly_add(s, ld_val(z + f));
  }
  const float n = (float)F;
  const float k1 = a.Coef[0] / sqrtf(block_sum(s.s1, red) / n + a.eps), k2 = a.Coef[1] / sqrtf(block_sum(s.s2, red) / n + a.eps),
              k3 = a.Coef[2] / sqrtf(block_sum(s.s3, red) / n + a.eps), e = a.Coef[3];
  auto val4 = [&](const float4 v) {
    return make_float4(poly_value(v.x, k1, k2, k3, e), poly_value(v.y, k1, k2, k3, e), poly_value(v.z, k1, k2, k3, e), poly_value(v.w, k1, k2, k3, e));
  };
  if (vec) {
#pragma unroll
    for (int q = 0; q < Q; ++q) {
      const int f = (q * 256 + tid) * 4;
      if (f < F) st_val4(o + f, val4(keep[q]));
    }
    for (int f = (Q * 256 + tid) * 4; f < F; f += 1024) st_val4(o + f, val4(ld_val4(z + f)));
  } else {
    for (int f = tid; f < F; f += 256) st_val(o + f, poly_value(ld_val(z + f), k1, k2, k3, e));
  }
}
__global__ void __launch_bounds__(256) PolyNormRowsF32(const PolyNormRowsArgs a) {
  pdl_launch_dependents();
  poly_norm_rows_body<float>(a);
}
__global__ void __launch_bounds__(256) PolyNormRowsB16(const PolyNormRowsArgs a) {
  pdl_launch_dependents();
  poly_norm_rows_body<uint16_t>(a);
}
#define F(f) AINFER_ARG(PolyNormRowsArgs, f)
AINFER_REGISTER(PolyNormRowsF32, PolyNormRowsArgs, 256, 1, 0, nullptr, F(Z), F(Coef), F(A), F(F), F(ldz), F(lda), F(eps));
AINFER_REGISTER(PolyNormRowsB16, PolyNormRowsArgs, 256, 1, 0, nullptr, F(Z), F(Coef), F(A), F(F), F(ldz), F(lda), F(eps));
#undef F

struct PolyStreamGemvArgs {
  const float *Z;          // [K]
  const float *Coef;       // a, b, c, e
  const uint16_t *W;
  float *Y;                // [N]
  int32_t N, K, ldw, rows_pb;
  float eps;
};
__global__ void __launch_bounds__(kSgThreads, 3) PolyStreamGemv(const PolyStreamGemvArgs a) {
  __shared__ GemvShared sh;
  __shared__ float red[3][8];
  pdl_launch_dependents();
  const GemvDims d = gemv_dims(a.ldw);
  const GemvShape c{a.W, nullptr, a.Y, a.N, a.ldw, a.rows_pb, ACT_NONE, 0.0f};
  const int K = a.K, tid = threadIdx.x, nth = kSgWarps * 32;
  float *lo = reinterpret_cast<float *>(sg_smem + d.nst * d.stage_bytes), *hi = lo + a.ldw / 2, *part = hi + a.ldw / 2;
  gemv_init(&sh, d.nst);
  if (tid >= nth) {
    gemv_produce(c, d, &sh, sg_smem);
  } else {
    const float ca = a.Coef[0], cb = a.Coef[1], cc = a.Coef[2], e = a.Coef[3];
    pdl_wait();
    PolySums s{0.0f, 0.0f, 0.0f};
    const bool vec = (K & 7) == 0;   // then ldw = K
    if (vec) {
      for (int k = tid * 4; k < K; k += nth * 4) {
        const float4 z = ld_val4(a.Z + k);
        poly_add(s, z.x); poly_add(s, z.y); poly_add(s, z.z); poly_add(s, z.w);
        st_val4(((k & 4) ? hi : lo) + (k >> 3) * 4, z);
      }
    } else {
      for (int k = tid; k < a.ldw; k += nth) {
        const float z = k < K ? a.Z[k] : 0.0f;
        poly_add(s, z);
        sg_put(lo, hi, k, z);
      }
    }
    const float n = (float)K;
    const float k1 = ca / sqrtf(consumers_sum(s.s1, red[0]) / n + a.eps), k2 = cb / sqrtf(consumers_sum(s.s2, red[1]) / n + a.eps),
                k3 = cc / sqrtf(consumers_sum(s.s3, red[2]) / n + a.eps);
    if (vec) {
      for (int k = tid * 4; k < K; k += nth * 4) {
        float *p = ((k & 4) ? hi : lo) + (k >> 3) * 4;
        const float4 z = ld_val4(p);
        st_val4(p, make_float4(poly_value(z.x, k1, k2, k3, e), poly_value(z.y, k1, k2, k3, e), poly_value(z.z, k1, k2, k3, e),
                               poly_value(z.w, k1, k2, k3, e)));
      }
    } else {
      for (int k = tid; k < K; k += nth) {
        float *p = ((k & 4) ? hi : lo) + (k >> 3) * 4 + (k & 3);
        *p = poly_value(*p, k1, k2, k3, e);
      }
    }
    asm volatile("bar.sync 1, 256;" ::: "memory");
    gemv_consume(c, d, &sh, sg_smem, lo, hi, part);
  }
  __syncthreads();
  gemv_store(c, d, part);
}
static uint32_t poly_gemv_smem(const void *args) {
  const PolyStreamGemvArgs *a = (const PolyStreamGemvArgs *)args;
  return gemv_smem(a->ldw, a->rows_pb, 0);
}
#define F(f) AINFER_ARG(PolyStreamGemvArgs, f)
AINFER_REGISTER(PolyStreamGemv, PolyStreamGemvArgs, kSgThreads, 0, 0, poly_gemv_smem, F(Z), F(Coef), F(W), F(Y), F(N), F(K), F(ldw), F(rows_pb),
                F(eps));
#undef F

AINFER_EARLY_LAUNCH(PostNormRowsF32);
AINFER_EARLY_LAUNCH(PostNormRowsB16);
AINFER_EARLY_LAUNCH(PostNormStreamGemv);
AINFER_EARLY_LAUNCH(PolyNormRowsF32);
AINFER_EARLY_LAUNCH(PolyNormRowsB16);
AINFER_EARLY_LAUNCH(PolyStreamGemv);

}  // namespace ainfer
