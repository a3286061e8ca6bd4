// Residual streams (hyper-connections): the arithmetic one row needs between two sublayers.
//
// A row's residual is S vectors x_0 .. x_{S-1} of width W. A sublayer reads u = sum_s in[s] x_s and,
// given its output y, turns the streams into x'_t = sum_s mix[s][t] x_s + out[t] y. The update of one
// sublayer and the read of the next touch the same elements, so they run as one step per element:
// the S values are loaded once, updated, stored once, and the next sublayer's u falls out.
#pragma once
#include "row_types.cuh"

namespace ainfer {

constexpr int kMaxStreams = 16;

// Coefficients of one step, in shared memory: [0, S*S) mix (row = from), [S*S, S*S+S) out, then in [S].
struct StreamCoef {
  float mix[kMaxStreams * kMaxStreams], out[kMaxStreams], in[kMaxStreams];
};
// Mix / Out may be null (no pending update); In null: the plain sum of the streams.
__device__ __forceinline__ void load_stream_coef(StreamCoef &c, const float *Mix, const float *Out, const float *In, int S) {
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) c.mix[i] = Mix ? Mix[i] : 0.0f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    c.out[i] = Out ? Out[i] : 0.0f;
    c.in[i] = In ? In[i] : 1.0f;
  }
}

// V consecutive elements of a row (V = 4: 16-byte accesses, 1: single elements), ST streams. Returns
// u; writes the updated streams when dst != null.
template <int ST, int V>
__device__ __forceinline__ void stream_step(const float *src, const float *y, float *dst, const StreamCoef &c, int W, bool update, float (&u)[V]) {
  float x[ST][V];
#pragma unroll
  for (int s = 0; s < ST; ++s) {
    if constexpr (V == 4) {
      const float4 v = *reinterpret_cast<const float4 *>(src + (size_t)s * W);
      x[s][0] = v.x; x[s][1] = v.y; x[s][2] = v.z; x[s][3] = v.w;
    } else {
      x[s][0] = src[(size_t)s * W];
    }
  }
#pragma unroll
  for (int i = 0; i < V; ++i) u[i] = 0.0f;
  if (!update) {
#pragma unroll
    for (int s = 0; s < ST; ++s)
#pragma unroll
      for (int i = 0; i < V; ++i) u[i] = fmaf(c.in[s], x[s][i], u[i]);
    return;
  }
  float yv[V];
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4 *>(y);
    yv[0] = v.x; yv[1] = v.y; yv[2] = v.z; yv[3] = v.w;
  } else {
    yv[0] = y[0];
  }
#pragma unroll
  for (int t = 0; t < ST; ++t) {
    float a[V];
#pragma unroll
    for (int i = 0; i < V; ++i) a[i] = c.out[t] * yv[i];
#pragma unroll
    for (int s = 0; s < ST; ++s) {
      const float m = c.mix[s * ST + t];
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] = fmaf(m, x[s][i], a[i]);
    }
    if (dst) {
      if constexpr (V == 4) *reinterpret_cast<float4 *>(dst + (size_t)t * W) = make_float4(a[0], a[1], a[2], a[3]);
      else dst[(size_t)t * W] = a[0];
    }
#pragma unroll
    for (int i = 0; i < V; ++i) u[i] = fmaf(c.in[t], a[i], u[i]);
  }
}
// Any number of streams, one element.
__device__ __forceinline__ float stream_step_n(const float *src, const float *y, float *dst, const StreamCoef &c, int S, int W, bool update) {
  float u = 0.0f;
  if (!update) {
    for (int s = 0; s < S; ++s) u = fmaf(c.in[s], src[(size_t)s * W], u);
    return u;
  }
  for (int t = 0; t < S; ++t) {
    float a = c.out[t] * y[0];
    for (int s = 0; s < S; ++s) a = fmaf(c.mix[s * S + t], src[(size_t)s * W], a);
    if (dst) dst[(size_t)t * W] = a;
    u = fmaf(c.in[t], a, u);
  }
  return u;
}

// How a row's elements are dealt to threads: four consecutive ones each, or one.
__host__ __device__ __forceinline__ bool stream_vec(int S, int W) { return (W & 3) == 0 && S >= 1 && S <= 4; }

template <int ST>
__device__ __forceinline__ float stream_row(const float *src, const float *y, float *dst, const StreamCoef &c, int W, bool update, float *hs,
                                            int tid, int nth) {
  float ss = 0.0f;
  for (int w = tid * 4; w < W; w += nth * 4) {
    float u[4];
    stream_step<ST, 4>(src + w, y + w, dst ? dst + w : nullptr, c, W, update, u);
    *reinterpret_cast<float4 *>(hs + w) = make_float4(u[0], u[1], u[2], u[3]);
#pragma unroll
    for (int i = 0; i < 4; ++i) ss = fmaf(u[i], u[i], ss);
  }
  return ss;
}
// One row of W elements over nth threads: streams -> u in hs[] (each thread its own elements); returns
// this thread's sum of u^2.
__device__ __forceinline__ float stream_row_any(const float *src, const float *y, float *dst, const StreamCoef &c, int S, int W, bool update,
                                                float *hs, int tid, int nth) {
  if (stream_vec(S, W)) {
    if (S == 4) return stream_row<4>(src, y, dst, c, W, update, hs, tid, nth);
    if (S == 3) return stream_row<3>(src, y, dst, c, W, update, hs, tid, nth);
    if (S == 2) return stream_row<2>(src, y, dst, c, W, update, hs, tid, nth);
    return stream_row<1>(src, y, dst, c, W, update, hs, tid, nth);
  }
  float ss = 0.0f;
  for (int w = tid; w < W; w += nth) {
    const float u = stream_step_n(src + w, y + w, dst ? dst + w : nullptr, c, S, W, update);
    hs[w] = u;
    ss = fmaf(u, u, ss);
  }
  return ss;
}

}  // namespace ainfer
