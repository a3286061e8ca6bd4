// Attention over a sliding window of tokens and, beside it, one mean key and value per block of `pool`
// tokens that lies wholly before the window; all in one softmax, whose denominator may have one more
// term per head (a sink). Scores may be capped: cap tanh(score / cap).
//
//   row i sees the tokens j with 0 <= i - j < window, and the blocks b with (b + 1) pool - 1 <= i - window
//
// The tokens of a sequence are a ring of `cap` positions (position p in slot p % cap; cap is a multiple
// of 64 and holds a window, a block and the rows of a pass), the blocks an array. A block is averaged
// when its last token arrives, from the keys and values as the ring holds them; it becomes visible
// `window` positions later.
#pragma once
#include "row_types.cuh"

namespace ainfer {

// Blocks that row i sees.
__device__ __forceinline__ int blocks_seen(int i, int window, int pool) {
  if (pool <= 0 || i - window + 1 < pool) return 0;
  return (i - window + 1) / pool;
}
__device__ __forceinline__ float cap_score(float s, float cap) { return cap > 0.0f ? cap * tanhf(s / cap) : s; }

// Neighbouring values (d even) of a row; as one access where the row is aligned to pairs.
__device__ __forceinline__ void st_pair(float *p, float x, float y, bool both) {
  if (both && (reinterpret_cast<unsigned long long>(p) & 7) == 0) *reinterpret_cast<float2 *>(p) = make_float2(x, y);
  else { p[0] = x; if (both) p[1] = y; }
}
__device__ __forceinline__ void st_pair(uint16_t *p, float x, float y, bool both) {
  if (both && (reinterpret_cast<unsigned long long>(p) & 3) == 0)
    *reinterpret_cast<uint32_t *>(p) = (uint32_t)f32_to_bf16(x) | ((uint32_t)f32_to_bf16(y) << 16);
  else { p[0] = f32_to_bf16(x); if (both) p[1] = f32_to_bf16(y); }
}

// One warp: a head's D values at src, divided by their root mean square and times w (w null: as they
// are), then the first rd of them turned in neighbouring pairs by rot (cosine, sine per pair);
// put(d, x, y, both): values d and d + 1, the second only if `both`. D <= 512.
constexpr int kHeadPairs = 8;   // pairs of a lane
template <typename P>
__device__ __forceinline__ void head_norm_turn(const float *src, int D, const float *w, float eps, const float2 *rot, int rd, P put) {
  const int lane = threadIdx.x & 31;
  float2 v[kHeadPairs];
  float ss = 0.0f;
  const bool wide = (reinterpret_cast<unsigned long long>(src) & 7) == 0;
#pragma unroll
  for (int i = 0; i < kHeadPairs; ++i) {
    const int d = (i * 32 + lane) * 2;
    v[i] = make_float2(0.0f, 0.0f);
    if (d + 1 < D && wide) v[i] = *reinterpret_cast<const float2 *>(src + d);
    else {
      if (d < D) v[i].x = src[d];
      if (d + 1 < D) v[i].y = src[d + 1];
    }
    if (i * 64 >= D) break;
  }
#pragma unroll
  for (int i = 0; i < kHeadPairs; ++i) {
    if (i * 64 >= D) break;
    ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, ss));
  }
  const float inv = w ? 1.0f / sqrtf(warp_tree_sum(ss) / (float)D + eps) : 1.0f;
#pragma unroll
  for (int i = 0; i < kHeadPairs; ++i) {
    if (i * 64 >= D) break;
    const int d = (i * 32 + lane) * 2;
    float x = v[i].x, y = v[i].y;
    if (w) {
      if (d < D) x = x * inv * w[d];
      if (d + 1 < D) y = y * inv * w[d + 1];
    }
    if (d < rd) {
      const float2 r = rot[d >> 1];
      const float t = x * r.x - y * r.y;
      y = y * r.x + x * r.y;
      x = t;
    }
    if (d < D) put(d, x, y, d + 1 < D);
  }
}

}  // namespace ainfer
