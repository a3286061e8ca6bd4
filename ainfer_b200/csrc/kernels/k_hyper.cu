// Row kernels of models with several residual streams: embedding with a learned position vector,
// the fused step between two sublayers (stream update of the one, weighted read + RMS norm +
// optional token shift of the other), and the commit of what a sequence carries over a pass.
//
// Rows of a pass: row r belongs to sequence Seq[r], its position is Ctrl[4 r + 1], and First[r] is
// the first row of the same sequence in this pass; rows of a sequence are consecutive. Nothing of a
// sequence's carried state is written while a pass still reads it: the pass leaves its last rows in
// pending buffers and SeqTailCommit, the pass's last launch, moves them into the state.
#include "hyper_core.cuh"

namespace ainfer {

// x_s[row] = Emb[token] * scale + Pos[position], the same in every stream.
struct EmbedPosRowsArgs {
  float *X;               // [rows][S][W]
  const uint16_t *Emb;    // [V][W] bf16
  const uint16_t *Pos;    // [P][W] bf16, or null
  const int32_t *Ctrl;    // [rows][4]
  int32_t W, V, P, S;
  float scale;
};
__global__ void __launch_bounds__(256) EmbedPosRows(const EmbedPosRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  int tok = a.Ctrl[4 * row + CTRL_TOKEN], pos = a.Ctrl[4 * row + CTRL_POS];
  tok = tok < 0 ? 0 : (tok >= a.V ? a.V - 1 : tok);
  pos = pos < 0 ? 0 : (pos >= a.P ? a.P - 1 : pos);
  const uint16_t *e = a.Emb + (size_t)tok * a.W, *p = a.Pos ? a.Pos + (size_t)pos * a.W : nullptr;
  float *x = a.X + (size_t)row * a.S * a.W;
  for (int w = threadIdx.x; w < a.W; w += 256) {
    float v = bf16_to_f32(e[w]) * a.scale;
    if (p) v = v + bf16_to_f32(p[w]);
    for (int s = 0; s < a.S; ++s) x[(size_t)s * a.W + w] = v;
  }
}
#define F(f) AINFER_ARG(EmbedPosRowsArgs, f)
AINFER_REGISTER(EmbedPosRows, EmbedPosRowsArgs, 256, 1, 0, nullptr, F(X), F(Emb), F(Pos), F(Ctrl), F(W), F(V), F(P), F(S), F(scale));
#undef F

struct HyperNormRowsArgs {
  const float *Xin;        // [rows][S][W]
  const float *Y;          // [rows][W] output of the sublayer whose update is pending; null: none
  const float *Mix, *Out;  // [S][S] (from, to), [S] of that sublayer
  float *Xout;             // [rows][S][W] updated streams (another buffer than Xin); null: not stored
  const float *In;         // [S] of the sublayer that reads; null: plain sum
  const float *NormW;      // [W]
  const float *Shift;      // [W] token-shift amounts; null: no shift
  const float *State;      // [seq][2][W]: normalised row of position p in slot p & 1 (unshifted); null without shift
  float *Pend;             // [seq][W] the sequence's last normalised row of this pass; null without shift
  const int32_t *Ctrl, *Seq, *First;
  const int32_t *Idx;      // input row of output row r (only without shift and without stored streams); null: r
  void *H;                 // [rows][ldh] output
  int32_t W, S, rows, per, ldh;   // per: rows of a block
  float eps;
};

template <typename T>
__device__ __forceinline__ void hyper_norm_body(const HyperNormRowsArgs &a) {
  extern __shared__ __align__(16) float hy_smem[];   // [2][W rounded to 4]
  __shared__ StreamCoef coef;
  __shared__ float red[33];
  const int W = a.W, Wp = (W + 3) & ~3, tid = threadIdx.x;
  load_stream_coef(coef, a.Mix, a.Out, a.In, a.S);   // weights: they do not depend on the predecessor
  pdl_wait();
  __syncthreads();
  const bool update = a.Y != nullptr;
  const int r0 = blockIdx.x * a.per, r1 = min(a.rows, r0 + a.per);
  float *prev = hy_smem, *cur = hy_smem + Wp;
  T *H = reinterpret_cast<T *>(a.H);
  const bool vec = stream_vec(a.S, W);
  auto norm_row = [&](int r, bool own, float *hs) {
    if (a.Idx) r = a.Idx[r];
    const float *src = a.Xin + (size_t)r * a.S * W;
    float *dst = own && a.Xout ? a.Xout + (size_t)r * a.S * W : nullptr;
    const float ss = stream_row_any(src, a.Y + (update ? (size_t)r * W : 0), dst, coef, a.S, W, update, hs, tid, 256);
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps);
    // every thread touches only the elements it wrote
    if (vec) {
      for (int w = tid * 4; w < W; w += blockDim.x * 4)
#pragma unroll
        for (int i = 0; i < 4; ++i) hs[w + i] = hs[w + i] * inv * a.NormW[w + i];
    } else {
      for (int w = tid; w < W; w += blockDim.x) hs[w] = hs[w] * inv * a.NormW[w];
    }
  };
  auto each = [&](auto f) {
    if (vec) {
      for (int w = tid * 4; w < W; w += blockDim.x * 4)
#pragma unroll
        for (int i = 0; i < 4; ++i) f(w + i);
    } else {
      for (int w = tid; w < W; w += blockDim.x) f(w);
    }
  };
  bool have_prev = false;
  if (a.Shift && r0 < r1 && a.First[r0] != r0) {   // the row before the block's first: no stores
    norm_row(r0 - 1, false, prev);
    have_prev = true;
  }
  for (int r = r0; r < r1; ++r) {
    int seq = 0, pos = 0, fr = 0, fn = 0;
    if (a.Shift) {
      seq = a.Seq[r]; pos = a.Ctrl[4 * r + CTRL_POS]; fr = a.First[r];
      fn = r + 1 == a.rows ? r + 1 : a.First[r + 1];
    }
    norm_row(r, true, cur);
    T *h = H + (size_t)r * a.ldh;
    if (!a.Shift) {
      each([&](int w) { st_val(h + w, cur[w]); });
      continue;
    }
    if (fr == r || !have_prev) {
      const float *st = a.State + ((size_t)seq * 2 + ((pos - 1) & 1)) * W;
      each([&](int w) { prev[w] = pos > 0 ? st[w] : 0.0f; });
    }
    each([&](int w) { st_val(h + w, fmaf(prev[w] - cur[w], a.Shift[w], cur[w])); });
    if (fn == r + 1) {
      float *pd = a.Pend + (size_t)seq * W;
      each([&](int w) { pd[w] = cur[w]; });
    }
    float *t = prev; prev = cur; cur = t;
    have_prev = true;
  }
}
__global__ void __launch_bounds__(256) HyperNormRowsF32(const HyperNormRowsArgs a) {
  pdl_launch_dependents();
  hyper_norm_body<float>(a);
}
__global__ void __launch_bounds__(256) HyperNormRowsB16(const HyperNormRowsArgs a) {
  pdl_launch_dependents();
  hyper_norm_body<uint16_t>(a);
}
static uint32_t hyper_norm_smem_fn(const void *args) { return 2u * 4u * (uint32_t)((((const HyperNormRowsArgs *)args)->W + 3) & ~3); }
#define F(f) AINFER_ARG(HyperNormRowsArgs, f)
#define HYPER_FIELDS                                                                                                            \
  F(Xin), F(Y), F(Mix), F(Out), F(Xout), F(In), F(NormW), F(Shift), F(State), F(Pend), F(Ctrl), F(Seq), F(First), F(Idx), F(H), F(W), \
      F(S), F(rows), F(per), F(ldh), F(eps)
AINFER_REGISTER(HyperNormRowsF32, HyperNormRowsArgs, 256, 0, 0, hyper_norm_smem_fn, HYPER_FIELDS);
AINFER_REGISTER(HyperNormRowsB16, HyperNormRowsArgs, 256, 0, 0, hyper_norm_smem_fn, HYPER_FIELDS);
#undef F

// Dst[row] = sum of the row's streams after a pending update (diagnostics: the residual a layer leaves).
struct StreamSumRowsArgs {
  const float *X, *Y, *Mix, *Out;   // Y null: no pending update
  float *Dst;                       // [rows][W]
  int32_t W, S;
};
__global__ void __launch_bounds__(256) StreamSumRows(const StreamSumRowsArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ StreamCoef coef;
  load_stream_coef(coef, a.Mix, a.Out, nullptr, a.S);
  __syncthreads();
  const size_t row = blockIdx.x;
  for (int w = threadIdx.x; w < a.W; w += 256)
    a.Dst[row * a.W + w] = stream_step_n(a.X + row * a.S * a.W + w, a.Y + (a.Y ? row * a.W + w : 0), nullptr, coef, a.S, a.W, a.Y != nullptr);
}
#define F(f) AINFER_ARG(StreamSumRowsArgs, f)
AINFER_REGISTER(StreamSumRows, StreamSumRowsArgs, 256, 1, 0, nullptr, F(X), F(Y), F(Mix), F(Out), F(Dst), F(W), F(S));
#undef F

// Moves a pass's last rows of every sequence into its state, all layers in one launch: the shift row
// of the sequence's last position q into slot q & 1, and the projections of the last taps - 1
// positions (as far as the pass holds them) into slots position % taps. One block per (layer, row from
// row0 on); rows that are not their sequence's last do nothing.
struct SeqTailLayer {
  const float *pend_shift;   // [seq][W]
  float *shift;              // [seq][2][W]
  const float *pend_conv;    // [seq][taps][C]
  float *conv;               // [seq][taps][C]
  int32_t C, taps;
};
struct SeqTailCommitArgs {
  const SeqTailLayer *L;
  const int32_t *Ctrl, *Seq, *First;
  int32_t layers, rows, W, row0;
};
__global__ void __launch_bounds__(256) SeqTailCommit(const SeqTailCommitArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int n_rows = a.rows - a.row0, l = blockIdx.x / n_rows, r = a.row0 + blockIdx.x % n_rows;
  if (l >= a.layers) return;
  if (r + 1 < a.rows && a.First[r + 1] != r + 1) return;
  const SeqTailLayer L = a.L[l];
  const int seq = a.Seq[r], q = a.Ctrl[4 * r + CTRL_POS], n = r - a.First[r] + 1;
  for (int w = threadIdx.x; w < a.W; w += 256) L.shift[((size_t)seq * 2 + (q & 1)) * a.W + w] = L.pend_shift[(size_t)seq * a.W + w];
  for (int i = 0; i < L.taps - 1 && i < n; ++i) {
    const size_t o = ((size_t)seq * L.taps + (q - i) % L.taps) * L.C;
    for (int c = threadIdx.x; c < L.C; c += 256) L.conv[o + c] = L.pend_conv[o + c];
  }
}
#define F(f) AINFER_ARG(SeqTailCommitArgs, f)
AINFER_REGISTER(SeqTailCommit, SeqTailCommitArgs, 256, 1, 0, nullptr, F(L), F(Ctrl), F(Seq), F(First), F(layers), F(rows), F(W), F(row0));
#undef F

AINFER_EARLY_LAUNCH(EmbedPosRows);
AINFER_EARLY_LAUNCH(HyperNormRowsF32);
AINFER_EARLY_LAUNCH(HyperNormRowsB16);
AINFER_EARLY_LAUNCH(SeqTailCommit);
AINFER_EARLY_LAUNCH(StreamSumRows);

}  // namespace ainfer
