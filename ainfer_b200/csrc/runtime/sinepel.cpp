// Sinepel: pre-norm decoder whose residual is several streams mixed around every sublayer
// (hyper-connections), with a token shift on the mixer's input, short convolutions on q and k,
// chunk-local attention in which the keys are also the values (learned temperature and logarithmic
// distance penalty per head), squared-ReLU feed-forward, learned positions and capped logits.
//
// This file holds what is particular to it: configuration, tensor list, prepared weights, and the
// sequence of launches of a row pass and of a decode step (RowEngine). The mechanisms are kernels of
// their own with their constants as arguments: k_hyper.cu, k_chunk_attn.cu, k_linear.cu,
// k_linear_tc.cu, k_chunk_mma.cu.
#include <algorithm>
#include <cmath>
#include <cstring>

#include "json.h"
#include "row_engine.h"
#include "../common/detmath.h"

namespace ainfer {

namespace {

// ---------------------------------------------------------------- configuration ---
bool parse(const Json &js, ModelConfig &c, std::string &err) {
  auto bad = [&](const std::string &m) { err = "config: " + m; return false; };
  c = ModelConfig();
  c.arch = "Sinepel";
  c.hidden = js.at("width").integer(0);
  c.vocab = js.at("vocab").integer(0);
  c.streams = js.at("streams").integer(1);
  c.max_positions = js.at("max_positions").integer(0);
  c.rms_eps = js.at("norm").at("eps").num(-1);
  c.embed_scale = js.at("embedding").at("scale").num(1.0);
  c.logit_softcap = js.at("logit_softcap").num(0.0);
  if (js.at("layers").kind != Json::ARR) return bad("no list of layers");
  for (const Json &l : js.at("layers").a) {
    RowLayerConfig r;
    if (l.at("type").str() != "attention") return bad("unknown layer type \"" + l.at("type").str() + "\"");
    const Json &x = l.at("mixer");
    r.heads = x.at("heads").integer(0);
    r.kv_heads = x.at("kv_heads").integer(0);
    r.dim = x.at("dim").integer(0);
    r.taps = x.at("conv").integer(0);
    r.scale = x.at("scale").num(NAN);
    r.chunk = x.at("mask").at("size").integer(0);
    if (x.at("vdim").integer(r.dim) != r.dim) return bad("the keys are the values, so vdim must equal dim");
    const Json &f = l.at("mlp");
    if (!f.is_null()) {
      if (f.at("kind").str() != "dense") return bad("unknown feed-forward \"" + f.at("kind").str() + "\"");
      r.ff = f.at("ff").integer(0);
      if (r.ff < 1) return bad("feed-forward without a size");
    }
    c.row_layers.push_back(r);
  }
  c.layers = (int)c.row_layers.size();
  return true;
}

std::string to_json(const ModelConfig &c) {
  std::string s = "{\"architecture\":\"Sinepel\",\"embedding\":{\"scale\":" + json_num(c.embed_scale) + "},\"layers\":[";
  for (size_t i = 0; i < c.row_layers.size(); ++i) {
    const RowLayerConfig &r = c.row_layers[i];
    s += (i ? "," : "") + std::string("{\"mixer\":{\"conv\":") + std::to_string(r.taps) + ",\"dim\":" + std::to_string(r.dim) +
         ",\"heads\":" + std::to_string(r.heads) + ",\"kv_heads\":" + std::to_string(r.kv_heads) + ",\"mask\":{\"size\":" +
         std::to_string(r.chunk) + "},\"scale\":" + json_num(r.scale) + ",\"vdim\":" + std::to_string(r.dim) + "},\"mlp\":" +
         (r.ff ? "{\"ff\":" + std::to_string(r.ff) + ",\"kind\":\"dense\"}" : std::string("null")) + ",\"type\":\"attention\"}";
  }
  return s + "],\"logit_softcap\":" + json_num(c.logit_softcap) + ",\"max_positions\":" + std::to_string(c.max_positions) +
         ",\"norm\":{\"eps\":" + json_num(c.rms_eps) + "},\"streams\":" + std::to_string(c.streams) + ",\"vocab\":" + std::to_string(c.vocab) +
         ",\"width\":" + std::to_string(c.hidden) + "}";
}

bool check(const ModelConfig &c, std::string &err) {
  auto bad = [&](const std::string &m) { err = "unsupported architecture: " + m; return false; };
  if (c.row_layers.empty()) return bad("no layers");
  if (c.hidden < 1 || c.hidden > 16384) return bad("width must be in [1, 16384]");
  if (c.vocab < 1) return bad("vocab");
  if (c.streams < 1 || c.streams > 16) return bad("streams must be in [1, 16]");
  if (c.max_positions < 1) return bad("max_positions");
  if (!(c.rms_eps >= 0)) return bad("norm.eps");
  for (const RowLayerConfig &r : c.row_layers) {
    if (r.heads < 1 || r.kv_heads < 1 || r.heads % r.kv_heads) return bad("heads must be a multiple of kv_heads");
    if (r.dim < 1 || r.dim > 512) return bad("dim must be in [1, 512]");
    if (r.taps < 1 || r.taps > 64) return bad("conv must be in [1, 64] taps");
    if (r.chunk < 0) return bad("mask.size");
    if (!std::isfinite(r.scale)) return bad("mixer.scale");
    if (r.ff > 24576 || r.heads * r.dim > 24576) return bad("a layer's inner size exceeds 24576");
    // shared memory of the decode step's attention: queries, sums, a tile of keys, scores
    const long hg = r.heads / r.kv_heads;
    if (4 * (2 * hg * r.dim + r.dim + 64L * (r.dim + 1) + 64 * hg + 3 * hg) > 220 * 1024) return bad("too many query heads per key head at this dim");
  }
  return true;
}

// Every tensor with its shape, in storage order (q directly before k: one matrix when rows align).
std::vector<RowTensor> tensors(const ModelConfig &c) {
  std::vector<RowTensor> t;
  const uint64_t W = c.hidden, S = c.streams, V = c.vocab;
  auto add = [&](const std::string &n, std::vector<uint64_t> sh, float sd, float cst) { t.push_back({n, sh, sd, cst}); };
  add("embed", {V, W}, 0.5f, 0);
  add("pos", {(uint64_t)c.max_positions, W}, 0.5f, 0);
  for (int L = 0; L < c.layers; ++L) {
    const RowLayerConfig &r = c.row_layers[L];
    const std::string p = layer_name(L), x = p + "mix.";
    const uint64_t Q = (uint64_t)r.heads * r.dim, K = (uint64_t)r.kv_heads * r.dim, J = r.taps, H = r.heads, F = r.ff;
    const float iw = 1.0f / std::sqrt((float)W);
    add(p + "norm1", {W}, 0, 1);
    add(x + "q", {Q, W}, iw, 0);
    add(x + "k", {K, W}, iw, 0);
    add(x + "q.b", {Q}, 0.02f, 0);
    add(x + "k.b", {K}, 0.02f, 0);
    add(x + "q.conv", {Q, J}, 0.5f, 0);
    add(x + "k.conv", {K, J}, 0.5f, 0);
    add(x + "r1", {H}, 0, 0.5f);
    add(x + "r2", {H}, 0, 0.5f);
    add(x + "temp", {H}, 0, 1);
    add(x + "o", {W, Q}, 1.0f / std::sqrt((float)Q), 0);
    add(p + "shift", {W}, 0, 0.25f);
    for (int q = 1; q <= (F ? 2 : 1); ++q) {
      const std::string h = p + "hc" + std::to_string(q) + ".";
      add(h + "in", {S}, 0, 1.0f / (float)S);
      add(h + "out", {S}, 0, 1);
      add(h + "mix", {S, S}, 0.2f, 0);
    }
    if (F) {
      add(p + "norm2", {W}, 0, 1);
      add(p + "mlp.up", {F, W}, iw, 0);
      add(p + "mlp.down", {W, F}, 1.0f / std::sqrt((float)F), 0);
    }
  }
  add("final.norm", {W}, 0, 1);
  add("head", {V, W}, 1.0f / std::sqrt((float)W), 0);
  return t;
}

void plan(const ModelConfig &c, Container &dir, std::vector<SynthSpec> &specs) { plan_row_tensors(tensors(c), to_json(c), c.vocab, dir, specs); }
int check_directory(const Container &dir, const ModelConfig &c, std::string &err) { return check_row_tensors(dir, tensors(c), err); }

}  // namespace

// ------------------------------------------------------------- prepared weights ---
struct RowSublayer { const float *in, *out, *mix, *norm; };
struct RowLayerWeights {
  RowMatrix qk, o, up, down;
  RowSublayer sub[2];
  const float *shift, *conv /* [taps][C] */, *temp, *lb /* [H][lb_len] */;
  int lb_len;
};
struct SinepelWeights : RowWeights {
  std::vector<RowLayerWeights> L;
  RowMatrix head;
  const float *final_norm = nullptr;
  const uint16_t *embed = nullptr, *pos = nullptr;
};

namespace {

int prepare(DeviceModel *m, std::string &err) {
  const ModelConfig &c = m->cfg;
  auto w = std::make_shared<SinepelWeights>();
  RowLoader k(m, &err);
  for (int L = 0; L < c.layers && !k.status; ++L) {
    const RowLayerConfig &r = c.row_layers[L];
    const std::string p = layer_name(L), x = p + "mix.";
    const int Q = r.heads * r.dim, Kn = r.kv_heads * r.dim, C = Q + Kn;
    RowLayerWeights lw{};
    lw.qk = k.stack({x + "q", x + "k"});
    std::vector<float> bias((size_t)C), conv((size_t)C * r.taps);
    int at = 0;
    for (const char *n : {"q", "k"}) {
      const auto b = k.host(x + n + ".b"), cv = k.host(x + n + std::string(".conv"));
      for (size_t i = 0; i < b.size(); ++i) {
        bias[(size_t)at + i] = bf16_to_f32(b[i]);
        for (int j = 0; j < r.taps; ++j) conv[(size_t)j * C + at + i] = bf16_to_f32(cv[i * r.taps + j]);
      }
      at += (int)b.size();
    }
    lw.qk.bias = k.upload(bias);
    lw.conv = k.upload(conv);
    lw.o = k.stack({x + "o"});
    lw.temp = k.widen(x + "temp");
    // distances that occur: below the chunk length and below the number of positions
    lw.lb_len = r.chunk ? std::min(r.chunk, c.max_positions) : c.max_positions;
    float *lb = (float *)k.alloc((size_t)r.heads * lw.lb_len * 4);
    const float *r1 = k.widen(x + "r1"), *r2 = k.widen(x + "r2");
    if (!k.status) k.launch("LogDistanceTable", 1024, lb, r1, r2, (int32_t)r.heads, (int32_t)lw.lb_len);
    lw.lb = lb;
    lw.shift = k.widen(p + "shift");
    for (int q = 0; q < (r.ff ? 2 : 1); ++q) {
      const std::string h = p + "hc" + std::to_string(q + 1) + ".";
      lw.sub[q].in = k.widen(h + "in");
      lw.sub[q].out = k.widen(h + "out");
      lw.sub[q].mix = k.widen(h + "mix");
      lw.sub[q].norm = k.widen(p + (q ? "norm2" : "norm1"));
    }
    if (r.ff) {
      lw.up = k.stack({p + "mlp.up"});
      lw.down = k.stack({p + "mlp.down"});
    }
    w->L.push_back(lw);
  }
  if (!k.status) {
    w->head = k.stack({"head"});
    w->final_norm = k.widen("final.norm");
    w->embed = (const uint16_t *)m->tensor("embed").data;
    w->pos = (const uint16_t *)m->tensor("pos").data;
  }
  k.finish();
  m->rows = w;
  return k.status;
}

// ------------------------------------------------------------------- row engine ---
struct TailRecord {   // SeqTailLayer of k_hyper.cu
  const float *pend_shift;
  float *shift;
  const float *pend_conv;
  float *conv;
  int32_t C, taps;
};

struct Engine : RowEngineBase {
  const SinepelWeights *w;
  struct LayerState { float *shift, *conv, *pend_shift, *pend_conv; char *k; int cap, chunk; };
  std::vector<LayerState> st;
  char *state = nullptr;
  size_t state_bytes = 0, k_off = 0, conv_off = 0;
  // pass buffers
  float *X[2] = {nullptr, nullptr}, *U = nullptr, *Y = nullptr, *AttPart = nullptr;
  char *H = nullptr, *Q = nullptr, *Att = nullptr, *Act = nullptr;
  uint32_t *AttCount = nullptr;
  void *tail_rows = nullptr, *tail_steps = nullptr;
  int ldw = 0, ldq = 0, ldf = 0, maxC = 0, att_splits = 1;
  // recording of a decode step
  int cur = 0;
  const RowSublayer *pending = nullptr;

  int create(DeviceModel *model, int n, int ctx, int cap_rows, bool in_f32, std::string &err) override {
    if (begin(model, n, ctx, cap_rows, in_f32, err)) return 1;
    w = static_cast<const SinepelWeights *>(m->rows.get());
    const ModelConfig &c = m->cfg;
    const size_t W = c.hidden, S = c.streams, R = rows_cap;
    int maxQ = 1, maxF = 1, maxHGD = 1, maxG = 1;
    // one block of state: shift rows, convolution rings, key rings, layer after layer
    size_t off = 0;
    auto take = [&](size_t bytes) { const size_t o = off; off += (bytes + 255) / 256 * 256; return o; };
    std::vector<size_t> so, co, ko;
    for (int L = 0; L < c.layers; ++L) so.push_back(take((size_t)nseq * 2 * W * 4));
    conv_off = off;
    for (const RowLayerConfig &r : c.row_layers) co.push_back(take((size_t)nseq * r.taps * (r.heads + r.kv_heads) * r.dim * 4));
    k_off = off;
    for (const RowLayerConfig &r : c.row_layers) {
      LayerState s{};
      s.chunk = r.chunk ? r.chunk : c.max_positions;
      // keys of the current chunk plus those of a pass; a multiple of the attention kernels' key tile
      s.cap = round_up((int)std::min<long>(max_ctx, (long)s.chunk + rows_cap), 128);
      ko.push_back(take((size_t)nseq * s.cap * r.kv_heads * r.dim * esz()));
      st.push_back(s);
      maxQ = std::max(maxQ, r.heads * r.dim);
      maxF = std::max(maxF, r.ff);
      maxC = std::max(maxC, (r.heads + r.kv_heads) * r.dim);
      maxG = std::max(maxG, r.kv_heads);
      maxHGD = std::max(maxHGD, r.heads * (r.dim + 4));
    }
    state_bytes = off;
    int e = alloc(state_bytes, &state);
    std::vector<TailRecord> tr, ts;
    for (int L = 0; L < c.layers && !e; ++L) {
      const RowLayerConfig &r = c.row_layers[L];
      LayerState &s = st[L];
      const int C = (r.heads + r.kv_heads) * r.dim;
      s.shift = (float *)(state + so[L]);
      s.conv = (float *)(state + co[L]);
      s.k = state + ko[L];
      e |= alloc((size_t)nseq * W, &s.pend_shift);
      e |= alloc((size_t)nseq * r.taps * C, &s.pend_conv);
      tr.push_back({s.pend_shift, s.shift, s.pend_conv, s.conv, C, r.taps});
      ts.push_back({s.pend_shift, s.shift, nullptr, nullptr, C, 1});   // steps keep their convolution ring themselves
    }
    ldw = round_up((int)W, 8); ldq = round_up(maxQ, 8); ldf = round_up(maxF, 8);
    att_splits = step_splits(maxG);
    for (int i = 0; i < 2; ++i) e |= alloc(R * S * W, &X[i]);
    e |= alloc(R * ldw * esz(), &H); e |= alloc(R * maxC, &U); e |= alloc(R * ldq * esz(), &Q);
    e |= alloc(R * ldq * 4, &Att); e |= alloc(R * W, &Y); e |= alloc(R * ldf * 4, &Act);
    e |= alloc((size_t)nseq * att_splits * maxHGD, &AttPart);
    e |= alloc((size_t)nseq * maxG, &AttCount);
    TailRecord *d = nullptr;
    e |= alloc(tr.size(), &d); tail_rows = d;
    if (!e) e |= ainfer_memcpy_h2d(dev, d, tr.data(), tr.size() * sizeof(TailRecord)) != AINFER_OK;
    e |= alloc(ts.size(), &d); tail_steps = d;
    if (!e) e |= ainfer_memcpy_h2d(dev, d, ts.data(), ts.size() * sizeof(TailRecord)) != AINFER_OK;
    if (e) { err = "row engine: " + (alloc_err.empty() ? std::string(ainfer_last_error(dev)) : alloc_err); return 1; }
    return 0;
  }
  int reset(std::string &err) override {
    if (ainfer_mem_fill(dev, state, 0, state_bytes) != AINFER_OK) { err = ainfer_last_error(dev); return 1; }
    return 0;
  }
  bool buffer(const std::string &which, void **p, uint64_t *n) override {
    if (which == "state") { *p = state; *n = state_bytes; }
    else if (which == "shift") { *p = state; *n = conv_off; }
    else if (which == "conv") { *p = state + conv_off; *n = k_off - conv_off; }
    else if (which == "Kc") { *p = state + k_off; *n = state_bytes - k_off; }
    else return false;
    return true;
  }

  // stream update of the pending sublayer (if any), then the read + norm (+ shift) of the next
  void hyper(KernelCalls &k, const RowSpan &sp, const float *in, const float *norm, const RowLayerWeights *lw, const LayerState *s, int rows,
             const int32_t *idx, bool store) {
    const ModelConfig &c = m->cfg;
    // a run of rows per block when rows are plentiful: the token shift re-reads one row per run
    const int per = lw ? std::max(1, std::min(8, rows / (2 * sm_count))) : 1;
    k.launch(f32 ? "HyperNormRowsF32" : "HyperNormRowsB16", (uint32_t)((rows + per - 1) / per), (const float *)X[cur],
             (const float *)(pending ? Y : nullptr), (const float *)(pending ? pending->mix : nullptr),
             (const float *)(pending ? pending->out : nullptr), (float *)(pending && store ? X[cur ^ 1] : nullptr), in, norm,
             (const float *)(lw ? lw->shift : nullptr), (const float *)(s ? s->shift : nullptr), (float *)(s ? s->pend_shift : nullptr), sp.ctrl,
             sp.seq, sp.first, idx, (void *)H, (int32_t)c.hidden, (int32_t)c.streams, (int32_t)rows, (int32_t)per, (int32_t)ldw, (float)c.rms_eps);
    if (pending && store) { cur ^= 1; pending = nullptr; }
  }

  void emit(KernelCalls &k, const RowSpan &sp) override {
    const ModelConfig &c = m->cfg;
    const int R = sp.rows, W = c.hidden;
    const bool b16 = !f32;
    cur = 0;
    pending = nullptr;
    k.launch("EmbedPosRows", (uint32_t)R, X[0], w->embed, w->pos, sp.ctrl, (int32_t)W, (int32_t)c.vocab, (int32_t)c.max_positions,
             (int32_t)c.streams, (float)c.embed_scale);
    for (int L = 0; L < c.layers && !k.status; ++L) {
      const RowLayerConfig &r = c.row_layers[L];
      const RowLayerWeights &lw = w->L[L];
      const LayerState &s = st[L];
      const int C = (r.heads + r.kv_heads) * r.dim, Qc = r.heads * r.dim;
      const int64_t kv_stride = (int64_t)s.cap * r.kv_heads * r.dim;
      const int ldo = round_up(Qc, 8);
      hyper(k, sp, lw.sub[0].in, lw.sub[0].norm, &lw, &s, R, nullptr, true);
      linear(k, lw.qk, H, ldw, R, U, C, ACT_NONE, false);
      if (sp.one_sequence) {
        const int per = std::max(1, std::min(8, R / 16));
        const int cblk = C % 4 == 0 && Qc % 4 == 0 && r.taps >= 2 && r.taps <= 4 ? 1024 : 256;   // channels of a block
        k.launch(f32 ? "ShortConvRowsF32" : "ShortConvRowsB16", (uint32_t)(((R + per - 1) / per) * ((C + cblk - 1) / cblk)), (const float *)U, lw.conv,
                 (const float *)s.conv, s.pend_conv, sp.ctrl, sp.seq, sp.first, (void *)Q, (void *)s.k, kv_stride, (int32_t)R, (int32_t)C,
                 (int32_t)Qc, (int32_t)r.taps, (int32_t)s.cap, (int32_t)C, (int32_t)per);
        if (mma_dim(r))
          k.launch(sized("ChunkAttnMma", r.dim).c_str(), (uint32_t)(((R + 63) / 64) * r.heads), (const uint16_t *)Q, (const uint16_t *)s.k, lw.lb,
                   lw.temp, sp.ctrl, (uint16_t *)Att, (int32_t)R, (int32_t)r.heads, (int32_t)r.kv_heads, (int32_t)r.dim, (int32_t)s.cap,
                   (int32_t)s.chunk, (int32_t)lw.lb_len, (int32_t)ldo, (float)r.scale);
        else
          k.launch(f32 ? "ChunkAttnRowsF32" : "ChunkAttnRowsB16", (uint32_t)(((R + 15) / 16) * r.heads), (const void *)Q, (const void *)s.k, lw.lb,
                   lw.temp, sp.ctrl, (void *)Att, (int32_t)R, (int32_t)r.heads, (int32_t)r.kv_heads, (int32_t)r.dim, (int32_t)s.cap,
                   (int32_t)s.chunk, (int32_t)lw.lb_len, (int32_t)ldo, (float)r.scale);
      } else {
        attn_step(k, r, lw, s, sp.ctrl, R, C, ldo, b16);
      }
      linear(k, lw.o, Att, ldo, R, Y, W, ACT_NONE, false);
      pending = &lw.sub[0];
      if (r.ff) {
        const int ldx = round_up(r.ff, 8);
        hyper(k, sp, lw.sub[1].in, lw.sub[1].norm, nullptr, nullptr, R, nullptr, true);
        linear(k, lw.up, H, ldw, R, Act, ldx, ACT_RELU2, b16);
        linear(k, lw.down, Act, ldx, R, Y, W, ACT_NONE, false);
        pending = &lw.sub[1];
      }
    }
    if (sp.n_want > 0) {
      hyper(k, sp, nullptr, w->final_norm, nullptr, nullptr, sp.n_want, sp.want, false);
      linear(k, w->head, H, ldw, sp.n_want, sp.logits, c.vocab, c.logit_softcap > 0 ? ACT_SOFTCAP : ACT_NONE, false, (float)c.logit_softcap);
    }
    const int row0 = sp.one_sequence ? R - 1 : 0;   // the first row that may be its sequence's last
    k.launch("SeqTailCommit", (uint32_t)(c.layers * (R - row0)), (const void *)(sp.one_sequence ? tail_rows : tail_steps), sp.ctrl, sp.seq, sp.first,
             (int32_t)c.layers, (int32_t)R, (int32_t)W, (int32_t)row0);
  }

  // head sizes the tensor-core attention takes (bf16)
  bool mma_dim(const RowLayerConfig &r) const { return !f32 && r.dim % 8 == 0 && r.dim <= 256; }
  void attn_step(KernelCalls &k, const RowLayerConfig &r, const RowLayerWeights &lw, const LayerState &s, const int32_t *ctrl, int n, int C, int ldo,
                 bool out16) {
    const std::string name = mma_dim(r) && r.heads / r.kv_heads <= 16 ? sized("ChunkAttnStepMma", r.dim)
                                                                      : std::string(f32 ? "ChunkAttnStepF32" : "ChunkAttnStepB16");
    k.launch(name.c_str(), (uint32_t)(n * r.kv_heads * att_splits), (const float *)U, lw.conv, s.conv, ctrl,
             (void *)s.k, (int64_t)s.cap * r.kv_heads * r.dim, lw.lb, lw.temp, AttPart, AttCount, (void *)Att, (int32_t)n, (int32_t)r.heads,
             (int32_t)r.kv_heads, (int32_t)r.dim, (int32_t)r.taps, (int32_t)s.cap, (int32_t)s.chunk, (int32_t)lw.lb_len, (int32_t)att_splits,
             (int32_t)C, (int32_t)ldo, (int32_t)(out16 ? 1 : 0), (float)r.scale);
  }

  // ---- one decode step of sequence 0 ----
  void hyper_gemv(KernelCalls &k, const RowMatrix &mt, const float *in, const float *norm, const float *shift, float *shift_state,
                  const int32_t *ctrl, float *y, int act, float cap) {
    const ModelConfig &c = m->cfg;
    const int rows_pb = gemv_rows(mt.N);
    k.launch("HyperStreamGemv", gemv_blocks(mt.N), (const float *)X[cur], (const float *)(pending ? Y : nullptr),
             (const float *)(pending ? pending->mix : nullptr), (const float *)(pending ? pending->out : nullptr),
             (float *)(pending ? X[cur ^ 1] : nullptr), in, norm, shift, shift_state, ctrl, mt.w, mt.bias, y, (int32_t)c.streams, (int32_t)mt.N,
             (int32_t)mt.K, (int32_t)mt.ldw, (int32_t)rows_pb, (int32_t)act, (float)c.rms_eps, cap);
    if (pending) { cur ^= 1; pending = nullptr; }
  }
  void record_embed(KernelCalls &k, const int32_t *ctrl) override {
    const ModelConfig &c = m->cfg;
    cur = 0;
    pending = nullptr;
    k.launch("EmbedPosRows", 1, X[0], w->embed, w->pos, ctrl, (int32_t)c.hidden, (int32_t)c.vocab, (int32_t)c.max_positions, (int32_t)c.streams,
             (float)c.embed_scale);
  }
  void record_layer(KernelCalls &k, int L, const int32_t *ctrl) override {
    const ModelConfig &c = m->cfg;
    const RowLayerConfig &r = c.row_layers[L];
    const RowLayerWeights &lw = w->L[L];
    const LayerState &s = st[L];
    const int C = (r.heads + r.kv_heads) * r.dim;
    hyper_gemv(k, lw.qk, lw.sub[0].in, lw.sub[0].norm, lw.shift, s.shift, ctrl, U, ACT_NONE, 0.0f);
    attn_step(k, r, lw, s, ctrl, 1, C, r.heads * r.dim, false);
    gemv(k, lw.o, (const float *)Att, Y, ACT_NONE);
    pending = &lw.sub[0];
    if (r.ff) {
      hyper_gemv(k, lw.up, lw.sub[1].in, lw.sub[1].norm, nullptr, nullptr, ctrl, (float *)Act, ACT_RELU2, 0.0f);
      gemv(k, lw.down, (const float *)Act, Y, ACT_NONE);
      pending = &lw.sub[1];
    }
  }
  void record_residual(KernelCalls &k, float *dst) override {
    k.launch("StreamSumRows", 1, (const float *)X[cur], (const float *)(pending ? Y : nullptr), (const float *)(pending ? pending->mix : nullptr),
             (const float *)(pending ? pending->out : nullptr), dst, (int32_t)m->cfg.hidden, (int32_t)m->cfg.streams);
  }
  void record_head(KernelCalls &k, float *logits) override {
    const ModelConfig &c = m->cfg;
    hyper_gemv(k, w->head, nullptr, w->final_norm, nullptr, nullptr, nullptr, logits, c.logit_softcap > 0 ? ACT_SOFTCAP : ACT_NONE,
               (float)c.logit_softcap);
  }
};

}  // namespace

const ModelArch *sinepel_model_arch() {
  static const ModelArch a = {"Sinepel", false, parse, to_json, check, plan, check_directory, prepare, []() -> RowEngine * { return new Engine; }};
  return &a;
}

bool sinepel_preset(const std::string &name, ModelConfig &c) {
  auto layer = [](int heads, int kv_heads, int dim, int taps, int chunk, int ff) {
    RowLayerConfig r;
    r.heads = heads; r.kv_heads = kv_heads; r.dim = dim; r.taps = taps; r.chunk = chunk; r.ff = ff;
    r.scale = 1.0 / std::sqrt((double)dim);
    return r;
  };
  c = ModelConfig();
  c.arch = "Sinepel";
  c.logit_softcap = 30.0;
  if (name == "sinepel-tiny") {
    c.hidden = 96; c.vocab = 512; c.streams = 3; c.max_positions = 1024;
    c.row_layers = {layer(4, 2, 32, 3, 48, 160), layer(6, 2, 16, 2, 100, 0), layer(3, 1, 40, 4, 32, 128)};
  } else if (name == "sinepel-small") {
    c.hidden = 2048; c.vocab = 32000; c.streams = 4; c.max_positions = 8192;
    c.row_layers.assign(4, layer(16, 4, 128, 4, 2048, 8192));
  } else {
    return false;
  }
  c.layers = (int)c.row_layers.size();
  return true;
}

}  // namespace ainfer
