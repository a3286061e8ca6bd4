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

#include "arch.h"
#include "json.h"
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

std::string num(double v) {
  char b[40];
  std::snprintf(b, sizeof b, "%.17g", v);
  return b;
}

std::string to_json(const ModelConfig &c) {
  std::string s = "{\"architecture\":\"Sinepel\",\"embedding\":{\"scale\":" + num(c.embed_scale) + "},\"layers\":[";
  for (size_t i = 0; i < c.row_layers.size(); ++i) {
    const RowLayerConfig &r = c.row_layers[i];
    s += (i ? "," : "") + std::string("{\"mixer\":{\"conv\":") + std::to_string(r.taps) + ",\"dim\":" + std::to_string(r.dim) +
         ",\"heads\":" + std::to_string(r.heads) + ",\"kv_heads\":" + std::to_string(r.kv_heads) + ",\"mask\":{\"size\":" +
         std::to_string(r.chunk) + "},\"scale\":" + num(r.scale) + ",\"vdim\":" + std::to_string(r.dim) + "},\"mlp\":" +
         (r.ff ? "{\"ff\":" + std::to_string(r.ff) + ",\"kind\":\"dense\"}" : std::string("null")) + ",\"type\":\"attention\"}";
  }
  return s + "],\"logit_softcap\":" + num(c.logit_softcap) + ",\"max_positions\":" + std::to_string(c.max_positions) +
         ",\"norm\":{\"eps\":" + num(c.rms_eps) + "},\"streams\":" + std::to_string(c.streams) + ",\"vocab\":" + std::to_string(c.vocab) +
         ",\"width\":" + std::to_string(c.hidden) + "}";
}

int round_up(int v, int m) { return (v + m - 1) / m * m; }

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

std::string layer_name(int L) { return "l" + std::to_string(L) + "."; }

// Every tensor with its shape, in storage order (q directly before k: one matrix when rows align).
struct Named { std::string name; std::vector<uint64_t> shape; float std_, constant; };
std::vector<Named> tensors(const ModelConfig &c) {
  std::vector<Named> t;
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

void plan(const ModelConfig &c, Container &dir, std::vector<SynthSpec> &specs) {
  dir = Container();
  specs.clear();
  for (const Named &n : tensors(c)) {
    TensorEntry e;
    e.name = n.name;
    e.ndim = (int)n.shape.size();
    for (int i = 0; i < e.ndim; ++i) e.shape[i] = n.shape[i];
    e.logical = e.storage = DT_BF16;
    e.d_bytes = e.numel() * 2;
    dir.index[e.name] = dir.entries.size();
    dir.entries.push_back(e);
    SynthSpec sp;
    sp.std_ = n.std_;
    sp.constant = n.constant;
    specs.push_back(sp);
  }
  dir.identity_json =
      "{\"converter\":\"ainfer_b200 synthetic writer\",\"converter_version\":\"1.0\",\"created_date\":\"1970-01-01\",\"source_repo\":"
      "\"synthetic\",\"source_revision\":\"0000000000000000000000000000000000000000\",\"source_total_bytes\":0}";
  dir.arch_json = to_json(c);
  dir.tokenizer_json = "{\"format\":\"none\",\"vocab_size\":" + std::to_string(c.vocab) + "}";
  dir.policy_json = "{\"default\":\"BF16\"}";
  container_layout(dir);
}

int check_directory(const Container &dir, const ModelConfig &c, std::string &err) {
  for (const Named &n : tensors(c)) {
    const TensorEntry *e = dir.find(n.name);
    if (!e) { err = "missing " + n.name; return 1; }
    if (e->storage != DT_BF16) { err = "unexpected storage of " + n.name; return 2; }
    bool same = e->ndim == (int)n.shape.size();
    for (int i = 0; same && i < e->ndim; ++i) same = e->shape[i] == n.shape[i];
    if (!same) { err = "unexpected shape of " + n.name; return 2; }
  }
  return 0;
}

}  // namespace

// ------------------------------------------------------------- prepared weights ---
struct RowMatrix {           // bf16 rows of ldw values (ldw a multiple of 8, zero padding)
  const uint16_t *w = nullptr;
  const float *bias = nullptr;
  int N = 0, K = 0, ldw = 0;
};
struct RowSublayer { const float *in, *out, *mix, *norm; };
struct RowLayerWeights {
  RowMatrix qk, o, up, down;
  RowSublayer sub[2];
  const float *shift, *conv /* [taps][C] */, *temp, *lb /* [H][lb_len] */;
  int lb_len;
};
struct RowWeights {
  std::vector<RowLayerWeights> L;
  RowMatrix head;
  const float *final_norm = nullptr;
  const uint16_t *embed = nullptr, *pos = nullptr;
};

namespace {

int prepare(DeviceModel *m, std::string &err) {
  const ModelConfig &c = m->cfg;
  ainfer_device_t dev = m->dev;
  auto w = std::make_shared<RowWeights>();
  std::map<std::string, ainfer_kernel_t> kernels;
  KernelCalls k(dev, &kernels, &err);
  auto alloc = [&](size_t bytes) -> void * {
    void *p = nullptr;
    if (k.status) return nullptr;
    if (ainfer_mem_alloc(dev, std::max<size_t>(bytes, 16), 256, &p) != AINFER_OK) { k.fail(1, ainfer_last_error(dev)); return nullptr; }
    m->owned.push_back(p);
    return p;
  };
  auto widen = [&](const std::string &name) -> const float * {
    DeviceTensor t = m->tensor(name);
    const uint64_t n = t.entry->numel();
    float *p = (float *)alloc(n * 4);
    if (p) k.launch("WidenBf16", (uint32_t)std::min<uint64_t>((n + 255) / 256, 1024), p, (const void *)t.data, n);
    return p;
  };
  // rows of one or two tensors as one matrix; copied only when rows need padding or the two do not adjoin
  auto matrix = [&](const std::string &a, const std::string &b) {
    DeviceTensor ta = m->tensor(a), tb = b.empty() ? DeviceTensor() : m->tensor(b);
    RowMatrix r;
    const int Na = (int)ta.entry->shape[0], Nb = b.empty() ? 0 : (int)tb.entry->shape[0];
    r.K = (int)ta.entry->shape[1];
    r.N = Na + Nb;
    r.ldw = round_up(r.K, 8);
    if (r.ldw == r.K && (b.empty() || (char *)ta.data + (size_t)Na * r.K * 2 == (char *)tb.data)) {
      r.w = (const uint16_t *)ta.data;
      return r;
    }
    uint16_t *p = (uint16_t *)alloc((size_t)r.N * r.ldw * 2);
    r.w = p;
    if (!p) return r;
    k.launch("PackRowsBf16", (uint32_t)std::min(Na, 4096), p, (const uint16_t *)ta.data, (int32_t)Na, (int32_t)r.K, (int32_t)r.ldw);
    if (Nb)
      k.launch("PackRowsBf16", (uint32_t)std::min(Nb, 4096), p + (size_t)Na * r.ldw, (const uint16_t *)tb.data, (int32_t)Nb, (int32_t)r.K,
               (int32_t)r.ldw);
    return r;
  };
  auto host_bf16 = [&](const std::string &name) {
    DeviceTensor t = m->tensor(name);
    std::vector<uint16_t> v(t.entry->numel());
    if (ainfer_memcpy_d2h(dev, v.data(), t.data, v.size() * 2) != AINFER_OK) k.fail(1, ainfer_last_error(dev));
    return v;
  };
  auto upload = [&](const std::vector<float> &v) -> const float * {
    float *p = (float *)alloc(v.size() * 4);
    if (p && ainfer_memcpy_h2d(dev, p, v.data(), v.size() * 4) != AINFER_OK) k.fail(1, ainfer_last_error(dev));
    return p;
  };
  for (int L = 0; L < c.layers && !k.status; ++L) {
    const RowLayerConfig &r = c.row_layers[L];
    const std::string p = layer_name(L), x = p + "mix.";
    const int Q = r.heads * r.dim, Kn = r.kv_heads * r.dim, C = Q + Kn;
    RowLayerWeights lw{};
    lw.qk = matrix(x + "q", x + "k");
    std::vector<float> bias((size_t)C), conv((size_t)C * r.taps);
    int at = 0;
    for (const char *n : {"q", "k"}) {
      const auto b = host_bf16(x + n + ".b"), cv = host_bf16(x + n + std::string(".conv"));
      for (size_t i = 0; i < b.size(); ++i) {
        bias[(size_t)at + i] = bf16_to_f32(b[i]);
        for (int j = 0; j < r.taps; ++j) conv[(size_t)j * C + at + i] = bf16_to_f32(cv[i * r.taps + j]);
      }
      at += (int)b.size();
    }
    lw.qk.bias = upload(bias);
    lw.conv = upload(conv);
    lw.o = matrix(x + "o", "");
    lw.temp = widen(x + "temp");
    // distances that occur: below the chunk length and below the number of positions
    lw.lb_len = r.chunk ? std::min(r.chunk, c.max_positions) : c.max_positions;
    float *lb = (float *)alloc((size_t)r.heads * lw.lb_len * 4);
    const float *r1 = widen(x + "r1"), *r2 = widen(x + "r2");
    if (!k.status) k.launch("LogDistanceTable", 1024, lb, r1, r2, (int32_t)r.heads, (int32_t)lw.lb_len);
    lw.lb = lb;
    lw.shift = widen(p + "shift");
    for (int q = 0; q < (r.ff ? 2 : 1); ++q) {
      const std::string h = p + "hc" + std::to_string(q + 1) + ".";
      lw.sub[q].in = widen(h + "in");
      lw.sub[q].out = widen(h + "out");
      lw.sub[q].mix = widen(h + "mix");
      lw.sub[q].norm = widen(p + (q ? "norm2" : "norm1"));
    }
    if (r.ff) {
      lw.up = matrix(p + "mlp.up", "");
      lw.down = matrix(p + "mlp.down", "");
    }
    w->L.push_back(lw);
  }
  if (!k.status) {
    w->head = matrix("head", "");
    w->final_norm = widen("final.norm");
    w->embed = (const uint16_t *)m->tensor("embed").data;
    w->pos = (const uint16_t *)m->tensor("pos").data;
    if (!k.status && ainfer_sync(dev, UINT64_MAX) != AINFER_OK) k.fail(1, ainfer_last_error(dev));
  }
  for (auto &kv : kernels) ainfer_kernel_release(kv.second);
  m->rows = w;
  return k.status;
}

const ModelArch kModel = {"Sinepel", false, parse, to_json, check, plan, check_directory, prepare};

// ------------------------------------------------------------------- row engine ---
struct alignas(64) TensorMap { unsigned char b[128]; };
enum { ACT_NONE = 0, ACT_RELU2 = 1, ACT_SOFTCAP = 2 };

struct TailRecord {   // SeqTailLayer of k_hyper.cu
  const float *pend_shift;
  float *shift;
  const float *pend_conv;
  float *conv;
  int32_t C, taps;
};

struct Engine : RowEngine {
  DeviceModel *m;
  ainfer_device_t dev;
  const RowWeights *w;
  int nseq, max_ctx, sm_count = 1;
  bool f32;
  std::vector<void *> owned;
  std::string alloc_err;
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

  size_t esz() const { return f32 ? 4 : 2; }

  template <typename T>
  int alloc(size_t count, T **out) {
    void *p = nullptr;
    const size_t bytes = std::max<size_t>(count * sizeof(T), 16);
    if (ainfer_mem_alloc(dev, bytes, 256, &p) != AINFER_OK || ainfer_mem_fill(dev, p, 0, bytes) != AINFER_OK) {
      alloc_err = ainfer_last_error(dev);
      return 1;
    }
    owned.push_back(p);
    *out = (T *)p;
    return 0;
  }

  int create(DeviceModel *model, int n, int ctx, int cap_rows, bool in_f32, std::string &err) {
    m = model; dev = m->dev; w = m->rows.get();
    nseq = n; f32 = in_f32;
    const ModelConfig &c = m->cfg;
    max_ctx = std::min(ctx, c.max_positions);
    rows_cap = std::max(1, cap_rows);
    ainfer_device_info info;
    if (ainfer_device_get_info(dev, &info) != AINFER_OK) { err = ainfer_last_error(dev); return 1; }
    sm_count = info.sm_count;
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
    // blocks of a step's attention over sequences, key heads and splits: few tiles each when there are many sequences
    att_splits = nseq == 1 ? std::max(1, std::min(16, 2 * sm_count / maxG)) : std::max(1, std::min(16, 8 * sm_count / (std::min(nseq, 8 * sm_count) * maxG)));
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
  ~Engine() override {
    ainfer_sync(dev, UINT64_MAX);
    for (void *p : owned) ainfer_mem_free(dev, p);
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

  // Y[rows][N] = act(X W^T + bias); X in the activation type, out16: Y bf16 (else fp32)
  void linear(KernelCalls &k, const RowMatrix &mt, const char *Xp, int ldx, int rows, void *Yp, int ldy, int act, bool out16, float cap = 0.0f) {
    if (k.status) return;
    if (f32) {
      k.launch("LinearRows", (uint32_t)(((mt.N + 63) / 64) * ((rows + 63) / 64)), (const float *)Xp, mt.w, mt.bias, (float *)Yp, (int32_t)rows,
               (int32_t)mt.N, (int32_t)mt.K, (int32_t)ldx, (int32_t)mt.ldw, (int32_t)ldy, (int32_t)act, cap);
      return;
    }
    const int n_tiles = (mt.N + 127) / 128, kb = (mt.K + 63) / 64;
    int nt = rows <= 16 ? 16 : rows <= 32 ? 32 : rows <= 64 ? 64 : 128;
    if (rows > 128) {
      // rows of a tile: as large as possible (operand traffic), but a launch lasts whole rounds of tiles over the SMs
      long best = -1;
      for (int t = 256; t >= 96; t -= 16) {
        const long rounds = ((long)n_tiles * ((rows + t - 1) / t) + sm_count - 1) / sm_count, cost = rounds * (t + 48);
        if (best < 0 || cost < best) { best = cost; nt = t; }
      }
    }
    const int tiles = n_tiles * ((rows + nt - 1) / nt);
    int splits = 1;   // few tiles: a cluster of blocks per tile, each a part of K
    while (rows <= 128 && splits < 8 && tiles * splits * 2 <= sm_count && kb >= splits * 4) splits *= 2;
    TensorMap wm, xm;
    if (ainfer_tensor_map_bf16(dev, &wm, mt.w, (uint64_t)mt.N, (uint64_t)mt.K, (uint64_t)mt.ldw, 128) != AINFER_OK ||
        ainfer_tensor_map_bf16(dev, &xm, Xp, (uint64_t)rows, (uint64_t)mt.K, (uint64_t)ldx, (uint32_t)nt) != AINFER_OK) {
      k.fail(1, ainfer_last_error(dev));
      return;
    }
    static const char *const names[] = {"LinearTc", "LinearTcSplit2", "LinearTcSplit4", "LinearTcSplit8"};
    const int which = splits == 8 ? 3 : splits == 4 ? 2 : splits == 2 ? 1 : 0;
    k.launch(names[which], (uint32_t)(splits > 1 ? tiles * splits : std::min(tiles, sm_count)), wm, xm, mt.bias, Yp, (int32_t)rows, (int32_t)mt.N,
             (int32_t)mt.K, (int32_t)nt, (int32_t)ldy, (int32_t)act, (int32_t)(out16 ? 1 : 0), cap);
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

  // head sizes the tensor-core attention takes (bf16), and the name of the instance that holds one
  bool mma_dim(const RowLayerConfig &r) const { return !f32 && r.dim % 8 == 0 && r.dim <= 256; }
  static std::string sized(const char *base, int dim) {
    for (int d : {32, 64, 96, 128, 192})
      if (dim <= d) return base + std::to_string(d);
    return base + std::string("256");
  }
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
  void gemv(KernelCalls &k, const RowMatrix &mt, const float *x, float *y, int act) {
    const int rows_pb = (mt.N + 2 * sm_count - 1) / (2 * sm_count);
    k.launch("StreamGemv", (uint32_t)((mt.N + rows_pb - 1) / rows_pb), x, mt.w, mt.bias, y, (int32_t)mt.N, (int32_t)mt.K, (int32_t)mt.ldw,
             (int32_t)rows_pb, (int32_t)act, 0.0f);
  }
  void hyper_gemv(KernelCalls &k, const RowMatrix &mt, const float *in, const float *norm, const float *shift, float *shift_state,
                  const int32_t *ctrl, float *y, int act, float cap) {
    const ModelConfig &c = m->cfg;
    const int rows_pb = (mt.N + 2 * sm_count - 1) / (2 * sm_count);
    k.launch("HyperStreamGemv", (uint32_t)((mt.N + rows_pb - 1) / rows_pb), (const float *)X[cur], (const float *)(pending ? Y : nullptr),
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

const ModelArch *sinepel_model_arch() { return &kModel; }

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

int row_engine_create(DeviceModel *m, int nseq, int max_ctx, int rows_cap, bool f32, RowEngine **out, std::string &err) {
  *out = nullptr;
  if (!m->rows) { err = "usage: this architecture has no row engine"; return 2; }
  Engine *e = new Engine;
  const int r = e->create(m, nseq, max_ctx, rows_cap, f32, err);
  if (r) { delete e; return r; }
  *out = e;
  return 0;
}

}  // namespace ainfer
