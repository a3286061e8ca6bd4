// Robopel: decoder whose sublayers read the residual itself and are normalised on their output. Layers
// mix tokens by a minGRU recurrence, or by attention over a sliding window of tokens and pooled blocks
// before it (per-head query and key norms, interleaved rotary positions with scaled long wavelengths,
// capped scores, sinks, an output gate; a layer may read an earlier layer's keys and values). The
// feed-forward is dense with a polynomial of normalised powers, a mixture of squared-ReLU experts with
// identity experts, or absent.
//
// This file holds what is particular to it: configuration, tensor list, prepared weights, and the
// sequence of launches of a row pass and of a decode step (RowEngine). The mechanisms are kernels of
// their own with their constants as arguments: k_post_norm.cu, k_mingru.cu, k_moe16.cu,
// k_window_attn.cu, k_window_mma.cu, and the products of k_linear.cu and k_linear_tc.cu.
#include <algorithm>
#include <climits>
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
  c.arch = "Robopel";
  c.hidden = js.at("width").integer(0);
  c.vocab = js.at("vocab").integer(0);
  c.rms_eps = js.at("norm").at("eps").num(-1);
  c.embed_scale = js.at("embedding").at("scale").num(1.0);
  if (js.at("layers").kind != Json::ARR) return bad("no list of layers");
  for (const Json &l : js.at("layers").a) {
    RowLayerConfig r;
    const std::string type = l.at("type").str();
    const Json &x = l.at("mixer");
    if (type == "attention") {
      r.heads = x.at("heads").integer(0);
      r.kv_heads = x.at("kv_heads").integer(0);
      r.dim = x.at("dim").integer(0);
      r.vdim = x.at("vdim").integer(r.dim);
      r.scale = x.at("scale").num(NAN);
      r.softcap = x.at("softcap").num(0.0);
      r.window = x.at("mask").at("size").integer(0);
      r.pool = x.at("mask").at("pool").integer(0);
      r.kv_from = x.at("kv_from").integer(-1);
      if (x.has("kv_from") && !x.at("kv_from").is_null() && r.kv_from < 0) return bad("kv_from must be a layer");
      const Json &t = x.at("rot");
      if (!t.is_null()) {
        r.rot.dims = t.at("dims").integer(r.dim);
        r.rot.base = t.at("base").num(NAN);
        const Json &s = t.at("scaling");
        if (!s.is_null()) {
          r.rot.scaled = true;
          r.rot.factor = s.at("factor").num(NAN);
          r.rot.low = s.at("low").num(NAN);
          r.rot.high = s.at("high").num(NAN);
          r.rot.original = s.at("original").num(NAN);
        }
      }
    } else if (type == "mingru") {
      r.mixer = RowLayerConfig::MINGRU;
      r.width = x.at("width").integer(0);
    } else {
      return bad("unknown layer type \"" + type + "\"");
    }
    const Json &f = l.at("mlp");
    if (!f.is_null()) {
      const std::string kind = f.at("kind").str();
      if (kind == "dense") {
        r.ff = f.at("ff").integer(0);
      } else if (kind == "moe") {
        r.ff = f.at("expert").at("ff").integer(0);
        r.experts = f.at("router").at("experts").integer(0);
        r.identity = f.at("router").at("identity").integer(0);
        r.top = f.at("router").at("top").integer(0);
        if (r.experts < 1 || r.identity < 0 || r.top < 1) return bad("a mixture needs experts and a choice among them");
      } else {
        return bad("unknown feed-forward \"" + kind + "\"");
      }
      if (r.ff < 1) return bad("feed-forward without a size");
    }
    c.row_layers.push_back(r);
  }
  c.layers = (int)c.row_layers.size();
  return true;
}

std::string to_json(const ModelConfig &c) {
  auto i = [](int v) { return std::to_string(v); };
  std::string s = "{\"architecture\":\"Robopel\",\"embedding\":{\"scale\":" + json_num(c.embed_scale) + "},\"layers\":[";
  for (size_t n = 0; n < c.row_layers.size(); ++n) {
    const RowLayerConfig &r = c.row_layers[n];
    s += n ? "," : "";
    if (r.mixer == RowLayerConfig::MINGRU) {
      s += "{\"mixer\":{\"width\":" + i(r.width) + "}";
    } else {
      s += "{\"mixer\":{\"dim\":" + i(r.dim) + ",\"heads\":" + i(r.heads) + (r.kv_from >= 0 ? ",\"kv_from\":" + i(r.kv_from) : std::string()) +
           ",\"kv_heads\":" + i(r.kv_heads) + ",\"mask\":{" + (r.pool ? "\"pool\":" + i(r.pool) + "," : std::string()) + "\"size\":" + i(r.window) + "}";
      if (r.rot.dims) {
        s += ",\"rot\":{\"base\":" + json_num(r.rot.base) + ",\"dims\":" + i(r.rot.dims);
        if (r.rot.scaled)
          s += ",\"scaling\":{\"factor\":" + json_num(r.rot.factor) + ",\"high\":" + json_num(r.rot.high) + ",\"low\":" + json_num(r.rot.low) +
               ",\"original\":" + json_num(r.rot.original) + "}";
        s += "}";
      }
      s += ",\"scale\":" + json_num(r.scale) + (r.softcap > 0 ? ",\"softcap\":" + json_num(r.softcap) : std::string()) + ",\"vdim\":" + i(r.vdim) + "}";
    }
    if (!r.ff) s += ",\"mlp\":null";
    else if (!r.experts) s += ",\"mlp\":{\"ff\":" + i(r.ff) + ",\"kind\":\"dense\"}";
    else
      s += ",\"mlp\":{\"expert\":{\"ff\":" + i(r.ff) + "},\"kind\":\"moe\",\"router\":{\"experts\":" + i(r.experts) + ",\"identity\":" + i(r.identity) +
           ",\"top\":" + i(r.top) + "}}";
    s += std::string(",\"type\":\"") + (r.mixer == RowLayerConfig::MINGRU ? "mingru" : "attention") + "\"}";
  }
  return s + "],\"norm\":{\"eps\":" + json_num(c.rms_eps) + "},\"vocab\":" + i(c.vocab) + ",\"width\":" + i(c.hidden) + "}";
}

bool check(const ModelConfig &c, std::string &err) {
  auto bad = [&](const std::string &m) { err = "unsupported architecture: " + m; return false; };
  if (c.row_layers.empty()) return bad("no layers");
  if (c.hidden < 1 || c.hidden > 16384) return bad("width must be in [1, 16384]");
  if (c.vocab < 1) return bad("vocab");
  if (!(c.rms_eps >= 0)) return bad("norm.eps");
  for (size_t n = 0; n < c.row_layers.size(); ++n) {
    const RowLayerConfig &r = c.row_layers[n];
    if (r.mixer == RowLayerConfig::MINGRU) {
      if (r.width < 1 || r.width > 24576) return bad("a recurrence's width must be in [1, 24576]");
    } else {
      if (r.heads < 1 || r.kv_heads < 1 || r.heads % r.kv_heads) return bad("heads must be a multiple of kv_heads");
      if (r.dim < 1 || r.dim > 512 || r.vdim < 1 || r.vdim > 512) return bad("dim and vdim must be in [1, 512]");
      if (r.heads * r.vdim > 24576) return bad("a layer's inner size exceeds 24576");
      if (r.window < 0 || r.pool < 0) return bad("mask");
      if (!std::isfinite(r.scale)) return bad("mixer.scale");
      if (!(r.softcap >= 0) || !std::isfinite(r.softcap)) return bad("mixer.softcap");
      const RotaryConfig &t = r.rot;
      if (t.dims < 0 || t.dims % 2 || t.dims > r.dim) return bad("rot.dims must be even and at most dim");
      if (t.dims && !(t.base > 0)) return bad("rot.base");
      if (t.scaled && !(t.factor > 0 && t.original > 0 && t.low > 0 && t.high > t.low)) return bad("rot.scaling");
      if (r.kv_from >= 0) {
        if (r.kv_from >= (int)n) return bad("kv_from must be an earlier layer");
        const RowLayerConfig &s = c.row_layers[(size_t)r.kv_from];
        if (s.mixer != RowLayerConfig::ATTENTION || s.kv_from >= 0) return bad("kv_from must be a layer with keys and values of its own");
        if (s.kv_heads != r.kv_heads || s.dim != r.dim || s.vdim != r.vdim) return bad("kv_from: key and value heads differ");
      }
      // shared memory of the CUDA-core step's attention: queries, sums, a tile of keys and values, scores
      const long hg = r.heads / r.kv_heads;
      if (4 * (hg * (r.dim + r.vdim) + r.dim + r.vdim + 64L * (r.dim + 1 + r.vdim) + 64 * hg + 3 * hg) > 220 * 1024)
        return bad("too many query heads per key head at these sizes");
    }
    if (r.ff > 24576) return bad("a feed-forward's size exceeds 24576");
    if (r.experts) {
      if (r.experts + r.identity > 1024) return bad("more than 1024 experts");
      if (r.top > 32 || r.top > r.experts + r.identity) return bad("router.top must be at most 32 and the number of experts");
      if ((long)r.top * round_up(r.ff, 8) > 32768) return bad("router.top times the expert size exceeds 32768");
    }
  }
  return true;
}

// Every tensor with its shape, in storage order (matrices that are used as one lie side by side).
std::vector<RowTensor> tensors(const ModelConfig &c) {
  std::vector<RowTensor> t;
  const uint64_t W = c.hidden, V = c.vocab;
  auto add = [&](const std::string &n, std::vector<uint64_t> sh, float sd, float cst) { t.push_back({n, sh, sd, cst}); };
  const float iw = 1.0f / std::sqrt((float)W);
  add("embed", {V, W}, 0.5f, 0);
  for (int L = 0; L < c.layers; ++L) {
    const RowLayerConfig &r = c.row_layers[L];
    const std::string p = layer_name(L), x = p + "mix.", f = p + "mlp.";
    const uint64_t F = r.ff;
    add(p + "norm1", {W}, 0, 0);
    if (r.mixer == RowLayerConfig::MINGRU) {
      const uint64_t K = r.width;
      add(x + "z", {K, W}, iw, 0);
      add(x + "x", {K, W}, iw, 0);
      add(x + "g", {K, W}, iw, 0);
      add(x + "z.b", {K}, 0.02f, 0);
      add(x + "x.b", {K}, 0.02f, 0);
      add(x + "o", {W, K}, 1.0f / std::sqrt((float)K), 0);
    } else {
      const uint64_t H = r.heads, G = r.kv_heads, D = r.dim, E = r.vdim;
      add(x + "q", {H * D, W}, iw, 0);
      if (r.kv_from < 0) {
        add(x + "k", {G * D, W}, iw, 0);
        add(x + "v", {G * E, W}, iw, 0);
      }
      add(x + "g", {H * E, W}, iw, 0);
      add(x + "q.norm", {D}, 0, 1);
      if (r.kv_from < 0) add(x + "k.norm", {D}, 0, 1);
      add(x + "sink", {H}, 0, 0);
      add(x + "o", {W, H * E}, 1.0f / std::sqrt((float)(H * E)), 0);
    }
    if (!r.ff) continue;
    add(p + "norm2", {W}, 0, 0);
    const float fw = 1.0f / std::sqrt((float)F);
    if (!r.experts) {
      add(f + "up", {F, W}, iw, 0);
      add(f + "down", {W, F}, fw, 0);
      add(f + "act", {4}, 0, 0.5f);
    } else {
      add(f + "router", {(uint64_t)(r.experts + r.identity), W}, iw, 0);
      add(f + "correction", {(uint64_t)(r.experts + r.identity)}, 0, 0);
      for (int e = 0; e < r.experts; ++e) add(f + "e" + std::to_string(e) + ".up", {F, W}, iw, 0);
      for (int e = 0; e < r.experts; ++e) add(f + "e" + std::to_string(e) + ".down", {W, F}, fw, 0);
    }
  }
  add("final.norm", {W}, 0, 0);
  add("head", {V, W}, iw, 0);
  return t;
}

void plan(const ModelConfig &c, Container &dir, std::vector<SynthSpec> &specs) { plan_row_tensors(tensors(c), to_json(c), c.vocab, dir, specs); }
int check_directory(const Container &dir, const ModelConfig &c, std::string &err) { return check_row_tensors(dir, tensors(c), err); }

// ------------------------------------------------------------- prepared weights ---
struct LayerWeights {
  RowMatrix in, o;                       // mixer: the projections of its input (attention: q, k, v, gate; recurrence: z, u, gate), the output's
  const float *q_norm, *k_norm, *sink;
  const float *gain1, *gain2;            // of the output norms
  RowMatrix up, down, router;            // experts: rows of all experts, one after the other
  const float *act, *correction;
};
struct Weights : RowWeights {
  std::vector<LayerWeights> L;
  RowMatrix head;
  const float *final_gain = nullptr;
  const uint16_t *embed = nullptr;
};

int prepare(DeviceModel *m, std::string &err) {
  const ModelConfig &c = m->cfg;
  auto w = std::make_shared<Weights>();
  RowLoader k(m, &err);
  for (int L = 0; L < c.layers && !k.status; ++L) {
    const RowLayerConfig &r = c.row_layers[L];
    const std::string p = layer_name(L), x = p + "mix.", f = p + "mlp.";
    LayerWeights lw{};
    if (r.mixer == RowLayerConfig::MINGRU) {
      lw.in = k.stack({x + "z", x + "x", x + "g"});
      std::vector<float> bias((size_t)3 * r.width, 0.0f);
      const auto zb = k.host(x + "z.b"), xb = k.host(x + "x.b");
      for (int i = 0; i < r.width; ++i) {
        bias[(size_t)i] = bf16_to_f32(zb[(size_t)i]);
        bias[(size_t)r.width + i] = bf16_to_f32(xb[(size_t)i]);
      }
      lw.in.bias = k.upload(bias);
    } else {
      if (r.kv_from < 0) {
        lw.in = k.stack({x + "q", x + "k", x + "v", x + "g"});
        lw.k_norm = k.widen(x + "k.norm");
      } else {
        lw.in = k.stack({x + "q", x + "g"});
      }
      lw.q_norm = k.widen(x + "q.norm");
      lw.sink = k.widen(x + "sink");
    }
    lw.o = k.stack({x + "o"});
    lw.gain1 = k.gain(p + "norm1");
    if (r.ff) {
      lw.gain2 = k.gain(p + "norm2");
      if (r.experts) {
        std::vector<std::string> up, down;
        for (int e = 0; e < r.experts; ++e) {
          up.push_back(f + "e" + std::to_string(e) + ".up");
          down.push_back(f + "e" + std::to_string(e) + ".down");
        }
        lw.up = k.stack(up);
        lw.down = k.stack(down);
        lw.router = k.stack({f + "router"});
        lw.correction = k.widen(f + "correction");
      } else {
        lw.up = k.stack({f + "up"});
        lw.down = k.stack({f + "down"});
        lw.act = k.widen(f + "act");
      }
    }
    w->L.push_back(lw);
  }
  if (!k.status) {
    w->head = k.stack({"head"});
    w->final_gain = k.gain("final.norm");
    w->embed = (const uint16_t *)m->tensor("embed").data;
  }
  k.finish();
  m->rows = w;
  return k.status;
}

// Angle per position of every rotated pair.
std::vector<double> rotary_frequencies(const RotaryConfig &t) {
  const double two_pi = 6.283185307179586476925;
  std::vector<double> f;
  for (int i = 0; i < t.dims / 2; ++i) {
    double v = std::pow(t.base, -2.0 * i / t.dims);
    if (t.scaled) {
      const double wave = two_pi / v;
      if (wave > t.original / t.low) {
        v /= t.factor;
      } else if (wave >= t.original / t.high) {
        const double s = (t.original / wave - t.low) / (t.high - t.low);
        v = (1.0 - s) * v / t.factor + s * v;
      }
    }
    f.push_back(v);
  }
  return f;
}

// ------------------------------------------------------------------- row engine ---
struct Engine : RowEngineBase {
  const Weights *w;
  // keys and values of a layer that has its own: rings of `cap` positions; block means per (layer, block size)
  struct Ring { char *k = nullptr, *v = nullptr; int cap = 0; };
  struct Means { int layer = -1, pool = 0; char *k = nullptr, *v = nullptr; int blocks = 0; };
  struct LayerState {
    Ring ring;               // of the layer the keys come from
    int means = -1;          // index into `means`
    bool own_means = false;  // the first layer in the order that uses them averages
    float *gru = nullptr;    // [seq][2][width]
    const void *rot = nullptr;
  };
  std::vector<LayerState> st;
  std::vector<Means> means;
  char *state = nullptr;
  size_t state_bytes = 0, ring_off = 0, means_off = 0;   // recurrences, rings, means
  // pass buffers
  float *X[2] = {nullptr, nullptr}, *U = nullptr, *Y = nullptr, *Pair = nullptr, *Logits = nullptr, *SelW = nullptr, *AttPart = nullptr;
  char *H = nullptr, *Q = nullptr, *Att = nullptr, *Z = nullptr, *Act = nullptr, *Hp = nullptr;
  int32_t *Sel = nullptr, *Place = nullptr, *RowOf = nullptr, *Count = nullptr;
  void *Tiles = nullptr;
  uint32_t *AttCount = nullptr;
  int ldw = 0, ldq = 0, ldf = 0, att_splits = 1;
  // the update that the residual still waits for
  struct Pending { const float *gain = nullptr; int top = 0; };
  Pending pending;
  int cur = 0;   // decode step: the buffer that holds the residual

  static int inner(const RowLayerConfig &r) { return r.mixer == RowLayerConfig::MINGRU ? r.width : r.heads * r.vdim; }
  static int window_of(const RowLayerConfig &r) { return r.window > 0 ? r.window : INT_MAX / 2; }

  int create(DeviceModel *model, int n, int ctx, int cap_rows, bool in_f32, std::string &err) override {
    if (begin(model, n, ctx, cap_rows, in_f32, err)) return 1;
    w = static_cast<const Weights *>(m->rows.get());
    const ModelConfig &c = m->cfg;
    const size_t W = c.hidden, R = rows_cap;
    // ---- state: one block, layer after layer ----
    size_t off = 0;
    auto take = [&](size_t bytes) { const size_t o = off; off += (bytes + 255) / 256 * 256; return o; };
    st.resize((size_t)c.layers);
    std::vector<size_t> gru((size_t)c.layers), rk((size_t)c.layers), rv((size_t)c.layers), mk, mv;
    for (int L = 0; L < c.layers; ++L)
      if (c.row_layers[L].mixer == RowLayerConfig::MINGRU) gru[L] = take((size_t)nseq * 2 * c.row_layers[L].width * 4);
    ring_off = off;
    for (int L = 0; L < c.layers; ++L) {
      const RowLayerConfig &r = c.row_layers[L];
      if (r.mixer != RowLayerConfig::ATTENTION || r.kv_from >= 0) continue;
      long need = 1;   // positions any reader looks back to
      for (int i = L; i < c.layers; ++i) {
        const RowLayerConfig &q = c.row_layers[i];
        if (i == L || (q.mixer == RowLayerConfig::ATTENTION && q.kv_from == L)) need = std::max(need, (long)std::max(window_of(q), q.pool));
      }
      // those plus the rows of a pass; a multiple of the attention kernels' key tile
      st[L].ring.cap = round_up((int)std::min<long>(max_ctx, need + rows_cap), 64);
      rk[L] = take((size_t)nseq * st[L].ring.cap * r.kv_heads * r.dim * esz());
      rv[L] = take((size_t)nseq * st[L].ring.cap * r.kv_heads * r.vdim * esz());
    }
    means_off = off;
    for (int L = 0; L < c.layers; ++L) {
      const RowLayerConfig &r = c.row_layers[L];
      if (r.mixer != RowLayerConfig::ATTENTION || !r.pool) continue;
      const int src = r.kv_from >= 0 ? r.kv_from : L;
      for (size_t i = 0; i < means.size() && st[L].means < 0; ++i)
        if (means[i].layer == src && means[i].pool == r.pool) st[L].means = (int)i;
      if (st[L].means >= 0) continue;
      Means x;
      x.layer = src;
      x.pool = r.pool;
      x.blocks = round_up(max_ctx / r.pool + 1, 64);
      st[L].means = (int)means.size();
      st[L].own_means = true;
      means.push_back(x);
      mk.push_back(take((size_t)nseq * x.blocks * r.kv_heads * r.dim * esz()));
      mv.push_back(take((size_t)nseq * x.blocks * r.kv_heads * r.vdim * esz()));
    }
    state_bytes = off;
    int e = alloc(state_bytes, &state);
    for (int L = 0; L < c.layers && !e; ++L) {
      const RowLayerConfig &r = c.row_layers[L];
      if (r.mixer == RowLayerConfig::MINGRU) { st[L].gru = (float *)(state + gru[L]); continue; }
      if (r.kv_from < 0) { st[L].ring.k = state + rk[L]; st[L].ring.v = state + rv[L]; }
      else st[L].ring = st[r.kv_from].ring;
    }
    for (size_t i = 0; i < means.size() && !e; ++i) { means[i].k = state + mk[i]; means[i].v = state + mv[i]; }
    // ---- rotary tables, one per distinct setting ----
    if (!e) e = rotary_tables(err);
    // ---- buffers of a pass ----
    size_t maxU = 1, maxQ = 1, maxA = 1, maxF = 1, maxKe = 0, maxEI = 1, maxS = 1, maxK = 1, maxHE = 1, maxHp = 0, y_rows = R, tiles = 1;
    int maxG = 1;
    for (const RowLayerConfig &r : c.row_layers) {
      maxA = std::max(maxA, (size_t)inner(r));
      if (r.mixer == RowLayerConfig::MINGRU) {
        maxU = std::max(maxU, (size_t)3 * r.width);
        maxK = std::max(maxK, (size_t)r.width);
      } else {
        maxU = std::max(maxU, (size_t)r.heads * (r.dim + r.vdim) + (size_t)r.kv_heads * (r.dim + r.vdim));
        maxQ = std::max(maxQ, (size_t)r.heads * r.dim);
        maxHE = std::max(maxHE, (size_t)r.heads * (r.vdim + 4));
        maxG = std::max(maxG, r.kv_heads);
      }
      if (r.experts) {
        const size_t slots = R * r.top;
        maxKe = std::max(maxKe, slots * round_up(r.ff, 8));
        maxHp = std::max(maxHp, slots);
        y_rows = std::max(y_rows, slots);
        maxEI = std::max(maxEI, (size_t)(r.experts + r.identity));
        maxS = std::max(maxS, slots);
        tiles = std::max(tiles, slots / 16 + r.experts + 1);
      } else {
        maxF = std::max(maxF, (size_t)r.ff);
      }
    }
    ldw = round_up((int)W, 8);
    ldq = round_up((int)maxA, 8);
    ldf = round_up((int)maxF, 8);
    att_splits = step_splits(maxG);
    for (int i = 0; i < 2; ++i) e |= alloc(R * W, &X[i]);
    e |= alloc(R * ldw * esz(), &H); e |= alloc(R * maxU, &U); e |= alloc(R * maxQ * esz(), &Q);
    e |= alloc(R * ldq * 4, &Att); e |= alloc(y_rows * W, &Y); e |= alloc(R * ldf * 4, &Z);
    e |= alloc(std::max(R * ldf, maxKe) * 4, &Act);
    e |= alloc((R / 32 + 2) * 2 * maxK, &Pair);
    e |= alloc(R * maxEI, &Logits); e |= alloc(maxS, &Sel); e |= alloc(maxS, &SelW); e |= alloc(maxS, &Place); e |= alloc(maxS, &RowOf);
    e |= alloc(tiles * 4, (int32_t **)&Tiles); e |= alloc(2, &Count);
    e |= alloc(maxHp * ldw * esz(), &Hp);
    e |= alloc((size_t)nseq * att_splits * maxHE, &AttPart);
    e |= alloc((size_t)nseq * maxG, &AttCount);
    if (e) { if (err.empty()) err = "row engine: " + (alloc_err.empty() ? std::string(ainfer_last_error(dev)) : alloc_err); return 1; }
    return 0;
  }

  int rotary_tables(std::string &err) {
    const ModelConfig &c = m->cfg;
    std::map<std::string, ainfer_kernel_t> handles;
    KernelCalls k(dev, &handles, &err);
    std::vector<std::pair<std::vector<double>, const void *>> known;
    for (int L = 0; L < c.layers && !k.status; ++L) {
      const RowLayerConfig &r = c.row_layers[L];
      if (r.mixer != RowLayerConfig::ATTENTION || !r.rot.dims) continue;
      const std::vector<double> f = rotary_frequencies(r.rot);
      for (const auto &x : known)
        if (x.first == f) st[L].rot = x.second;
      if (st[L].rot) continue;
      double *fd = nullptr;
      float *t = nullptr;
      if (alloc(f.size(), &fd) || alloc((size_t)max_ctx * f.size() * 2, &t)) return 1;
      if (ainfer_memcpy_h2d(dev, fd, f.data(), f.size() * 8) != AINFER_OK) return 1;
      k.launch("RotaryTable", (uint32_t)std::min<size_t>(((size_t)max_ctx * f.size() + 255) / 256, 4096), (void *)t, (const double *)fd, (int32_t)max_ctx,
               (int32_t)f.size());
      st[L].rot = t;
      known.push_back({f, t});
    }
    if (!k.status && ainfer_sync(dev, UINT64_MAX) != AINFER_OK) k.fail(1, ainfer_last_error(dev));
    for (auto &kv : handles) ainfer_kernel_release(kv.second);
    return k.status;
  }

  int reset(std::string &err) override {
    if (ainfer_mem_fill(dev, state, 0, state_bytes) != AINFER_OK) { err = ainfer_last_error(dev); return 1; }
    return 0;
  }
  bool buffer(const std::string &which, void **p, uint64_t *n) override {
    if (which == "state") { *p = state; *n = state_bytes; }
    else if (which == "gru") { *p = state; *n = ring_off; }
    else if (which == "Kc") { *p = state + ring_off; *n = means_off - ring_off; }
    else if (which == "means") { *p = state + means_off; *n = state_bytes - means_off; }
    else return false;
    return true;
  }

  // ---- rows ----
  // The rows' operand of the products: the residual itself in 32-bit, its bf16 copy else.
  const char *operand() const { return f32 ? (const char *)X[0] : H; }
  int operand_ld() const { return f32 ? m->cfg.hidden : ldw; }

  // x += norm(y) gain for the pending sublayer; then the operand, or (final) the head's input of chosen rows.
  void post_norm(KernelCalls &k, int rows, const float *final_gain, const int32_t *idx) {
    const bool last = final_gain != nullptr;
    if (f32 && !last && !pending.gain) return;
    k.launch(f32 ? "PostNormRowsF32" : "PostNormRowsB16", (uint32_t)rows, (const float *)X[0], (const void *)(pending.gain ? Y : nullptr), pending.gain,
             (float *)(last ? nullptr : X[0]), (const int32_t *)Place, (const float *)SelW, final_gain, idx, (void *)(f32 && !last ? nullptr : H),
             (int32_t)m->cfg.hidden, (int32_t)rows, (int32_t)pending.top, (int32_t)ldw, (float)m->cfg.rms_eps);
    pending = Pending();
  }
  void attention_rows(KernelCalls &k, const RowSpan &sp, const RowLayerConfig &r, const LayerWeights &lw, const LayerState &s, int ldo) {
    const int R = sp.rows, Hd = r.heads * r.dim, Gd = r.kv_heads * r.dim, Ge = r.kv_heads * r.vdim;
    const bool own = r.kv_from < 0;
    const int koff = own ? Hd : -1, voff = Hd + Gd, goff = own ? voff + Ge : Hd, ldu = lw.in.N;
    const int units = R * (r.heads + (own ? 2 * r.kv_heads : 0));
    k.launch(f32 ? "QkvRowsF32" : "QkvRowsB16", (uint32_t)((units + 7) / 8), (const float *)U, lw.q_norm, lw.k_norm, s.rot, sp.ctrl, (void *)Q,
             (void *)s.ring.k, (void *)s.ring.v, (int32_t)R, (int32_t)r.heads, (int32_t)r.kv_heads, (int32_t)r.dim, (int32_t)r.vdim,
             (int32_t)r.rot.dims, (int32_t)s.ring.cap, (int32_t)ldu, (int32_t)koff, (int32_t)voff, (float)m->cfg.rms_eps);
    const Means *mn = s.means >= 0 ? &means[(size_t)s.means] : nullptr;
    if (s.own_means)
      k.launch(f32 ? "PoolRowsF32" : "PoolRowsB16", (uint32_t)((R / r.pool + 1) * ((Gd + Ge + 255) / 256)), (const void *)s.ring.k, (const void *)s.ring.v,
               (void *)mn->k, (void *)mn->v, sp.ctrl, (int32_t)R, (int32_t)Gd, (int32_t)Ge, (int32_t)s.ring.cap, (int32_t)r.pool);
    const bool mma = mma_dims(r);
    const std::string name = mma ? sized("WindowAttnMma", std::max(r.dim, r.vdim)) : std::string(f32 ? "WindowAttnRowsF32" : "WindowAttnRowsB16");
    const int per = mma ? 64 : 16;
    k.launch(name.c_str(), (uint32_t)(((R + per - 1) / per) * r.heads), (const void *)Q, (const void *)s.ring.k, (const void *)s.ring.v,
             (const void *)(mn ? mn->k : nullptr), (const void *)(mn ? mn->v : nullptr), lw.sink, (const float *)(U + goff), sp.ctrl, (void *)Att,
             (int32_t)R, (int32_t)r.heads, (int32_t)r.kv_heads, (int32_t)r.dim, (int32_t)r.vdim, (int32_t)s.ring.cap, (int32_t)window_of(r),
             (int32_t)r.pool, (int32_t)ldu, (int32_t)ldo, (float)r.scale, (float)r.softcap);
  }
  void recurrence_rows(KernelCalls &k, const RowSpan &sp, const RowLayerConfig &r, const LayerState &s, int lda) {
    const uint32_t cb = (uint32_t)((r.width + 255) / 256);
    if (!sp.one_sequence) {
      k.launch(f32 ? "MinGruStepRowsF32" : "MinGruStepRowsB16", cb * (uint32_t)sp.rows, (const float *)U, s.gru, sp.ctrl, (void *)Att, (int32_t)sp.rows,
               (int32_t)r.width, (int32_t)lda);
      return;
    }
    const uint32_t chunks = (uint32_t)((sp.rows + 31) / 32);
    k.launch(f32 ? "MinGruChunkF32" : "MinGruChunkB16", cb * chunks, (const float *)U, (const float *)s.gru, sp.ctrl, Pair, (int32_t)sp.rows, (int32_t)r.width);
    k.launch(f32 ? "MinGruScanF32" : "MinGruScanB16", cb * chunks, (const float *)U, (const float *)Pair, s.gru, sp.ctrl, (void *)Att, (int32_t)sp.rows,
             (int32_t)r.width, (int32_t)lda);
  }
  // Rows of a tile: an expert's rows, two standard deviations above their mean, in as few even tiles as possible.
  static int expert_tile_rows(double mean) {
    const double most = mean + 2.0 * std::sqrt(mean);
    const int tiles = (int)std::ceil(most / 256.0);
    return std::max(16, std::min(256, round_up((int)std::ceil(most / tiles), 16)));
  }
  void mixture_rows(KernelCalls &k, const RowLayerConfig &r, const LayerWeights &lw, int R) {
    const int EI = r.experts + r.identity, slots = R * r.top, lde = round_up(r.ff, 8), W = m->cfg.hidden;
    linear(k, lw.router, operand(), operand_ld(), R, Logits, EI, ACT_NONE, false);
    k.launch("RouterTopRows", (uint32_t)((R + 3) / 4), (const float *)Logits, lw.correction, Sel, SelW, (int32_t)R, (int32_t)EI, (int32_t)r.top);
    const int nt = f32 ? 64 : expert_tile_rows((double)slots / EI);
    k.launch("MoePlanRows", 1, (const int32_t *)Sel, Place, RowOf, Tiles, Count, (int32_t)R, (int32_t)r.top, (int32_t)r.experts, (int32_t)nt);
    k.launch("GatherRows", (uint32_t)std::min(slots, 8 * sm_count), (void *)Hp, (const void *)operand(), (const int32_t *)RowOf, (const int32_t *)Count,
             (int64_t)(operand_ld() * esz()), (int64_t)(ldw * esz()), (int32_t)(operand_ld() * esz()));
    grouped(k, lw.up, r, Hp, ldw, slots, Act, lde, ACT_RELU2, !f32, nt);
    grouped(k, lw.down, r, Act, lde, slots, Y, W, ACT_NONE, !f32, nt);
  }
  // the experts' products over their rows: Y[place][N] = act(X W_e^T)
  void grouped(KernelCalls &k, const RowMatrix &mt, const RowLayerConfig &r, const char *Xp, int ldx, int slots, void *Yp, int ldy, int act, bool out16,
               int nt) {
    if (k.status) return;
    const int N = mt.N / r.experts, tile_n = f32 ? 64 : 128;
    const long units = (long)(slots / nt + std::min(r.experts, slots)) * ((N + tile_n - 1) / tile_n);
    if (f32) {
      k.launch("LinearRowsGrouped", (uint32_t)std::min<long>(units, 8 * sm_count), (const float *)Xp, mt.w, (float *)Yp, (const void *)Tiles,
               (const int32_t *)Count, (int32_t)N, (int32_t)mt.K, (int32_t)ldx, (int32_t)mt.ldw, (int32_t)ldy, (int32_t)act);
      return;
    }
    TensorMap wm, xm;
    if (ainfer_tensor_map_bf16(dev, &wm, mt.w, (uint64_t)mt.N, (uint64_t)mt.K, (uint64_t)mt.ldw, 128) != AINFER_OK ||
        ainfer_tensor_map_bf16(dev, &xm, Xp, (uint64_t)slots, (uint64_t)mt.K, (uint64_t)ldx, (uint32_t)nt) != AINFER_OK) {
      k.fail(1, ainfer_last_error(dev));
      return;
    }
    k.launch("LinearTcGrouped", (uint32_t)std::min<long>(units, sm_count), wm, xm, Yp, (const void *)Tiles, (const int32_t *)Count, (int32_t)N,
             (int32_t)mt.K, (int32_t)nt, (int32_t)ldy, (int32_t)act, (int32_t)(out16 ? 1 : 0));
  }

  void emit(KernelCalls &k, const RowSpan &sp) override {
    const ModelConfig &c = m->cfg;
    const int R = sp.rows, W = c.hidden;
    pending = Pending();
    k.launch("EmbedPosRows", (uint32_t)R, X[0], w->embed, (const uint16_t *)nullptr, sp.ctrl, (int32_t)W, (int32_t)c.vocab, (int32_t)1, (int32_t)1,
             (float)c.embed_scale);
    for (int L = 0; L < c.layers && !k.status; ++L) {
      const RowLayerConfig &r = c.row_layers[L];
      const LayerWeights &lw = w->L[L];
      const int lda = round_up(inner(r), 8);
      post_norm(k, R, nullptr, nullptr);
      linear(k, lw.in, operand(), operand_ld(), R, U, lw.in.N, ACT_NONE, false);
      if (r.mixer == RowLayerConfig::MINGRU) recurrence_rows(k, sp, r, st[L], lda);
      else if (sp.one_sequence) attention_rows(k, sp, r, lw, st[L], lda);
      else attention_step(k, r, lw, st[L], sp.ctrl, R, lda, !f32);
      linear(k, lw.o, Att, lda, R, Y, W, ACT_NONE, false);
      pending.gain = lw.gain1;
      if (!r.ff) continue;
      post_norm(k, R, nullptr, nullptr);
      if (r.experts) {
        mixture_rows(k, r, lw, R);
        pending.top = r.top;
      } else {
        const int ldz = round_up(r.ff, 8);
        linear(k, lw.up, operand(), operand_ld(), R, Z, ldz, ACT_NONE, !f32);
        k.launch(f32 ? "PolyNormRowsF32" : "PolyNormRowsB16", (uint32_t)R, (const void *)Z, lw.act, (void *)Act, (int32_t)r.ff, (int32_t)ldz, (int32_t)ldz,
                 (float)c.rms_eps);
        linear(k, lw.down, Act, ldz, R, Y, W, ACT_NONE, false);
      }
      pending.gain = lw.gain2;
    }
    if (sp.n_want > 0) {
      post_norm(k, sp.n_want, w->final_gain, sp.want);
      linear(k, w->head, H, ldw, sp.n_want, sp.logits, c.vocab, ACT_NONE, false);
    }
  }

  // sizes the tensor-core attention takes (bf16)
  bool mma_dims(const RowLayerConfig &r) const { return !f32 && r.dim % 8 == 0 && r.vdim % 8 == 0 && std::max(r.dim, r.vdim) <= 256; }
  void attention_step(KernelCalls &k, const RowLayerConfig &r, const LayerWeights &lw, const LayerState &s, const int32_t *ctrl, int n, int ldo, bool out16) {
    const int Hd = r.heads * r.dim, Gd = r.kv_heads * r.dim, Ge = r.kv_heads * r.vdim;
    const bool own = r.kv_from < 0;
    const int koff = own ? Hd : -1, voff = Hd + Gd, goff = own ? voff + Ge : Hd;
    const Means *mn = s.means >= 0 ? &means[(size_t)s.means] : nullptr;
    const int64_t blocks = mn ? mn->blocks : 0;
    const std::string name = mma_dims(r) && r.heads / r.kv_heads <= 16 ? sized("WindowAttnStepMma", std::max(r.dim, r.vdim))
                                                                       : std::string(f32 ? "WindowAttnStepF32" : "WindowAttnStepB16");
    k.launch(name.c_str(), (uint32_t)(n * r.kv_heads * (att_splits + 1)), (const float *)U, lw.q_norm, lw.k_norm, s.rot, ctrl, (void *)s.ring.k,
             (void *)s.ring.v, (void *)(mn ? mn->k : nullptr), (void *)(mn ? mn->v : nullptr), (int64_t)s.ring.cap * Gd, (int64_t)s.ring.cap * Ge,
             blocks * Gd, blocks * Ge, lw.sink, AttPart, AttCount, (void *)Att, (int32_t)n, (int32_t)r.heads, (int32_t)r.kv_heads, (int32_t)r.dim,
             (int32_t)r.vdim, (int32_t)r.rot.dims, (int32_t)s.ring.cap, (int32_t)window_of(r), (int32_t)r.pool, (int32_t)koff, (int32_t)voff,
             (int32_t)goff, (int32_t)(s.own_means ? 1 : 0), (int32_t)att_splits, (int32_t)lw.in.N, (int32_t)ldo, (int32_t)(out16 ? 1 : 0), (float)r.scale,
             (float)r.softcap, (float)m->cfg.rms_eps);
  }

  // ---- one decode step of sequence 0 ----
  // the pending update of the residual in the prologue of the next product, whose input is the residual (or its norm)
  void post_gemv(KernelCalls &k, const RowMatrix &mt, const float *final_gain, float *y) {
    k.launch("PostNormStreamGemv", gemv_blocks(mt.N), (const float *)X[cur], (const float *)(pending.gain ? Y : nullptr), pending.gain,
             (float *)(pending.gain ? X[cur ^ 1] : nullptr), final_gain, mt.w, mt.bias, y, (int32_t)mt.N, (int32_t)mt.K, (int32_t)mt.ldw,
             (int32_t)gemv_rows(mt.N), (int32_t)ACT_NONE, (float)m->cfg.rms_eps, 0.0f);
    if (pending.gain) { cur ^= 1; pending = Pending(); }
  }
  void record_embed(KernelCalls &k, const int32_t *ctrl) override {
    const ModelConfig &c = m->cfg;
    cur = 0;
    pending = Pending();
    k.launch("EmbedPosRows", 1, X[0], w->embed, (const uint16_t *)nullptr, ctrl, (int32_t)c.hidden, (int32_t)c.vocab, (int32_t)1, (int32_t)1,
             (float)c.embed_scale);
  }
  void record_layer(KernelCalls &k, int L, const int32_t *ctrl) override {
    const ModelConfig &c = m->cfg;
    const RowLayerConfig &r = c.row_layers[L];
    const LayerWeights &lw = w->L[L];
    post_gemv(k, lw.in, nullptr, U);
    if (r.mixer == RowLayerConfig::MINGRU) {
      k.launch("MinGruStreamGemv", gemv_blocks(c.hidden), (const float *)U, st[L].gru, ctrl, lw.o.w, Y, (int32_t)c.hidden, (int32_t)r.width,
               (int32_t)lw.o.ldw, (int32_t)gemv_rows(c.hidden));
    } else {
      attention_step(k, r, lw, st[L], ctrl, 1, inner(r), false);
      gemv(k, lw.o, (const float *)Att, Y, ACT_NONE);
    }
    pending.gain = lw.gain1;
    if (!r.ff) return;
    if (r.experts) {
      const int per = std::max(1, 2 * sm_count / r.top), rows_up = (r.ff + per - 1) / per;
      post_gemv(k, lw.router, nullptr, Logits);
      k.launch("ExpertUpStreamGemv", (uint32_t)(r.top * ((r.ff + rows_up - 1) / rows_up)), (const float *)Logits, lw.correction, (const float *)X[cur],
               lw.up.w, (float *)Act, Sel, SelW, (int32_t)r.experts, (int32_t)(r.experts + r.identity), (int32_t)r.top, (int32_t)r.ff, (int32_t)lw.up.K,
               (int32_t)lw.up.ldw, (int32_t)rows_up, (int32_t)ACT_RELU2);
      k.launch("ExpertDownStreamGemv", gemv_blocks(c.hidden), (const float *)Act, (const float *)X[cur], (const int32_t *)Sel, (const float *)SelW,
               lw.down.w, Y, (int32_t)r.experts, (int32_t)r.top, (int32_t)c.hidden, (int32_t)r.ff, (int32_t)lw.down.ldw, (int32_t)gemv_rows(c.hidden));
    } else {
      post_gemv(k, lw.up, nullptr, (float *)Z);
      k.launch("PolyStreamGemv", gemv_blocks(c.hidden), (const float *)Z, lw.act, lw.down.w, Y, (int32_t)c.hidden, (int32_t)r.ff, (int32_t)lw.down.ldw,
               (int32_t)gemv_rows(c.hidden), (float)c.rms_eps);
    }
    pending.gain = lw.gain2;
  }
  void record_residual(KernelCalls &k, float *dst) override {
    const int W = m->cfg.hidden;
    k.launch("PostNormRowsF32", 1, (const float *)X[cur], (const void *)(pending.gain ? Y : nullptr), pending.gain, dst, (const int32_t *)nullptr,
             (const float *)nullptr, (const float *)nullptr, (const int32_t *)nullptr, (void *)nullptr, (int32_t)W, (int32_t)1, (int32_t)0, (int32_t)W,
             (float)m->cfg.rms_eps);
  }
  void record_head(KernelCalls &k, float *logits) override { post_gemv(k, w->head, w->final_gain, logits); }
};

}  // namespace

const ModelArch *robopel_model_arch() {
  static const ModelArch a = {"Robopel", false, parse, to_json, check, plan, check_directory, prepare, []() -> RowEngine * { return new Engine; }};
  return &a;
}

bool robopel_preset(const std::string &name, ModelConfig &c) {
  auto attention = [](int heads, int kv_heads, int dim, int vdim, int window, int pool, int rot, int kv_from) {
    RowLayerConfig r;
    r.heads = heads; r.kv_heads = kv_heads; r.dim = dim; r.vdim = vdim; r.window = window; r.pool = pool; r.kv_from = kv_from;
    r.scale = 1.0 / std::sqrt((double)dim);
    r.softcap = 30.0;
    r.rot.dims = rot; r.rot.base = 10000.0; r.rot.scaled = true; r.rot.factor = 8.0; r.rot.original = 2048.0;
    return r;
  };
  auto recurrence = [](int width) {
    RowLayerConfig r;
    r.mixer = RowLayerConfig::MINGRU;
    r.width = width;
    return r;
  };
  auto dense = [](RowLayerConfig r, int ff) { r.ff = ff; return r; };
  auto mixture = [](RowLayerConfig r, int ff, int experts, int identity, int top) {
    r.ff = ff; r.experts = experts; r.identity = identity; r.top = top;
    return r;
  };
  c = ModelConfig();
  c.arch = "Robopel";
  if (name == "robopel-tiny") {
    c.hidden = 80; c.vocab = 512; c.embed_scale = 9.0;
    c.row_layers = {dense(recurrence(112), 160), mixture(attention(6, 2, 24, 40, 20, 6, 16, -1), 56, 5, 1, 2), attention(4, 2, 24, 40, 32, 5, 16, 1)};
  } else if (name == "robopel-small") {
    c.hidden = 2048; c.vocab = 32000; c.embed_scale = 1.0;
    c.row_layers = {dense(attention(16, 4, 128, 128, 1024, 16, 128, -1), 8192), mixture(recurrence(2048), 1024, 32, 2, 4),
                    dense(attention(16, 4, 128, 128, 1024, 16, 128, 0), 8192), mixture(recurrence(2048), 1024, 32, 2, 4)};
  } else {
    return false;
  }
  c.layers = (int)c.row_layers.size();
  return true;
}

}  // namespace ainfer
