#include "row_engine.h"

#include <cstdio>

#include "../common/detmath.h"

namespace ainfer {

std::string json_num(double v) {
  char b[40];
  std::snprintf(b, sizeof b, "%.17g", v);
  return b;
}

// ----------------------------------------------------------------- tensors ---
void plan_row_tensors(const std::vector<RowTensor> &t, const std::string &arch_json, int vocab, Container &dir, std::vector<SynthSpec> &specs) {
  dir = Container();
  specs.clear();
  for (const RowTensor &n : t) {
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
  dir.arch_json = arch_json;
  dir.tokenizer_json = "{\"format\":\"none\",\"vocab_size\":" + std::to_string(vocab) + "}";
  dir.policy_json = "{\"default\":\"BF16\"}";
  container_layout(dir);
}

int check_row_tensors(const Container &dir, const std::vector<RowTensor> &t, std::string &err) {
  for (const RowTensor &n : t) {
    const TensorEntry *e = dir.find(n.name);
    if (!e) { err = "missing " + n.name; return 1; }
    if (e->storage != DT_BF16) { err = "unexpected storage of " + n.name; return 2; }
    bool same = e->ndim == (int)n.shape.size();
    for (int i = 0; same && i < e->ndim; ++i) same = e->shape[i] == n.shape[i];
    if (!same) { err = "unexpected shape of " + n.name; return 2; }
  }
  return 0;
}

// ------------------------------------------------------------------ loader ---
RowLoader::RowLoader(DeviceModel *model, std::string *e) : KernelCalls(model->dev, nullptr, e), m(model) { kernels = &handles; }

void *RowLoader::alloc(size_t bytes) {
  void *p = nullptr;
  if (status) return nullptr;
  if (ainfer_mem_alloc(dev, std::max<size_t>(bytes, 16), 256, &p) != AINFER_OK) { fail(1, ainfer_last_error(dev)); return nullptr; }
  m->owned.push_back(p);
  return p;
}
const float *RowLoader::widen(const std::string &name) {
  DeviceTensor t = m->tensor(name);
  const uint64_t n = t.entry->numel();
  float *p = (float *)alloc(n * 4);
  if (p) launch("WidenBf16", (uint32_t)std::min<uint64_t>((n + 255) / 256, 1024), p, (const void *)t.data, n);
  return p;
}
std::vector<uint16_t> RowLoader::host(const std::string &name) {
  DeviceTensor t = m->tensor(name);
  std::vector<uint16_t> v(t.entry->numel());
  if (!status && ainfer_memcpy_d2h(dev, v.data(), t.data, v.size() * 2) != AINFER_OK) fail(1, ainfer_last_error(dev));
  return v;
}
const float *RowLoader::upload(const std::vector<float> &v) {
  float *p = (float *)alloc(v.size() * 4);
  if (p && ainfer_memcpy_h2d(dev, p, v.data(), v.size() * 4) != AINFER_OK) fail(1, ainfer_last_error(dev));
  return p;
}
const float *RowLoader::gain(const std::string &name) {
  std::vector<float> g;
  for (uint16_t b : host(name)) g.push_back(1.0f + bf16_to_f32(b));
  return upload(g);
}
RowMatrix RowLoader::stack(const std::vector<std::string> &names) {
  RowMatrix r;
  std::vector<DeviceTensor> parts;
  bool adjoin = true;
  const char *end = nullptr;
  for (const std::string &n : names) {
    DeviceTensor t = m->tensor(n);
    if (end && (const char *)t.data != end) adjoin = false;
    end = (const char *)t.data + t.entry->numel() * 2;
    r.N += (int)t.entry->shape[0];
    r.K = (int)t.entry->shape[1];
    parts.push_back(t);
  }
  r.ldw = round_up(r.K, 8);
  if (adjoin && r.ldw == r.K) {
    r.w = (const uint16_t *)parts[0].data;
    return r;
  }
  uint16_t *p = (uint16_t *)alloc((size_t)r.N * r.ldw * 2);
  r.w = p;
  for (const DeviceTensor &t : parts) {
    const int n = (int)t.entry->shape[0];
    if (p) launch("PackRowsBf16", (uint32_t)std::min(n, 4096), p, (const uint16_t *)t.data, (int32_t)n, (int32_t)r.K, (int32_t)r.ldw);
    if (p) p += (size_t)n * r.ldw;
  }
  return r;
}
void RowLoader::finish() {
  if (!status && ainfer_sync(dev, UINT64_MAX) != AINFER_OK) fail(1, ainfer_last_error(dev));
  for (auto &kv : handles) ainfer_kernel_release(kv.second);
  handles.clear();
}

// ------------------------------------------------------------------ engine ---
RowEngineBase::~RowEngineBase() {
  if (!dev) return;
  ainfer_sync(dev, UINT64_MAX);
  for (void *p : owned) ainfer_mem_free(dev, p);
}
int RowEngineBase::begin(DeviceModel *model, int n, int ctx, int cap_rows, bool in_f32, std::string &err) {
  m = model; dev = m->dev;
  nseq = n; f32 = in_f32;
  max_ctx = m->cfg.positions(ctx);
  rows_cap = std::max(1, cap_rows);
  ainfer_device_info info;
  if (ainfer_device_get_info(dev, &info) != AINFER_OK) { err = ainfer_last_error(dev); return 1; }
  sm_count = info.sm_count;
  return 0;
}
int RowEngineBase::alloc_bytes(size_t bytes, void **out) {
  void *p = nullptr;
  bytes = std::max<size_t>(bytes, 16);
  if (ainfer_mem_alloc(dev, bytes, 256, &p) != AINFER_OK || ainfer_mem_fill(dev, p, 0, bytes) != AINFER_OK) {
    alloc_err = ainfer_last_error(dev);
    return 1;
  }
  owned.push_back(p);
  *out = p;
  return 0;
}

void RowEngineBase::linear(KernelCalls &k, const RowMatrix &mt, const char *Xp, int ldx, int rows, void *Yp, int ldy, int act, bool out16, float cap) {
  if (k.status) return;
  if (f32) {
    k.launch("LinearRows", (uint32_t)(((mt.N + 63) / 64) * ((rows + 63) / 64)), (const float *)Xp, mt.w, mt.bias, (float *)Yp, (int32_t)rows,
             (int32_t)mt.N, (int32_t)mt.K, (int32_t)ldx, (int32_t)mt.ldw, (int32_t)ldy, (int32_t)act, cap);
    return;
  }
  const int n_tiles = (mt.N + 127) / 128, kb = (mt.K + 63) / 64;
  int nt = rows <= 16 ? 16 : rows <= 32 ? 32 : rows <= 64 ? 64 : 128;
  const bool few = 2 * n_tiles * ((rows + 127) / 128) <= sm_count;   // tiles of 128 rows leave most SMs idle: split K instead
  if (rows > 128 && !few) {
    // rows of a tile: as large as possible (operand traffic), but a launch lasts whole rounds of tiles over the SMs
    long best = -1;
    for (int t = 256; t >= 96; t -= 16) {
      const long rounds = ((long)n_tiles * ((rows + t - 1) / t) + sm_count - 1) / sm_count, cost = rounds * (t + 48);
      if (best < 0 || cost < best) { best = cost; nt = t; }
    }
  }
  const int tiles = n_tiles * ((rows + nt - 1) / nt);
  int splits = 1;   // few tiles: a cluster of blocks per tile, each a part of K
  while ((rows <= 128 || few) && splits < 8 && tiles * splits * 2 <= sm_count && kb >= splits * 4) splits *= 2;
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

void RowEngineBase::gemv(KernelCalls &k, const RowMatrix &mt, const float *x, float *y, int act) {
  k.launch("StreamGemv", gemv_blocks(mt.N), x, mt.w, mt.bias, y, (int32_t)mt.N, (int32_t)mt.K, (int32_t)mt.ldw, (int32_t)gemv_rows(mt.N), (int32_t)act,
           0.0f);
}

}  // namespace ainfer
