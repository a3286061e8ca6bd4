// What the row engines share: tensor lists, prepared matrices, device buffers, and the products of rows
// and of a decode step's single row.
#pragma once
#include <algorithm>
#include <string>
#include <vector>

#include "arch.h"

namespace ainfer {

inline int round_up(int v, int m) { return (v + m - 1) / m * m; }
inline std::string layer_name(int L) { return "l" + std::to_string(L) + "."; }
std::string json_num(double v);   // every digit

// ----------------------------------------------------------------- tensors ---
// One bf16 tensor of an architecture and how a synthetic model fills it (N(0, std^2), or a constant).
struct RowTensor { std::string name; std::vector<uint64_t> shape; float std_, constant; };
void plan_row_tensors(const std::vector<RowTensor> &t, const std::string &arch_json, int vocab, Container &dir, std::vector<SynthSpec> &specs);
int check_row_tensors(const Container &dir, const std::vector<RowTensor> &t, std::string &err);

struct RowMatrix {           // bf16 rows of ldw values (ldw a multiple of 8, zero padding)
  const uint16_t *w = nullptr;
  const float *bias = nullptr;
  int N = 0, K = 0, ldw = 0;
};

// Preparation of a model's weights; what it allocates belongs to the model.
struct RowLoader : KernelCalls {
  DeviceModel *m;
  std::map<std::string, ainfer_kernel_t> handles;
  RowLoader(DeviceModel *model, std::string *err);
  void *alloc(size_t bytes);
  const float *widen(const std::string &name);                 // fp32 copy on the device
  std::vector<uint16_t> host(const std::string &name);         // bf16 values on the host
  const float *upload(const std::vector<float> &v);
  const float *gain(const std::string &name);                  // 1 + the stored weight
  // the rows of matrices with the same row length as one; copied only when rows need padding or do not adjoin
  RowMatrix stack(const std::vector<std::string> &names);
  void finish();                                               // waits, releases the handles
};

// ------------------------------------------------------------------ engine ---
enum { ACT_NONE = 0, ACT_RELU2 = 1, ACT_SOFTCAP = 2 };
struct alignas(64) TensorMap { unsigned char b[128]; };

struct RowEngineBase : RowEngine {
  DeviceModel *m = nullptr;
  ainfer_device_t dev = nullptr;
  int nseq = 0, max_ctx = 0, sm_count = 1;
  bool f32 = false;
  std::vector<void *> owned;
  std::string alloc_err;

  ~RowEngineBase() override;
  int begin(DeviceModel *model, int n, int ctx, int cap_rows, bool in_f32, std::string &err);
  size_t esz() const { return f32 ? 4 : 2; }
  int alloc_bytes(size_t bytes, void **out);
  template <typename T>
  int alloc(size_t count, T **out) {
    void *p = nullptr;
    if (alloc_bytes(count * sizeof(T), &p)) return 1;
    *out = (T *)p;
    return 0;
  }
  // Y[rows][N] = act(X W^T + bias); X in the activation type, out16: Y bf16 (else fp32)
  void linear(KernelCalls &k, const RowMatrix &mt, const char *Xp, int ldx, int rows, void *Yp, int ldy, int act, bool out16, float cap = 0.0f);
  // one fp32 row; the same for kernels that prepare the row themselves: rows per block and blocks
  int gemv_rows(int N) const { return (N + 2 * sm_count - 1) / (2 * sm_count); }
  uint32_t gemv_blocks(int N) const { return (uint32_t)((N + gemv_rows(N) - 1) / gemv_rows(N)); }
  void gemv(KernelCalls &k, const RowMatrix &mt, const float *x, float *y, int act);
  // name of the instance of a kernel family whose padded head size holds `dim`
  static std::string sized(const char *base, int dim) {
    for (int d : {32, 64, 96, 128, 192})
      if (dim <= d) return base + std::to_string(d);
    return base + std::string("256");
  }
  // blocks of a step's attention over sequences, key heads and splits: few tiles each when there are many sequences
  int step_splits(int max_kv_heads) const {
    if (nseq == 1) return std::max(1, std::min(16, 2 * sm_count / max_kv_heads));
    return std::max(1, std::min(16, 8 * sm_count / (std::min(nseq, 8 * sm_count) * max_kv_heads)));
  }
};

}  // namespace ainfer
