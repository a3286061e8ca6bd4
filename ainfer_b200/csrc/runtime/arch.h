// Architectures the runtime serves. A model names its architecture in its configuration; the loader
// (model.cpp) and the block executor (executor.cpp, prefill.cpp, batch.cpp) look it up here and call
// what differs between architectures through these tables. The token loop, control block, prompt
// passes, sampler, batch interface, command line and server are common to all.
#pragma once
#include <string>
#include <vector>

#include "launcher.h"
#include "model.h"

namespace ainfer {

struct Session;
struct Json;
struct RowEngine;

// Configuration and weights.
struct ModelArch {
  const char *name;
  bool int4;                                                             // projection weights are INT4 g128 (else bf16)
  bool (*parse)(const Json &js, ModelConfig &out, std::string &err);     // null: the flat INT4 form
  std::string (*to_json)(const ModelConfig &c);
  bool (*check)(const ModelConfig &c, std::string &err);
  void (*plan)(const ModelConfig &c, Container &dir, std::vector<SynthSpec> &specs);
  int (*check_directory)(const Container &dir, const ModelConfig &c, std::string &err);
  int (*prepare)(DeviceModel *m, std::string &err);                      // after the weights are on the device
  RowEngine *(*engine)();                                                // null: the block executor of the INT4 hybrid
};
const ModelArch *model_arch(const std::string &name);                    // null: unknown

// Rows of a prompt pass or of a batched step, as the architecture's row path sees them.
struct RowSpan {
  const int32_t *ctrl = nullptr, *seq = nullptr, *first = nullptr;   // device: [rows][4], [rows], [rows]
  int rows = 0;
  bool one_sequence = true;       // rows are consecutive positions of one sequence; else one row per sequence
  const int32_t *want = nullptr;  // device: rows whose logits are asked for
  int n_want = 0;
  float *logits = nullptr;        // device: [n_want][vocab]
};
struct RowEngine {                // state of `nseq` sequences plus the buffers of a pass of `rows_cap` rows
  virtual ~RowEngine() {}
  // max_ctx: positions a sequence may reach; f32: activations and cache in 32-bit. 0, 1 (device) or 2 (usage).
  virtual int create(DeviceModel *m, int nseq, int max_ctx, int rows_cap, bool f32, std::string &err) = 0;
  virtual void emit(KernelCalls &k, const RowSpan &span) = 0;
  virtual int reset(std::string &err) = 0;
  virtual bool buffer(const std::string &which, void **dptr, uint64_t *bytes) = 0;
  // one decode step of sequence 0 as recorded launches: embedding, one layer, final norm + head
  virtual void record_embed(KernelCalls &k, const int32_t *ctrl) = 0;
  virtual void record_layer(KernelCalls &k, int layer, const int32_t *ctrl) = 0;
  virtual void record_residual(KernelCalls &k, float *dst) = 0;   // after a layer: the residual it leaves [hidden]
  virtual void record_head(KernelCalls &k, float *logits) = 0;
  int rows_cap = 0;
};
// Makes and creates the row engine of a model's architecture (usage error where it has none).
int row_engine_create(DeviceModel *m, int nseq, int max_ctx, int rows_cap, bool f32, RowEngine **out, std::string &err);

bool sinepel_preset(const std::string &name, ModelConfig &c);   // "sinepel-tiny", "sinepel-small"
bool robopel_preset(const std::string &name, ModelConfig &c);   // "robopel-tiny", "robopel-small"
const ModelArch *sinepel_model_arch();
const ModelArch *robopel_model_arch();
const ModelArch *int4_hybrid_model_arch();

}  // namespace ainfer
