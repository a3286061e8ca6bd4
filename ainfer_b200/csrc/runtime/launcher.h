// Kernel calls by name with arguments by index in member order, handed to a list being recorded or
// (list == null) straight to the execution queue. What the session's recorder, the batch engine and
// the prefill passes build on.
#pragma once
#include <cstdint>
#include <map>
#include <string>

#include "../../../include/ainfer_cuda.h"

namespace ainfer {

struct KernelCalls {
  ainfer_device_t dev = nullptr;
  std::map<std::string, ainfer_kernel_t> *kernels = nullptr;   // handles by name, filled on first use, owned by the caller
  std::string *err = nullptr;
  ainfer_list_t list = nullptr;
  int status = 0;             // first failure; later calls do nothing
  uint64_t launches = 0;

  KernelCalls(ainfer_device_t d, std::map<std::string, ainfer_kernel_t> *k, std::string *e, ainfer_list_t l = nullptr)
      : dev(d), kernels(k), err(e), list(l) {}

  void fail(int code, const std::string &msg) {
    if (!status) { status = code; *err = msg; }
  }
  ainfer_kernel_t kernel(const char *name) {
    auto it = kernels->find(name);
    if (it != kernels->end()) return it->second;
    ainfer_kernel_t k = nullptr;
    if (ainfer_kernel_get(dev, name, &k) != AINFER_OK) {
      fail(1, std::string("entry ") + name + " not found");
      return nullptr;
    }
    (*kernels)[name] = k;
    return k;
  }
  template <typename T>
  void set(ainfer_kernel_t k, uint32_t &idx, const T &v) {
    if (!status && ainfer_kernel_set_arg(k, idx, sizeof(T), &v) != AINFER_OK) fail(1, ainfer_last_error(dev));
    ++idx;
  }
  template <typename... A>
  void launch(const char *name, uint32_t groups, const A &...args) {
    if (status) return;
    ainfer_kernel_t k = kernel(name);
    if (!k) return;
    uint32_t idx = 0;
    (set(k, idx, args), ...);
    if (status) return;
    if (groups == 0) groups = 1;
    const int rc = list ? ainfer_list_append_launch(list, k, groups) : ainfer_kernel_launch(dev, k, groups);
    if (rc != AINFER_OK) fail(1, std::string(name) + ": " + ainfer_last_error(dev));
    ++launches;
  }
  void copy(void *dst, const void *src, size_t bytes) {   // recorded lists only
    if (!status && ainfer_list_append_memcpy(list, dst, src, bytes) != AINFER_OK) fail(1, std::string("append failed: ") + ainfer_last_error(dev));
  }
};

}  // namespace ainfer
