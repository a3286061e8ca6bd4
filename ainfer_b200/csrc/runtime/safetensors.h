// SafeTensors files and sharded directories, mapped into memory (ingest.cpp).
#pragma once
#include <cstddef>
#include <cstdint>
#include <string>
#include <vector>

namespace ainfer {

struct SrcTensor {
  std::string name, dtype;
  std::vector<uint64_t> shape;
  const uint8_t *data = nullptr;
  uint64_t bytes = 0;
};

struct Shard {
  int fd = -1;
  const uint8_t *map = nullptr;
  size_t size = 0;
  Shard() = default;
  Shard(const Shard &) = delete;
  Shard &operator=(const Shard &) = delete;
  ~Shard();
};

struct SafeTensors {
  std::vector<Shard> shards;
  std::vector<SrcTensor> tensors;
  // A file, or a directory holding model.safetensors or model.safetensors.index.json with its shards.
  bool open(const char *src, std::string &err);
};

// Bytes of one element of a floating-point source (0: another type).
int st_elem_bytes(const std::string &dtype);
// Writes tensor t as bf16 (exact for BF16 sources, rounded to nearest even otherwise).
void st_to_bf16(const SrcTensor &t, uint16_t *out);

}  // namespace ainfer
