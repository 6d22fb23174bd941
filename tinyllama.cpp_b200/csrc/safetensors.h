// Read-only view of a safetensors file: an 8-byte little-endian header length, a JSON header (name -> dtype, shape,
// data_offsets) and the data. The file is mapped; tensors point into the mapping.
#pragma once
#include <cstdint>
#include <map>
#include <string>
#include <vector>

namespace b200 {

struct StTensor {
  std::string dtype;  // "BF16", "F32", "I32", ...
  std::vector<int64_t> shape;
  const uint8_t* data = nullptr;
  size_t bytes = 0;
  int64_t elems() const {
    int64_t n = 1;
    for (int64_t d : shape) n *= d;
    return n;
  }
};

struct StFile {
  std::map<std::string, StTensor> tensors;
  const uint8_t* map_base = nullptr;
  size_t map_size = 0;
  int fd = -1;
  StFile() = default;
  StFile(const StFile&) = delete;
  StFile& operator=(const StFile&) = delete;
  ~StFile();
};

// Throws std::runtime_error on malformed input.
void safetensors_open(const std::string& path, StFile& out);

}  // namespace b200
