// The safetensors reader behind lg_safetensors_*, for the checkpoint loaders of the executors.
#pragma once
#include <cstddef>
#include <cstdint>
#include <initializer_list>
#include <map>
#include <string>
#include <vector>

#include "logismos_model.h"

namespace lgm {

struct ArchiveEntry {
  int dtype = 0;
  std::vector<int64_t> shape;
  size_t start = 0, end = 0;  // absolute byte range in the mapping
};

struct Archive {
  std::string path;
  const uint8_t* map = nullptr;
  size_t len = 0;
  size_t data_start = 0;
  std::vector<std::string> ordering;  // by on-disk offset
  std::map<std::string, ArchiveEntry> index;
  ~Archive();
};

// sets lg_last_error() and returns `code`
uint32_t fail(uint32_t code, const std::string& msg);
uint32_t open_archive(const char* path, Archive** out);
uint32_t get_view(const Archive* r, const char* name, lg_tensor_view_t* out);
// the tensor must exist with exactly this dtype and shape (LG_EMB_COMPUTE with the reason otherwise)
uint32_t want_tensor(const Archive* r, const std::string& name, int dtype, std::initializer_list<int64_t> shape, const void** out);
// read_f32 of crates/encoders/src/stella.rs:376-400: F32, the exact shape and 4-byte aligned data
uint32_t want_f32(const Archive* r, const std::string& name, std::initializer_list<int64_t> shape, const float** out);

}  // namespace lgm
