// Host-side packing of bf16 weights for the executors that keep dense matrices (zero-padded at load), and the route
// of a projection by its number of rows.
#pragma once
#include <cstdint>
#include <cstring>
#include <vector>

#include "logismos_kernels.h"
#include "model_util.h"

namespace lgm {

inline int round_up(int v, int to) { return (v + to - 1) / to * to; }
inline int r64(int v) { return round_up(v, 64); }

// Whether a projection of few rows streams its weights (linear_small) instead of running on the tcgen05 tiles. Measured
// (us, small / tiles): accumulating into the residual, where the tiles split k, 2048 x 10240 at 1 / 8 / 32 rows 14.6 /
// 12.6, 15.6 / 12.6, 29.0 / 12.6; gated 16384 x 2048 at 8 / 16 / 32 rows 17.8 / 22.7, 19.0 / 22.0, 28.5 / 17.9; head 32768
// x 2048 at 16 / 32 rows 39.5 / 41.5, 57.2 / 41.1; 1536 x 2048 at 8 / 32 / 64 rows 5.7 / 17.4, 11.6 / 18.2, 20.8 / 19.1.
inline bool stream_weights(int rows, int n, int k, int epi) {
  if (epi == LG_EPI_RESID_F32) return logismos_get_deterministic() && rows <= 32;
  return rows <= ((int64_t)n * k >= (1 << 23) ? 16 : 32);
}

// ---- weights: bf16 on the host, read bytewise (file data may be unaligned) -------------------------

inline uint16_t bf_at(const void* p, size_t i) {
  uint16_t v;
  std::memcpy(&v, (const uint8_t*)p + 2 * i, 2);
  return v;
}
inline float f_at(const void* p, size_t i) {
  const uint32_t u = (uint32_t)bf_at(p, i) << 16;
  float f;
  std::memcpy(&f, &u, 4);
  return f;
}

// offset + w over n values, zero in the padding
inline bool upload_vec(Buf& b, const void* src, int n, int padded, float offset) {
  std::vector<float> v((size_t)padded, 0.0f);
  for (int i = 0; i < n; ++i) v[(size_t)i] = offset + f_at(src, (size_t)i);
  return b.upload(v.data(), v.size() * 4);
}

// filters [n, taps] -> fp32 [taps, padded]
inline bool upload_conv(Buf& b, const void* src, int n, int padded, int taps) {
  std::vector<float> v((size_t)taps * padded, 0.0f);
  for (int i = 0; i < n; ++i)
    for (int j = 0; j < taps; ++j) v[(size_t)j * padded + i] = f_at(src, (size_t)i * taps + j);
  return b.upload(v.data(), v.size() * 4);
}

struct Mat {  // zero-initialised bf16 matrix under construction
  int ld;
  std::vector<uint16_t> v;
  Mat(int rows, int cols) : ld(cols), v((size_t)rows * cols, 0) {}
  void row(int dst_row, int dst_col, const void* src, size_t src_elem, int n) {
    std::memcpy(v.data() + (size_t)dst_row * ld + dst_col, (const uint8_t*)src + 2 * src_elem, (size_t)n * 2);
  }
  bool up(Buf& b) { return b.upload(v.data(), v.size() * 2); }
};

// [heads, d] values, every head padded to dp
inline bool upload_heads(Buf& b, const void* src, int heads, int d, int dp) {
  std::vector<float> v((size_t)heads * dp, 0.0f);
  for (int h = 0; h < heads; ++h)
    for (int i = 0; i < d; ++i) v[(size_t)h * dp + i] = f_at(src, (size_t)h * d + i);
  return b.upload(v.data(), v.size() * 4);
}

}  // namespace lgm
