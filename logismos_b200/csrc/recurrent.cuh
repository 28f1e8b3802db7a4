// Pieces shared by the token-serial recurrences whose per-head state is a matrix [rows][cols] in fp32: a CTA of
// 256 threads holds it as float4 pieces, thread -> four columns and every (1024 / cols)-th row. cols is a power of
// two from 16 to 1024. PT pieces per thread stay in registers over the tokens of a call; PT = 0: too many for that,
// the state is read and written in memory for every token.
#pragma once
#include "common.cuh"

namespace lg {
namespace rec {

constexpr int kThreads = 256;

template <typename T> struct Io;
template <> struct Io<float> {
  static LG_DEVINL float load(const float* p) { return *p; }
  static LG_DEVINL void store(float* p, float v) { *p = v; }
};
template <> struct Io<__nv_bfloat16> {
  static LG_DEVINL float load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
  static LG_DEVINL void store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
};

LG_DEVINL float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
LG_DEVINL float silu_f(float z) { return z / (1.0f + expf(-z)); }
LG_DEVINL float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

struct Tile {
  int rows, cols, c4, r0, step;   // first column and row of this thread, distance of its rows
  LG_DEVINL Tile(int rows_, int cols_) : rows(rows_), cols(cols_) {
    const int nv = cols_ >> 2;
    c4 = 4 * ((int)threadIdx.x % nv);
    r0 = (int)threadIdx.x / nv;
    step = kThreads / nv;
  }
};

// pieces per thread that hold a state of this size, or 0
inline int pieces(int rows, int cols) {
  const int n = (rows * cols + 4 * kThreads - 1) / (4 * kThreads);
  return n <= 1 ? 1 : n <= 2 ? 2 : n <= 4 ? 4 : n <= 8 ? 8 : n <= 16 ? 16 : 0;
}

// sum over the threads that share columns; the result of column c is in out[c] for every thread after the barrier.
// red: [8][cols] floats (cols <= 128) or [kThreads / (cols / 4)][cols]
LG_DEVINL int reduce_groups(int cols) { const int nv = cols >> 2; return kThreads / (nv < 32 ? 32 : nv); }
LG_DEVINL void reduce_store(const Tile& t, float4 v, float* red) {
  const int nv = t.cols >> 2;
  for (int o = nv; o < 32; o <<= 1) {
    v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
    v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
    v.z += __shfl_xor_sync(0xffffffffu, v.z, o);
    v.w += __shfl_xor_sync(0xffffffffu, v.w, o);
  }
  const int g = (int)threadIdx.x / (nv < 32 ? 32 : nv);
  if (nv >= 32 || (threadIdx.x & 31) < (unsigned)nv) *reinterpret_cast<float4*>(red + (size_t)g * t.cols + t.c4) = v;
}
LG_DEVINL float reduce_load(int cols, const float* red, int c) {
  float s = 0.0f;
  const int n = reduce_groups(cols);
  for (int g = 0; g < n; ++g) s += red[(size_t)g * cols + c];
  return s;
}

}  // namespace rec
}  // namespace lg
