// Pieces shared by the kernels of recurrences whose per-head state is a matrix [rows][cols] in fp32.
//
// Token-serial forms: a CTA of 256 threads, thread -> four columns (cols: a power of two from 16 to 1024) and every
// (1024 / cols)-th row. The state waits in shared memory, every thread fetching its own pieces asynchronously and
// reading back only those: what is in flight takes no registers and needs no barrier, so that many CTAs of a step
// stream their states at once. A state too large for that is read and written in memory for every token.
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

// shared memory that holds a state, or 0: too large
inline size_t state_smem(int rows, int cols) {
  const size_t bytes = ((size_t)rows * cols * 4 + 16 * kThreads - 1) / (16 * kThreads) * (16 * kThreads);
  return bytes <= 160 * 1024 ? bytes : 0;
}

// the state of one head: requested (or zeroed) at once, then visited row piece by row piece
struct State {
  float4* own;        // this thread's pieces in shared memory, kThreads apart; NULL: in memory
  float* st;
  LG_DEVINL State(void* smem, bool in_smem, float* st_) : own(in_smem ? reinterpret_cast<float4*>(smem) + threadIdx.x : nullptr), st(st_) {}
  LG_DEVINL void request(const Tile& t, bool fresh) {
    if (!own) return;
    int i = 0;
    for (int r = t.r0; r < t.rows; r += t.step, ++i) {
      if (fresh) own[i * kThreads] = make_float4(0.f, 0.f, 0.f, 0.f);
      else cp_async16(smem_u32(own + i * kThreads), st + (size_t)r * t.cols + t.c4);
    }
    cp_async_commit();
  }
  LG_DEVINL void arrived() { if (own) cp_async_wait<0>(); }
  // f(row, piece) updates each piece; `first`: the first token of a sequence that starts here; `last`: leaves for memory
  template <typename F>
  LG_DEVINL void visit(const Tile& t, bool first, bool last, F f) {
    int i = 0;
#pragma unroll 4
    for (int r = t.r0; r < t.rows; r += t.step, ++i) {
      float4* at = reinterpret_cast<float4*>(st + (size_t)r * t.cols + t.c4);
      float4 s = own ? own[i * kThreads] : first ? make_float4(0.f, 0.f, 0.f, 0.f) : *at;
      f(r, s);
      if (own && !last) own[i * kThreads] = s;
      else *at = s;
    }
  }
};

// sum over the threads that share columns; the result of column c is in out[c] for every thread after the barrier.
// red: 1024 floats
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

// ---- pieces of the chunk-parallel forms: 64 tokens of a sequence at a time, one head per CTA, a warp owns eight
// value columns and its slice of the state as mma accumulators --------------------------------------------------

constexpr int kChunk = 64;

// transposes an 8 x 8 tile of 16-bit values held one row pair per lane
LG_DEVINL uint32_t movmatrix_trans(uint32_t v) {
  uint32_t r;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;\n" : "=r"(r) : "r"(v));
  return r;
}
// two fp32 values as bf16 plus what rounding dropped: together about 16 significant bits
LG_DEVINL void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - h.x, b - h.y);
}
// accumulators of a 16 (state channels) x 8 (values) tile as the B operand of a product over its channels
LG_DEVINL void state_operand(const float (&s)[4], uint32_t (&hi)[2], uint32_t (&lo)[2]) {
  uint32_t h0, l0, h1, l1;
  split2(s[0], s[1], h0, l0);
  split2(s[2], s[3], h1, l1);
  hi[0] = movmatrix_trans(h0); hi[1] = movmatrix_trans(h1);
  lo[0] = movmatrix_trans(l0); lo[1] = movmatrix_trans(l1);
}
// tiles of bf16 rows with a pitch of `pitch` bytes (row length + 16: rows start in different banks)
// A operand: rows r0 .. r0 + 15, columns k0 .. k0 + 15
LG_DEVINL void frag_a(uint32_t (&a)[4], uint32_t base, int pitch, int r0, int k0, int lane) {
  ldmatrix_x4(a, base + (uint32_t)((r0 + (lane & 7) + 8 * ((lane >> 3) & 1)) * pitch + (k0 + 8 * (lane >> 4)) * 2));
}
// A operand, the transpose of the tile: rows = columns m0 .. m0 + 15 of it, k = its rows k0 .. k0 + 15
LG_DEVINL void frag_at(uint32_t (&a)[4], uint32_t base, int pitch, int m0, int k0, int lane) {
  ldmatrix_x4_trans(a, base + (uint32_t)((k0 + (lane & 7) + 8 * (lane >> 4)) * pitch + (m0 + 8 * ((lane >> 3) & 1)) * 2));
}
// B operands of two neighbouring n8 tiles: n = rows n0 .. n0 + 15, k = columns k0 .. k0 + 15; tile i at b[2 i]
LG_DEVINL void frag_b(uint32_t (&b)[4], uint32_t base, int pitch, int n0, int k0, int lane) {
  ldmatrix_x4(b, base + (uint32_t)((n0 + (lane & 7) + 8 * (lane >> 4)) * pitch + (k0 + 8 * ((lane >> 3) & 1)) * 2));
}
// B operands of one n8 tile for two neighbouring k16 steps: k = rows k0 .. k0 + 31, n = columns n0 .. n0 + 7; step i at b[2 i]
LG_DEVINL void frag_bt(uint32_t (&b)[4], uint32_t base, int pitch, int k0, int n0, int lane) {
  ldmatrix_x4_trans(b, base + (uint32_t)((k0 + lane) * pitch + n0 * 2));
}
LG_DEVINL void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  const uint32_t b[2] = {b0, b1};
  mma_bf16_16816(d, a, b, d);
}
// 64 rows of a [rows][width] bf16 block at src (row stride ld elements; width a power of two) into a tile; rows >= n are zero
LG_DEVINL void stage_tile(uint8_t* tile, int pitch, const __nv_bfloat16* src, int64_t ld, int n, int width) {
  const int pieces = width >> 3, lg = 31 - __clz(pieces);
  for (int e = threadIdx.x; e < kChunk * pieces; e += blockDim.x) {
    const int row = e >> lg, piece = e & (pieces - 1);
    uint8_t* dst = tile + row * pitch + piece * 16;
    if (row < n) cp_async16(smem_u32(dst), src + row * ld + piece * 8);
    else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
  }
}

}  // namespace rec
}  // namespace lg
