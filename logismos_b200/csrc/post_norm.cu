// The residual stream of a stack that normalises what a sublayer returns (fp32), and the inputs of the next
// sublayer made from it:
//   output norm   x += (y - mean(y)) / sqrt(var(y) + eps) * w + b
//   inputs        copy 0 = x; copies 1.. = x + (x' - x) * mu_s with x' the previous token's row (zero for the first)
// One token per sequence: all of it in one launch (a CTA per row). Ragged steps: the norm, then a second kernel
// for the mixes. The last row of a sequence is its state. A state slot holds two copies; a step reads the one its
// phase names and writes the other, so that a step that failed or is replayed finds its input unchanged.
// Rows are ld columns wide (a multiple of 4); columns from n on are zero in y, x, w and b.
#include "common.cuh"
#include "logismos_kernels.h"

namespace {

using namespace lg;

constexpr int kMaxThreads = 512, kMaxVec = 8, kMaxMix = 5;

LG_DEVINL void store4(void* out, size_t i4, float4 v, bool f32) {
  if (f32) reinterpret_cast<float4*>(out)[i4] = v;
  else reinterpret_cast<uint2*>(out)[i4] = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
LG_DEVINL float4 mix4(float4 x, float4 p, float4 mu) {
  return make_float4(fmaf(p.x - x.x, mu.x, x.x), fmaf(p.y - x.y, mu.y, x.y), fmaf(p.z - x.z, mu.z, x.z), fmaf(p.w - x.w, mu.w, x.w));
}

struct NormArgs {
  float* src;             // y, or with row_idx the stream itself
  int zero_src;           // src is an accumulation buffer: cleared once read
  const int* row_idx;
  int n_src_rows;
  float* x;               // residual stream (NULL: the normalised row is the result)
  const float* w;         // NULL: no norm, the row of x passes through
  const float* b;
  void* h;                // copy 0 in the activation format (NULL: none)
  int rows, n, ld, f32;
  float eps;
  int* status;
};

struct ShiftArgs {
  const float* mu;        // [n_mix][ld]
  int n_mix;              // copies 1 .. n_mix at h + s * rows * ld
  float* state;           // [n_slots][2][ld]
  const int* state_slots;
  const uint8_t* fresh;
  const uint8_t* phase;
};

template <int NV, bool SHIFT>
__global__ void __launch_bounds__(kMaxThreads)
post_norm_kernel(NormArgs p, ShiftArgs c) {
  lg::pdl_trigger();
  __shared__ float red[32];
  const int r = blockIdx.x, nv = p.ld >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  // gains, mixing weights and the state of an earlier step do not depend on the kernels before this one
  float4 w4 = zero, b4 = zero, prev = zero, mu[SHIFT ? kMaxMix : 1];
  const float4* old = nullptr;
  float4* next = nullptr;
  if (SHIFT) {
    float4* slot = reinterpret_cast<float4*>(c.state) + (size_t)c.state_slots[r] * 2 * nv;
    const int ph = c.phase[r] & 1;
    old = c.fresh[r] ? nullptr : slot + (size_t)ph * nv;
    next = slot + (size_t)(1 - ph) * nv;
  }
  auto fetch = [&](int v) {
    if (p.w) { w4 = __ldg(reinterpret_cast<const float4*>(p.w) + v); b4 = __ldg(reinterpret_cast<const float4*>(p.b) + v); }
    if (SHIFT) {
      prev = old ? old[v] : zero;
#pragma unroll
      for (int s = 0; s < kMaxMix; ++s) mu[s] = s < c.n_mix ? __ldg(reinterpret_cast<const float4*>(c.mu) + (size_t)s * nv + v) : zero;
    }
  };
  if (NV == 1 && (int)threadIdx.x < nv) fetch(threadIdx.x);
  lg::pdl_wait();
  int src_row = p.row_idx ? p.row_idx[r] : r;
  if (src_row < 0 || src_row >= p.n_src_rows) {
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, 1);
    src_row = 0;
  }
  float4 y[NV], x[NV];
  float inv = 0.0f, mean = 0.0f;
  float4* src = reinterpret_cast<float4*>(p.src) + (size_t)src_row * nv;
  float4* xr = p.x ? reinterpret_cast<float4*>(p.x) + (size_t)r * nv : nullptr;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    y[i] = p.w && v < nv ? src[v] : zero;
    x[i] = xr && v < nv ? xr[v] : zero;
  }
  if (p.w) {
    float s = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += (y[i].x + y[i].y) + (y[i].z + y[i].w);
    mean = block_sum(s, red) / (float)p.n;
    float q = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c0 = 4 * (threadIdx.x + i * blockDim.x);
      const float d0 = y[i].x - mean, d1 = y[i].y - mean, d2 = y[i].z - mean, d3 = y[i].w - mean;
      if (c0 + 4 <= p.n) q += (d0 * d0 + d1 * d1) + (d2 * d2 + d3 * d3);
      else q += (c0 < p.n ? d0 * d0 : 0.f) + (c0 + 1 < p.n ? d1 * d1 : 0.f) + (c0 + 2 < p.n ? d2 * d2 : 0.f);
    }
    inv = 1.0f / sqrtf(block_sum(q, red) / (float)p.n + p.eps);
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= nv) continue;
    if (NV > 1) fetch(v);
    float4 o = x[i];
    if (p.w) {  // zero gains keep the padding zero
      o.x += (y[i].x - mean) * inv * w4.x + b4.x;
      o.y += (y[i].y - mean) * inv * w4.y + b4.y;
      o.z += (y[i].z - mean) * inv * w4.z + b4.z;
      o.w += (y[i].w - mean) * inv * w4.w + b4.w;
      if (xr) xr[v] = o;
      if (p.zero_src) src[v] = zero;
    }
    if (p.h) store4(p.h, (size_t)r * nv + v, o, p.f32);
    if (SHIFT) {
      next[v] = o;
#pragma unroll
      for (int s = 0; s < kMaxMix; ++s)
        if (s < c.n_mix) store4(p.h, ((size_t)(s + 1) * p.rows + r) * nv + v, mix4(o, prev, mu[s]), p.f32);
    }
  }
}

// Copies 0 .. n_mix of ragged sequences: a thread owns four columns and a run of consecutive token rows.
constexpr int kRun = 8;
__global__ void __launch_bounds__(128)
token_shift_kernel(const float* __restrict__ x, const int* __restrict__ seq_ids, const int* __restrict__ cu, void* __restrict__ h, ShiftArgs c,
                   int rows, int ld, int f32) {
  lg::pdl_prologue();
  const int nv = ld >> 2, v = blockIdx.y * blockDim.x + threadIdx.x;
  if (v >= nv) return;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 mu[kMaxMix];
#pragma unroll
  for (int s = 0; s < kMaxMix; ++s) mu[s] = s < c.n_mix ? __ldg(reinterpret_cast<const float4*>(c.mu) + (size_t)s * nv + v) : zero;
  const float4* xs = reinterpret_cast<const float4*>(x);
  const int first = blockIdx.x * kRun, last = min(rows, first + kRun);
  float4 in[kRun];
#pragma unroll
  for (int i = 0; i < kRun; ++i) in[i] = first + i < last ? xs[(size_t)(first + i) * nv + v] : zero;
  float4 prev = zero;
  int cur = -1, t1 = 0;
  float4* next = nullptr;
#pragma unroll
  for (int i = 0; i < kRun; ++i) {
    const int t = first + i;
    if (t >= last) break;
    const int s = seq_ids[t];
    if (s != cur) {
      cur = s;
      t1 = cu[s + 1];
      float4* slot = reinterpret_cast<float4*>(c.state) + (size_t)c.state_slots[s] * 2 * nv;
      const int ph = c.phase[s] & 1;
      next = slot + (size_t)(1 - ph) * nv;
      prev = t > cu[s] ? xs[(size_t)(t - 1) * nv + v] : c.fresh[s] ? zero : slot[(size_t)ph * nv + v];
    }
    store4(h, (size_t)t * nv + v, in[i], f32);
#pragma unroll
    for (int m = 0; m < kMaxMix; ++m)
      if (m < c.n_mix) store4(h, ((size_t)(m + 1) * rows + t) * nv + v, mix4(in[i], prev, mu[m]), f32);
    if (t + 1 == t1) next[v] = in[i];
    prev = in[i];
  }
}

struct Shape { int threads, nv; };
Shape shape_of(int ld) {
  const int v = ld / 4;
  for (int nv = 1;; nv *= 2)
    if (v <= kMaxThreads * nv) return {((v + nv - 1) / nv + 31) / 32 * 32, nv};
}

template <bool SHIFT>
uint32_t launch_norm(const NormArgs& p, const ShiftArgs& c, cudaStream_t s) {
  const Shape sh = shape_of(p.ld);
  auto go = [&](auto kern) {
    lg::launch(kern, dim3((unsigned)p.rows), dim3((unsigned)sh.threads), 0, s, p, c);
    return lg::launch_status();
  };
  return sh.nv == 1 ? go(post_norm_kernel<1, SHIFT>) : sh.nv == 2 ? go(post_norm_kernel<2, SHIFT>) : sh.nv == 4 ? go(post_norm_kernel<4, SHIFT>)
       : go(post_norm_kernel<8, SHIFT>);
}

bool rows_ok(int rows, int n, int ld) { return rows > 0 && n > 0 && ld >= n && ld % 4 == 0 && ld / 4 <= kMaxThreads * kMaxVec; }

}  // namespace

extern "C" {

uint32_t logismos_launch_post_norm(void* src_f32, int32_t zero_src, const void* row_idx_i32, int32_t n_src_rows, void* x_f32, const void* w_f32,
                                   const void* b_f32, void* h, int32_t out_f32, int32_t rows, int32_t n, int32_t ld, float eps,
                                   void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!rows_ok(rows, n, ld) || (w_f32 && (!b_f32 || !src_f32)) || (!w_f32 && !x_f32) || n_src_rows <= 0 || (!row_idx_i32 && rows > n_src_rows) || (!x_f32 && !h))
    return lg::kInvalidValue;
  const NormArgs p{(float*)src_f32, zero_src, (const int*)row_idx_i32, n_src_rows, (float*)x_f32, (const float*)w_f32, (const float*)b_f32, h,
                   rows, n, ld, out_f32, eps, (int*)status_i32};
  return launch_norm<false>(p, ShiftArgs{}, (cudaStream_t)stream);
}

uint32_t logismos_launch_post_norm_shift_decode(void* src_f32, int32_t zero_src, void* x_f32, const void* w_f32, const void* b_f32, void* h,
                                                int32_t out_f32, const void* mu_f32, int32_t n_mix, void* state_f32, const void* state_slots_i32,
                                                const void* fresh_u8, const void* phase_u8, int32_t rows, int32_t n, int32_t ld, float eps,
                                                void* stream) {
  lg::LaunchScope launch_scope_;
  if (!rows_ok(rows, n, ld) || (w_f32 && (!b_f32 || !src_f32)) || !x_f32 || !h || !mu_f32 || n_mix < 1 || n_mix > kMaxMix || !state_f32 || !state_slots_i32 ||
      !fresh_u8 || !phase_u8)
    return lg::kInvalidValue;
  const NormArgs p{(float*)src_f32, zero_src, nullptr, rows, (float*)x_f32, (const float*)w_f32, (const float*)b_f32, h, rows, n, ld, out_f32, eps, nullptr};
  const ShiftArgs c{(const float*)mu_f32, n_mix, (float*)state_f32, (const int*)state_slots_i32, (const uint8_t*)fresh_u8, (const uint8_t*)phase_u8};
  return launch_norm<true>(p, c, (cudaStream_t)stream);
}

uint32_t logismos_launch_token_shift(const void* x_f32, void* h, int32_t out_f32, const void* mu_f32, int32_t n_mix, void* state_f32,
                                     const void* state_slots_i32, const void* fresh_u8, const void* phase_u8, const void* seq_ids_i32,
                                     const void* cu_seqlens_i32, int32_t rows, int32_t ld, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!x_f32 || !h || rows <= 0 || ld <= 0 || ld % 4 || !mu_f32 || n_mix < 1 || n_mix > kMaxMix || !state_f32 || !state_slots_i32 || !fresh_u8 || !phase_u8 ||
      !seq_ids_i32 || !cu_seqlens_i32)
    return lg::kInvalidValue;
  const ShiftArgs c{(const float*)mu_f32, n_mix, (float*)state_f32, (const int*)state_slots_i32, (const uint8_t*)fresh_u8, (const uint8_t*)phase_u8};
  const dim3 grid((unsigned)((rows + kRun - 1) / kRun), (unsigned)((ld / 4 + 127) / 128));
  lg::launch(token_shift_kernel, grid, dim3(128), 0, (cudaStream_t)stream, (const float*)x_f32, (const int*)seq_ids_i32, (const int*)cu_seqlens_i32, h, c, rows,
             ld, out_f32);
  return lg::launch_status();
}

}  // extern "C"
