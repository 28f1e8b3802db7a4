// Residual-stream mechanisms around a parallel block, all fp32:
//   depth average      x = sum_j coef[j] X_j over the snapshots X_0 .. X_{n-1} of the residual stream
//   offset RMS norm    h = x / sqrt(mean(x^2) + eps) * gain     (gain = offset + w, folded at load)
//   input convolution  o = h + sum_j w[j] * h_(t - taps + 1 + j), depthwise and causal over a sequence's
//                      tokens, for up to two filters over the same h (two sublayers that read one norm)
// The last taps - 1 rows h of a sequence are its convolution state. A state slot holds two copies and a
// step reads the one its phase names and writes the other, so a step never overwrites what another
// thread still reads and a step that failed or is replayed finds its input unchanged.
// Rows are ld columns wide (a multiple of 4); columns from n on are padding with zero gain and filters.
#include "common.cuh"
#include "logismos_kernels.h"

namespace {

using namespace lg;

constexpr int kMaxThreads = 512, kMaxVec = 8;   // float4 per thread and row: 1, 2, 4 or 8
constexpr int kMaxTaps = 8;

LG_DEVINL float4 fma4(float a, float4 x, float4 c) { return make_float4(fmaf(a, x.x, c.x), fmaf(a, x.y, c.y), fmaf(a, x.z, c.z), fmaf(a, x.w, c.w)); }
LG_DEVINL float4 fma4(float4 a, float4 x, float4 c) { return make_float4(fmaf(a.x, x.x, c.x), fmaf(a.y, x.y, c.y), fmaf(a.z, x.z, c.z), fmaf(a.w, x.w, c.w)); }
LG_DEVINL float4 mul4(float a, float4 x, float4 g) { return make_float4(a * x.x * g.x, a * x.y * g.y, a * x.z * g.z, a * x.w * g.w); }
LG_DEVINL void store4(void* out, size_t i4, float4 v, bool f32) {
  if (f32) reinterpret_cast<float4*>(out)[i4] = v;
  else reinterpret_cast<uint2*>(out)[i4] = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

struct MixArgs {
  const float* hist;       // snapshot j at hist + j * hist_stride
  int64_t hist_stride;
  int n_hist;
  const float* coef;
  const int* row_idx;      // NULL: row r of the output is row r of the snapshots
  int n_src_rows;
  float* x;                // weighted sum (may be NULL)
  float* inv_rms;          // 1 / rms of every row (may be NULL)
  const float* gain;       // with norm_out
  void* norm_out;          // NULL: no normalised output
  int rows, n, ld, f32;
  float eps;
  int* status;
};

// the row sum of one CTA: acc[i] holds float4 tid + i * blockDim of the row; about eight loads in flight per thread
template <int NV>
LG_DEVINL void mix_row(const MixArgs& p, int src, float4 (&acc)[NV], float& ss) {
  constexpr int kAhead = NV >= 8 ? 1 : 8 / NV;
  const int nv = p.ld >> 2;
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = make_float4(0.f, 0.f, 0.f, 0.f);
  const float* base = p.hist + (size_t)src * p.ld;
  for (int j0 = 0; j0 < p.n_hist; j0 += kAhead) {
    float4 x[kAhead][NV];
    float c[kAhead];
#pragma unroll
    for (int a = 0; a < kAhead; ++a) {
      const bool in = j0 + a < p.n_hist;
      c[a] = in ? __ldg(p.coef + j0 + a) : 0.0f;
      const float4* row = reinterpret_cast<const float4*>(base + (size_t)(j0 + a) * p.hist_stride);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        x[a][i] = in && v < nv ? row[v] : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
#pragma unroll
    for (int a = 0; a < kAhead; ++a)
#pragma unroll
      for (int i = 0; i < NV; ++i) acc[i] = fma4(c[a], x[a][i], acc[i]);
  }
  ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) ss += acc[i].x * acc[i].x + acc[i].y * acc[i].y + acc[i].z * acc[i].z + acc[i].w * acc[i].w;
}

template <int NV>
__global__ void __launch_bounds__(kMaxThreads)
depth_mix_kernel(MixArgs p) {
  lg::pdl_prologue();
  __shared__ float red[32];
  const int r = blockIdx.x, nv = p.ld >> 2;
  int src = p.row_idx ? p.row_idx[r] : r;
  if (src < 0 || src >= p.n_src_rows) {
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, 1);
    src = 0;
  }
  float4 acc[NV];
  float ss;
  mix_row<NV>(p, src, acc, ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.n + p.eps);
  if (p.inv_rms && threadIdx.x == 0) p.inv_rms[r] = inv;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= nv) continue;
    if (p.x) reinterpret_cast<float4*>(p.x)[(size_t)r * nv + v] = acc[i];
    if (p.norm_out) store4(p.norm_out, (size_t)r * nv + v, mul4(inv, acc[i], __ldg(reinterpret_cast<const float4*>(p.gain) + v)), p.f32);
  }
}

struct ConvArgs {
  const float* gain;
  const float* w1;   // [taps, ld], tap taps - 1 is the current token; NULL: o1 = h
  const float* w2;   // second filter; o2 == NULL: none
  void* o1;
  void* o2;
  float* state;      // [n_slots][2][taps - 1][ld]
  const int* state_slots;
  const uint8_t* fresh;
  const uint8_t* phase;
  int taps;
};

// Depth average, norm and convolution of a step whose sequences bring one token each (row r = sequence r). Gains,
// filters and the state (left by an earlier step) do not depend on the kernels before this one in the step, so
// with one float4 per thread they are read ahead of the dependency wait.
template <int NV, int TAPS>
__global__ void __launch_bounds__(kMaxThreads)
depth_mix_conv_decode_kernel(MixArgs p, ConvArgs c) {
  lg::pdl_trigger();
  constexpr int HN = TAPS - 1;
  __shared__ float red[32];
  const int r = blockIdx.x, nv = p.ld >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const bool fresh = c.fresh[r] != 0;
  float4* slot = reinterpret_cast<float4*>(c.state) + (size_t)c.state_slots[r] * 2 * HN * nv;
  const int ph = c.phase[r] & 1;
  const float4* old = slot + (size_t)ph * HN * nv;
  float4* next = slot + (size_t)(1 - ph) * HN * nv;
  float4 gain = zero, w1[TAPS], w2[TAPS], prev[HN > 0 ? HN : 1];
  auto fetch = [&](int v) {
    gain = __ldg(reinterpret_cast<const float4*>(c.gain) + v);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      w1[j] = c.w1 ? __ldg(reinterpret_cast<const float4*>(c.w1) + (size_t)j * nv + v) : zero;
      w2[j] = c.w2 ? __ldg(reinterpret_cast<const float4*>(c.w2) + (size_t)j * nv + v) : zero;
    }
#pragma unroll
    for (int j = 0; j < HN; ++j) prev[j] = fresh ? zero : old[(size_t)j * nv + v];
  };
  if (NV == 1 && (int)threadIdx.x < nv) fetch(threadIdx.x);
  lg::pdl_wait();
  float4 acc[NV];
  float ss;
  mix_row<NV>(p, r, acc, ss);
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)p.n + p.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= nv) continue;
    if (NV > 1) fetch(v);
    reinterpret_cast<float4*>(p.x)[(size_t)r * nv + v] = acc[i];
    const float4 h = mul4(inv, acc[i], gain);
    float4 y1 = fma4(w1[TAPS - 1], h, h), y2 = fma4(w2[TAPS - 1], h, h);
#pragma unroll
    for (int j = 0; j < HN; ++j) {
      y1 = fma4(w1[j], prev[j], y1);
      y2 = fma4(w2[j], prev[j], y2);
      if (j > 0) next[(size_t)(j - 1) * nv + v] = prev[j];
    }
    if (HN > 0) next[(size_t)(HN > 0 ? HN - 1 : 0) * nv + v] = h;
    store4(c.o1, (size_t)r * nv + v, y1, p.f32);
    if (c.o2) store4(c.o2, (size_t)r * nv + v, y2, p.f32);
  }
}

// Norm and convolution of ragged sequences: a thread owns four columns and a run of consecutive token rows,
// carrying the previous taps - 1 rows h in registers.
constexpr int kRun = 8;
template <int TAPS>
__global__ void __launch_bounds__(128)
norm_conv_kernel(const float* __restrict__ x, const float* __restrict__ inv_rms, const int* __restrict__ seq_ids,
                 const int* __restrict__ cu, ConvArgs c, int rows, int ld, int f32) {
  lg::pdl_prologue();
  constexpr int HN = TAPS - 1;
  const int nv = ld >> 2, v = blockIdx.y * blockDim.x + threadIdx.x;
  if (v >= nv) return;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 gain = __ldg(reinterpret_cast<const float4*>(c.gain) + v);
  float4 w1[TAPS], w2[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    w1[j] = c.w1 ? __ldg(reinterpret_cast<const float4*>(c.w1) + (size_t)j * nv + v) : zero;
    w2[j] = c.w2 ? __ldg(reinterpret_cast<const float4*>(c.w2) + (size_t)j * nv + v) : zero;
  }
  const float4* xs = reinterpret_cast<const float4*>(x);
  float4 prev[HN > 0 ? HN : 1];  // prev[j] = h at (t - HN + j)
  int cur_seq = -1, t0 = 0, len = 0;
  bool fresh = false;
  const float4* old = nullptr;
  float4* next = nullptr;
  const int first = blockIdx.x * kRun, last = min(rows, first + kRun);
  for (int t = first; t < last; ++t) {
    const int s = seq_ids[t];
    if (s != cur_seq) {
      cur_seq = s;
      t0 = cu[s];
      len = cu[s + 1] - t0;
      fresh = c.fresh[s] != 0;
      float4* slot = reinterpret_cast<float4*>(c.state) + (size_t)c.state_slots[s] * 2 * HN * nv;
      const int ph = c.phase[s] & 1;
      old = slot + (size_t)ph * HN * nv;
      next = slot + (size_t)(1 - ph) * HN * nv;
#pragma unroll
      for (int j = 0; j < HN; ++j) {
        const int idx = t - t0 - HN + j;  // place inside the step's tokens of this sequence; negative: the state
        if (idx >= 0) prev[j] = mul4(inv_rms[t0 + idx], xs[(size_t)(t0 + idx) * nv + v], gain);
        else prev[j] = fresh ? zero : old[(size_t)(HN + idx) * nv + v];
      }
      if (t == t0) {  // rows of the old state that stay in the new one (fewer new tokens than the state holds)
#pragma unroll
        for (int j = 0; j < HN; ++j)
          if (j + len < HN) next[(size_t)j * nv + v] = fresh ? zero : old[(size_t)(j + len) * nv + v];
      }
    }
    const float4 h = mul4(inv_rms[t], xs[(size_t)t * nv + v], gain);
    float4 y1 = fma4(w1[TAPS - 1], h, h), y2 = fma4(w2[TAPS - 1], h, h);
#pragma unroll
    for (int j = 0; j < HN; ++j) { y1 = fma4(w1[j], prev[j], y1); y2 = fma4(w2[j], prev[j], y2); }
    store4(c.o1, (size_t)t * nv + v, y1, f32);
    if (c.o2) store4(c.o2, (size_t)t * nv + v, y2, f32);
    const int keep = HN - (len - (t - t0));  // row of the new state this token becomes, if any
    if (keep >= 0) next[(size_t)keep * nv + v] = h;
#pragma unroll
    for (int j = 0; j + 1 < HN; ++j) prev[j] = prev[j + 1];
    if (HN > 0) prev[HN > 0 ? HN - 1 : 0] = h;
  }
}

// threads of a row and float4 per thread
struct MixShape { int threads, nv; };
MixShape mix_shape(int ld) {
  const int v = ld / 4;
  for (int nv = 1;; nv *= 2)
    if (v <= kMaxThreads * nv) return {((v + nv - 1) / nv + 31) / 32 * 32, nv};
}

template <int NV>
uint32_t launch_decode(const MixArgs& p, const ConvArgs& c, int threads, cudaStream_t s) {
  auto go = [&](auto kern) {
    lg::launch(kern, dim3((unsigned)p.rows), dim3((unsigned)threads), 0, s, p, c);
    return lg::launch_status();
  };
  switch (c.taps) {
    case 1: return go(depth_mix_conv_decode_kernel<NV, 1>);
    case 2: return go(depth_mix_conv_decode_kernel<NV, 2>);
    case 3: return go(depth_mix_conv_decode_kernel<NV, 3>);
    case 4: return go(depth_mix_conv_decode_kernel<NV, 4>);
    case 5: return go(depth_mix_conv_decode_kernel<NV, 5>);
    case 6: return go(depth_mix_conv_decode_kernel<NV, 6>);
    case 7: return go(depth_mix_conv_decode_kernel<NV, 7>);
    default: return go(depth_mix_conv_decode_kernel<NV, 8>);
  }
}

bool mix_ok(const void* hist, int n_hist, const void* coef, int rows, int n, int ld) {
  return hist && coef && n_hist > 0 && rows > 0 && n > 0 && ld >= n && ld % 4 == 0 && ld / 4 <= kMaxThreads * kMaxVec;
}

}  // namespace

extern "C" {

uint32_t logismos_launch_depth_mix_f32(const void* hist_f32, int64_t hist_stride, int32_t n_hist, const void* coef_f32,
                                       const void* row_idx_i32, int32_t n_src_rows, void* x_f32, void* inv_rms_f32,
                                       const void* gain_f32, void* norm_out, int32_t out_f32, int32_t rows, int32_t n, int32_t ld,
                                       float eps, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!mix_ok(hist_f32, n_hist, coef_f32, rows, n, ld) || n_src_rows <= 0 || (!row_idx_i32 && rows > n_src_rows) || (norm_out && !gain_f32))
    return lg::kInvalidValue;
  const MixArgs p{(const float*)hist_f32, hist_stride, n_hist, (const float*)coef_f32, (const int*)row_idx_i32, n_src_rows, (float*)x_f32,
                  (float*)inv_rms_f32, (const float*)gain_f32, norm_out, rows, n, ld, out_f32, eps, (int*)status_i32};
  const MixShape sh = mix_shape(ld);
  auto go = [&](auto kern) {
    lg::launch(kern, dim3((unsigned)rows), dim3((unsigned)sh.threads), 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
  return sh.nv == 1 ? go(depth_mix_kernel<1>) : sh.nv == 2 ? go(depth_mix_kernel<2>) : sh.nv == 4 ? go(depth_mix_kernel<4>) : go(depth_mix_kernel<8>);
}

uint32_t logismos_launch_norm_conv(const void* x_f32, const void* inv_rms_f32, const void* gain_f32, const void* w1_f32,
                                   const void* w2_f32, void* o1, void* o2, int32_t out_f32, void* state_f32,
                                   const void* state_slots_i32, const void* fresh_u8, const void* phase_u8, const void* seq_ids_i32,
                                   const void* cu_seqlens_i32, int32_t rows, int32_t ld, int32_t taps, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!x_f32 || !inv_rms_f32 || !gain_f32 || !o1 || rows <= 0 || ld <= 0 || ld % 4 || taps < 1 || taps > kMaxTaps || (taps > 1 && !state_f32))
    return lg::kInvalidValue;
  const ConvArgs c{(const float*)gain_f32, (const float*)w1_f32, (const float*)w2_f32, o1, o2, (float*)state_f32, (const int*)state_slots_i32,
                   (const uint8_t*)fresh_u8, (const uint8_t*)phase_u8, taps};
  const dim3 grid((unsigned)((rows + kRun - 1) / kRun), (unsigned)((ld / 4 + 127) / 128));
  auto go = [&](auto kern) {
    lg::launch(kern, grid, dim3(128), 0, (cudaStream_t)stream, (const float*)x_f32, (const float*)inv_rms_f32, (const int*)seq_ids_i32,
               (const int*)cu_seqlens_i32, c, rows, ld, out_f32);
    return lg::launch_status();
  };
  switch (taps) {
    case 1: return go(norm_conv_kernel<1>);
    case 2: return go(norm_conv_kernel<2>);
    case 3: return go(norm_conv_kernel<3>);
    case 4: return go(norm_conv_kernel<4>);
    case 5: return go(norm_conv_kernel<5>);
    case 6: return go(norm_conv_kernel<6>);
    case 7: return go(norm_conv_kernel<7>);
    default: return go(norm_conv_kernel<8>);
  }
}

uint32_t logismos_launch_depth_mix_conv_decode(const void* hist_f32, int64_t hist_stride, int32_t n_hist, const void* coef_f32, void* x_f32,
                                               const void* gain_f32, const void* w1_f32, const void* w2_f32, void* o1, void* o2,
                                               int32_t out_f32, void* state_f32, const void* state_slots_i32, const void* fresh_u8,
                                               const void* phase_u8, int32_t rows, int32_t n, int32_t ld, float eps, int32_t taps,
                                               void* stream) {
  lg::LaunchScope launch_scope_;
  if (!mix_ok(hist_f32, n_hist, coef_f32, rows, n, ld) || !x_f32 || !gain_f32 || !o1 || taps < 1 || taps > kMaxTaps || (taps > 1 && !state_f32))
    return lg::kInvalidValue;
  const MixArgs p{(const float*)hist_f32, hist_stride, n_hist, (const float*)coef_f32, nullptr, rows, (float*)x_f32, nullptr,
                  nullptr, nullptr, rows, n, ld, out_f32, eps, nullptr};
  const ConvArgs c{(const float*)gain_f32, (const float*)w1_f32, (const float*)w2_f32, o1, o2, (float*)state_f32, (const int*)state_slots_i32,
                   (const uint8_t*)fresh_u8, (const uint8_t*)phase_u8, taps};
  const MixShape sh = mix_shape(ld);
  cudaStream_t s = (cudaStream_t)stream;
  return sh.nv == 1 ? launch_decode<1>(p, c, sh.threads, s) : sh.nv == 2 ? launch_decode<2>(p, c, sh.threads, s)
       : sh.nv == 4 ? launch_decode<4>(p, c, sh.threads, s) : launch_decode<8>(p, c, sh.threads, s);
}

}  // extern "C"
