// The residual stream (fp32) of a stack with RMS norms of one gain and gated sublayers, and the difference of two attentions:
//   y = a sublayer's output, half the sum of two branches each divided by its root mean square and times its gain, or the
//       rows of a mixture of experts still to be summed
//   x += y sigmoid(gate);   x += embedding + step (ahead of a pass over repeated layers);   h = x / rms(x) * gain
// A CTA owns a row, a thread NV times four columns of it; the padding columns are zero in all that is read.
#include "common.cuh"
#include "logismos_kernels.h"

namespace {

using namespace lg;

constexpr int kMaxThreads = 512, kMaxVec = 8;

LG_DEVINL void store4(void* out, size_t i4, float4 v, bool f32) {
  if (f32) reinterpret_cast<float4*>(out)[i4] = v;
  else reinterpret_cast<uint2*>(out)[i4] = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
LG_DEVINL float4 load4(const void* in, size_t i4, bool f32) {
  if (f32) return reinterpret_cast<const float4*>(in)[i4];
  const uint2 u = reinterpret_cast<const uint2*>(in)[i4];
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
LG_DEVINL float dot4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }
LG_DEVINL float gate_f(float z, bool exact) { return 1.0f / (1.0f + (exact ? expf(-z) : __expf(-z))); }

struct Args {
  float4* x;
  float4* branch[2];
  int zero;
  const float4* branch_gain[2];
  const void* expert_rows;     // mixture
  const int* pair_row;
  const float* weights;
  int n_pairs, top;
  int* counts;
  int n_counts;
  const void* gate;
  int ld_gate;
  float4* kept;
  const void* embed;
  const uint32_t* ids;
  const float4* step;
  int vocab;
  void* h;
  float gain, eps;
  const int* row_idx;
  int n_src_rows, n, nv, f32;
  int* status;
};

enum { kNone = 0, kOne = 1, kTwo = 2, kMixture = 3 };   // where y comes from

// two sums over the CTA at once; red: 64 floats
LG_DEVINL float2 block_sum2(float a, float b, float* red) {
  a = warp_sum(a);
  b = warp_sum(b);
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if (lane == 0) { red[2 * wid] = a; red[2 * wid + 1] = b; }
  __syncthreads();
  const float2 t = lane < nw ? make_float2(red[2 * lane], red[2 * lane + 1]) : make_float2(0.f, 0.f);
  const float2 r = make_float2(warp_sum(t.x), warp_sum(t.y));
  __syncthreads();
  return r;
}

template <int NV, int FROM>
__global__ void __launch_bounds__(kMaxThreads)
gated_residual_kernel(Args p) {
  lg::pdl_trigger();
  __shared__ float red[64];
  const int r = blockIdx.x, nv = p.nv;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 g0 = zero, g1 = zero;   // gains of the branches do not depend on the kernels before this one
  if (FROM == kTwo && NV == 1 && (int)threadIdx.x < nv) { g0 = __ldg(p.branch_gain[0] + threadIdx.x); g1 = __ldg(p.branch_gain[1] + threadIdx.x); }
  lg::pdl_wait();
  if (FROM == kMixture && r == 0 && p.counts)
    for (int g = threadIdx.x; g < p.n_counts; g += blockDim.x) p.counts[g] = 0;
  int src = p.row_idx ? p.row_idx[r] : r;
  if (src < 0 || src >= p.n_src_rows) {
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, 1);
    src = 0;
  }
  float4 x[NV], y[NV], z[FROM == kTwo ? NV : 1];
  float4* xr = p.x + (size_t)src * nv;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    const bool in = v < nv;
    x[i] = in ? xr[v] : zero;
    y[i] = zero;
    if (FROM == kOne || FROM == kTwo) {
      if (in) y[i] = p.branch[0][(size_t)r * nv + v];
    }
    if (FROM == kTwo) z[i] = in ? p.branch[1][(size_t)r * nv + v] : zero;
  }
  if (FROM == kMixture) {
    constexpr int kBatch = 4;   // experts' rows in flight
    for (int k0 = 0; k0 < p.n_pairs; k0 += kBatch) {
      int row[kBatch];
      float w[kBatch];
#pragma unroll
      for (int j = 0; j < kBatch; ++j) {
        const int k = k0 + j;
        row[j] = k < p.n_pairs ? p.pair_row[(size_t)r * p.n_pairs + k] : -1;
        w[j] = k < p.top ? p.weights[(size_t)r * p.top + k] : 1.0f;
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        float4 e[kBatch];
#pragma unroll
        for (int j = 0; j < kBatch; ++j) e[j] = row[j] >= 0 && v < nv ? load4(p.expert_rows, (size_t)row[j] * nv + v, p.f32) : zero;
#pragma unroll
        for (int j = 0; j < kBatch; ++j) {
          y[i].x = fmaf(w[j], e[j].x, y[i].x); y[i].y = fmaf(w[j], e[j].y, y[i].y); y[i].z = fmaf(w[j], e[j].z, y[i].z); y[i].w = fmaf(w[j], e[j].w, y[i].w);
        }
      }
    }
  }
  float m0 = 0.0f, m1 = 0.0f;
  if (FROM == kTwo) {
    float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; ++i) { s0 += dot4(y[i]); s1 += dot4(z[i]); }
    const float2 s = block_sum2(s0, s1, red);
    m0 = 0.5f / sqrtf(s.x / (float)p.n + p.eps);
    m1 = 0.5f / sqrtf(s.y / (float)p.n + p.eps);
  }
  const uint32_t id = p.embed ? min(p.ids[r], (uint32_t)p.vocab - 1) : 0;
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= nv) continue;
    float4 d = y[i];
    if (FROM == kTwo) {
      if (NV > 1) { g0 = __ldg(p.branch_gain[0] + v); g1 = __ldg(p.branch_gain[1] + v); }
      const float4 e = z[i];
      d = make_float4(d.x * m0 * g0.x + e.x * m1 * g1.x, d.y * m0 * g0.y + e.y * m1 * g1.y, d.z * m0 * g0.z + e.z * m1 * g1.z, d.w * m0 * g0.w + e.w * m1 * g1.w);
    }
    if (FROM != kNone) {
      const float4 g = load4(p.gate, (size_t)r * (p.ld_gate >> 2) + v, p.f32);
      const bool exact = p.f32 != 0;
      x[i].x = fmaf(d.x, gate_f(g.x, exact), x[i].x);
      x[i].y = fmaf(d.y, gate_f(g.y, exact), x[i].y);
      x[i].z = fmaf(d.z, gate_f(g.z, exact), x[i].z);
      x[i].w = fmaf(d.w, gate_f(g.w, exact), x[i].w);
      if (p.zero && FROM != kMixture) {
        p.branch[0][(size_t)r * nv + v] = zero;
        if (FROM == kTwo) p.branch[1][(size_t)r * nv + v] = zero;
      }
    }
    if (p.kept) p.kept[(size_t)r * nv + v] = x[i];
    if (p.embed) {
      const float4 e = load4(p.embed, (size_t)id * nv + v, false);
      x[i].x += e.x; x[i].y += e.y; x[i].z += e.z; x[i].w += e.w;
    }
    if (p.step) {
      const float4 e = __ldg(p.step + v);
      x[i].x += e.x; x[i].y += e.y; x[i].z += e.z; x[i].w += e.w;
    }
    if (FROM != kNone || p.embed || p.step) xr[v] = x[i];
    ss += dot4(x[i]);
  }
  if (!p.h) return;
  const float m = p.gain / sqrtf(block_sum(ss, red) / (float)p.n + p.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nv) store4(p.h, (size_t)r * nv + v, make_float4(x[i].x * m, x[i].y * m, x[i].z * m, x[i].w * m), p.f32 != 0);
  }
}

// a warp per (row, head); outputs of the two maps stand rep heads apart
template <typename T>
__global__ void __launch_bounds__(256)
attention_difference_kernel(const float* __restrict__ a, int ld_a, T* __restrict__ out, int ld_out, int rows, int heads, int rep, int v, int vp, float lambda, float scale,
                            float eps) {
  lg::pdl_prologue();
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= (int64_t)rows * heads) return;
  const int r = (int)(item / heads), h = (int)(item % heads), lane = threadIdx.x & 31, nv = vp >> 2;
  const float4* a1 = reinterpret_cast<const float4*>(a + (size_t)r * ld_a + (size_t)(h / rep * 2 * rep + h % rep) * vp);
  const float4* a2 = a1 + (size_t)rep * nv;
  float4 o[2];   // vp <= 256
  float ss = 0.0f;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int c = lane + 32 * i;
    o[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c >= nv) continue;
    const float4 x = a1[c], y = a2[c];
    o[i] = make_float4(x.x - lambda * y.x, x.y - lambda * y.y, x.z - lambda * y.z, x.w - lambda * y.w);
    ss += dot4(o[i]);
  }
  const float m = scale / sqrtf(warp_sum(ss) / (float)v + eps);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int c = lane + 32 * i;
    if (c < nv) store4(out, (size_t)r * (ld_out >> 2) + (size_t)h * nv + c, make_float4(o[i].x * m, o[i].y * m, o[i].z * m, o[i].w * m), sizeof(T) == 4);
  }
}

}  // namespace

extern "C" {

uint32_t logismos_launch_gated_residual(const lg_gated_residual_t* a, void* status, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!a || !a->x || a->rows <= 0 || a->n <= 0 || a->ld < a->n || a->ld % 4 || a->ld / 4 > kMaxThreads * kMaxVec || a->n_src_rows <= 0 || (!a->row_idx && a->rows > a->n_src_rows))
    return lg::kInvalidValue;
  const int from = a->mixture ? kMixture : a->branch[1] ? kTwo : a->branch[0] ? kOne : kNone;
  if ((from != kNone && (!a->gate || a->ld_gate < a->ld || a->ld_gate % 4 || a->row_idx)) || (a->mixture && a->branch[0]) || (from == kTwo && (!a->branch[0] || !a->branch_gain[0] || !a->branch_gain[1])) ||
      (a->mixture && (!a->mixture->rows || !a->mixture->pair_row || !a->mixture->weights || a->mixture->n_pairs <= 0 || a->mixture->top < 0 || a->mixture->top > a->mixture->n_pairs)) ||
      (a->embed && (!a->ids || a->vocab <= 0)) || (a->row_idx && (a->embed || a->step || a->kept)) ||
      (((uintptr_t)a->x | (uintptr_t)a->branch[0] | (uintptr_t)a->branch[1] | (uintptr_t)a->branch_gain[0] | (uintptr_t)a->branch_gain[1] | (uintptr_t)a->gate | (uintptr_t)a->kept |
        (uintptr_t)a->embed | (uintptr_t)a->step | (uintptr_t)a->h) & 15))
    return lg::kInvalidValue;
  Args p{(float4*)a->x, {(float4*)a->branch[0], (float4*)a->branch[1]}, a->zero_branches, {(const float4*)a->branch_gain[0], (const float4*)a->branch_gain[1]}};
  if (a->mixture) {
    const lg_mixture_out_t& x = *a->mixture;
    p.expert_rows = x.rows; p.pair_row = (const int*)x.pair_row; p.weights = (const float*)x.weights; p.n_pairs = x.n_pairs; p.top = x.top; p.counts = (int*)x.counts; p.n_counts = x.n_counts;
  }
  p.gate = a->gate; p.ld_gate = a->ld_gate; p.kept = (float4*)a->kept; p.embed = a->embed; p.ids = (const uint32_t*)a->ids; p.step = (const float4*)a->step; p.vocab = a->vocab;
  p.h = a->h; p.gain = a->gain; p.eps = a->eps; p.row_idx = (const int*)a->row_idx; p.n_src_rows = a->n_src_rows; p.n = a->n; p.nv = a->ld / 4; p.f32 = a->is_f32; p.status = (int*)status;
  int nv = 1;
  const int most = a->rows > 512 && p.nv <= 256 * kMaxVec ? 256 : kMaxThreads;   // many rows: smaller CTAs with more in flight per thread
  while (p.nv > most * nv) nv *= 2;
  const int threads = ((p.nv + nv - 1) / nv + 31) / 32 * 32;
  auto go = [&](auto kern) -> uint32_t {
    lg::launch(kern, dim3((unsigned)a->rows), dim3((unsigned)threads), 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
#define LG_FROM(NV) (from == kNone ? go(gated_residual_kernel<NV, kNone>) : from == kOne ? go(gated_residual_kernel<NV, kOne>) : from == kTwo ? go(gated_residual_kernel<NV, kTwo>) \
                                                                                                                               : go(gated_residual_kernel<NV, kMixture>))
  return nv == 1 ? LG_FROM(1) : nv == 2 ? LG_FROM(2) : nv == 4 ? LG_FROM(4) : LG_FROM(8);
#undef LG_FROM
}

uint32_t logismos_launch_attention_difference(const void* a, int32_t ld_a, void* out, int32_t ld_out, int32_t is_f32, int32_t rows, int32_t heads, int32_t n_kv, int32_t v,
                                              int32_t vp, float lambda, float scale, float eps, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!a || !out || rows <= 0 || heads <= 0 || n_kv <= 0 || heads % n_kv || v <= 0 || v > vp || vp > 256 || vp % 4 || ld_a < 2 * heads * vp || ld_a % 4 || ld_out < heads * vp ||
      ld_out % 4 || (((uintptr_t)a | (uintptr_t)out) & 15))
    return lg::kInvalidValue;
  const int64_t blocks = ((int64_t)rows * heads + 7) / 8;
  if (blocks > 0x7fffffff) return lg::kInvalidValue;
  const dim3 grid((unsigned)blocks);
  if (is_f32) lg::launch(attention_difference_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)a, ld_a, (float*)out, ld_out, rows, heads, heads / n_kv, v, vp, lambda, scale, eps);
  else lg::launch(attention_difference_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, (const float*)a, ld_a, (__nv_bfloat16*)out, ld_out, rows, heads, heads / n_kv, v, vp, lambda, scale, eps);
  return lg::launch_status();
}

}  // extern "C"
