// Norms that compute no statistics, tanh(alpha x) w + b, around the sublayers of a residual stack (fp32 stream):
//   x += post(y);  h = next(x)
// y is a sublayer's output, or the rows of a mixture of experts still to be summed with their weights. Everything is
// elementwise: a thread owns four columns of a few rows, the norms' vectors stay in registers.
#include "common.cuh"
#include "logismos_kernels.h"

namespace {

using namespace lg;

constexpr int kThreads = 128;

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
LG_DEVINL float4 norm4(float4 v, float alpha, float4 w, float4 b) {
  return make_float4(fmaf(tanhf(alpha * v.x), w.x, b.x), fmaf(tanhf(alpha * v.y), w.y, b.y), fmaf(tanhf(alpha * v.z), w.z, b.z),
                     fmaf(tanhf(alpha * v.w), w.w, b.w));
}
LG_DEVINL void add_scaled(float4& s, float w, float4 v) {
  s.x = fmaf(w, v.x, s.x); s.y = fmaf(w, v.y, s.y); s.z = fmaf(w, v.z, s.z); s.w = fmaf(w, v.w, s.w);
}

struct NormVec { float alpha; const float4 *w, *b; };  // w NULL: absent

struct Args {
  float4* y;
  int zero_y;
  const int* row_idx;
  int n_src_rows;
  float4* x;
  NormVec post, next;
  void* h;
  int f32, rows, nv;
  unsigned cols;  // CTAs per row
  // mixture
  const void* expert_rows;
  const int* pair_row;
  const float* weights;
  const float* identity;
  int n_pairs, top;
  int* counts;
  int n_counts;
  int* status;
};

// BATCH: 0, or rows of experts that a thread has in flight. They lie at scattered places, so many rows of tokens want as
// many threads as the SM takes (MANY) rather than many requests in each.
template <int BATCH, bool MANY, int RUN>
__global__ void __launch_bounds__(kThreads, BATCH && MANY ? 16 : 1)
tanh_norm_kernel(Args p) {
  constexpr bool MIX = BATCH != 0;
  lg::pdl_trigger();
  const int v = (int)(blockIdx.x % p.cols) * kThreads + threadIdx.x, r0 = (int)(blockIdx.x / p.cols) * RUN;
  const bool in = v < p.nv;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 w1 = zero, b1 = zero, w2 = zero, b2 = zero;
  const auto vectors = [&] {
    if (p.post.w) { w1 = __ldg(p.post.w + v); b1 = __ldg(p.post.b + v); }
    if (p.next.w) { w2 = __ldg(p.next.w + v); b2 = __ldg(p.next.b + v); }
  };
  if (!(MIX && MANY) && in) vectors();  // they do not depend on the kernels before this one
  lg::pdl_wait();
  if (MIX && blockIdx.x == 0 && p.counts)
    for (int g = threadIdx.x; g < p.n_counts; g += kThreads) p.counts[g] = 0;
  if (!in) return;
  float4 x[RUN], y[RUN];
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int r = r0 + i;
    x[i] = y[i] = zero;
    if (r >= p.rows) continue;
    int src = p.row_idx ? p.row_idx[r] : r;
    if (src < 0 || src >= p.n_src_rows) {
      if (v == 0 && p.status) atomicExch(p.status, 1);
      src = 0;
    }
    x[i] = p.x[(size_t)src * p.nv + v];
    if (!MIX && p.post.w) y[i] = p.y[(size_t)r * p.nv + v];
  }
  if (MIX) {
    // a few experts of every row at a time: first where their rows are, then all of these at once
    constexpr int kBatch = BATCH ? BATCH : 1;
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      const int r = r0 + i;
      const float id = r < p.rows ? p.identity[r] : 0.0f;
      if (id != 0.0f) add_scaled(y[i], id, load4(p.h, (size_t)r * p.nv + v, p.f32));
    }
    for (int k0 = 0; k0 < p.n_pairs; k0 += kBatch) {
      int row[RUN][kBatch];
      float w[RUN][kBatch];
#pragma unroll
      for (int i = 0; i < RUN; ++i)
#pragma unroll
        for (int j = 0; j < kBatch; ++j) {
          const int r = r0 + i, k = k0 + j;
          const bool ok = r < p.rows && k < p.n_pairs;
          row[i][j] = ok ? p.pair_row[(size_t)r * p.n_pairs + k] : -1;
          w[i][j] = ok && k < p.top ? p.weights[(size_t)r * p.top + k] : 1.0f;
        }
      float4 e[RUN][kBatch];
#pragma unroll
      for (int i = 0; i < RUN; ++i)
#pragma unroll
        for (int j = 0; j < kBatch; ++j) e[i][j] = row[i][j] >= 0 ? load4(p.expert_rows, (size_t)row[i][j] * p.nv + v, p.f32) : zero;
#pragma unroll
      for (int i = 0; i < RUN; ++i)
#pragma unroll
        for (int j = 0; j < kBatch; ++j) add_scaled(y[i], w[i][j], e[i][j]);
    }
    if (MANY) vectors();
  }
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int r = r0 + i;
    if (r >= p.rows) continue;
    const size_t at = (size_t)r * p.nv + v;
    float4 o = x[i];
    if (p.post.w) {
      const float4 d = norm4(y[i], p.post.alpha, w1, b1);
      o.x += d.x; o.y += d.y; o.z += d.z; o.w += d.w;
      p.x[at] = o;
      if (!MIX && p.zero_y) p.y[at] = zero;
    }
    if (p.next.w) store4(p.h, at, norm4(o, p.next.alpha, w2, b2), p.f32 != 0);
  }
}

NormVec vec(const lg_tanh_norm_t* n) { return n ? NormVec{n->alpha, (const float4*)n->w, (const float4*)n->b} : NormVec{0.0f, nullptr, nullptr}; }

}  // namespace

extern "C" uint32_t logismos_launch_tanh_norm(void* y, int32_t zero_y, const lg_mixture_out_t* mix, const void* row_idx, int32_t n_src_rows, void* x,
                                              const lg_tanh_norm_t* post, void* h, const lg_tanh_norm_t* next, int32_t out_f32, int32_t rows, int32_t ld,
                                              void* status, void* stream) {
  lg::LaunchScope launch_scope_;
  if (rows <= 0 || ld <= 0 || ld % 4 || !x || n_src_rows <= 0 || (!row_idx && rows > n_src_rows) || (!post && !next) || (row_idx && post) || (next && !h) ||
      (post && (!post->w || !post->b || (!y && !mix))) || (next && (!next->w || !next->b)) || (mix && (!post || !h || !mix->rows || !mix->pair_row || !mix->weights || !mix->identity || mix->n_pairs <= 0 ||
                                                                              mix->top < 0 || mix->top > mix->n_pairs)) ||
      (((uintptr_t)x | (uintptr_t)y | (uintptr_t)h) & 15))
    return lg::kInvalidValue;
  Args p{(float4*)y, zero_y, (const int*)row_idx, n_src_rows, (float4*)x, vec(post), vec(next), h, out_f32, rows, ld / 4, (unsigned)(ld / 4 + kThreads - 1) / kThreads};
  p.status = (int*)status;
  if (mix) {
    p.expert_rows = mix->rows; p.pair_row = (const int*)mix->pair_row; p.weights = (const float*)mix->weights; p.identity = (const float*)mix->identity;
    p.n_pairs = mix->n_pairs; p.top = mix->top; p.counts = (int*)mix->counts; p.n_counts = mix->n_counts;
  }
  const bool many = (int64_t)p.cols * rows >= 148 * 16;
  auto go = [&](auto kern, int per) -> uint32_t {
    const int64_t blocks = ((int64_t)rows + per - 1) / per * p.cols;
    if (blocks > INT32_MAX) return lg::kInvalidValue;
    lg::launch(kern, dim3((unsigned)blocks), dim3(kThreads), 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
  if (mix) return many ? go(tanh_norm_kernel<3, true, 1>, 1) : go(tanh_norm_kernel<4, false, 1>, 1);
  return many ? go(tanh_norm_kernel<0, true, 4>, 4) : go(tanh_norm_kernel<0, false, 1>, 1);
}
