// What the attention kernels share beyond the plain softmax: scores that are capped and biased by distance, with an
// output gate per channel (lg_score_bias_t), and windows: sliding or by chunks, with kept first keys or with blocks of
// tokens pooled behind them, one added to the softmax denominator and an output gate per head (lg_window_t).
#pragma once
#include <cmath>

#include "common.cuh"
#include "logismos_kernels.h"

namespace lg {

// 1 - 2 / (1 + e^(2x)), for x in units in which e^(2x) = 2^x: absolute error of a few 1e-7 over the whole range
LG_DEVINL float tanh_from_exp2(float x2) { return 1.0f - __fdividef(2.0f, 1.0f + fast_exp2(x2)); }

// What turns a product q . k into a score in log2 units, and what becomes of the attention output (lg_score_bias_t)
struct ScoreExt {
  const float* bias;             // [heads][far + 1]
  int far;
  float pre, post;               // capped: post tanh(.) + bias with the exponent pre q . k; else post q . k + bias
  int capped;
  float poly[5];                 // post tanh(.) as q . k (poly[0] + poly[1] s + ...) with s = (q . k)^2, where products are bounded
  const __nv_bfloat16* gate;
  int ld_gate;
  float gate_scale;
  int ld_q, ld_out;
  LG_DEVINL float score(float qk, float b) const { return fmaf(post, capped ? tanh_from_exp2(qk * pre) : qk, b); }
  LG_DEVINL float score_poly(float qk, float b) const {
    const float s = qk * qk;
    return fmaf(qk, fmaf(fmaf(fmaf(fmaf(poly[4], s, poly[3]), s, poly[2]), s, poly[1]), s, poly[0]), b);
  }
  LG_DEVINL float gated(float o, float g) const { return o * __fdividef(gate_scale, 1.0f + __expf(-g)); }
};

constexpr int kRawPartial = 2;

// The window form: where a query at position i looks, and what becomes of its output. What stands ahead of the window, kept
// first keys or pooled blocks, is numbered through with it: `lead` of them, then the window's keys from a place rounded down.
struct WindowExt {
  int size, keep, sink, chunked, pool;   // size INT_MAX: all keys
  const float* gate;             // [rows, ld_gate], NULL: none
  int ld_gate;
  int ld_q, ld_out;
  int raw;                       // the output is fp32 (kRawPartial: decode leaves all partial results to another merge)
  const void *kmean, *vmean;     // pooled keys and values, mean_rows() of them per cache block
  // first key of the window
  __host__ __device__ int first(int i) const { return chunked ? i - i % size : i < size ? 0 : i - size + 1; }
  LG_DEVINL bool sees(int i, int j) const { return j <= i && (j >= first(i) || j < keep); }
  // pooled blocks that lie wholly before the window
  __host__ __device__ int pooled(int i) const { return pool && i >= size ? (i - size + 1) / pool : 0; }
  // a pooled block is kept with the cache block that holds its last token
  __host__ __device__ int mean_rows() const { return (15 + pool) / pool; }
  LG_DEVINL int mean_block(int b) const { return ((b + 1) * pool - 1) >> 4; }
  LG_DEVINL int mean_row(int b) const { return b - (mean_block(b) << 4) / pool; }
  LG_DEVINL float head_gate(size_t row, int head) const { return gate ? 1.0f / (1.0f + __expf(-gate[row * ld_gate + head])) : 1.0f; }
  // leading blocks of 16 for the last of `ctx` tokens, and the distance by which the blocks after them are renumbered
  __host__ __device__ int lead_blocks(int ctx) const { return ((pool ? pooled(ctx - 1) : keep) + 15) / 16; }
  __host__ __device__ int gap_blocks(int ctx) const {
    const int gap = first(ctx - 1) / 16 - lead_blocks(ctx);
    return pool || gap > 0 ? gap : 0;
  }
  // the same of a prompt launch's gather, for queries at the last q_len of kv_len positions: leading rows come in tiles of
  // 128, the window of the first query begins at a multiple of 8
  __host__ __device__ int lead_keys(int kv_len) const { return ((pool ? pooled(kv_len - 1) : keep) + 127) / 128 * 128; }
  __host__ __device__ int gap_keys(int kv_len, int q_len) const {
    const int gap = (first(kv_len - q_len) & ~7) - lead_keys(kv_len);
    return pool || gap > 0 ? gap : 0;
  }
};

inline bool window_ok(const lg_window_t* w, int heads) {
  return w && w->scale > 0.0f && w->size >= 0 && w->keep_first >= 0 && w->keep_first < (1 << 30) && (!w->gate || w->ld_gate >= heads) && w->pool >= 0 &&
         (!(w->chunked || w->pool) || (w->size > 0 && !w->keep_first)) && !(w->chunked && w->pool) &&
         (!w->pool || (w->k_mean && w->v_mean && (((uintptr_t)w->k_mean | (uintptr_t)w->v_mean) & 15) == 0));
}
inline WindowExt window_ext(const lg_window_t* w, int ld_q, int ld_out) {
  return WindowExt{w->size ? w->size : 0x7fffffff, w->keep_first, w->sink, w->chunked, w->pool, (const float*)w->gate, w->ld_gate, ld_q, ld_out, w->out_f32 ? 1 : 0, w->k_mean, w->v_mean};
}

inline bool score_ok(const lg_score_bias_t* s, int width) {
  return s && s->scale > 0.0f && s->cap >= 0.0f && s->bias && s->far >= 0 && s->gate && s->ld_gate >= width;
}

// The polynomial above by interpolation of tanh(x) / x in x^2 at Chebyshev nodes on [0, limit^2]: for limit <= 0.7 within
// 2e-7 of it. False: products may be too large, and nothing is set.
inline bool fit_score_poly(const lg_score_bias_t* s, ScoreExt* e) {
  const double x_max = (double)s->max_abs_qk * s->scale / (s->cap > 0.0f ? s->cap : 1.0f);
  if (!(s->cap > 0.0f) || !(s->max_abs_qk > 0.0f) || x_max > 0.7) return false;
  const int n = 5;
  const double U = x_max * x_max, pi = 3.14159265358979323846;
  double node[n], coef[n];  // Newton's divided differences
  for (int i = 0; i < n; ++i) {
    node[i] = 0.5 * U * (1.0 + std::cos(pi * (2 * i + 1) / (2 * n)));
    const double x = std::sqrt(node[i]);
    coef[i] = x > 1e-9 ? std::tanh(x) / x : 1.0;
  }
  for (int k = 1; k < n; ++k)
    for (int i = n - 1; i >= k; --i) coef[i] = (coef[i] - coef[i - 1]) / (node[i] - node[i - k]);
  double p[n] = {coef[n - 1], 0, 0, 0, 0};  // to powers of u
  for (int k = n - 2; k >= 0; --k) {
    for (int i = n - 1; i > 0; --i) p[i] = p[i - 1] - node[k] * p[i];
    p[0] = coef[k] - node[k] * p[0];
  }
  const double a = (double)s->scale / s->cap;  // x = a q.k
  double f = (double)s->cap * 1.4426950408889634 * a;
  for (int i = 0; i < n; ++i, f *= a * a) e->poly[i] = (float)(p[i] * f);
  return true;
}

inline ScoreExt score_ext(const lg_score_bias_t* s, int ld_q, int ld_out) {
  const float log2e = 1.4426950408889634f;
  ScoreExt e{};
  e.bias = (const float*)s->bias;
  e.far = s->far;
  e.capped = s->cap > 0.0f ? 1 : 0;
  e.pre = e.capped ? 2.0f * log2e * s->scale / s->cap : 0.0f;
  e.post = e.capped ? s->cap * log2e : s->scale * log2e;
  e.gate = (const __nv_bfloat16*)s->gate;
  e.ld_gate = s->ld_gate;
  e.gate_scale = s->gate_scale;
  e.ld_q = ld_q;
  e.ld_out = ld_out;
  return e;
}

}  // namespace lg
