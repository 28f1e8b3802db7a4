// Scores that are capped and biased by distance, and the output gate, shared by the attention kernels
// (lg_score_bias_t).
#pragma once
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
  const __nv_bfloat16* gate;
  int ld_gate;
  float gate_scale;
  int ld_q, ld_out;
  LG_DEVINL float score(float qk, float b) const { return fmaf(post, capped ? tanh_from_exp2(qk * pre) : qk, b); }
  LG_DEVINL float gated(float o, float g) const { return o * __fdividef(gate_scale, 1.0f + __expf(-g)); }
};

inline bool score_ok(const lg_score_bias_t* s, int width) {
  return s && s->scale > 0.0f && s->cap >= 0.0f && s->bias && s->far >= 0 && s->gate && s->ld_gate >= width;
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
