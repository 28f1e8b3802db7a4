// Host-side executor of one continuous-batching step over a stack of mixers and feed-forwards; see lg_mixer_* in
// logismos_model.h and mixer_stack.h. The contract is that of the other executors: a packed step equals running every
// sequence alone.
//
// A step packs decode tokens first and prefill chunks after them (step_batch.h):
//   embed -> per layer
//     mixer (mixer_parallel.cu, mixer_gated.cu, mixer_paired.cu) -> output GEMM
//     norm + residual + the next sublayer's input; feed-forward likewise (a mixture's sum rides in that norm)
//   -> wanted rows: final norm -> head (fp32) -> greedy argmax
// Every matrix is padded at load with zeros (inputs and outputs to multiples of 64, heads to powers of two), which
// keeps the padding of every activation zero.
#include "mixer_stack.h"

namespace lgm {

void MWeights::release() {
  Buf* wb[] = {&norm1, &norm1_b, &norm2, &norm2_b, &w_up, &w_down, &w_in, &w_out, &pre1.w, &pre1.b, &post1.w, &post1.b, &pre2.w, &pre2.b, &post2.w, &post2.b,
               &conv, &conv_b, &dt_bias, &A_log, &D, &gain, &bias, &mu, &w2, &w0, &u, &b_in, &gain_q, &gain_k, &w_uq, &w_uk, &w_ukt, &w_uv, &w_router, &correction,
               &w_gate2, &b_gate2, &w_out2, &branch_gain[0], &branch_gain[1], &decay};
  for (Buf* b : wb) b->release();
}

bool zeroed(Buf& b, size_t bytes) { return b.alloc(bytes) && (bytes == 0 || cudaMemset(b.p, 0, bytes) == cudaSuccess); }

uint32_t linear(Mixer* m, const void* a, int lda, const Buf& w, int n, int k, void* out, int ldc, int epi, int rows, cudaStream_t s, const Buf* bias) {
  m->launches += 1;
  const void* b = bias ? bias->p : nullptr;
  if (m->cfg.is_f32) {
    if (epi == LG_EPI_SWIGLU)  // the clamped form without its limit
      return logismos_launch_linear_f32(a, w.p, b, out, rows, n, k, lda, ldc, 1, 0, 0, 0, LG_EPI_GLU_CLAMP, 1.0f, INFINITY, 0.0f, s);
    return logismos_launch_linear_f32(a, w.p, b, out, rows, n, k, lda, ldc, 1, 0, 0, 0, epi == LG_EPI_BF16 ? (int)LG_EPI_F32 : epi, 0, 0, 0, s);
  }
  if (stream_weights(rows, n, k, epi))
    return logismos_launch_linear_small_bf16(a, w.p, b, out, rows, n, k, lda, ldc, 1, 0, 0, 0, epi, 0, 0, 0, s);
  return logismos_launch_linear_t_act_bf16(a, w.p, b, out, rows, n, k, lda, ldc, epi | LG_EPI_STATIC_W, 0, 0, 0, m->status.p, s);
}

uint32_t head_linear(Mixer* m, const void* a, int lda, const Buf& w, int heads, int n, int k, void* out, int ldc, int rows, cudaStream_t s) {
  m->launches += 1;
  if (m->cfg.is_f32)
    return logismos_launch_linear_f32(a, w.p, nullptr, out, rows, n, k, lda, ldc, heads, k, (int64_t)n * k, n, LG_EPI_F32, 0, 0, 0, s);
  return logismos_launch_linear_small_bf16(a, w.p, nullptr, out, rows, n, k, lda, ldc, heads, k, (int64_t)n * k, n, LG_EPI_BF16, 0, 0, 0, s);
}

// Whether an input projection of a few dozen rows is summed over slices of k, with a launch that finishes it: its tiles alone
// would leave most SMs idle (3088 x 2048 at 64 rows: 16.1 us in tiles; summed 5.2, finished 2.5)
bool splits_projections(const lg_linear_groups_t& g, int n, int rows) { return g.n_groups == 1 && rows > 32 && rows <= kAccRows && (n + 127) / 128 * ((rows + 127) / 128) <= 74; }

uint32_t grouped_projection(Mixer* m, const Buf& w, int n, const lg_linear_groups_t& g, cudaStream_t s) {
  m->launches += 1;
  const int Hp = m->Hp, rows = m->batch.T;
  if (m->cfg.is_f32) return logismos_launch_linear_groups_f32(m->h.p, w.p, m->proj.p, rows, n, Hp, Hp, g.n_main, &g, s);
  if (splits_projections(g, n, rows) && m->accumulates(rows)) {
    m->launches += 1;
    if (uint32_t rc = logismos_launch_linear_t_act_bf16(m->h.p, w.p, nullptr, m->raw_acc.p, rows, n, Hp, Hp, n, LG_EPI_RESID_F32 | LG_EPI_STATIC_W, 0, 0, 0, m->status.p, s)) return rc;
    return logismos_launch_linear_groups_finish(m->raw_acc.p, m->proj.p, rows, n, n, g.n_main, &g, s);
  }
  if (stream_weights(rows, n, Hp, LG_EPI_BF16)) return logismos_launch_linear_groups_small_bf16(m->h.p, w.p, m->proj.p, rows, n, Hp, Hp, g.n_main, &g, s);
  return logismos_launch_linear_groups_tc_bf16(m->h.p, w.p, m->proj.p, rows, n, Hp, Hp, g.n_main, &g, m->status.p, s);
}

uint32_t projections(Mixer* m, const MLayer& L, const MWeights& W, bool tail_parts, cudaStream_t s) {
  lg_linear_groups_t g = L.groups;
  g.tail = m->tail.p;
  g.tail_parts = tail_parts ? m->low2.p : nullptr;
  g.bias = W.b_in.p;
  return grouped_projection(m, W.w_in, L.N, g, s);
}

// rows of head h of src [heads * d, k] -> rows of dst at row0 + h * dp
void head_rows(Mat& dst, int row0, const void* src, int heads, int d, int dp, int k) {
  for (int h = 0; h < heads; ++h)
    for (int i = 0; i < d; ++i) dst.row(row0 + h * dp + i, 0, src, ((size_t)h * d + i) * k, k);
}
// columns of head h of src [n, heads * d] -> columns of dst at col0 + h * dp
void head_cols(Mat& dst, int col0, const void* src, int n, int heads, int d, int dp) {
  for (int i = 0; i < n; ++i)
    for (int h = 0; h < heads; ++h) dst.row(i, col0 + h * dp, src, ((size_t)i * heads + h) * d, d);
}

}  // namespace lgm

namespace {

using namespace lgm;

// Output projection of a sublayer, its norm and the residual, then the inputs of what follows: `next` is the layer
// whose mixer reads the stream (kPlain: a feed-forward, kNone: nothing).
constexpr int kNone = -1, kPlain = -2;

uint32_t shift_inputs(Mixer* m, MLayer& N, const MWeights& NW, cudaStream_t s) {
  StepBatch& B = m->batch;
  m->launches += 1;
  return logismos_launch_token_shift(m->x.p, m->h.p, m->cfg.is_f32, NW.mu.p, kMixes, N.shift.p, m->dev(B.state), m->dev(B.fresh), m->dev(B.phase),
                                     m->dev(B.seq_ids), m->dev(B.cu), B.T, m->Hp, s);
}

uint32_t norm_and_inputs(Mixer* m, void* y, int zero_y, const Buf* w, const Buf* b, int next, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const void *wp = w ? w->p : nullptr, *bp = b ? b->p : nullptr;
  const bool shift = next >= 0 && m->layers[(size_t)next].c.kind == LG_MIXER_PARALLEL;
  if (shift && B.n_pre == 0) {
    MLayer& N = m->layers[(size_t)next];
    m->launches += 1;
    return logismos_launch_post_norm_shift_decode(y, zero_y, m->x.p, wp, bp, m->h.p, c.is_f32, m->weights[(size_t)N.owner].mu.p, kMixes, N.shift.p,
                                                  m->dev(B.state), m->dev(B.fresh), m->dev(B.phase), B.T, c.width, m->Hp, c.norm_eps, s);
  }
  if (w || (next != kNone && !shift)) {
    m->launches += 1;
    if (uint32_t rc = logismos_launch_post_norm(y, zero_y, nullptr, B.T, m->x.p, wp, bp, shift || next == kNone ? nullptr : m->h.p, c.is_f32, B.T, c.width,
                                                m->Hp, c.norm_eps, m->status.p, s))
      return rc;
  }
  if (!shift) return 0;
  MLayer& N = m->layers[(size_t)next];
  return shift_inputs(m, N, m->weights[(size_t)N.owner], s);
}

// x += post(y) (or the sum of a mixture), then the next sublayer's input
uint32_t tanh_norms(Mixer* m, void* y, bool zero_y, const lg_mixture_out_t* mix, const TanhNorm* post, const TanhNorm* next, cudaStream_t s) {
  lg_tanh_norm_t a, b;
  if (post) a = post->view();
  if (next) b = next->view();
  m->launches += 1;
  return logismos_launch_tanh_norm(y, zero_y, mix, nullptr, m->batch.T, m->x.p, post ? &a : nullptr, m->h.p, next ? &b : nullptr, m->cfg.is_f32, m->batch.T, m->Hp,
                                   m->status.p, s);
}

// the norm of a sublayer's output, and that of the next sublayer's input (NULL: none)
void norms_after(Mixer* m, int l, bool second, const TanhNorm** post, const TanhNorm** next) {
  const MWeights& W = m->weights[(size_t)m->layers[(size_t)l].owner];
  *post = second ? &W.post2 : &W.post1;
  *next = !second && m->layers[(size_t)l].c.ff > 0 ? &W.pre2 : l + 1 < m->cfg.n_layers ? &m->weights[(size_t)m->layers[(size_t)l + 1].owner].pre1 : nullptr;
}

// Gated RMS stack. What precedes the norm of layer `next` (the last one's end: nothing): the embedding again and the
// vector of the pass that begins there
void begin_layer(Mixer* m, int next, lg_gated_residual_t* a) {
  if (next >= m->cfg.n_layers) return;
  const int pass = m->layer_cfg[(size_t)next].pass;
  if (pass > 1) { a->embed = m->embed.p; a->ids = m->dev(m->batch.ids); a->vocab = m->cfg.vocab; }
  if (pass > 0) a->step = (const float*)m->loop_step.p + (size_t)(pass - 1) * m->Hp;
  a->h = m->h.p;
  a->gain = m->weights[(size_t)m->layers[(size_t)next].owner].gain1;
}

lg_gated_residual_t residual_args(Mixer* m) {
  lg_gated_residual_t a{};
  a.x = m->x.p; a.eps = m->cfg.norm_eps; a.rows = a.n_src_rows = m->batch.T; a.n = m->cfg.width; a.ld = m->Hp; a.is_f32 = m->cfg.is_f32;
  return a;
}

// The residual after a sublayer of layer l and the input of the next one; y: its branches one after the other, or mix
uint32_t gated_residual(Mixer* m, int l, bool second, void* y, bool zero_y, const lg_mixture_out_t* mix, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  const MLayer& L = m->layers[(size_t)l];
  const MWeights& W = m->weights[(size_t)L.owner];
  lg_gated_residual_t a = residual_args(m);
  const size_t esz = c.is_f32 ? 4 : 2;
  a.branch[0] = y; a.zero_branches = zero_y; a.mixture = mix;
  if (!second && L.c.kind == LG_MIXER_PAIR) {
    a.branch[1] = (float*)y + (zero_y ? m->acc_bytes / 8 : (size_t)c.max_step_tokens * m->Hp);
    a.branch_gain[0] = W.branch_gain[0].p; a.branch_gain[1] = W.branch_gain[1].p;
  }
  a.gate = second ? m->proj.p : (uint8_t*)m->proj.p + (size_t)L.off_gate * esz;
  a.ld_gate = second ? L.gate2.n_main : L.groups.n_main;
  if (!second && L.c.ff > 0) {
    a.h = m->h.p;
    a.gain = W.gain2;
  } else {
    if (c.keep_layers) a.kept = (float*)m->hist.p + (size_t)(l + 1) * c.max_step_tokens * m->Hp;
    begin_layer(m, l + 1, &a);
  }
  m->launches += 1;
  return logismos_launch_gated_residual(&a, m->status.p, s);
}

constexpr int kStreamRows = 16;   // up to so many rows the output projections of a gated stack stream their weights (us, small / tiles that split k: 1024 x 1024 2.6 / 4.8, 4096 x 4096 8.9 / 10.8)
constexpr int kFusedNormRows = 16;   // up to so many rows the norms around the residual ride on the output projection

// What follows a sublayer of layer l: the norm of its output y, the residual, and the input of the next sublayer.
// second: the feed-forward; mix: instead of y.
uint32_t finish_sublayer(Mixer* m, int l, bool second, void* y, bool zero_y, const lg_mixture_out_t* mix, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  const MWeights& W = m->weights[(size_t)m->layers[(size_t)l].owner];
  const bool ff_next = !second && m->layers[(size_t)l].c.ff > 0;
  const int next = l + 1 < c.n_layers ? l + 1 : kNone;
  if (c.norm == LG_NORM_LAYER_POST)
    return norm_and_inputs(m, y, zero_y, second ? &W.norm2 : &W.norm1, second ? &W.norm2_b : &W.norm1_b, ff_next ? kPlain : next, s);
  if (c.norm == LG_NORM_RMS_GATED) return gated_residual(m, l, second, y, zero_y, mix, s);
  const TanhNorm *post, *in;
  norms_after(m, l, second, &post, &in);
  return tanh_norms(m, y, zero_y, mix, post, in, s);
}

uint32_t output_projection(Mixer* m, int l, bool second, const void* a, int k, const Buf& w, cudaStream_t s) {
  const int T = m->batch.T, Hp = m->Hp;
  const bool acc = m->accumulates(T) && !(m->cfg.norm == LG_NORM_RMS_GATED && T <= kStreamRows);
  void* y = acc ? m->y_acc.p : m->y.p;
  if (m->cfg.norm == LG_NORM_TANH_AROUND && !m->cfg.is_f32 && T <= kFusedNormRows) {  // the norms in the product's epilogue
    const TanhNorm *post, *next;
    norms_after(m, l, second, &post, &next);
    const lg_tanh_norm_t p = post->view(), n = next ? next->view() : lg_tanh_norm_t{};
    m->launches += 1;
    LG_TRY(logismos_launch_linear_small_tanh_norm(a, w.p, m->x.p, &p, m->h.p, next ? &n : nullptr, T, Hp, k, k, Hp, s), "output projection with norms");
    return 0;
  }
  LG_TRY(linear(m, a, k, w, Hp, k, y, Hp, acc ? LG_EPI_RESID_F32 : LG_EPI_F32, T, s), "output projection");
  LG_TRY(finish_sublayer(m, l, second, y, acc, nullptr, s), "output norm");
  return 0;
}

// of a mixer: the output projection, or those of a pair
uint32_t mixer_output(Mixer* m, int l, cudaStream_t s) {
  const MLayer& L = m->layers[(size_t)l];
  const MWeights& W = m->weights[(size_t)L.owner];
  if (L.c.kind != LG_MIXER_PAIR) return output_projection(m, l, false, m->act.p, L.Kout, W.w_out, s);
  const int T = m->batch.T, Hp = m->Hp;
  const bool acc = m->accumulates(T) && T > kStreamRows, both = L.Kout == 2 * L.Kleft;
  float *y = (float*)(acc ? m->y_acc.p : m->y.p), *y2 = y + (acc ? m->acc_bytes / 8 : (size_t)m->cfg.max_step_tokens * Hp);
  const int epi = acc ? LG_EPI_RESID_F32 : LG_EPI_F32;
  if (both && !m->cfg.is_f32 && T <= kStreamRows) {
    LG_TRY(logismos_launch_linear_small_bf16(m->act.p, W.w_out.p, nullptr, y, T, Hp, L.Kleft, L.Kout, Hp, 2, L.Kleft, (int64_t)Hp * L.Kleft, y2 - y, LG_EPI_F32, 0, 0, 0, s),
           "output projections");
    m->launches += 1;
  } else {
    LG_TRY(linear(m, m->act.p, L.Kout, W.w_out, Hp, L.Kleft, y, Hp, epi, T, s), "left output projection");
    const void* right = (const uint8_t*)m->act.p + (size_t)L.Kleft * (m->cfg.is_f32 ? 4 : 2);
    Buf second = W.w_out2;
    if (both) second.p = (uint16_t*)W.w_out.p + (size_t)Hp * L.Kleft;
    LG_TRY(linear(m, right, L.Kout, second, Hp, L.Kout - L.Kleft, y2, Hp, epi, T, s), "right output projection");
  }
  LG_TRY(finish_sublayer(m, l, false, y, acc, nullptr, s), "output norm");
  return 0;
}

uint32_t run_mixer(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  if (is_paired_kind(L.c.kind)) return run_paired_kinds(m, L, W, s);
  if (is_gated_kind(L.c.kind)) return run_gated_kinds(m, L, W, s);
  LG_TRY(projections(m, L, W, L.c.kind == LG_MIXER_PARALLEL && m->batch.n_pre > 0, s), "input projections");
  return L.c.kind == LG_MIXER_SSD ? run_ssd(m, L, W, s) : run_parallel(m, L, W, s);
}

uint32_t run_feed_forward(Mixer* m, int l, cudaStream_t s) {
  const MLayer& L = m->layers[(size_t)l];
  const MWeights& W = m->weights[(size_t)L.owner];
  const int T = m->batch.T, Hp = m->Hp;
  if (m->cfg.norm == LG_NORM_RMS_GATED) {
    lg_linear_groups_t g = L.gate2;
    g.tail = m->route.p;
    g.bias = W.b_gate2.p;
    LG_TRY(grouped_projection(m, W.w_gate2, g.end[0], g, s), "gate and router");
  }
  if (L.c.ff_kind == LG_FF_MIXTURE) {
    lg_mixture_out_t mix;
    if (uint32_t rc = run_mixture(m, L, W, &mix, s)) return rc;
    LG_TRY(finish_sublayer(m, l, true, nullptr, false, &mix, s), "sum of the experts and output norm");
    return 0;
  }
  if (L.c.ff_kind == LG_FF_GATED) LG_TRY(linear(m, m->h.p, Hp, W.w_up, 2 * L.Fp, Hp, m->ffb.p, L.Fp, LG_EPI_SWIGLU, T, s), "feed-forward");
  else LG_TRY(linear(m, m->h.p, Hp, W.w_up, L.Fp, Hp, m->ffb.p, L.Fp, LG_EPI_RELU2, T, s), "feed-forward");
  return output_projection(m, l, true, m->ffb.p, L.Fp, W.w_down, s);
}

uint32_t run_device(Mixer* m, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int Hp = m->Hp, T = B.T, f32 = c.is_f32;
  void* st = m->status.p;
  m->launches = 1;
  if (m->acc_dirty) {
    const struct { const Buf* b; size_t bytes; } sums[] = {{&m->y_acc, m->acc_bytes}, {&m->raw_acc, m->raw_acc_bytes}, {&m->route_acc, m->route_acc_bytes}, {&m->counts, m->counts_bytes}};
    for (const auto& z : sums)
      if (z.bytes) LG_TRY(cudaMemsetAsync(z.b->p, 0, z.bytes, s), "clear accumulation workspace");
    m->acc_dirty = false;
  }
  auto keep = [&](int j) -> cudaError_t {
    if (!c.keep_layers) return cudaSuccess;
    return cudaMemcpyAsync((float*)m->hist.p + (size_t)j * c.max_step_tokens * Hp, m->x.p, (size_t)T * Hp * 4, cudaMemcpyDeviceToDevice, s);
  };
  LG_TRY(logismos_launch_embed_lookup_bf16(m->embed.p, m->dev(B.ids), m->x.p, T, Hp, c.vocab, s), "embed_lookup");
  LG_TRY(keep(0), "snapshot");
  if (c.norm == LG_NORM_LAYER_POST) LG_TRY(norm_and_inputs(m, nullptr, 0, nullptr, nullptr, c.n_layers > 0 ? 0 : kNone, s), "inputs");
  else if (c.norm == LG_NORM_RMS_GATED && c.n_layers > 0) {
    lg_gated_residual_t a = residual_args(m);
    begin_layer(m, 0, &a);
    LG_TRY(logismos_launch_gated_residual(&a, st, s), "inputs");
    m->launches += 1;
  } else if (c.n_layers > 0) LG_TRY(tanh_norms(m, nullptr, false, nullptr, nullptr, &m->weights[(size_t)m->layers[0].owner].pre1, s), "inputs");
  for (int l = 0; l < c.n_layers; ++l) {
    MLayer& L = m->layers[(size_t)l];
    const MWeights& W = m->weights[(size_t)L.owner];
    if (uint32_t rc = run_mixer(m, L, W, s)) return rc;
    if (uint32_t rc = mixer_output(m, l, s)) return rc;
    if (L.c.ff)
      if (uint32_t rc = run_feed_forward(m, l, s)) return rc;
    if (c.norm != LG_NORM_RMS_GATED) LG_TRY(keep(l + 1), "snapshot");  // there the residual's launch keeps it
  }
  if (m->n_out > 0) {
    const int32_t* rows = m->dev((int32_t*)B.extra) + m->views.size() * (size_t)(c.max_step_seqs + 1);
    if (c.norm == LG_NORM_LAYER_POST) {
      LG_TRY(logismos_launch_post_norm(m->x.p, 0, rows, T, nullptr, m->final_norm.p, m->final_norm_b.p, m->last.p, f32, m->n_out, c.width, Hp, c.norm_eps, st, s), "final norm");
    } else if (c.norm == LG_NORM_RMS_GATED) {
      lg_gated_residual_t a = residual_args(m);
      a.row_idx = rows; a.rows = m->n_out; a.h = m->last.p; a.gain = m->final_gain * c.logit_scale;
      LG_TRY(logismos_launch_gated_residual(&a, st, s), "final norm");
    } else {
      const lg_tanh_norm_t n = m->final_tanh.view();
      LG_TRY(logismos_launch_tanh_norm(nullptr, 0, nullptr, rows, T, m->x.p, nullptr, m->last.p, &n, f32, m->n_out, Hp, st, s), "final norm");
    }
    LG_TRY(linear(m, m->last.p, Hp, m->head, c.vocab, Hp, m->logits.p, c.vocab, LG_EPI_F32, m->n_out, s), "head");
    LG_TRY(logismos_launch_greedy_argmax(m->logits.p, 1, m->tokens.p, m->n_out, c.vocab, s), "greedy");
    m->launches += 2;
  }
  return 0;
}

// Chunks of the decode contexts, one split per kind of attention; false: more than the scratch holds
bool split_contexts(Mixer* m) {
  StepBatch& B = m->batch;
  std::vector<int32_t> ctx((size_t)B.n_dec);
  int32_t* at = (int32_t*)B.extra;
  for (DecodeView& V : m->views) {
    V.chunks = at;
    at += m->cfg.max_step_seqs + 1;
    if (m->cfg.is_f32 || B.n_dec == 0) continue;
    for (int i = 0; i < B.n_dec; ++i) ctx[(size_t)i] = logismos_window_view_context(&V.shape, B.ctx[i]);
    V.chunk_tokens = V.latent ? logismos_pick_latent_chunk(ctx.data(), B.n_dec, V.heads) : logismos_pick_decode_chunk(ctx.data(), B.n_dec, V.kv, V.hd);
    if (V.shape.size && V.chunk_tokens == 512) {  // few sequences: what a window shows is cut in smaller pieces, down to a block per warp
      auto pieces = [&](int c) {
        int64_t n = 0;
        for (int32_t v : ctx) n += (v + c - 1) / c;
        return n;
      };
      while (V.chunk_tokens > 64 && pieces(V.chunk_tokens) * V.kv < 32768 / V.hd) V.chunk_tokens /= 2;
    }
    V.total = logismos_build_decode_chunks(ctx.data(), B.n_dec, V.chunk_tokens, V.chunks);
    if (V.total < 0 || V.total > V.max_chunks) return false;
  }
  return true;
}

// ---- weights and configuration -----------------------------------------------------------------------

bool upload_tanh(Mixer* m, TanhNorm& n, const void* w, const void* b, const void* alpha) {
  n.alpha = f_at(alpha, 0);
  return upload_vec(n.w, w, m->cfg.width, m->Hp, 0.0f) && upload_vec(n.b, b, m->cfg.width, m->Hp, 0.0f);
}

bool upload_layer(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w) {
  const int H = m->cfg.width, Hp = m->Hp;
  bool ok;
  if (m->cfg.norm == LG_NORM_RMS_GATED) {
    W.gain1 = f_at(w.norm1, 0);
    if (L.c.ff) W.gain2 = f_at(w.norm2, 0);
    ok = upload_paired_kinds(m, L, W, w);
    if (!L.c.ff) return ok;
    const int n = L.gate2.end[0], routed = n > L.gate2.n_main ? L.c.experts + L.c.identity : 0;
    Mat g(n, Hp);
    for (int i = 0; i < H; ++i) g.row(i, 0, w.rg2, (size_t)i * H, H);
    for (int i = 0; i < routed; ++i) g.row(L.gate2.n_main + i, 0, w.router, (size_t)i * H, H);
    return ok && g.up(W.w_gate2) && upload_vec(W.b_gate2, w.rg2_b, H, L.gate2.n_main, 0.0f) && upload_feed_forward(m, L, W, w);
  }
  if (m->cfg.norm == LG_NORM_TANH_AROUND) {
    ok = upload_tanh(m, W.pre1, w.norm1, w.norm1_b, w.norm1_alpha) && upload_tanh(m, W.post1, w.norm1b, w.norm1b_b, w.norm1b_alpha);
    if (L.c.ff) ok = ok && upload_tanh(m, W.pre2, w.norm2, w.norm2_b, w.norm2_alpha) && upload_tanh(m, W.post2, w.norm2b, w.norm2b_b, w.norm2b_alpha);
  } else {
    ok = upload_vec(W.norm1, w.norm1, H, Hp, 0.0f) && upload_vec(W.norm1_b, w.norm1_b, H, Hp, 0.0f);
    if (L.c.ff) ok = ok && upload_vec(W.norm2, w.norm2, H, Hp, 0.0f) && upload_vec(W.norm2_b, w.norm2_b, H, Hp, 0.0f);
  }
  if (L.c.ff) ok = ok && upload_feed_forward(m, L, W, w);
  Mat out(Hp, L.Kout);
  if (is_gated_kind(L.c.kind)) {
    ok = ok && upload_gated_kinds(m, L, W, w, out);
  } else {
    Mat in(L.N, Hp);
    ok = ok && upload_parallel_kinds(m, L, W, w, in, out);
  }
  return ok && out.up(W.w_out);
}

const char* check_layer(const lg_mixer_layer_config_t& y, int norm) {
  if (const char* what = check_feed_forward(y)) return what;
  if (y.kind == LG_MIXER_PARALLEL && norm != LG_NORM_LAYER_POST) return "a parallel mixer in a stack that is not post-norm";
  if (y.ff && y.ff_kind == LG_FF_MIXTURE && norm == LG_NORM_LAYER_POST) return "a mixture of experts in a post-norm stack";
  if (is_paired_kind(y.kind) != (norm == LG_NORM_RMS_GATED)) return "a kind of mixer that its stack's norm does not go with";
  if (norm == LG_NORM_RMS_GATED) return y.ff && y.ff_kind == LG_FF_MIXTURE && (y.identity || y.shared_ff) ? "identity or shared experts in a gated stack" : check_paired_kinds(y);
  return is_gated_kind(y.kind) ? check_gated_kinds(y) : check_parallel_kinds(y);
}

const char* check_tensor_sizes(const lg_mixer_layer_config_t& y) {
  if (y.kind == LG_MIXER_GLA && y.tm_rank <= 0) return "rank of the decay";
  return is_gated_kind(y.kind) || is_paired_kind(y.kind) ? nullptr : check_parallel_tensors(y);
}

const char* check_config(const lg_mixer_config_t& c) {
  if (c.vocab <= 0 || c.width <= 0 || c.width > 16384 || c.n_layers < 0 || (c.n_layers > 0 && !c.layers)) return "vocab, width (<= 16384) or layer count";
  if (c.norm < LG_NORM_LAYER_POST || c.norm > LG_NORM_RMS_GATED) return "kind of norm";
  if (c.passes < 0 || (c.passes && c.norm != LG_NORM_RMS_GATED)) return "repeated layers";
  if (c.n_pool_blocks <= 0 || c.max_blocks_per_seq <= 0 || c.max_step_tokens <= 0 || c.max_step_seqs <= 0 || c.max_step_seqs > 65535 ||
      c.n_state_slots <= 0 || c.max_out_rows <= 0)
    return "pool, step or slot sizes";
  for (int l = 0; l < c.n_layers; ++l) {
    if (const char* what = check_layer(c.layers[l], c.norm)) return what;
    const int o = c.layers[l].weights_of;
    if (c.layers[l].pass < 0 || c.layers[l].pass > c.passes) return "a pass that does not exist";
    if (o < 0 || o >= c.n_layers || c.layers[o].weights_of != o || c.layers[o].kind != c.layers[l].kind || (c.layers[o].ff > 0) != (c.layers[l].ff > 0))
      return "a layer that uses the tensors of a layer without own ones or of another kind";
  }
  return nullptr;
}

uint32_t unsupported(const char* what) { return fail(LG_EMB_COMPUTE, std::string("unsupported mixer-stack config: ") + what); }

void layout(const Mixer* m, MLayer& L) {
  L.Fp = r64(L.c.ff);
  if (L.c.ff && L.c.ff_kind == LG_FF_MIXTURE) {
    L.always = (L.c.shared_ff + L.c.ff - 1) / L.c.ff;
    L.route_ld = round_up(L.c.experts + L.c.identity, 16);
  }
  if (m->cfg.norm == LG_NORM_RMS_GATED && L.c.ff) {
    L.gate2.n_groups = 1;
    L.gate2.n_main = round_up(m->Hp, 128);
    L.gate2.ld_tail = L.route_ld;
    L.gate2.end[0] = L.gate2.n_main + L.route_ld;
  }
  if (is_paired_kind(L.c.kind)) layout_paired_kinds(m, L);
  else if (is_gated_kind(L.c.kind)) layout_gated_kinds(L);
  else layout_parallel_kinds(L);
}

// the decode view of a layer with a cache: layers with one window share one
int view_of(Mixer* m, const MLayer& L) {
  const lg_mixer_layer_config_t& y = L.c;
  if (y.kind == LG_MIXER_SSD || y.kind == LG_MIXER_GLA) return -1;
  const bool latent = y.kind == LG_MIXER_LATENT, paired = is_paired_kind(y.kind);
  const int window = y.kind == LG_MIXER_ATTENTION || paired ? y.window : 0, keep = window ? y.keep_first : 0, seqs = m->cfg.max_step_seqs;
  lg_window_t shape{};
  shape.size = window; shape.keep_first = keep; shape.chunked = paired ? y.chunked : 0; shape.pool = paired ? y.pool : 0;
  int i = 0;
  for (; i < (int)m->views.size(); ++i) {
    const lg_window_t& o = m->views[(size_t)i].shape;
    if (m->views[(size_t)i].latent == latent && o.size == window && o.keep_first == keep && o.chunked == shape.chunked && o.pool == shape.pool) break;
  }
  if (i == (int)m->views.size()) {
    DecodeView v;
    v.latent = latent;
    v.shape = shape;
    const int64_t longest = (int64_t)m->cfg.max_blocks_per_seq * kKvBlock + (shape.pool ? 3 * kKvBlock : 0);
    v.max_chunks = latent ? logismos_latent_max_chunks(seqs) : (int)(seqs * ((longest + 511) / 512));
    if (!latent && window) {  // cut in pieces of 64 while these are too few to fill the GPU
      const int64_t seen = std::min(longest, (int64_t)window + keep + (shape.pool ? longest / shape.pool : 0) + 4 * kKvBlock);
      v.max_chunks = std::max(v.max_chunks, (int)std::min((int64_t)seqs * ((seen + 63) / 64), (int64_t)seqs + 2048));
    }
    m->views.push_back(v);
  }
  DecodeView& V = m->views[(size_t)i];
  if (!latent && y.kv_heads * L.Dh > V.kv * V.hd) { V.kv = y.kv_heads; V.hd = L.Dh; }
  V.heads = std::max(V.heads, (int)y.heads);
  return i;
}

// cos and sin of every position's angles, evaluated in double. YaRN: pairs that turn less than `slow` times over the original
// context are stretched by the factor, those that turn more than `fast` times kept, with a linear ramp between; cos and sin
// carry the factor 0.1 ln(factor) + 1.
bool fill_table(RotationTable& t, int positions) {
  const int pairs = t.dims / 2;
  std::vector<double> f((size_t)pairs);
  double amp = 1.0, lo = 0.0, hi = 0.0;
  auto turns_at = [&](double turns) { return t.dims * std::log(t.original / (2.0 * 3.14159265358979323846 * turns)) / (2.0 * std::log(t.base)); };
  const bool linear = t.factor != 0.0 && t.original == 0.0;   // all pairs stretched alike
  if (t.factor != 0.0 && !linear) {
    lo = std::max(std::floor(turns_at(t.fast)), 0.0);
    hi = std::min(std::ceil(turns_at(t.slow)), t.dims - 1.0);
    amp = 0.1 * std::log(t.factor) + 1.0;
  }
  for (int i = 0; i < pairs; ++i) {
    f[(size_t)i] = std::pow(t.base, -2.0 * i / t.dims);
    if (linear) f[(size_t)i] /= t.factor;
    if (t.factor == 0.0 || linear) continue;
    const double ramp = std::min(std::max((i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
    f[(size_t)i] = f[(size_t)i] / t.factor * ramp + f[(size_t)i] * (1.0 - ramp);
  }
  std::vector<float> v((size_t)positions * t.dims);
  for (int p = 0; p < positions; ++p)
    for (int i = 0; i < pairs; ++i) {
      v[(size_t)p * t.dims + 2 * i] = (float)(amp * std::cos(p * f[(size_t)i]));
      v[(size_t)p * t.dims + 2 * i + 1] = (float)(amp * std::sin(p * f[(size_t)i]));
    }
  return t.angles.upload(v.data(), v.size() * 4);
}

// index of the layer's rotation table (-1: none, -2: out of memory); equal rotations share one
int table_of(Mixer* m, const lg_mixer_layer_config_t& y) {
  if ((!is_gated_kind(y.kind) && !is_paired_kind(y.kind)) || y.kind == LG_MIXER_GLA || y.rot_dims == 0) return -1;
  for (size_t i = 0; i < m->tables.size(); ++i) {
    const RotationTable& t = m->tables[i];
    if (t.dims == y.rot_dims && t.base == y.rot_base && t.factor == y.rot_factor && t.original == y.rot_original && t.fast == y.rot_fast && t.slow == y.rot_slow) return (int)i;
  }
  RotationTable t;
  t.dims = y.rot_dims; t.base = y.rot_base; t.factor = y.rot_factor; t.original = y.rot_original; t.fast = y.rot_fast; t.slow = y.rot_slow;
  const bool ok = fill_table(t, m->cfg.max_blocks_per_seq * kKvBlock);
  m->tables.push_back(t);
  return ok ? (int)m->tables.size() - 1 : -2;
}

}  // namespace

extern "C" {

uint32_t lg_mixer_create(int32_t device, const lg_mixer_config_t* cfg, const lg_mixer_weights_t* w, void** model) {
  if (!cfg || !w || !model) return fail(LG_EMB_COMPUTE, "null argument");
  *model = nullptr;
  if (const char* what = check_config(*cfg)) return unsupported(what);
  for (int l = 0; l < cfg->n_layers; ++l)
    if (const char* what = check_tensor_sizes(cfg->layers[cfg->layers[l].weights_of])) return unsupported(what);
  if (cudaSetDevice(device) != cudaSuccess) return fail(LG_EMB_COMPUTE, "cudaSetDevice failed");
  Mixer* m = new Mixer();
  m->layer_cfg.assign(cfg->layers, cfg->layers + cfg->n_layers);
  m->cfg = *cfg;
  m->cfg.layers = m->layer_cfg.data();
  const lg_mixer_config_t& c = m->cfg;
  m->device = device;
  m->Hp = r64(c.width);
  const int H = c.width, Hp = m->Hp;
  size_t branches = 1, copies = 1;           // outputs of a mixer; copies of the activations: parallel mixers read token-shift mixes too
  for (int l = 0; l < c.n_layers; ++l)
    if (c.layers[l].kind == LG_MIXER_PARALLEL) copies = 1 + kMixes;
  for (int l = 0; l < c.n_layers; ++l)
    if (c.layers[l].kind == LG_MIXER_PAIR) branches = 2;
  const size_t esz = c.is_f32 ? 4 : 2, T = (size_t)c.max_step_tokens, S = (size_t)c.max_step_seqs, MB = (size_t)c.max_blocks_per_seq, acc_rows = std::min(T, (size_t)kAccRows);
  bool ok = true;
  {
    Mat e(c.vocab, Hp), h(c.vocab, Hp);
    for (int i = 0; i < c.vocab; ++i) { e.row(i, 0, w->embed, (size_t)i * H, H); h.row(i, 0, w->head, (size_t)i * H, H); }
    ok = ok && e.up(m->embed) && h.up(m->head);
  }
  if (c.norm == LG_NORM_RMS_GATED) {
    m->final_gain = f_at(w->final_norm, 0);
    std::vector<float> steps((size_t)c.passes * Hp, 0.0f);
    for (int t = 0; t < c.passes; ++t)
      for (int i = 0; i < H; ++i) steps[(size_t)t * Hp + i] = f_at(w->loop_step, (size_t)t * H + i);
    ok = ok && m->loop_step.upload(steps.data(), steps.size() * 4);
  } else if (c.norm == LG_NORM_TANH_AROUND) ok = ok && upload_tanh(m, m->final_tanh, w->final_norm, w->final_norm_b, w->final_norm_alpha);
  else ok = ok && upload_vec(m->final_norm, w->final_norm, H, Hp, 0.0f) && upload_vec(m->final_norm_b, w->final_norm_b, H, Hp, 0.0f);
  m->layers.resize((size_t)c.n_layers);
  m->weights.resize((size_t)c.n_layers);
  Sizes z;
  for (int l = 0; l < c.n_layers; ++l) {
    MLayer& L = m->layers[(size_t)l];
    L.owner = c.layers[l].weights_of;
    L.c = c.layers[L.owner];
    layout(m, L);
    L.view = view_of(m, L);
  }
  for (int l = 0; l < c.n_layers && ok; ++l) {
    MLayer& L = m->layers[(size_t)l];
    if (L.owner == l) ok = ok && upload_layer(m, L, m->weights[(size_t)l], w->layers[l]);
    L.table = table_of(m, L.c);
    grow(z.proj, (size_t)L.groups.n_main);
    grow(z.tail, (size_t)L.groups.ld_tail);
    if (splits_projections(L.groups, L.N, 33)) grow(z.raw, (size_t)L.N);
    if (L.gate2.n_groups) {
      grow(z.proj, (size_t)L.gate2.n_main);
      if (splits_projections(L.gate2, L.gate2.end[0], 33)) grow(z.raw, (size_t)L.gate2.end[0]);
    }
    grow(z.act, (size_t)L.Kout);
    size_feed_forward(L, z);
    ok = ok && L.table != -2 && (is_paired_kind(L.c.kind) ? alloc_paired_kinds(m, L, z) : is_gated_kind(L.c.kind) ? alloc_gated_kinds(m, L, z) : alloc_parallel_kinds(m, L, z));
  }
  StepLimits lim;
  lim.max_pos = (int64_t)1 << 30;            // the block table is the limit, also of the rotation tables
  lim.max_blocks_per_seq = c.max_blocks_per_seq;
  lim.n_pool_blocks = c.n_pool_blocks;
  lim.max_step_tokens = c.max_step_tokens;
  lim.max_step_seqs = c.max_step_seqs;
  lim.n_state_slots = c.n_state_slots;
  lim.prefix_cap_tokens = std::max(MB * kKvBlock, T);
  lim.extra_bytes = ((size_t)c.max_out_rows + m->views.size() * (S + 1)) * 4;
  m->acc_bytes = branches * acc_rows * Hp * 4;
  m->raw_acc_bytes = c.is_f32 ? 0 : acc_rows * z.raw * 4;
  m->route_acc_bytes = c.is_f32 ? 0 : T * z.route * 4;
  m->segment_bytes = z.segments;
  m->counts_bytes = z.groups ? (z.groups + 1) * 4 : 0;  // the last one counts the router's finished tokens
  ok = ok && m->x.alloc(T * Hp * 4) && zeroed(m->h, copies * T * Hp * esz) && zeroed(m->proj, T * z.proj * esz) && m->tail.alloc(T * z.tail * 4) &&
       zeroed(m->act, T * z.act * esz) && zeroed(m->ffb, T * z.ff * esz) && zeroed(m->xbc, T * z.xbc * esz) && m->y.alloc(branches * T * Hp * 4) && zeroed(m->qx, T * z.maps * esz) && m->maps_out.alloc(T * z.maps * 4) && m->segments.alloc(z.segments) && m->y_acc.alloc(m->acc_bytes) && m->raw_acc.alloc(m->raw_acc_bytes) &&
       m->last.alloc((size_t)c.max_out_rows * Hp * esz) && m->logits.alloc((size_t)c.max_out_rows * c.vocab * 4) && m->tokens.alloc((size_t)c.max_out_rows * 4) &&
       m->status.alloc(4) && (!c.keep_layers || m->hist.alloc((size_t)(c.n_layers + 1) * T * Hp * 4));
  if (!c.is_f32)
    ok = ok && m->low2.alloc(T * z.low * 2) && m->z.alloc(T * z.z * 4) && m->attn_ws.alloc(z.attn_ws) && m->dec_scratch.alloc(z.scratch);
  if (z.lat) {  // latent attention
    const size_t rows = c.is_f32 ? T : S;    // that attend in the latent space
    ok = ok && m->cq.alloc(T * z.cq * esz) && m->gate.alloc(T * z.heads * 4) && m->qlat.alloc(rows * z.lat_q * esz) &&
         m->olat.alloc(rows * z.lat_q * esz);
    if (!c.is_f32) {
      const size_t tp = (size_t)logismos_latent_gather_rows((int32_t)lim.prefix_cap_tokens, c.max_step_seqs);
      ok = ok && m->lat.alloc(tp * z.lat * 2) && m->kbuf.alloc(tp * z.lat_heads * 2) && m->vt.alloc(tp * z.lat_heads * 2) && m->kv_start.alloc(S * 4);
    }
  }
  if (z.pairs) {  // a mixture
    const size_t pairs = T * z.pairs;
    ok = ok && m->route.alloc(T * z.route * 4) && m->route_acc.alloc(m->route_acc_bytes) && m->pair_w.alloc(T * z.top * 4) && m->pair_row.alloc(pairs * 4) &&
         m->pair_expert.alloc(T * z.top * 4) && m->identity.alloc(T * 4) && m->offsets.alloc((z.groups + 1) * 4) && m->row_token.alloc(pairs * 4) &&
         m->counts.alloc(m->counts_bytes) && m->expert_rows.alloc(pairs * Hp * esz);
    if (!c.is_f32) ok = ok && m->gathered.alloc(pairs * Hp * 2) && m->tiles.alloc((1 + pairs / 128 + z.groups + z.pairs) * 16);
  }
  ok = ok && cudaMemset(m->status.p, 0, 4) == cudaSuccess && m->batch.alloc(lim) && m->dev_batch.alloc(m->batch.capacity) &&
       cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking) == cudaSuccess;
  m->slot_phase.assign((size_t)c.n_state_slots, 0);
  if (!ok || cudaDeviceSynchronize() != cudaSuccess) {
    set_error(std::string("lg_mixer_create: allocation or upload failed: ") + cudaGetErrorString(cudaGetLastError()));
    lg_mixer_destroy(m);
    return LG_EMB_COMPUTE;
  }
  *model = m;
  return LG_EMB_OK;
}

uint32_t lg_mixer_load(int32_t device, const char* path, const lg_mixer_config_t* cfg, void** model) {
  if (!path || !cfg || !model) return fail(LG_EMB_COMPUTE, "null argument");
  *model = nullptr;
  if (const char* what = check_config(*cfg)) return unsupported(what);
  Archive* r = nullptr;
  if (uint32_t rc = open_archive(path, &r)) return rc;
  struct Guard { Archive* r; ~Guard() { delete r; } } guard{r};
  lg_mixer_config_t c = *cfg;
  std::vector<lg_mixer_layer_config_t> lc(cfg->layers, cfg->layers + cfg->n_layers);
  c.layers = lc.data();
  const bool tanh = c.norm == LG_NORM_TANH_AROUND, rms = c.norm == LG_NORM_RMS_GATED;
  Wanted t{r};
  auto want_norm = [&](const std::string& name, const void** wt, const void** bias, const void** alpha) {
    if (rms) return t.get(name, {}, wt);
    return t.get(name, {c.width}, wt) && t.get(name + ".b", {c.width}, bias) && (!tanh || t.get(name + ".alpha", {}, alpha));
  };
  const int64_t H = c.width, V = c.vocab;
  lg_mixer_weights_t w{};
  std::vector<lg_mixer_layer_weights_t> layers((size_t)c.n_layers);
  std::vector<std::vector<const void*>> experts((size_t)c.n_layers);
  if (!(t.get("embed", {V, H}, &w.embed) && want_norm("final.norm", &w.final_norm, &w.final_norm_b, &w.final_norm_alpha) && t.get("head", {V, H}, &w.head))) return t.rc;
  if (c.passes && !t.get("loop.step", {c.passes, H}, &w.loop_step)) return t.rc;
  for (int i = 0; i < c.n_layers; ++i) {
    lg_mixer_layer_config_t& y = lc[(size_t)i];
    if (y.weights_of != i) continue;
    lg_mixer_layer_weights_t& L = layers[(size_t)i];
    const std::string p = "l" + std::to_string(y.file_layer ? y.file_layer - 1 : i) + ".";
    if (rms && (!t.get(p + "rg1", {H, H}, &L.rg1) || !t.get(p + "rg1.b", {H}, &L.rg1_b))) return t.rc;
    // a layer without a feed-forward may still store its norm and gate
    if (rms && (y.ff || t.has(p + "rg2")) && (!t.get(p + "rg2", {H, H}, &L.rg2) || !t.get(p + "rg2.b", {H}, &L.rg2_b))) return t.rc;
    if (!want_norm(p + "norm1", &L.norm1, &L.norm1_b, &L.norm1_alpha) || (tanh && !want_norm(p + "norm1b", &L.norm1b, &L.norm1b_b, &L.norm1b_alpha))) return t.rc;
    // a layer without a feed-forward has nothing that these norms act on; a stack with norms around may still store them
    if (y.ff || ((tanh || rms) && t.has(p + "norm2")))
      if (!want_norm(p + "norm2", &L.norm2, &L.norm2_b, &L.norm2_alpha)) return t.rc;
    if (tanh && (y.ff || t.has(p + "norm2b")))
      if (!want_norm(p + "norm2b", &L.norm2b, &L.norm2b_b, &L.norm2b_alpha)) return t.rc;
    if (y.ff && !want_feed_forward(t, p + "mlp.", H, y, L, experts[(size_t)i])) return t.rc;
    if (!(is_paired_kind(y.kind) ? want_paired_kinds(t, p + "mix.", H, y, L) : is_gated_kind(y.kind) ? want_gated_kinds(t, p + "mix.", H, y, L) : want_parallel_kinds(t, p + "mix.", H, y, L))) return t.rc;
  }
  if (r->ordering.size() != t.count)
    return fail(LG_EMB_COMPUTE, "expected " + std::to_string(t.count) + " tensors in the archive, got " + std::to_string(r->ordering.size()));
  w.layers = layers.data();
  return lg_mixer_create(device, &c, &w, model);
}

void lg_mixer_destroy(void* model) {
  if (!model) return;
  Mixer* m = static_cast<Mixer*>(model);
  cudaSetDevice(m->device);
  Buf* bufs[] = {&m->embed, &m->head, &m->final_norm, &m->final_norm_b, &m->final_tanh.w, &m->final_tanh.b, &m->x, &m->h, &m->proj, &m->tail, &m->low2, &m->z, &m->xbc,
                 &m->act, &m->ffb, &m->y, &m->y_acc, &m->hist, &m->last, &m->logits, &m->tokens, &m->status, &m->attn_ws, &m->dec_scratch, &m->dev_batch, &m->raw_acc,
                 &m->cq, &m->gate, &m->qlat, &m->olat, &m->lat, &m->kbuf, &m->vt, &m->kv_start, &m->route, &m->route_acc, &m->pair_w, &m->pair_row, &m->pair_expert,
                 &m->identity, &m->offsets, &m->row_token, &m->counts, &m->tiles, &m->gathered, &m->expert_rows,
                 &m->loop_step, &m->qx, &m->maps_out, &m->segments};
  for (Buf* b : bufs) b->release();
  for (MWeights& W : m->weights) W.release();
  for (MLayer& L : m->layers) {
    Buf* lb[] = {&L.kpool, &L.vpool, &L.kmean, &L.vmean, &L.shift, &L.conv_state, &L.state};
    for (Buf* b : lb) b->release();
  }
  for (RotationTable& t : m->tables) t.angles.release();
  m->batch.release();
  if (m->stream) cudaStreamDestroy(m->stream);
  delete m;
}

uint32_t lg_mixer_step(void* model, const uint32_t* host_ids, const int32_t* cached, const int32_t* newl, int32_t n_seqs, const int32_t* tables,
                       const int32_t* state_slots, const int32_t* out_rows, int32_t n_out, uint32_t* next_tokens) {
  Mixer* m = static_cast<Mixer*>(model);
  if (!m) return fail(LG_EMB_COMPUTE, "lg_mixer_step: null model");
  const lg_mixer_config_t& c = m->cfg;
  if (!out_rows) n_out = n_seqs;
  if (n_out < 0 || n_out > c.max_out_rows || (n_out > 0 && !next_tokens))
    return fail(LG_EMB_COMPUTE, "lg_mixer_step: more output rows than max_out_rows, or no room for their tokens");
  std::lock_guard<std::mutex> lock(m->mu);
  if (cudaSetDevice(m->device) != cudaSuccess) return fail(LG_EMB_COMPUTE, "cudaSetDevice failed");
  StepBatch& B = m->batch;
  m->ready = false;
  if (uint32_t rc = B.build("lg_mixer_step", host_ids, cached, newl, n_seqs, tables, state_slots, false)) return rc;
  for (int s = 0; s < n_seqs; ++s) B.phase[s] = m->slot_phase[(size_t)B.state[s]];
  if (!split_contexts(m)) return fail(LG_EMB_COMPUTE, "lg_mixer_step: decode chunk count exceeds the scratch");
  int32_t* rows = (int32_t*)B.extra + m->views.size() * (size_t)(c.max_step_seqs + 1);
  if (!B.select_rows(out_rows, n_out, newl, rows)) return fail(LG_EMB_COMPUTE, "lg_mixer_step: an output row lies outside the step");
  m->n_out = n_out;
  cudaStream_t s = m->stream;
  LG_TRY(cudaMemsetAsync(m->status.p, 0, 4, s), "clear status");
  LG_TRY(cudaMemcpyAsync(m->dev_batch.p, B.pinned, (size_t)((uint8_t*)(rows + n_out) - B.pinned), cudaMemcpyHostToDevice, s), "H2D step");
  m->ready = true;
  if (uint32_t rc = run_device(m, s)) { m->acc_dirty = true; return rc; }
  if (n_out > 0) LG_TRY(cudaMemcpyAsync(next_tokens, m->tokens.p, (size_t)n_out * 4, cudaMemcpyDeviceToHost, s), "D2H tokens");
  LG_TRY(cudaStreamSynchronize(s), "stream synchronize");
  if (const int dev_status = lg_mixer_device_status(m)) {
    m->acc_dirty = true;
    char buf[256];
    std::snprintf(buf, sizeof(buf), "device status 0x%x after a step of %d tokens in %d sequences (low byte 1: a range check failed, 2: a bounded wait expired in kernel family <next byte>)",
                  dev_status, B.T, (int)n_seqs);
    return fail(LG_EMB_COMPUTE, buf);
  }
  for (int k = 0; k < n_seqs; ++k) m->slot_phase[(size_t)B.state[k]] ^= 1;  // the step is complete: its states are the current ones
  return LG_EMB_OK;
}

uint32_t lg_mixer_replay_device(void* model, void* stream) {
  Mixer* m = static_cast<Mixer*>(model);
  if (!m || !m->ready) return fail(LG_EMB_COMPUTE, "lg_mixer_replay_device: no step has run");
  if (cudaSetDevice(m->device) != cudaSuccess) return fail(LG_EMB_COMPUTE, "cudaSetDevice failed");
  return run_device(m, (cudaStream_t)stream);
}

uint32_t lg_mixer_last_logits(void* model, int32_t n_out, float* host_out) {
  Mixer* m = static_cast<Mixer*>(model);
  if (!m || n_out != m->n_out) return fail(LG_EMB_COMPUTE, "lg_mixer_last_logits: n_out differs from the last step");
  cudaSetDevice(m->device);
  LG_TRY(cudaDeviceSynchronize(), "device synchronize");
  if (n_out > 0) LG_TRY(cudaMemcpy(host_out, m->logits.p, (size_t)n_out * m->cfg.vocab * 4, cudaMemcpyDeviceToHost), "D2H logits");
  return LG_EMB_OK;
}

void* lg_mixer_logits_device(void* model) { return static_cast<Mixer*>(model)->logits.p; }

uint32_t lg_mixer_snapshot(void* model, int32_t j, int32_t n_tokens, float* host_out) {
  Mixer* m = static_cast<Mixer*>(model);
  if (!m || !m->ready || !m->cfg.keep_layers || j < 0 || j > m->cfg.n_layers || n_tokens != m->batch.T)
    return fail(LG_EMB_COMPUTE, "lg_mixer_snapshot: bad arguments, or a model without keep_layers");
  cudaSetDevice(m->device);
  LG_TRY(cudaDeviceSynchronize(), "device synchronize");
  LG_TRY(m->batch.rows_to_host((const float*)m->hist.p + (size_t)j * m->cfg.max_step_tokens * m->Hp, m->Hp, m->cfg.width, host_out), "D2H snapshot");
  return LG_EMB_OK;
}

int32_t lg_mixer_launches_last_step(const void* model) { return static_cast<const Mixer*>(model)->launches; }

int32_t lg_mixer_device_status(void* model) {
  Mixer* m = static_cast<Mixer*>(model);
  int32_t v = -1;
  cudaSetDevice(m->device);
  if (cudaMemcpy(&v, m->status.p, 4, cudaMemcpyDeviceToHost) != cudaSuccess) return -1;
  return v;
}

}  // extern "C"
