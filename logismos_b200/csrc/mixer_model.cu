// Host-side executor of one continuous-batching step over a post-norm stack of state-space layers and parallel
// layers (attention beside time mixing); see lg_mixer_* in logismos_model.h. The contract is that of the other
// executors: a packed step equals running every sequence alone.
//
// A step packs decode tokens first and prefill chunks after them (step_batch.h):
//   embed -> per layer
//     state-space: one GEMM to [z | x | B | C] and fp32 dt -> convolution -> recurrence, token by token for decode
//       rows, chunk-parallel for prefill rows -> gate + norm -> output GEMM
//     parallel: one GEMM over the stream and its five token-shift mixes to attention q | k | v | gate, time-mixing
//       r | k | v | g and the fp32 low-rank activations of the decay -> unit q, k + cache store -> attention with its
//       gate into the left columns of one activation row; time mixing with its norm and gate into the right ones ->
//       one GEMM over [left W_o | right W_o] (the branch scales ride on the gates)
//     output norm + residual (+ the next layer's inputs); feed-forward likewise
//   -> wanted rows: final norm -> head (fp32) -> greedy argmax
// Every matrix is padded at load with zeros (inputs and outputs to multiples of 64, heads to powers of two), which
// keeps the padding of every activation zero.
#include <cuda_runtime.h>

#include <algorithm>
#include <cmath>
#include <mutex>
#include <string>
#include <vector>

#include "logismos_kernels.h"
#include "logismos_model.h"

#include "model_util.h"
#include "safetensors.h"
#include "step_batch.h"
#include "weight_pack.h"

namespace {

using namespace lgm;

constexpr int kAccRows = 512;   // steps up to this size accumulate their output projections over slices of k
constexpr int kMixes = 5;       // r, k, v, g, w

inline int pow2_at_least(int v, int lo) {
  int p = lo;
  while (p < v) p *= 2;
  return p;
}

struct MWeights {   // of a layer that owns tensors
  Buf norm1, norm1_b, norm2, norm2_b, w_up, w_down, w_in, w_out;
  Buf conv, conv_b, dt_bias, A_log, D, gain;              // state-space (gain also: time mixing)
  Buf bias, mu, w2, w0, u;                                // parallel
  float max_bias = 0.0f;
};

struct MLayer {
  lg_mixer_layer_config_t c{};
  int owner = 0;
  lg_linear_groups_t groups{};
  int N = 0, Fp = 0, Kout = 0;          // projection width, feed-forward and output-projection inputs
  int Vp = 0, Np = 0, channels = 0;     // state-space
  int Dh = 0, Dp = 0, Rw = 0, Lr = 0;   // attention head, time-mixing head, padded block of its heads, padded rank
  Buf kpool, vpool, shift, conv_state, state;
};

struct Mixer {
  lg_mixer_config_t cfg{};
  std::vector<lg_mixer_layer_config_t> layer_cfg;
  int device = 0, Hp = 0;
  Buf embed, head, final_norm, final_norm_b;
  std::vector<MWeights> weights;
  std::vector<MLayer> layers;
  Buf x, h, proj, tail, low2, z, xbc, act, ffb, y, y_acc, hist, last, logits, tokens, status, attn_ws, dec_scratch, dev_batch;
  StepBatch batch;
  std::vector<uint8_t> slot_phase;      // per state slot: the copy that holds its convolution and shift states
  cudaStream_t stream = nullptr;
  std::mutex mu;
  int n_out = 0, total_chunks = 0, chunk_tokens = 512, max_chunks = 0, launches = 0;
  // `y_acc` is all zero between its uses (the norm that reads it zeroes it); a step that failed part-way may have
  // left sums there, so the next one clears it
  bool acc_dirty = true, ready = false;
  size_t acc_bytes = 0;
  template <typename T> T* dev(T* host) const { return (T*)((uint8_t*)dev_batch.p + ((uint8_t*)host - batch.pinned)); }
};

uint32_t linear(Mixer* m, const void* a, int lda, const Buf& w, int n, int k, void* out, int ldc, int epi, int rows, cudaStream_t s) {
  m->launches += 1;
  if (m->cfg.is_f32)
    return logismos_launch_linear_f32(a, w.p, nullptr, out, rows, n, k, lda, ldc, 1, 0, 0, 0, epi == LG_EPI_BF16 ? LG_EPI_F32 : epi, 0, 0, 0, s);
  if (stream_weights(rows, n, k, epi))
    return logismos_launch_linear_small_bf16(a, w.p, nullptr, out, rows, n, k, lda, ldc, 1, 0, 0, 0, epi, 0, 0, 0, s);
  return logismos_launch_linear_t_act_bf16(a, w.p, nullptr, out, rows, n, k, lda, ldc, epi | LG_EPI_STATIC_W, 0, 0, 0, m->status.p, s);
}

// input projections of a layer: main columns to proj, fp32 tail to `tail`
uint32_t projections(Mixer* m, const MLayer& L, const MWeights& W, int rows, cudaStream_t s) {
  lg_linear_groups_t g = L.groups;
  g.tail = m->tail.p;
  g.tail_parts = L.c.kind == LG_MIXER_PARALLEL && m->batch.n_pre > 0 ? m->low2.p : nullptr;
  m->launches += 1;
  const int Hp = m->Hp;
  if (m->cfg.is_f32) return logismos_launch_linear_groups_f32(m->h.p, W.w_in.p, m->proj.p, rows, L.N, Hp, Hp, g.n_main, &g, s);
  if (stream_weights(rows, L.N, Hp, LG_EPI_BF16))
    return logismos_launch_linear_groups_small_bf16(m->h.p, W.w_in.p, m->proj.p, rows, L.N, Hp, Hp, g.n_main, &g, s);
  return logismos_launch_linear_groups_tc_bf16(m->h.p, W.w_in.p, m->proj.p, rows, L.N, Hp, Hp, g.n_main, &g, m->status.p, s);
}

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

uint32_t output_projection(Mixer* m, const void* a, int k, const Buf& w, const Buf& nw, const Buf& nb, int next, cudaStream_t s) {
  const int T = m->batch.T, Hp = m->Hp;
  const bool acc = !m->cfg.is_f32 && T <= kAccRows && !logismos_get_deterministic();
  void* y = acc ? m->y_acc.p : m->y.p;
  LG_TRY(linear(m, a, k, w, Hp, k, y, Hp, acc ? LG_EPI_RESID_F32 : LG_EPI_F32, T, s), "output projection");
  LG_TRY(norm_and_inputs(m, y, acc, &nw, &nb, next, s), "output norm");
  return 0;
}

uint32_t ssd_mixer(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int T = B.T, inner = L.c.ssd_heads * L.Vp, f32 = c.is_f32;
  lg_ssd_t a{};
  a.proj = m->proj.p; a.ld = L.groups.n_main; a.dt = m->tail.p; a.ld_dt = L.groups.ld_tail;
  a.conv_w = W.conv.p; a.conv_b = W.conv_b.p; a.conv_state = L.conv_state.p; a.taps = L.c.ssd_taps;
  a.dt_bias = W.dt_bias.p; a.log_a = W.A_log.p; a.skip = W.D.p; a.state = L.state.p;
  a.state_slots = m->dev(B.state); a.fresh = m->dev(B.fresh); a.phase = m->dev(B.phase); a.cu = m->dev(B.cu);
  a.y = m->ffb.p; a.ld_y = inner; a.heads = L.c.ssd_heads; a.groups = L.c.ssd_groups; a.np = L.Np; a.vp = L.Vp;
  a.xbc = m->xbc.p; a.ld_xbc = L.channels;
  const bool chunked = !f32 && B.n_pre > 0 && logismos_ssd_has_chunked(L.Np, L.Vp);
  const int serial = chunked ? B.n_dec : B.n_seqs;  // sequences that go token by token
  if (B.n_dec > 0) LG_TRY(logismos_launch_ssd_conv(&a, m->dev(B.seq_ids), 0, B.n_dec, 1, f32, s), "state-space convolution");
  if (B.n_pre > 0) LG_TRY(logismos_launch_ssd_conv(&a, m->dev(B.seq_ids), B.n_dec, T, 0, f32, s), "state-space convolution");
  m->launches += (B.n_dec > 0) + (B.n_pre > 0);
  if (serial > 0) {
    LG_TRY(logismos_launch_ssd_step(&a, serial, f32, s), "state-space recurrence");
    m->launches += 1;
  }
  if (chunked) {
    a.state_slots = m->dev(B.state) + B.n_dec; a.fresh = m->dev(B.fresh) + B.n_dec; a.phase = m->dev(B.phase) + B.n_dec; a.cu = m->dev(B.cu) + B.n_dec;
    LG_TRY(logismos_launch_ssd_chunked_bf16(&a, B.n_pre, s), "state-space recurrence (prompts)");
    m->launches += 1;
  }
  LG_TRY(logismos_launch_gated_group_norm(m->ffb.p, inner, m->proj.p, L.groups.n_main, W.gain.p, m->act.p, L.Kout, f32, T, L.c.ssd_heads, L.c.ssd_vdim, L.Vp,
                                          L.c.ssd_norm_groups, c.norm_eps, s), "gate and norm");
  m->launches += 1;
  return 0;
}

uint32_t attention(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int T = B.T, MB = c.max_blocks_per_seq, P = L.groups.n_main, HD = L.c.heads * L.Dh, GD = L.c.kv_heads * L.Dh, f32 = c.is_f32;
  const size_t esz = f32 ? 4 : 2;
  void* st = m->status.p;
  uint8_t *proj = (uint8_t*)m->proj.p, *out = (uint8_t*)m->act.p;
  LG_TRY(logismos_launch_unit_qk_store(proj, P, L.kpool.p, L.vpool.p, m->dev(B.slots), m->dev(B.pos), T, L.c.heads, L.c.kv_heads, L.Dh, L.c.dim, c.norm_eps,
                                       L.c.temp_coef, L.c.temp_every, (int64_t)c.n_pool_blocks * kKvBlock, f32, st, s), "queries, keys and cache store");
  m->launches += 1;
  lg_score_bias_t sb{};
  sb.scale = L.c.scale; sb.cap = L.c.softcap; sb.bias = W.bias.p; sb.far = L.c.bias_max; sb.max_abs_bias = W.max_bias;
  {  // unit queries and keys: |q . k| <= dim times the largest temperature, with room for their rounding
    int longest = 1;
    for (int k = 0; k < B.n_seqs; ++k) longest = std::max(longest, B.cached[(size_t)k] + B.newl[(size_t)k]);
    const float t = L.c.temp_coef != 0.0f ? std::fabs(L.c.temp_coef) * std::log(std::floor(longest / L.c.temp_every) + 1.0f) : 0.0f;
    sb.max_abs_qk = 1.01f * L.c.dim * (1.0f + t);
  }
  sb.gate = proj + (size_t)(HD + 2 * GD) * esz; sb.ld_gate = P; sb.gate_scale = L.c.left_scale;
  if (f32) {
    LG_TRY(logismos_launch_bias_attention_f32(proj, P, L.kpool.p, L.vpool.p, m->dev(B.tables), m->dev(B.seq_ids), m->dev(B.pos), out, L.Kout, T, MB,
                                              c.n_pool_blocks, L.c.heads, L.c.kv_heads, L.Dh, &sb, st, s), "attention");
    m->launches += 1;
    return 0;
  }
  if (B.n_dec > 0) {
    LG_TRY(logismos_launch_bias_attention_decode_bf16(proj, P, L.kpool.p, L.vpool.p, m->dev(B.tables), m->dev(B.ctx), m->dev(B.chunks), out, L.Kout,
                                                      m->dec_scratch.p, B.n_dec, m->total_chunks, m->chunk_tokens, MB, c.n_pool_blocks, L.c.heads,
                                                      L.c.kv_heads, L.Dh, &sb, st, s), "decode attention");
    m->launches += m->total_chunks > B.n_dec ? 2 : 1;
  }
  const size_t row0 = (size_t)B.n_dec;
  sb.gate = (const uint8_t*)sb.gate + row0 * P * esz;
  for (const PrefixRun& r : B.runs) {
    LG_TRY(logismos_launch_bias_attention_prefix_bf16(proj + row0 * P * esz, P, m->dev(B.cu_pre) + r.s0, m->dev(B.pre_kv) + r.s0, L.kpool.p, L.vpool.p,
                                                      m->dev(B.tables) + (row0 + r.s0) * MB, MB, c.n_pool_blocks, out + row0 * L.Kout * esz, L.Kout,
                                                      m->attn_ws.p, T - B.n_dec, r.total_kv, r.s1 - r.s0, r.max_q, r.max_kv, L.c.heads, L.c.kv_heads,
                                                      L.Dh, &sb, st, s), "attention");
    m->launches += 2;
  }
  return 0;
}

uint32_t time_mixing(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  StepBatch& B = m->batch;
  const int left = L.c.heads * L.Dh, f32 = m->cfg.is_f32;
  lg_time_mix_t a{};
  a.proj = m->proj.p; a.ld = L.groups.n_main;
  a.off_r = L.groups.end[0]; a.off_k = L.groups.end[1]; a.off_v = L.groups.end[2]; a.off_g = L.groups.end[3];
  a.low = m->tail.p; a.ld_low = L.groups.ld_tail; a.w2 = W.w2.p; a.ld_w2 = 2 * L.Lr; a.rank = L.Lr; a.w0 = W.w0.p; a.u = W.u.p; a.gain = W.gain.p;
  a.state = L.state.p; a.state_slots = m->dev(B.state); a.fresh = m->dev(B.fresh); a.cu = m->dev(B.cu);
  a.out = (uint8_t*)m->act.p + (size_t)left * (f32 ? 4 : 2); a.ld_out = L.Kout; a.heads = L.c.tm_heads; a.d = L.c.tm_dim; a.dp = L.Dp;
  a.scale = L.c.right_scale; a.eps = m->cfg.norm_eps;
  const bool chunked = !f32 && B.n_pre > 0 && logismos_time_mix_has_chunked(L.Dp);
  const int serial = chunked ? B.n_dec : B.n_seqs;  // sequences that go token by token
  if (serial > 0) {
    LG_TRY(logismos_launch_time_mix_step(&a, serial, f32, s), "time mixing");
    m->launches += 1;
  }
  if (chunked) {
    const int rows = B.T - B.n_dec, w = L.Lr;
    LG_TRY(logismos_launch_linear_t_act_bf16((const uint16_t*)m->low2.p + (size_t)B.n_dec * 2 * w, W.w2.p, W.w0.p, (float*)m->z.p + (size_t)B.n_dec * L.Rw, rows, L.Rw, 2 * w, 2 * w, L.Rw,
                                             LG_EPI_F32 | LG_EPI_STATIC_W, 0, 0, 0, m->status.p, s), "decay");
    a.z = m->z.p; a.ld_z = L.Rw;
    a.state_slots = m->dev(B.state) + B.n_dec; a.fresh = m->dev(B.fresh) + B.n_dec; a.cu = m->dev(B.cu) + B.n_dec;
    LG_TRY(logismos_launch_time_mix_chunked_bf16(&a, B.n_pre, s), "time mixing (prompts)");
    m->launches += 2;
  }
  return 0;
}

uint32_t run_device(Mixer* m, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int Hp = m->Hp, T = B.T, f32 = c.is_f32;
  void* st = m->status.p;
  m->launches = 1;
  if (m->acc_dirty) {
    LG_TRY(cudaMemsetAsync(m->y_acc.p, 0, m->acc_bytes, s), "clear accumulation workspace");
    m->acc_dirty = false;
  }
  auto keep = [&](int j) -> cudaError_t {
    if (!c.keep_layers) return cudaSuccess;
    return cudaMemcpyAsync((float*)m->hist.p + (size_t)j * c.max_step_tokens * Hp, m->x.p, (size_t)T * Hp * 4, cudaMemcpyDeviceToDevice, s);
  };
  LG_TRY(logismos_launch_embed_lookup_bf16(m->embed.p, m->dev(B.ids), m->x.p, T, Hp, c.vocab, s), "embed_lookup");
  LG_TRY(keep(0), "snapshot");
  LG_TRY(norm_and_inputs(m, nullptr, 0, nullptr, nullptr, c.n_layers > 0 ? 0 : kNone, s), "inputs");
  for (int l = 0; l < c.n_layers; ++l) {
    MLayer& L = m->layers[(size_t)l];
    const MWeights& W = m->weights[(size_t)L.owner];
    const int next = l + 1 < c.n_layers ? l + 1 : kNone;
    LG_TRY(projections(m, L, W, T, s), "input projections");
    if (L.c.kind == LG_MIXER_SSD) {
      if (uint32_t rc = ssd_mixer(m, L, W, s)) return rc;
    } else {
      if (uint32_t rc = attention(m, L, W, s)) return rc;
      if (uint32_t rc = time_mixing(m, L, W, s)) return rc;
    }
    if (uint32_t rc = output_projection(m, m->act.p, L.Kout, W.w_out, W.norm1, W.norm1_b, L.c.ff ? kPlain : next, s)) return rc;
    if (L.c.ff) {
      LG_TRY(linear(m, m->h.p, Hp, W.w_up, L.Fp, Hp, m->ffb.p, L.Fp, LG_EPI_RELU2, T, s), "feed-forward");
      if (uint32_t rc = output_projection(m, m->ffb.p, L.Fp, W.w_down, W.norm2, W.norm2_b, next, s)) return rc;
    }
    LG_TRY(keep(l + 1), "snapshot");
  }
  if (m->n_out > 0) {
    LG_TRY(logismos_launch_post_norm(m->x.p, 0, m->dev((int32_t*)B.extra), T, nullptr, m->final_norm.p, m->final_norm_b.p, m->last.p, f32, m->n_out, c.width, Hp,
                                     c.norm_eps, st, s), "final norm");
    LG_TRY(linear(m, m->last.p, Hp, m->head, c.vocab, Hp, m->logits.p, c.vocab, LG_EPI_F32, m->n_out, s), "head");
    LG_TRY(logismos_launch_greedy_argmax(m->logits.p, 1, m->tokens.p, m->n_out, c.vocab, s), "greedy");
    m->launches += 2;
  }
  return 0;
}

// ---- weights ---------------------------------------------------------------------------------------

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

// row of the bias table for a distance: one per distance below rows / 2, then logarithmic up to `far`
int distance_bucket(int n, int rows, int far) {
  const int half = rows / 2;
  if (n < half) return n;
  const double at = std::log((double)n / half) / std::log((double)far / half) * (rows - half);
  const int b = half + (int)std::floor(at);
  return b < rows - 1 ? b : rows - 1;
}

bool upload_layer(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w) {
  const int H = m->cfg.width, Hp = m->Hp;
  const lg_mixer_layer_config_t& c = L.c;
  bool ok = upload_vec(W.norm1, w.norm1, H, Hp, 0.0f) && upload_vec(W.norm1_b, w.norm1_b, H, Hp, 0.0f);
  if (c.ff) {
    Mat up(L.Fp, Hp), down(Hp, L.Fp);
    for (int i = 0; i < c.ff; ++i) up.row(i, 0, w.up, (size_t)i * H, H);
    for (int i = 0; i < H; ++i) down.row(i, 0, w.down, (size_t)i * c.ff, c.ff);
    ok = ok && up.up(W.w_up) && down.up(W.w_down) && upload_vec(W.norm2, w.norm2, H, Hp, 0.0f) && upload_vec(W.norm2_b, w.norm2_b, H, Hp, 0.0f);
  }
  Mat in(L.N, Hp), out(Hp, L.Kout);
  if (c.kind == LG_MIXER_SSD) {
    const int heads = c.ssd_heads, V = c.ssd_vdim, N = c.ssd_state, G = c.ssd_groups, taps = c.ssd_taps, inner = heads * V;
    const size_t bc = (size_t)2 * inner;  // first row of B
    head_rows(in, 0, w.in, heads, V, L.Vp, H);
    head_rows(in, heads * L.Vp, (const uint8_t*)w.in + (size_t)inner * H * 2, heads, V, L.Vp, H);
    head_rows(in, 2 * heads * L.Vp, (const uint8_t*)w.in + bc * H * 2, 2 * G, N, L.Np, H);
    for (int h = 0; h < heads; ++h) in.row(L.groups.n_main + h, 0, w.in, (bc + (size_t)2 * G * N + h) * H, H);
    std::vector<float> cw((size_t)taps * L.channels, 0.0f), cb((size_t)L.channels, 0.0f);
    auto channel = [&](int src, int dst) {
      for (int j = 0; j < taps; ++j) cw[(size_t)j * L.channels + dst] = f_at(w.conv, (size_t)src * taps + j);
      cb[(size_t)dst] = f_at(w.conv_b, (size_t)src);
    };
    for (int h = 0; h < heads; ++h)
      for (int v = 0; v < V; ++v) channel(h * V + v, h * L.Vp + v);
    for (int g = 0; g < 2 * G; ++g)
      for (int n = 0; n < N; ++n) channel(inner + g * N + n, heads * L.Vp + g * L.Np + n);
    head_cols(out, 0, w.o, H, heads, V, L.Vp);
    return ok && in.up(W.w_in) && out.up(W.w_out) && W.conv.upload(cw.data(), cw.size() * 4) && W.conv_b.upload(cb.data(), cb.size() * 4) &&
           upload_vec(W.dt_bias, w.dt_bias, heads, heads, 0.0f) && upload_vec(W.A_log, w.A_log, heads, heads, 0.0f) && upload_vec(W.D, w.D, heads, heads, 0.0f) &&
           upload_heads(W.gain, w.norm, heads, V, L.Vp);
  }
  const int heads = c.heads, G = c.kv_heads, tm = c.tm_heads, D = c.tm_dim, R = c.tm_rank;
  head_rows(in, 0, w.left_q, heads, c.dim, L.Dh, H);
  head_rows(in, heads * L.Dh, w.left_k, G, c.dim, L.Dh, H);
  head_rows(in, (heads + G) * L.Dh, w.left_v, G, c.vdim, L.Dh, H);
  head_rows(in, (heads + 2 * G) * L.Dh, w.left_g, heads, c.vdim, L.Dh, H);
  const void* right[4] = {w.right_r, w.right_k, w.right_v, w.right_g};
  for (int i = 0; i < 4; ++i) head_rows(in, L.groups.end[i], right[i], tm, D, L.Dp, H);
  for (int i = 0; i < R; ++i) in.row(L.groups.n_main + i, 0, w.right_w1, (size_t)i * H, H);
  head_cols(out, 0, w.left_o, H, heads, c.vdim, L.Dh);
  head_cols(out, heads * L.Dh, w.right_o, H, tm, D, L.Dp);
  // the low-rank matrix twice over: the chunked form multiplies rounded activations and what rounding dropped
  Mat w2(L.Rw, 2 * L.Lr);
  for (int h = 0; h < tm; ++h)
    for (int d = 0; d < D; ++d)
      for (int half = 0; half < 2; ++half) w2.row(h * L.Dp + d, half * L.Lr, w.right_w2, ((size_t)h * D + d) * R, R);
  std::vector<float> mu((size_t)kMixes * Hp, 0.0f);
  for (int i = 0; i < kMixes; ++i)
    for (int d = 0; d < H; ++d) mu[(size_t)i * Hp + d] = f_at(w.mu[i], (size_t)d);
  const int far = c.bias_max;
  std::vector<float> bias((size_t)heads * (far + 1));
  for (int n = 0; n <= far; ++n) {
    const int b = distance_bucket(n, c.bias_rows, far);
    for (int h = 0; h < heads; ++h) {
      const float v = f_at(w.left_rel, (size_t)b * heads + h);
      if (std::fabs(v) > W.max_bias) W.max_bias = std::fabs(v);
      bias[(size_t)h * (far + 1) + n] = v * 1.4426950408889634f;
    }
  }
  std::vector<float> w0((size_t)L.Rw, 0.0f);
  for (int h = 0; h < tm; ++h)
    for (int d = 0; d < D; ++d) w0[(size_t)h * L.Dp + d] = f_at(w.right_w0, (size_t)h * D + d);
  return ok && in.up(W.w_in) && out.up(W.w_out) && w2.up(W.w2) && W.mu.upload(mu.data(), mu.size() * 4) && W.bias.upload(bias.data(), bias.size() * 4) &&
         W.w0.upload(w0.data(), w0.size() * 4) && upload_heads(W.u, w.right_u, tm, D, L.Dp) && upload_heads(W.gain, w.right_norm, tm, D, L.Dp);
}

const char* check_layer(const lg_mixer_layer_config_t& y) {
  if (y.ff < 0) return "feed-forward size";
  if (y.kind == LG_MIXER_SSD) {
    if (y.ssd_heads <= 0 || y.ssd_vdim <= 0 || y.ssd_vdim > 256 || y.ssd_state <= 0 || y.ssd_state > 256) return "state-space heads, or vdim / state above 256";
    if (y.ssd_groups <= 0 || y.ssd_heads % y.ssd_groups) return "state-space groups do not divide the heads";
    if (y.ssd_norm_groups <= 0 || (y.ssd_heads * y.ssd_vdim) % y.ssd_norm_groups) return "norm groups do not divide the channels";
    if (y.ssd_taps < 1 || y.ssd_taps > 8) return "convolution taps must be 1..8";
    return nullptr;
  }
  if (y.kind != LG_MIXER_PARALLEL) return "kind of mixer";
  if (y.heads <= 0 || y.kv_heads <= 0 || y.heads % y.kv_heads) return "attention heads";
  if (y.dim <= 0 || y.dim > 256 || y.vdim <= 0 || y.vdim > 256) return "attention head dimensions above 256";
  if (!(y.scale > 0.0f) || !(y.softcap >= 0.0f)) return "a score scale that is not positive, or a negative cap";
  if (y.temp_coef != 0.0f && !(y.temp_every > 0.0f)) return "query temperature";
  if (y.tm_heads <= 0 || y.tm_dim <= 0 || y.tm_dim > 256) return "time-mixing heads, or a head above 256";
  return nullptr;
}
// sizes that a file's tensors give
const char* check_tensor_sizes(const lg_mixer_layer_config_t& y) {
  if (y.kind != LG_MIXER_PARALLEL) return nullptr;
  if (y.bias_rows < 2 || y.bias_max <= y.bias_rows / 2) return "bias table: at least two rows, and bias_max above half of them";
  if (y.tm_rank <= 0) return "rank of the decay";
  return nullptr;
}

const char* check_config(const lg_mixer_config_t& c) {
  if (c.vocab <= 0 || c.width <= 0 || c.width > 16384 || c.n_layers < 0 || (c.n_layers > 0 && !c.layers)) return "vocab, width (<= 16384) or layer count";
  if (c.n_pool_blocks <= 0 || c.max_blocks_per_seq <= 0 || c.max_step_tokens <= 0 || c.max_step_seqs <= 0 || c.max_step_seqs > 65535 ||
      c.n_state_slots <= 0 || c.max_out_rows <= 0)
    return "pool, step or slot sizes";
  for (int l = 0; l < c.n_layers; ++l) {
    if (const char* what = check_layer(c.layers[l])) return what;
    const int o = c.layers[l].weights_of;
    if (o < 0 || o >= c.n_layers || c.layers[o].weights_of != o || c.layers[o].kind != c.layers[l].kind || (c.layers[o].ff > 0) != (c.layers[l].ff > 0))
      return "a layer that uses the tensors of a layer without own ones or of another kind";
  }
  return nullptr;
}

uint32_t unsupported(const char* what) { return fail(LG_EMB_COMPUTE, std::string("unsupported mixer-stack config: ") + what); }

void layout(MLayer& L) {
  const lg_mixer_layer_config_t& c = L.c;
  lg_linear_groups_t& g = L.groups;
  L.Fp = r64(c.ff);
  if (c.kind == LG_MIXER_SSD) {
    L.Vp = pow2_at_least(c.ssd_vdim, 16);
    L.Np = pow2_at_least(c.ssd_state, 32);
    L.channels = c.ssd_heads * L.Vp + 2 * c.ssd_groups * L.Np;
    L.Kout = r64(c.ssd_heads * L.Vp);
    g.n_groups = 1;
    g.n_main = round_up(c.ssd_heads * L.Vp + L.channels, 128);
    g.ld_tail = round_up(c.ssd_heads, 16);
    L.N = g.end[0] = g.n_main + g.ld_tail;
    return;
  }
  const int d = c.dim > c.vdim ? c.dim : c.vdim;
  L.Dh = pow2_at_least(d, 64);
  L.Dp = pow2_at_least(c.tm_dim, 32);
  L.Rw = round_up(c.tm_heads * L.Dp, 128);
  L.Lr = round_up(c.tm_rank, 32);
  L.Kout = c.heads * L.Dh + r64(c.tm_heads * L.Dp);
  g.n_groups = 1 + kMixes;
  g.end[0] = round_up((2 * c.heads + 2 * c.kv_heads) * L.Dh, 128);
  for (int i = 1; i < kMixes; ++i) g.end[i] = g.end[i - 1] + L.Rw;
  g.n_main = g.end[kMixes - 1];
  g.ld_tail = L.Lr;
  g.tail_cap = 1.0f;
  L.N = g.end[kMixes] = g.n_main + L.Lr;
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
  const size_t esz = c.is_f32 ? 4 : 2, T = (size_t)c.max_step_tokens, S = (size_t)c.max_step_seqs, MB = (size_t)c.max_blocks_per_seq, slots = (size_t)c.n_state_slots;
  bool ok = true;
  {
    Mat e(c.vocab, Hp), h(c.vocab, Hp);
    for (int i = 0; i < c.vocab; ++i) { e.row(i, 0, w->embed, (size_t)i * H, H); h.row(i, 0, w->head, (size_t)i * H, H); }
    ok = ok && e.up(m->embed) && h.up(m->head) && upload_vec(m->final_norm, w->final_norm, H, Hp, 0.0f) && upload_vec(m->final_norm_b, w->final_norm_b, H, Hp, 0.0f);
  }
  auto zeroed = [&](Buf& b, size_t bytes) { return b.alloc(bytes) && (bytes == 0 || cudaMemset(b.p, 0, bytes) == cudaSuccess); };
  auto grow = [](size_t& a, size_t b) { if (b > a) a = b; };
  m->layers.resize((size_t)c.n_layers);
  m->weights.resize((size_t)c.n_layers);
  size_t proj_w = 0, tail_w = 0, act_w = 0, ff_w = 0, z_w = 0, low_w = 0, xbc_w = 0, ws = 0, scratch = 0;
  const size_t cap_tokens = MB * kKvBlock > T ? MB * kKvBlock : T;
  m->max_chunks = (int)(S * ((MB * kKvBlock + 511) / 512));
  for (int l = 0; l < c.n_layers && ok; ++l) {
    MLayer& L = m->layers[(size_t)l];
    L.owner = c.layers[l].weights_of;
    L.c = c.layers[L.owner];
    layout(L);
    if (L.owner == l) ok = ok && upload_layer(m, L, m->weights[(size_t)l], w->layers[l]);
    grow(proj_w, (size_t)L.groups.n_main);
    grow(tail_w, (size_t)L.groups.ld_tail);
    grow(act_w, (size_t)L.Kout);
    grow(ff_w, (size_t)L.Fp);
    if (L.c.kind == LG_MIXER_SSD) {
      grow(ff_w, (size_t)L.c.ssd_heads * L.Vp);
      grow(xbc_w, (size_t)L.channels);
      ok = ok && zeroed(L.state, slots * L.c.ssd_heads * L.Np * L.Vp * 4) && zeroed(L.conv_state, slots * 2 * (L.c.ssd_taps - 1) * L.channels * 4);
    } else {
      const size_t pool = (size_t)c.n_pool_blocks * kKvBlock * L.c.kv_heads * L.Dh * esz;
      grow(z_w, (size_t)L.Rw);
      grow(low_w, (size_t)2 * L.Lr);
      if (!c.is_f32) {
        grow(ws, logismos_paged_prefix_attention_scratch_bytes((int32_t)cap_tokens, c.max_step_seqs, L.c.kv_heads, L.Dh));
        grow(scratch, logismos_paged_decode_scratch_bytes(m->max_chunks, L.c.heads, L.Dh));
      }
      ok = ok && zeroed(L.kpool, pool) && zeroed(L.vpool, pool) && zeroed(L.shift, slots * 2 * Hp * 4) && zeroed(L.state, slots * L.c.tm_heads * L.Dp * L.Dp * 4);
    }
  }
  StepLimits lim;
  lim.max_pos = (int64_t)1 << 30;            // no positional table: the block table is the limit
  lim.max_blocks_per_seq = c.max_blocks_per_seq;
  lim.n_pool_blocks = c.n_pool_blocks;
  lim.max_step_tokens = c.max_step_tokens;
  lim.max_step_seqs = c.max_step_seqs;
  lim.n_state_slots = c.n_state_slots;
  lim.prefix_cap_tokens = cap_tokens;
  lim.extra_bytes = (size_t)c.max_out_rows * 4;
  m->acc_bytes = (T < (size_t)kAccRows ? T : (size_t)kAccRows) * Hp * 4;
  ok = ok && m->x.alloc(T * Hp * 4) && zeroed(m->h, (1 + kMixes) * T * Hp * esz) && zeroed(m->proj, T * proj_w * esz) && m->tail.alloc(T * tail_w * 4) &&
       zeroed(m->act, T * act_w * esz) && zeroed(m->ffb, T * ff_w * esz) && zeroed(m->xbc, T * xbc_w * esz) && m->y.alloc(T * Hp * 4) && m->y_acc.alloc(m->acc_bytes) &&
       m->last.alloc((size_t)c.max_out_rows * Hp * esz) && m->logits.alloc((size_t)c.max_out_rows * c.vocab * 4) && m->tokens.alloc((size_t)c.max_out_rows * 4) &&
       m->status.alloc(4) && (!c.keep_layers || m->hist.alloc((size_t)(c.n_layers + 1) * T * Hp * 4));
  if (!c.is_f32)
    ok = ok && m->low2.alloc(T * low_w * 2) && m->z.alloc(T * z_w * 4) && m->attn_ws.alloc(ws) && m->dec_scratch.alloc(scratch);
  ok = ok && cudaMemset(m->status.p, 0, 4) == cudaSuccess && m->batch.alloc(lim) && m->dev_batch.alloc(m->batch.capacity) &&
       cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking) == cudaSuccess;
  m->slot_phase.assign(slots, 0);
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
  uint32_t rc = 0;
  size_t count = 0;
  auto want = [&](const std::string& name, std::initializer_list<int64_t> shape, const void** out) {
    ++count;
    return (rc = want_tensor(r, name, LG_DT_BF16, shape, out)) == 0;
  };
  auto want_norm = [&](const std::string& name, const void** wt, const void** bias) {
    return want(name, {c.width}, wt) && want(name + ".b", {c.width}, bias);
  };
  auto first_dim = [&](const std::string& name, int32_t* out) {
    lg_tensor_view_t v;
    if ((rc = get_view(r, name.c_str(), &v))) return false;
    if (v.rank != 2 || v.shape[0] <= 0 || v.shape[0] > 1 << 20) { rc = fail(LG_EMB_COMPUTE, name + ": expected a matrix"); return false; }
    *out = (int32_t)v.shape[0];
    return true;
  };
  const int64_t H = c.width, V = c.vocab;
  lg_mixer_weights_t w{};
  std::vector<lg_mixer_layer_weights_t> layers((size_t)c.n_layers);
  if (!(want("embed", {V, H}, &w.embed) && want_norm("final.norm", &w.final_norm, &w.final_norm_b) && want("head", {V, H}, &w.head))) return rc;
  for (int i = 0; i < c.n_layers; ++i) {
    lg_mixer_layer_config_t& y = lc[(size_t)i];
    if (y.weights_of != i) continue;
    lg_mixer_layer_weights_t& L = layers[(size_t)i];
    const std::string p = "l" + std::to_string(i) + ".", mix = p + "mix.";
    if (!want_norm(p + "norm1", &L.norm1, &L.norm1_b)) return rc;
    if (y.ff && !(want_norm(p + "norm2", &L.norm2, &L.norm2_b) && want(p + "mlp.up", {y.ff, H}, &L.up) && want(p + "mlp.down", {H, y.ff}, &L.down))) return rc;
    if (y.kind == LG_MIXER_SSD) {
      const int64_t heads = y.ssd_heads, inner = heads * y.ssd_vdim, ch = inner + 2 * (int64_t)y.ssd_groups * y.ssd_state;
      if (!(want(mix + "in", {inner + ch + heads, H}, &L.in) && want(mix + "conv", {ch, y.ssd_taps}, &L.conv) && want(mix + "conv.b", {ch}, &L.conv_b) &&
            want(mix + "dt_bias", {heads}, &L.dt_bias) && want(mix + "A_log", {heads}, &L.A_log) && want(mix + "D", {heads}, &L.D) &&
            want(mix + "norm", {inner}, &L.norm) && want(mix + "o", {H, inner}, &L.o)))
        return rc;
      continue;
    }
    const std::string a = mix + "left.", b = mix + "right.";
    if (!first_dim(a + "rel", &y.bias_rows) || !first_dim(b + "w1", &y.tm_rank)) return rc;
    if (const char* what = check_tensor_sizes(y)) return unsupported(what);
    const int64_t QD = (int64_t)y.heads * y.dim, HV = (int64_t)y.heads * y.vdim, HD = (int64_t)y.tm_heads * y.tm_dim, R = y.tm_rank;
    if (!(want(a + "q", {QD, H}, &L.left_q) && want(a + "k", {(int64_t)y.kv_heads * y.dim, H}, &L.left_k) && want(a + "v", {(int64_t)y.kv_heads * y.vdim, H}, &L.left_v) &&
          want(a + "rel", {y.bias_rows, y.heads}, &L.left_rel) && want(a + "g", {HV, H}, &L.left_g) && want(a + "o", {H, HV}, &L.left_o)))
      return rc;
    const char* order[kMixes] = {"mu.r", "mu.k", "mu.v", "mu.g", "mu.w"};
    for (int s = 0; s < kMixes; ++s)
      if (!want(b + order[s], {H}, &L.mu[s])) return rc;
    if (!(want(b + "r", {HD, H}, &L.right_r) && want(b + "k", {HD, H}, &L.right_k) && want(b + "v", {HD, H}, &L.right_v) && want(b + "g", {HD, H}, &L.right_g) &&
          want(b + "w1", {R, H}, &L.right_w1) && want(b + "w2", {HD, R}, &L.right_w2) && want(b + "w0", {HD}, &L.right_w0) &&
          want(b + "u", {y.tm_heads, y.tm_dim}, &L.right_u) && want(b + "norm", {HD}, &L.right_norm) && want(b + "o", {H, HD}, &L.right_o)))
      return rc;
  }
  if (r->ordering.size() != count)
    return fail(LG_EMB_COMPUTE, "expected " + std::to_string(count) + " tensors in the archive, got " + std::to_string(r->ordering.size()));
  w.layers = layers.data();
  return lg_mixer_create(device, &c, &w, model);
}

void lg_mixer_destroy(void* model) {
  if (!model) return;
  Mixer* m = static_cast<Mixer*>(model);
  cudaSetDevice(m->device);
  Buf* bufs[] = {&m->embed, &m->head, &m->final_norm, &m->final_norm_b, &m->x, &m->h, &m->proj, &m->tail, &m->low2, &m->z, &m->xbc, &m->act, &m->ffb, &m->y,
                 &m->y_acc, &m->hist, &m->last, &m->logits, &m->tokens, &m->status, &m->attn_ws, &m->dec_scratch, &m->dev_batch};
  for (Buf* b : bufs) b->release();
  for (MWeights& W : m->weights) {
    Buf* wb[] = {&W.norm1, &W.norm1_b, &W.norm2, &W.norm2_b, &W.w_up, &W.w_down, &W.w_in, &W.w_out, &W.conv, &W.conv_b, &W.dt_bias, &W.A_log, &W.D, &W.gain,
                 &W.bias, &W.mu, &W.w2, &W.w0, &W.u};
    for (Buf* b : wb) b->release();
  }
  for (MLayer& L : m->layers) {
    Buf* lb[] = {&L.kpool, &L.vpool, &L.shift, &L.conv_state, &L.state};
    for (Buf* b : lb) b->release();
  }
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
  int32_t* rows = (int32_t*)B.extra;
  if (!B.select_rows(out_rows, n_out, newl, rows)) return fail(LG_EMB_COMPUTE, "lg_mixer_step: an output row lies outside the step");
  if (!c.is_f32 && B.n_dec > 0) {
    int kv = 1, hd = 64;
    for (const MLayer& L : m->layers)
      if (L.c.kind == LG_MIXER_PARALLEL && L.c.kv_heads * L.Dh > kv * hd) { kv = L.c.kv_heads; hd = L.Dh; }
    m->chunk_tokens = logismos_pick_decode_chunk(B.ctx, B.n_dec, kv, hd);
    m->total_chunks = logismos_build_decode_chunks(B.ctx, B.n_dec, m->chunk_tokens, B.chunks);
    if (m->total_chunks < 0 || m->total_chunks > m->max_chunks) return fail(LG_EMB_COMPUTE, "lg_mixer_step: decode chunk count exceeds the scratch");
  }
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
