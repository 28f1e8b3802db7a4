// Host-side executor of one continuous-batching step over a latent-attention decoder stack (parallel
// blocks with an input convolution and a depth average; see lg_latent_* in logismos_model.h). The
// reference has no decoder model; the contract is that of the other executors: a packed step equals
// running every sequence alone.
//
// A step packs decode tokens first and prefill chunks after them (step_batch.h):
//   embed -> X_0; per layer [ depth average + norm + both input convolutions (one launch in a pure decode
//   step) -> query and key/value latents (one GEMM, fp32 out) -> norms + cache store -> queries -> attention
//   into the left columns of one activation row, gated feed-forward into the right columns -> one GEMM over
//   [W_o | W_down] accumulates both sublayers into the residual row, which holds the averaged stream ]
//   -> wanted rows: depth average + final norm -> head with soft cap (fp32) -> greedy argmax
// Attention, bf16: decode rows stay in the latent space (W_uk folded into the query, W_uv applied to the
// output, batched per head) over the paged latents; prefill rows gather their sequence's latents, expand them
// to keys and transposed values with two GEMMs and run the tcgen05 attention kernel. fp32: every row in the
// latent space with the fp32 kernels.
// Every matrix is padded at load (inputs and outputs to multiples of 64, heads to 64 / 128 / 256) with zeros,
// which keeps the padding of every activation zero.
#include <cuda_runtime.h>

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

constexpr int kAccRows = 512;

struct LLayer {
  lg_latent_layer_config_t c{};
  int D = 0, Qp = 0, Rp = 0, Fp = 0, Cw = 0;  // padded head, latent and ff sizes; width of an activation row
  Buf gain, conv1, conv2, gain_q, gain_c, dwa;
  Buf w_in, w_uq, w_ukt, w_uk, w_uv, w_gu, b_gu, w_out, b_out;
  Buf pool, state;
};

struct Latent {
  lg_latent_config_t cfg{};
  std::vector<lg_latent_layer_config_t> layer_cfg;
  int device = 0, Hp = 0;
  Buf embed, final_gain, head, one;
  std::vector<LLayer> layers;
  Buf hist, h1, h2, raw, raw_acc, cq, q, qlat, olat, cat, last, logits, tokens, status, inv_rms;
  Buf lat, kbuf, vt, kv_start, dec_scratch, dev_batch;
  StepBatch batch;
  std::vector<uint8_t> slot_phase;  // per state slot: the copy that holds its state
  cudaStream_t stream = nullptr;
  std::mutex mu;
  int n_out = 0, total_chunks = 0, chunk_tokens = 64, launches = 0;
  // `raw_acc` is all zero between its uses (the kernel that reads it zeroes it); a step that failed part-way may have left
  // sums there, so the next one clears it
  bool acc_dirty = true;
  size_t acc_bytes = 0;
  bool ready = false;               // a step's indices are on the device (replay)
  template <typename T> T* dev(T* host) const { return (T*)((uint8_t*)dev_batch.p + ((uint8_t*)host - batch.pinned)); }
};

struct Lin { const void* a; int lda; const Buf* w; int n, k; const Buf* bias; void* out; int ldc; int epi; float p0 = 0, p1 = 0, p2 = 0; };

uint32_t linear(Latent* m, const Lin& l, int rows, cudaStream_t s) {
  const void* b = l.bias ? l.bias->p : nullptr;
  m->launches += 1;
  if (m->cfg.is_f32)
    return logismos_launch_linear_f32(l.a, l.w->p, b, l.out, rows, l.n, l.k, l.lda, l.ldc, 1, 0, 0, 0, l.epi == LG_EPI_BF16 ? LG_EPI_F32 : l.epi,
                                      l.p0, l.p1, l.p2, s);
  if (stream_weights(rows, l.n, l.k, l.epi))
    return logismos_launch_linear_small_bf16(l.a, l.w->p, b, l.out, rows, l.n, l.k, l.lda, l.ldc, 1, 0, 0, 0, l.epi, l.p0, l.p1, l.p2, s);
  return logismos_launch_linear_t_act_bf16(l.a, l.w->p, b, l.out, rows, l.n, l.k, l.lda, l.ldc, l.epi | LG_EPI_STATIC_W, l.p0, l.p1, l.p2,
                                           m->status.p, s);
}

// one small matrix per head: out[r, h, :n] = W_h a[r, h, :k]
uint32_t head_linear(Latent* m, const void* a, int lda, const Buf& w, int heads, int n, int k, void* out, int ldc, int rows, cudaStream_t s) {
  m->launches += 1;
  if (m->cfg.is_f32)
    return logismos_launch_linear_f32(a, w.p, nullptr, out, rows, n, k, lda, ldc, heads, k, (int64_t)n * k, n, LG_EPI_F32, 0, 0, 0, s);
  return logismos_launch_linear_small_bf16(a, w.p, nullptr, out, rows, n, k, lda, ldc, heads, k, (int64_t)n * k, n, LG_EPI_BF16, 0, 0, 0, s);
}

uint32_t attention(Latent* m, LLayer& L, cudaStream_t s) {
  const lg_latent_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int HD = L.c.heads * L.D, HR = L.c.heads * L.Rp, MB = c.max_blocks_per_seq;
  void* st = m->status.p;
  if (c.is_f32) {
    LG_TRY(head_linear(m, m->q.p, HD, L.w_ukt, L.c.heads, L.Rp, L.D, m->qlat.p, HR, B.T, s), "latent queries");
    LG_TRY(logismos_launch_latent_attention_f32(m->qlat.p, L.pool.p, m->dev(B.tables), m->dev(B.seq_ids), m->dev(B.pos), m->olat.p, B.T, MB,
                                                c.n_pool_blocks, L.c.heads, L.Rp, L.c.scale, nullptr, 0, st, s), "latent attention");
    m->launches += 1;
    LG_TRY(head_linear(m, m->olat.p, HR, L.w_uv, L.c.heads, L.D, L.Rp, m->cat.p, L.Cw, B.T, s), "latent values");
    return 0;
  }
  if (B.n_dec > 0) {
    LG_TRY(head_linear(m, m->q.p, HD, L.w_ukt, L.c.heads, L.Rp, L.D, m->qlat.p, HR, B.n_dec, s), "latent queries");
    LG_TRY(logismos_launch_latent_decode_bf16(m->qlat.p, L.pool.p, m->dev(B.tables), m->dev(B.ctx), m->dev(B.chunks), m->olat.p, m->dec_scratch.p,
                                              B.n_dec, m->total_chunks, m->chunk_tokens, MB, c.n_pool_blocks, L.c.heads, L.Rp, L.c.scale, nullptr, 0, nullptr, 0, 0, st, s),
           "latent decode");
    m->launches += m->total_chunks > B.n_dec ? 2 : 1;
    LG_TRY(head_linear(m, m->olat.p, HR, L.w_uv, L.c.heads, L.D, L.Rp, m->cat.p, L.Cw, B.n_dec, s), "latent values");
  }
  const uint16_t* q = (const uint16_t*)m->q.p + (size_t)B.n_dec * HD;
  uint16_t* out = (uint16_t*)m->cat.p + (size_t)B.n_dec * L.Cw;
  for (const PrefixRun& r : B.runs) {
    const int ns = r.s1 - r.s0, tp = logismos_latent_gather_rows(r.total_kv, ns);
    const int32_t* kv_lens = m->dev(B.pre_kv) + r.s0;
    LG_TRY(logismos_launch_latent_gather_bf16(L.pool.p, m->dev(B.tables) + (size_t)(B.n_dec + r.s0) * MB, MB, c.n_pool_blocks, kv_lens, m->lat.p,
                                              m->kv_start.p, r.total_kv, ns, r.max_kv, L.Rp, st, s), "latent gather");
    LG_TRY(logismos_launch_linear_t_act_bf16(m->lat.p, L.w_uk.p, nullptr, m->kbuf.p, tp, HD, L.Rp, L.Rp, HD, LG_EPI_BF16 | LG_EPI_STATIC_W, 0, 0, 0,
                                             st, s), "keys");
    LG_TRY(logismos_launch_linear_t_act_bf16(L.w_uv.p, m->lat.p, nullptr, m->vt.p, HD, tp, L.Rp, L.Rp, tp, LG_EPI_BF16, 0, 0, 0, st, s), "values");
    LG_TRY(logismos_launch_varlen_attention_kv_tc_bf16(q, HD, m->dev(B.cu_pre) + r.s0, kv_lens, m->kv_start.p, m->kbuf.p, m->vt.p, tp, out, L.Cw,
                                                       B.T - B.n_dec, ns, r.max_q, L.c.heads, L.c.heads, L.D, L.c.scale, nullptr, 0, st, s), "attention");
    m->launches += 4;
  }
  return 0;
}

uint32_t run_device(Latent* m, cudaStream_t s) {
  const lg_latent_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int Hp = m->Hp, T = B.T, f32 = c.is_f32;
  const size_t esz = f32 ? 4 : 2;
  const int64_t snap = (int64_t)c.max_step_tokens * Hp;
  float* hist = (float*)m->hist.p;
  void* st = m->status.p;
  m->launches = 1;
  if (m->acc_dirty) {
    LG_TRY(cudaMemsetAsync(m->raw_acc.p, 0, m->acc_bytes, s), "clear accumulation workspace");
    m->acc_dirty = false;
  }
  LG_TRY(logismos_launch_embed_lookup_bf16(m->embed.p, m->dev(B.ids), hist, T, Hp, c.vocab, s), "embed_lookup");
  const Buf* coef = &m->one;
  for (int l = 0; l < c.n_layers; ++l) {
    LLayer& L = m->layers[(size_t)l];
    const int HD = L.c.heads * L.D;
    float* x = hist + (size_t)(l + 1) * snap;
    void* h2 = L.c.ff ? m->h2.p : nullptr;
    if (B.n_pre == 0) {
      LG_TRY(logismos_launch_depth_mix_conv_decode(hist, snap, l + 1, coef->p, x, L.gain.p, L.conv1.p, L.conv2.p, m->h1.p, h2, f32, L.state.p,
                                                   m->dev(B.state), m->dev(B.fresh), m->dev(B.phase), T, c.width, Hp, c.rms_eps, c.conv_taps, s),
             "depth average, norm and convolution");
      m->launches += 1;
    } else {
      LG_TRY(logismos_launch_depth_mix_f32(hist, snap, l + 1, coef->p, nullptr, T, x, m->inv_rms.p, nullptr, nullptr, f32, T, c.width, Hp, c.rms_eps, st, s),
             "depth average");
      LG_TRY(logismos_launch_norm_conv(x, m->inv_rms.p, L.gain.p, L.conv1.p, L.conv2.p, m->h1.p, h2, f32, L.state.p, m->dev(B.state), m->dev(B.fresh),
                                       m->dev(B.phase), m->dev(B.seq_ids), m->dev(B.cu), T, Hp, c.conv_taps, s), "norm and convolution");
      m->launches += 2;
    }
    // a few dozen rows: the narrow projection is accumulated, so that the tiles split its reduction over the idle SMs
    const bool acc = !f32 && T > 32 && T <= kAccRows && !logismos_get_deterministic();
    float* raw = (float*)(acc ? m->raw_acc.p : m->raw.p);
    LG_TRY(linear(m, {m->h1.p, Hp, &L.w_in, L.Qp + L.Rp, Hp, nullptr, raw, L.Qp + L.Rp, acc ? LG_EPI_RESID_F32 : LG_EPI_F32}, T, s), "latent projections");
    LG_TRY(logismos_launch_latent_norm_store(raw, L.Qp + L.Rp, L.gain_q.p, L.gain_c.p, m->cq.p, L.pool.p, m->dev(B.slots), T, L.Qp, L.c.q_rank,
                                             L.Rp, L.c.kv_rank, c.rms_eps, (int64_t)c.n_pool_blocks * kKvBlock, f32, acc, nullptr, st, s), "latent norm and store");
    m->launches += 1;
    LG_TRY(linear(m, {m->cq.p, L.Qp, &L.w_uq, HD, L.Qp, nullptr, m->q.p, HD, LG_EPI_BF16}, T, s), "queries");
    if (uint32_t rc = attention(m, L, s)) return rc;
    if (L.c.ff)
      LG_TRY(linear(m, {m->h2.p, Hp, &L.w_gu, 2 * L.Fp, Hp, &L.b_gu, (uint8_t*)m->cat.p + (size_t)HD * esz, L.Cw, LG_EPI_GLU_CLAMP, c.glu_alpha,
                        L.c.glu_limit, c.glu_shift}, T, s), "gated feed-forward");
    LG_TRY(linear(m, {m->cat.p, L.Cw, &L.w_out, Hp, L.Cw, L.c.ff ? &L.b_out : nullptr, x, Hp, LG_EPI_RESID_F32}, T, s), "output projection");
    coef = &L.dwa;
  }
  if (m->n_out > 0) {
    LG_TRY(logismos_launch_depth_mix_f32(hist, snap, c.n_layers + 1, coef->p, m->dev((int32_t*)B.extra), T, nullptr, nullptr, m->final_gain.p, m->last.p,
                                         f32, m->n_out, c.width, Hp, c.rms_eps, st, s), "final depth average and norm");
    LG_TRY(linear(m, {m->last.p, Hp, &m->head, c.vocab, Hp, nullptr, m->logits.p, c.vocab, LG_EPI_F32, c.logit_softcap}, m->n_out, s), "head");
    LG_TRY(logismos_launch_greedy_argmax(m->logits.p, 1, m->tokens.p, m->n_out, c.vocab, s), "greedy");
    m->launches += 2;
  }
  return 0;
}

bool upload_layer(Latent* m, LLayer& L, const lg_latent_layer_weights_t& w, int index) {
  const lg_latent_config_t& c = m->cfg;
  const int H = c.width, Hp = m->Hp, heads = L.c.heads, D = L.D, HD = heads * D, F = L.c.ff;
  const int dim = L.c.dim, vdim = L.c.vdim, Q = L.c.q_rank, R = L.c.kv_rank;
  bool ok = upload_vec(L.gain, w.norm1, H, Hp, c.norm_offset) && upload_conv(L.conv1, w.conv1, H, Hp, c.conv_taps) &&
            upload_vec(L.gain_q, w.dq_norm, Q, L.Qp, 0.0f) && upload_vec(L.gain_c, w.dkv_norm, R, L.Rp, 0.0f) &&
            upload_vec(L.dwa, w.dwa, index + 2, index + 2, 0.0f);
  {
    Mat a(L.Qp + L.Rp, Hp);
    for (int i = 0; i < Q; ++i) a.row(i, 0, w.dq, (size_t)i * H, H);
    for (int i = 0; i < R; ++i) a.row(L.Qp + i, 0, w.dkv, (size_t)i * H, H);
    ok = ok && a.up(L.w_in);
  }
  {
    Mat a(HD, L.Qp);
    for (int h = 0; h < heads; ++h)
      for (int d = 0; d < dim; ++d) a.row(h * D + d, 0, w.uq, ((size_t)h * dim + d) * Q, Q);
    ok = ok && a.up(L.w_uq);
  }
  {
    Mat k(HD, L.Rp), kt(heads * L.Rp, D), v(HD, L.Rp);
    for (int h = 0; h < heads; ++h) {
      for (int d = 0; d < dim; ++d) {
        k.row(h * D + d, 0, w.uk, ((size_t)h * dim + d) * R, R);
        for (int r = 0; r < R; ++r) kt.v[((size_t)h * L.Rp + r) * D + d] = bf_at(w.uk, ((size_t)h * dim + d) * R + r);
      }
      for (int d = 0; d < vdim; ++d) v.row(h * D + d, 0, w.uv, ((size_t)h * vdim + d) * R, R);
    }
    ok = ok && (c.is_f32 || k.up(L.w_uk)) && kt.up(L.w_ukt) && v.up(L.w_uv);
  }
  {
    Mat a(Hp, L.Cw);
    for (int i = 0; i < H; ++i) {
      for (int h = 0; h < heads; ++h) a.row(i, h * D, w.o, (size_t)i * heads * vdim + (size_t)h * vdim, vdim);
      if (F) a.row(i, HD, w.down, (size_t)i * F, F);
    }
    ok = ok && a.up(L.w_out);
  }
  if (F) {  // gate and up rows interleaved in blocks of 32, as the gated epilogue reads them
    Mat a(2 * L.Fp, Hp);
    std::vector<float> b((size_t)2 * L.Fp, 0.0f);
    for (int i = 0; i < F; ++i) {
      const int g = (i / 32) * 64 + i % 32;
      a.row(g, 0, w.gate, (size_t)i * H, H);
      a.row(g + 32, 0, w.up, (size_t)i * H, H);
      b[(size_t)g] = f_at(w.gate_b, (size_t)i);
      b[(size_t)g + 32] = f_at(w.up_b, (size_t)i);
    }
    ok = ok && a.up(L.w_gu) && L.b_gu.upload(b.data(), b.size() * 4) && upload_vec(L.b_out, w.down_b, H, Hp, 0.0f) &&
         upload_conv(L.conv2, w.conv2, H, Hp, c.conv_taps);
  }
  return ok;
}

const char* check_config(const lg_latent_config_t& c) {
  if (c.vocab <= 0 || c.width <= 0 || c.width > 16384 || c.n_layers < 0 || (c.n_layers > 0 && !c.layers)) return "vocab, width (<= 16384) or layer count";
  if (c.conv_taps < 1 || c.conv_taps > 8) return "convolution taps must be 1..8";
  if (c.n_pool_blocks <= 0 || c.max_blocks_per_seq <= 0 || c.max_step_tokens <= 0 || c.max_step_seqs <= 0 || c.max_step_seqs > 65535 ||
      c.n_state_slots <= 0 || c.max_out_rows <= 0)
    return "pool, step or slot sizes";
  for (int l = 0; l < c.n_layers; ++l) {
    const lg_latent_layer_config_t& y = c.layers[l];
    if (y.heads <= 0 || y.dim <= 0 || y.vdim <= 0 || y.dim > 256 || y.vdim > 256) return "heads, or head dimensions above 256";
    if (y.q_rank <= 0 || y.kv_rank <= 0 || y.kv_rank > 1024) return "latent sizes (kv_rank <= 1024)";
    if (y.ff < 0 || !(y.scale > 0.0f)) return "feed-forward size, or a score scale that is not positive";
  }
  return nullptr;
}

}  // namespace

extern "C" {

uint32_t lg_latent_create(int32_t device, const lg_latent_config_t* cfg, const lg_latent_weights_t* w, void** model) {
  if (!cfg || !w || !model) { set_error("null argument"); return LG_EMB_COMPUTE; }
  *model = nullptr;
  if (const char* what = check_config(*cfg)) { set_error(std::string("unsupported latent-attention config: ") + what); return LG_EMB_COMPUTE; }
  if (cudaSetDevice(device) != cudaSuccess) { set_error("cudaSetDevice failed"); return LG_EMB_COMPUTE; }
  Latent* m = new Latent();
  m->layer_cfg.assign(cfg->layers, cfg->layers + cfg->n_layers);
  m->cfg = *cfg;
  m->cfg.layers = m->layer_cfg.data();
  const lg_latent_config_t& c = m->cfg;
  m->device = device;
  m->Hp = r64(c.width);
  const int H = c.width, Hp = m->Hp;
  const size_t esz = c.is_f32 ? 4 : 2;
  bool ok = true;
  {
    Mat e(c.vocab, Hp), h(c.vocab, Hp);
    for (int i = 0; i < c.vocab; ++i) { e.row(i, 0, w->embed, (size_t)i * H, H); h.row(i, 0, w->head, (size_t)i * H, H); }
    const float one = 1.0f;
    ok = ok && e.up(m->embed) && h.up(m->head) && m->one.upload(&one, 4) && upload_vec(m->final_gain, w->final_norm, H, Hp, c.norm_offset);
  }
  m->layers.resize((size_t)c.n_layers);
  size_t in_w = 0, q_w = 0, hd_w = 0, hr_w = 0, cat_w = 0, r_w = 0, scratch = 0;
  const int max_chunks = logismos_latent_max_chunks(c.max_step_seqs);
  for (int l = 0; l < c.n_layers && ok; ++l) {
    LLayer& L = m->layers[(size_t)l];
    L.c = c.layers[l];
    const int d = L.c.dim > L.c.vdim ? L.c.dim : L.c.vdim;
    L.D = d <= 64 ? 64 : d <= 128 ? 128 : 256;
    L.Qp = r64(L.c.q_rank);
    L.Rp = r64(L.c.kv_rank);
    L.Fp = r64(L.c.ff);
    L.Cw = L.c.heads * L.D + L.Fp;
    ok = ok && upload_layer(m, L, w->layers[l], l);
    const size_t pool_bytes = (size_t)c.n_pool_blocks * kKvBlock * L.Rp * esz;
    const size_t state_bytes = (size_t)c.n_state_slots * 2 * (c.conv_taps - 1) * Hp * 4;
    ok = ok && L.pool.alloc(pool_bytes) && cudaMemset(L.pool.p, 0, pool_bytes) == cudaSuccess;
    ok = ok && L.state.alloc(state_bytes) && (state_bytes == 0 || cudaMemset(L.state.p, 0, state_bytes) == cudaSuccess);
    auto grow = [](size_t& a, size_t b) { if (b > a) a = b; };
    grow(in_w, (size_t)(L.Qp + L.Rp));
    grow(q_w, (size_t)L.Qp);
    grow(hd_w, (size_t)L.c.heads * L.D);
    grow(hr_w, (size_t)L.c.heads * L.Rp);
    grow(cat_w, (size_t)L.Cw);
    grow(r_w, (size_t)L.Rp);
    grow(scratch, logismos_latent_decode_scratch_bytes(max_chunks, L.c.heads, L.Rp));
  }
  const size_t T = (size_t)c.max_step_tokens, S = (size_t)c.max_step_seqs, MB = (size_t)c.max_blocks_per_seq;
  const size_t lat_rows = c.is_f32 ? T : S;  // rows that attend in the latent space
  StepLimits lim;
  lim.max_pos = (int64_t)1 << 30;            // no positional table: the block table is the limit
  lim.max_blocks_per_seq = c.max_blocks_per_seq;
  lim.n_pool_blocks = c.n_pool_blocks;
  lim.max_step_tokens = c.max_step_tokens;
  lim.max_step_seqs = c.max_step_seqs;
  lim.n_state_slots = c.n_state_slots;
  lim.prefix_cap_tokens = MB * kKvBlock > T ? MB * kKvBlock : T;
  lim.extra_bytes = (size_t)c.max_out_rows * 4;
  m->acc_bytes = (T < (size_t)kAccRows ? T : (size_t)kAccRows) * in_w * 4;
  ok = ok && m->hist.alloc((size_t)(c.n_layers + 1) * T * Hp * 4) && m->h1.alloc(T * Hp * esz) && m->h2.alloc(T * Hp * esz) && m->raw.alloc(T * in_w * 4) && m->raw_acc.alloc(m->acc_bytes) &&
       m->cq.alloc(T * q_w * esz) && m->q.alloc(T * hd_w * esz) && m->qlat.alloc(lat_rows * hr_w * esz) && m->olat.alloc(lat_rows * hr_w * esz) &&
       m->cat.alloc(T * cat_w * esz) && m->last.alloc((size_t)c.max_out_rows * Hp * esz) && m->logits.alloc((size_t)c.max_out_rows * c.vocab * 4) &&
       m->tokens.alloc((size_t)c.max_out_rows * 4) && m->status.alloc(4) && m->inv_rms.alloc(T * 4);
  if (!c.is_f32) {
    const size_t tp = (size_t)logismos_latent_gather_rows((int32_t)lim.prefix_cap_tokens, c.max_step_seqs);
    ok = ok && m->lat.alloc(tp * r_w * 2) && m->kbuf.alloc(tp * hd_w * 2) && m->vt.alloc(tp * hd_w * 2) && m->kv_start.alloc(S * 4) && m->dec_scratch.alloc(scratch);
  }
  ok = ok && cudaMemset(m->status.p, 0, 4) == cudaSuccess && m->batch.alloc(lim) && m->dev_batch.alloc(m->batch.capacity) &&
       cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking) == cudaSuccess;
  m->slot_phase.assign((size_t)c.n_state_slots, 0);
  if (!ok || cudaDeviceSynchronize() != cudaSuccess) {
    set_error(std::string("lg_latent_create: allocation or upload failed: ") + cudaGetErrorString(cudaGetLastError()));
    lg_latent_destroy(m);
    return LG_EMB_COMPUTE;
  }
  *model = m;
  return LG_EMB_OK;
}

uint32_t lg_latent_load(int32_t device, const char* path, const lg_latent_config_t* cfg, void** model) {
  if (!path || !cfg || !model) return fail(LG_EMB_COMPUTE, "null argument");
  *model = nullptr;
  const lg_latent_config_t& c = *cfg;
  if (const char* what = check_config(c)) return fail(LG_EMB_COMPUTE, std::string("unsupported latent-attention config: ") + what);
  Archive* r = nullptr;
  if (uint32_t rc = open_archive(path, &r)) return rc;
  struct Guard { Archive* r; ~Guard() { delete r; } } guard{r};
  uint32_t rc = 0;
  size_t count = 0;
  auto want = [&](const std::string& name, std::initializer_list<int64_t> shape, const void** out) {
    ++count;
    return (rc = want_tensor(r, name, LG_DT_BF16, shape, out)) == 0;
  };
  const int64_t H = c.width, V = c.vocab, taps = c.conv_taps;
  lg_latent_weights_t w{};
  std::vector<lg_latent_layer_weights_t> layers((size_t)c.n_layers);
  if (!(want("embed", {V, H}, &w.embed) && want("final.norm", {H}, &w.final_norm) && want("head", {V, H}, &w.head))) return rc;
  for (int i = 0; i < c.n_layers; ++i) {
    const std::string p = "l" + std::to_string(i) + ".";
    const lg_latent_layer_config_t& y = c.layers[i];
    lg_latent_layer_weights_t& L = layers[(size_t)i];
    const int64_t Q = y.q_rank, R = y.kv_rank, HD = (int64_t)y.heads * y.dim, HV = (int64_t)y.heads * y.vdim, F = y.ff;
    if (!(want(p + "norm1", {H}, &L.norm1) && want(p + "mix.dq", {Q, H}, &L.dq) && want(p + "mix.dq.norm", {Q}, &L.dq_norm) &&
          want(p + "mix.uq", {HD, Q}, &L.uq) && want(p + "mix.dkv", {R, H}, &L.dkv) && want(p + "mix.dkv.norm", {R}, &L.dkv_norm) &&
          want(p + "mix.uk", {HD, R}, &L.uk) && want(p + "mix.uv", {HV, R}, &L.uv) && want(p + "mix.o", {H, HV}, &L.o) &&
          want(p + "canon1", {H, taps}, &L.conv1) && want(p + "dwa", {(int64_t)i + 2}, &L.dwa)))
      return rc;
    if (F && !(want(p + "mlp.gate", {F, H}, &L.gate) && want(p + "mlp.gate.b", {F}, &L.gate_b) && want(p + "mlp.up", {F, H}, &L.up) &&
               want(p + "mlp.up.b", {F}, &L.up_b) && want(p + "mlp.down", {H, F}, &L.down) && want(p + "mlp.down.b", {H}, &L.down_b) &&
               want(p + "canon2", {H, taps}, &L.conv2)))
      return rc;
    // a layer without a feed-forward has nothing that reads a second filter; its tensor may still be stored
    if (!F && r->index.count(p + "canon2") && !want(p + "canon2", {H, taps}, &L.conv2)) return rc;
  }
  if (r->ordering.size() != count)
    return fail(LG_EMB_COMPUTE, "expected " + std::to_string(count) + " tensors in the archive, got " + std::to_string(r->ordering.size()));
  w.layers = layers.data();
  return lg_latent_create(device, cfg, &w, model);
}

void lg_latent_destroy(void* model) {
  if (!model) return;
  Latent* m = static_cast<Latent*>(model);
  cudaSetDevice(m->device);
  Buf* bufs[] = {&m->embed, &m->final_gain, &m->head, &m->one, &m->hist, &m->h1, &m->h2, &m->raw, &m->raw_acc, &m->cq, &m->q, &m->qlat, &m->olat, &m->cat,
                 &m->last, &m->logits, &m->tokens, &m->status, &m->inv_rms, &m->lat, &m->kbuf, &m->vt, &m->kv_start, &m->dec_scratch, &m->dev_batch};
  for (Buf* b : bufs) b->release();
  for (LLayer& L : m->layers) {
    Buf* lb[] = {&L.gain, &L.conv1, &L.conv2, &L.gain_q, &L.gain_c, &L.dwa, &L.w_in, &L.w_uq, &L.w_ukt, &L.w_uk, &L.w_uv, &L.w_gu, &L.b_gu,
                 &L.w_out, &L.b_out, &L.pool, &L.state};
    for (Buf* b : lb) b->release();
  }
  m->batch.release();
  if (m->stream) cudaStreamDestroy(m->stream);
  delete m;
}

uint32_t lg_latent_step(void* model, const uint32_t* host_ids, const int32_t* cached, const int32_t* newl, int32_t n_seqs, const int32_t* tables,
                        const int32_t* state_slots, const int32_t* out_rows, int32_t n_out, uint32_t* next_tokens) {
  Latent* m = static_cast<Latent*>(model);
  if (!m) { set_error("lg_latent_step: null model"); return LG_EMB_COMPUTE; }
  const lg_latent_config_t& c = m->cfg;
  if (!out_rows) n_out = n_seqs;
  if (n_out < 0 || n_out > c.max_out_rows || (n_out > 0 && !next_tokens)) {
    set_error("lg_latent_step: more output rows than max_out_rows, or no room for their tokens");
    return LG_EMB_COMPUTE;
  }
  std::lock_guard<std::mutex> lock(m->mu);
  if (cudaSetDevice(m->device) != cudaSuccess) { set_error("cudaSetDevice failed"); return LG_EMB_COMPUTE; }
  StepBatch& B = m->batch;
  m->ready = false;
  if (uint32_t rc = B.build("lg_latent_step", host_ids, cached, newl, n_seqs, tables, state_slots, false)) return rc;
  for (int s = 0; s < n_seqs; ++s) B.phase[s] = m->slot_phase[(size_t)B.state[s]];
  int32_t* rows = (int32_t*)B.extra;
  if (!B.select_rows(out_rows, n_out, newl, rows)) { set_error("lg_latent_step: an output row lies outside the step"); return LG_EMB_COMPUTE; }
  if (!c.is_f32 && B.n_dec > 0) {
    int heads = 1;
    for (const LLayer& L : m->layers) if (L.c.heads > heads) heads = L.c.heads;
    m->chunk_tokens = logismos_pick_latent_chunk(B.ctx, B.n_dec, heads);
    m->total_chunks = logismos_build_decode_chunks(B.ctx, B.n_dec, m->chunk_tokens, B.chunks);
    if (m->total_chunks < 0 || m->total_chunks > logismos_latent_max_chunks(c.max_step_seqs)) {
      set_error("lg_latent_step: decode chunk count exceeds the scratch");
      return LG_EMB_COMPUTE;
    }
  }
  m->n_out = n_out;
  cudaStream_t s = m->stream;
  LG_TRY(cudaMemsetAsync(m->status.p, 0, 4, s), "clear status");
  LG_TRY(cudaMemcpyAsync(m->dev_batch.p, B.pinned, (size_t)((uint8_t*)(rows + n_out) - B.pinned), cudaMemcpyHostToDevice, s), "H2D step");
  m->ready = true;
  if (uint32_t rc = run_device(m, s)) { m->acc_dirty = true; return rc; }
  if (n_out > 0) LG_TRY(cudaMemcpyAsync(next_tokens, m->tokens.p, (size_t)n_out * 4, cudaMemcpyDeviceToHost, s), "D2H tokens");
  LG_TRY(cudaStreamSynchronize(s), "stream synchronize");
  if (const int dev_status = lg_latent_device_status(m)) {
    m->acc_dirty = true;
    char buf[256];
    std::snprintf(buf, sizeof(buf), "device status 0x%x after a step of %d tokens in %d sequences (low byte 1: a range check failed, 2: a bounded wait expired in kernel family <next byte>)",
                  dev_status, B.T, (int)n_seqs);
    set_error(buf);
    return LG_EMB_COMPUTE;
  }
  for (int k = 0; k < n_seqs; ++k) m->slot_phase[(size_t)B.state[k]] ^= 1;  // the step is complete: its states are the current ones
  return LG_EMB_OK;
}

uint32_t lg_latent_replay_device(void* model, void* stream) {
  Latent* m = static_cast<Latent*>(model);
  if (!m || !m->ready) { set_error("lg_latent_replay_device: no step has run"); return LG_EMB_COMPUTE; }
  if (cudaSetDevice(m->device) != cudaSuccess) { set_error("cudaSetDevice failed"); return LG_EMB_COMPUTE; }
  return run_device(m, (cudaStream_t)stream);
}

uint32_t lg_latent_last_logits(void* model, int32_t n_out, float* host_out) {
  Latent* m = static_cast<Latent*>(model);
  if (!m || n_out != m->n_out) { set_error("lg_latent_last_logits: n_out differs from the last step"); return LG_EMB_COMPUTE; }
  cudaSetDevice(m->device);
  LG_TRY(cudaDeviceSynchronize(), "device synchronize");
  if (n_out > 0) LG_TRY(cudaMemcpy(host_out, m->logits.p, (size_t)n_out * m->cfg.vocab * 4, cudaMemcpyDeviceToHost), "D2H logits");
  return LG_EMB_OK;
}

void* lg_latent_logits_device(void* model) { return static_cast<Latent*>(model)->logits.p; }

uint32_t lg_latent_snapshot(void* model, int32_t j, int32_t n_tokens, float* host_out) {
  Latent* m = static_cast<Latent*>(model);
  if (!m || !m->ready || j < 0 || j > m->cfg.n_layers || n_tokens != m->batch.T) { set_error("lg_latent_snapshot: bad arguments"); return LG_EMB_COMPUTE; }
  cudaSetDevice(m->device);
  LG_TRY(cudaDeviceSynchronize(), "device synchronize");
  LG_TRY(m->batch.rows_to_host((const float*)m->hist.p + (size_t)j * m->cfg.max_step_tokens * m->Hp, m->Hp, m->cfg.width, host_out), "D2H snapshot");
  return LG_EMB_OK;
}

int32_t lg_latent_launches_last_step(const void* model) { return static_cast<const Latent*>(model)->launches; }

int32_t lg_latent_device_status(void* model) {
  Latent* m = static_cast<Latent*>(model);
  int32_t v = -1;
  cudaSetDevice(m->device);
  if (cudaMemcpy(&v, m->status.p, 4, cudaMemcpyDeviceToHost) != cudaSuccess) return -1;
  return v;
}

}  // extern "C"
