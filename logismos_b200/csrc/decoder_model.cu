// Host-side executor of one continuous-batching step over a Qwen2-style decoder stack with int4
// group-32 weights and a paged KV cache (block 16). The reference has neither a decoder executor
// (crates/decoders/src/lib.rs:1-15) nor a scheduler (crates/sched/src/lib.rs:1-30); the contract
// kept is "a packed step equals running every sequence alone" through the causal variant of
// StellaLayer::forward (crates/encoders/src/stella.rs:190-206), lm_head and decode::greedy
// (crates/decode/src/lib.rs:73-83).
//
// A step packs decode tokens (one per sequence) first and prefill chunks after them:
//   embed -> per layer [ rms_norm -> QKV (int4 weights) + bias -> RoPE at each token's position ->
//   K/V rows scattered into the paged cache by slot mapping -> attention: paged decode kernel for
//   the decode rows, ragged causal attention for the prefill rows (over the chunk's own rows when every
//   chunk starts its sequence, else over keys and values gathered from the cache through the block
//   tables, so a chunk may continue a cached sequence) -> o_proj + residual ->
//   rms_norm -> gate/up with SwiGLU fused in the GEMM epilogue -> down + residual ] -> last token rows -> final norm ->
//   lm_head (int4 GEMV) -> greedy argmax.
// Contractions over the packed rows run on the tcgen05 GEMM over a per-layer bf16 expansion of the
// int4 codes; the lm_head, whose batch is the number of sequences, runs on the int4 GEMV kernel.
#include <cuda_runtime.h>

#include <cmath>
#include <cstdio>
#include <cstring>
#include <mutex>
#include <string>
#include <vector>

#include "logismos_kernels.h"
#include "logismos_model.h"

#include "model_util.h"
#include "step_batch.h"

namespace {

using namespace lgm;

struct DLayer {
  Buf norm1, norm2, bqkv, kpool, vpool;
  QMat wqkv, wo, wgu, wdown;
};

constexpr int kChunkTokens = 512;
constexpr int kBlock = kKvBlock;

struct Decoder {
  lg_decoder_config_t cfg{};
  int device = 0, head_dim = 0, qkv_dim = 0, kv_dim = 0;
  Buf tok_embed, final_norm, cos, sin;
  QMat lm_head;
  std::vector<DLayer> layers;
  // workspace
  Buf x, h, qkv, attn, qdec, gu, act, wscratch, accws, last, last_bf16, logits, tokens, status;
  Buf ids, pos, slots, cu_prefill, last_idx, dec_ctx, dec_tables, dec_chunks, dec_scratch, attn_ws, pre_kv;
  StepBatch batch;  // the last step (kept for replay and diagnostics)
  cudaStream_t stream = nullptr;
  std::mutex mu;
  int T = 0, n_dec = 0, n_pre = 0, n_seqs = 0, max_pre_len = 0, total_chunks = 0, chunk_tokens = kChunkTokens, launches = 0, logits_f32 = 0;
  size_t max_chunks = 0;
  // the fused int4 linears rely on `accws` being all zero between calls, which their finishing kernels
  // restore; a step that failed part-way may have left partial sums there, so the next one clears it
  bool acc_dirty = false;
  size_t accws_bytes = 0;
  size_t prefix_cap_tokens = 0;
};

uint32_t qlinear(Decoder* m, const void* a, const QMat& w, const void* bias, void* out, int T, int lda, int ldc,
                 int epi, cudaStream_t s) {
  LG_TRY(qlinear_any(a, w, bias, out, T, lda, ldc, epi, m->wscratch.p, m->accws.p, m->status.p, &m->launches, s), "int4 linear");
  return 0;
}

uint32_t run_device(Decoder* m, cudaStream_t s) {
  const lg_decoder_config_t& c = m->cfg;
  const int H = c.hidden, I = c.intermediate, D = m->head_dim, QKV = m->qkv_dim, KV = m->kv_dim, T = m->T;
  void* st = m->status.p;
  m->launches = 0;
  if (m->acc_dirty) {
    LG_TRY(cudaMemsetAsync(m->accws.p, 0, m->accws_bytes, s), "clear accumulation workspace");
    m->acc_dirty = false;
  }
  LG_TRY(logismos_launch_embed_lookup_bf16(m->tok_embed.p, m->ids.p, m->x.p, T, H, c.vocab, s), "embed_lookup");
  m->launches += 1;
  for (int l = 0; l < c.n_layers; ++l) {
    DLayer& L = m->layers[l];
    LG_TRY(logismos_launch_rms_norm_f32(m->x.p, L.norm1.p, m->h.p, T, H, c.rms_eps, 0, s), "rms_norm");
    if (uint32_t rc = qlinear(m, m->h.p, L.wqkv, L.bqkv.p, m->qkv.p, T, H, QKV, LG_EPI_BF16, s)) return rc;
    LG_TRY(logismos_launch_rope_halves_bf16(m->qkv.p, m->cos.p, m->sin.p, m->pos.p, T, c.n_heads + c.n_kv_heads, D, QKV,
                                            c.max_pos, st, s), "rope");
    const uint16_t* qkv16 = (const uint16_t*)m->qkv.p;
    if (c.kv_turbo3) {
      // TurboQuant 3-bit cache: rows are encoded on the way in and every sequence of the step (decode
      // tokens are chunks of one query) attends through the decoding gather, run by run
      LG_TRY(logismos_launch_paged_kv_store_turbo3(qkv16 + H, qkv16 + H + KV, QKV, L.kpool.p, L.vpool.p, m->slots.p, T, KV,
                                                   (int64_t)c.n_pool_blocks * kBlock, st, s), "paged_kv_store_turbo3");
      m->launches += 3;
      for (const PrefixRun& r : m->batch.runs) {
        LG_TRY(logismos_launch_paged_prefix_attention_turbo3_bf16(
                   qkv16, QKV, (const int32_t*)m->cu_prefill.p + r.s0, (const int32_t*)m->pre_kv.p + r.s0, L.kpool.p, L.vpool.p,
                   (const int32_t*)m->dec_tables.p + (size_t)r.s0 * c.max_blocks_per_seq, c.max_blocks_per_seq, c.n_pool_blocks, m->attn.p,
                   m->attn_ws.p, T, r.total_kv, r.s1 - r.s0, r.max_q, r.max_kv, c.n_heads, c.n_kv_heads, D, st, s),
               "paged_prefix_attention_turbo3");
        m->launches += 2;
      }
    } else {
    LG_TRY(logismos_launch_paged_kv_store_bf16(qkv16 + H, qkv16 + H + KV, QKV, L.kpool.p, L.vpool.p, m->slots.p, T, KV,
                                               (int64_t)c.n_pool_blocks * kBlock, st, s), "paged_kv_store");
    m->launches += 3;
    if (m->n_dec > 0) {
      // decode rows are the first n_dec rows of the packed batch: gather their q heads contiguously
      LG_TRY(cudaMemcpy2DAsync(m->qdec.p, (size_t)H * 2, m->qkv.p, (size_t)QKV * 2, (size_t)H * 2, m->n_dec,
                               cudaMemcpyDeviceToDevice, s), "q gather");
      LG_TRY(logismos_launch_paged_attention_decode_bf16(m->qdec.p, L.kpool.p, L.vpool.p, nullptr, nullptr, m->dec_tables.p,
                                                         m->dec_ctx.p, m->dec_chunks.p, m->attn.p, m->dec_scratch.p, st, m->n_dec,
                                                         m->total_chunks, m->chunk_tokens, c.max_blocks_per_seq, c.n_pool_blocks,
                                                         c.n_heads, c.n_kv_heads, D, s), "paged_attention_decode");
      m->launches += 2;
    }
    if (m->n_pre > 0 && m->batch.has_prefix) {
      // some chunk continues a cached sequence: keys and values come from the cache (the chunk's own rows
      // were stored above), gathered per run of sequences into attn_ws
      const int32_t* tabs = (const int32_t*)m->dec_tables.p + (size_t)m->n_dec * c.max_blocks_per_seq;
      for (const PrefixRun& r : m->batch.runs) {
        LG_TRY(logismos_launch_paged_prefix_attention_tc_bf16(
                   qkv16 + (size_t)m->n_dec * QKV, QKV, (const int32_t*)m->cu_prefill.p + r.s0, (const int32_t*)m->pre_kv.p + r.s0,
                   L.kpool.p, L.vpool.p, tabs + (size_t)r.s0 * c.max_blocks_per_seq, c.max_blocks_per_seq, c.n_pool_blocks,
                   (uint16_t*)m->attn.p + (size_t)m->n_dec * H, m->attn_ws.p, T - m->n_dec, r.total_kv, r.s1 - r.s0, r.max_q, r.max_kv,
                   c.n_heads, c.n_kv_heads, D, st, s),
               "paged_prefix_attention");
        m->launches += 2;
      }
    } else if (m->n_pre > 0) {  // tcgen05 kernel; V transposed into attn_ws first
      LG_TRY(logismos_launch_varlen_attention_tc_bf16(qkv16 + (size_t)m->n_dec * QKV, m->cu_prefill.p,
                                                      (uint16_t*)m->attn.p + (size_t)m->n_dec * H, m->attn_ws.p, T - m->n_dec,
                                                      m->n_pre, m->max_pre_len, c.n_heads, c.n_kv_heads, D, QKV, H, H + KV, 1, st, s),
             "varlen_attention");
      m->launches += 2;
    }
    }
    if (uint32_t rc = qlinear(m, m->attn.p, L.wo, nullptr, m->x.p, T, H, H, LG_EPI_RESID_F32, s)) return rc;
    LG_TRY(logismos_launch_rms_norm_f32(m->x.p, L.norm2.p, m->h.p, T, H, c.rms_eps, 0, s), "rms_norm");
    if (uint32_t rc = qlinear(m, m->h.p, L.wgu, nullptr, m->act.p, T, H, I, LG_EPI_SWIGLU, s)) return rc;
    if (uint32_t rc = qlinear(m, m->act.p, L.wdown, nullptr, m->x.p, T, I, H, LG_EPI_RESID_F32, s)) return rc;
    m->launches += 1;
  }
  LG_TRY(logismos_launch_gather_rows_f32(m->x.p, m->last_idx.p, m->last.p, m->n_seqs, H, T, st, s), "gather_rows");
  LG_TRY(logismos_launch_rms_norm_f32(m->last.p, m->final_norm.p, m->last_bf16.p, m->n_seqs, H, c.rms_eps, 0, s), "final_norm");
  m->launches += 2;
  if (uint32_t rc = lm_head_and_greedy(m->lm_head, m->last_bf16.p, m->logits.p, m->tokens.p, m->n_seqs, H, st, &m->logits_f32,
                                       &m->launches, s)) {
    char buf[96];
    std::snprintf(buf, sizeof(buf), "lm_head / greedy failed: %s (code %u)", cudaGetErrorString((cudaError_t)rc), rc);
    set_error(buf);
    return LG_EMB_COMPUTE;
  }
  return 0;
}

}  // namespace

extern "C" {

uint32_t lg_decoder_create(int32_t device, const lg_decoder_config_t* cfg, const lg_decoder_weights_t* w, void** model) {
  if (!cfg || !w || !model) { set_error("null argument"); return LG_EMB_COMPUTE; }
  *model = nullptr;
  const lg_decoder_config_t& c = *cfg;
  if (c.hidden <= 0 || c.n_heads <= 0 || c.n_kv_heads <= 0 || c.hidden % c.n_heads || c.n_heads % c.n_kv_heads ||
      c.hidden / c.n_heads != 128 || c.hidden % 128 || c.intermediate % 128 || c.n_layers < 0 || c.n_pool_blocks <= 0 ||
      c.max_blocks_per_seq <= 0 || c.max_step_tokens <= 0 || c.max_step_seqs <= 0 || c.max_pos <= 0 || c.vocab <= 0 ||
      c.n_heads / c.n_kv_heads > 16) {
    set_error("unsupported decoder config (head_dim must be 128; hidden and intermediate multiples of 128)");
    return LG_EMB_COMPUTE;
  }
  if (cudaSetDevice(device) != cudaSuccess) { set_error("cudaSetDevice failed"); return LG_EMB_COMPUTE; }
  Decoder* m = new Decoder();
  m->cfg = c;
  m->device = device;
  m->head_dim = c.hidden / c.n_heads;
  m->kv_dim = c.n_kv_heads * m->head_dim;
  m->qkv_dim = c.hidden + 2 * m->kv_dim;
  const size_t H = c.hidden, I = c.intermediate, KV = m->kv_dim, QKV = m->qkv_dim;
  bool ok = true;
  {
    std::vector<uint16_t> tmp((size_t)c.vocab * H);
    for (size_t i = 0; i < tmp.size(); ++i) tmp[i] = f32_to_bf16(w->tok_embed[i]);
    ok = ok && m->tok_embed.upload(tmp.data(), tmp.size() * 2);
  }
  ok = ok && m->final_norm.upload(w->final_norm, H * 4);
  ok = ok && upload_q(m->lm_head, {&w->lm_head}, {c.vocab}, (int)H);
  m->layers.resize(c.n_layers);
  const size_t pool_bytes = (size_t)c.n_pool_blocks * kBlock * (c.kv_turbo3 ? logismos_turbo3_row_bytes((int32_t)KV) : KV * 2);
  for (int l = 0; l < c.n_layers && ok; ++l) {
    const lg_decoder_layer_weights_t& lw = w->layers[l];
    DLayer& L = m->layers[l];
    ok = ok && L.norm1.upload(lw.norm1, H * 4) && L.norm2.upload(lw.norm2, H * 4);
    std::vector<float> b(QKV);
    std::memcpy(b.data(), lw.bq, H * 4);
    std::memcpy(b.data() + H, lw.bk, KV * 4);
    std::memcpy(b.data() + H + KV, lw.bv, KV * 4);
    ok = ok && L.bqkv.upload(b.data(), QKV * 4);
    ok = ok && upload_q(L.wqkv, {&lw.wq, &lw.wk, &lw.wv}, {(int)H, (int)KV, (int)KV}, (int)H);
    ok = ok && upload_q(L.wo, {&lw.wo}, {(int)H}, (int)H);
    ok = ok && upload_q_gate_up(L.wgu, lw.w_gate, lw.w_up, (int)I, (int)H);
    ok = ok && upload_q(L.wdown, {&lw.w_down}, {(int)H}, (int)I);
    if (c.keep_bf16_copy) ok = ok && make_dense_copy(L.wqkv) && make_dense_copy(L.wo) && make_dense_copy(L.wgu) && make_dense_copy(L.wdown);
    ok = ok && L.kpool.alloc(pool_bytes) && L.vpool.alloc(pool_bytes);
    ok = ok && cudaMemset(L.kpool.p, 0, pool_bytes) == cudaSuccess && cudaMemset(L.vpool.p, 0, pool_bytes) == cudaSuccess;
  }
  if (ok) {  // RoPE table in f64 then f32 (cpu_f32/mod.rs:599-619)
    const size_t half = m->head_dim / 2;
    std::vector<float> cs((size_t)c.max_pos * half), sn((size_t)c.max_pos * half);
    for (int p = 0; p < c.max_pos; ++p)
      for (size_t i = 0; i < half; ++i) {
        const double ang = (double)p * std::pow(c.rope_theta, -(2.0 * (double)i) / (double)m->head_dim);
        cs[p * half + i] = (float)std::cos(ang);
        sn[p * half + i] = (float)std::sin(ang);
      }
    ok = ok && m->cos.upload(cs.data(), cs.size() * 4) && m->sin.upload(sn.data(), sn.size() * 4);
  }
  const size_t T = c.max_step_tokens, S = c.max_step_seqs, MB = c.max_blocks_per_seq;
  size_t wmax = QKV * H;
  if (2 * I * H > wmax) wmax = 2 * I * H;
  // every sequence of a step may be a decode sequence of up to max_blocks_per_seq blocks
  m->max_chunks = S * ((MB * kBlock + kChunkTokens - 1) / kChunkTokens);
  const size_t acc_n = QKV > 2 * I ? QKV : 2 * I;
  ok = ok && m->x.alloc(T * H * 4) && m->h.alloc(T * H * 2) && m->qkv.alloc(T * QKV * 2) && m->attn.alloc(T * H * 2) &&
       m->qdec.alloc(S * H * 2) && m->gu.alloc(16) && m->act.alloc(T * I * 2) && m->wscratch.alloc(wmax * 2) &&
       m->last.alloc(S * H * 4) && m->last_bf16.alloc(S * H * 2) && m->logits.alloc(S * (size_t)c.vocab * 4) && m->accws.alloc((size_t)kFusedDequantMaxRows * acc_n * 4) &&
       m->tokens.alloc(S * 4) && m->status.alloc(4) && m->ids.alloc(T * 4) && m->pos.alloc(T * 4) && m->slots.alloc(T * 8) &&
       m->cu_prefill.alloc((S + 1) * 4) && m->last_idx.alloc(S * 4) && m->dec_ctx.alloc(S * 4) && m->dec_tables.alloc(S * MB * 4) &&
       m->dec_chunks.alloc((S + 1) * 4) && m->pre_kv.alloc(S * 4) &&
       m->dec_scratch.alloc(logismos_paged_decode_scratch_bytes((int32_t)m->max_chunks, c.n_heads, m->head_dim));
  {
    // the attention workspace serves both prefill routes; the gather route holds one run of sequences at
    // a time, and any single sequence (at most a full block table) must fit
    m->prefix_cap_tokens = MB * kBlock > T ? MB * kBlock : T;
    if (c.kv_turbo3) {  // every sequence of a step goes through the gather: room for many contexts at once
      const size_t all = S * MB * kBlock, cap = (size_t)512 * 1024;
      m->prefix_cap_tokens = all < cap ? all : cap;
      if (m->prefix_cap_tokens < MB * kBlock) m->prefix_cap_tokens = MB * kBlock;
    }
    size_t ws = logismos_varlen_attention_tc_scratch_bytes((int32_t)T, (int32_t)S, c.n_kv_heads, 128);
    const size_t ws2 = logismos_paged_prefix_attention_scratch_bytes((int32_t)m->prefix_cap_tokens, (int32_t)S, c.n_kv_heads, 128);
    if (ws2 > ws) ws = ws2;
    ok = ok && m->attn_ws.alloc(ws);
  }
  ok = ok && cudaMemset(m->status.p, 0, 4) == cudaSuccess;
  m->accws_bytes = (size_t)kFusedDequantMaxRows * acc_n * 4;
  ok = ok && cudaMemset(m->accws.p, 0, m->accws_bytes) == cudaSuccess;
  StepLimits lim;
  lim.max_pos = c.max_pos; lim.max_blocks_per_seq = c.max_blocks_per_seq; lim.n_pool_blocks = c.n_pool_blocks;
  lim.max_step_tokens = c.max_step_tokens; lim.max_step_seqs = c.max_step_seqs; lim.prefix_cap_tokens = m->prefix_cap_tokens;
  ok = ok && m->batch.alloc(lim);
  ok = ok && cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking) == cudaSuccess;
  if (!ok) {
    set_error(std::string("lg_decoder_create: allocation or upload failed: ") + cudaGetErrorString(cudaGetLastError()));
    lg_decoder_destroy(m);
    return LG_EMB_COMPUTE;
  }
  *model = m;
  return LG_EMB_OK;
}

void lg_decoder_destroy(void* model) {
  if (!model) return;
  Decoder* m = static_cast<Decoder*>(model);
  cudaSetDevice(m->device);
  Buf* bufs[] = {&m->tok_embed, &m->final_norm, &m->cos, &m->sin, &m->lm_head.codes, &m->lm_head.scales, &m->x, &m->h, &m->qkv,
                 &m->attn, &m->qdec, &m->gu, &m->act, &m->wscratch, &m->accws, &m->last, &m->last_bf16, &m->logits, &m->tokens, &m->status,
                 &m->ids, &m->pos, &m->slots, &m->cu_prefill, &m->last_idx, &m->dec_ctx, &m->dec_tables, &m->dec_chunks, &m->dec_scratch, &m->attn_ws, &m->pre_kv};
  for (Buf* b : bufs) b->release();
  for (auto& L : m->layers) {
    Buf* lb[] = {&L.norm1, &L.norm2, &L.bqkv, &L.kpool, &L.vpool, &L.wqkv.codes, &L.wqkv.scales, &L.wo.codes, &L.wo.scales,
                 &L.wgu.codes, &L.wgu.scales, &L.wdown.codes, &L.wdown.scales, &L.wqkv.dense, &L.wo.dense, &L.wgu.dense, &L.wdown.dense};
    for (Buf* b : lb) b->release();
  }
  m->batch.release();
  if (m->stream) cudaStreamDestroy(m->stream);
  delete m;
}

uint32_t lg_decoder_step(void* model, const uint32_t* host_ids, const int32_t* cached, const int32_t* newl, int32_t n_seqs,
                         const int32_t* tables, uint32_t* next_tokens) {
  Decoder* m = static_cast<Decoder*>(model);
  const lg_decoder_config_t& c = m->cfg;
  if (!next_tokens) { set_error("lg_decoder_step: null argument"); return LG_EMB_COMPUTE; }
  std::lock_guard<std::mutex> lock(m->mu);
  if (cudaSetDevice(m->device) != cudaSuccess) { set_error("cudaSetDevice failed"); return LG_EMB_COMPUTE; }
  const int MB = c.max_blocks_per_seq;
  StepBatch& B = m->batch;
  m->T = 0;  // nothing to replay until this step is on the device
  if (uint32_t rc = B.build("lg_decoder_step", host_ids, cached, newl, n_seqs, tables, nullptr, c.kv_turbo3 != 0)) return rc;
  const int n_dec = B.n_dec;
  const bool has_prefix = B.has_prefix;
  const size_t total = (size_t)B.T;
  m->chunk_tokens = n_dec > 0 ? logismos_pick_decode_chunk(B.ctx, n_dec, m->cfg.n_kv_heads, m->head_dim) : kChunkTokens;
  const int total_chunks = n_dec > 0 ? logismos_build_decode_chunks(B.ctx, n_dec, m->chunk_tokens, B.chunks) : 0;
  if (total_chunks < 0 || (size_t)total_chunks > m->max_chunks) { set_error("lg_decoder_step: decode chunk count exceeds the scratch"); return LG_EMB_COMPUTE; }
  m->T = B.T; m->n_dec = n_dec; m->n_pre = B.n_pre; m->n_seqs = n_seqs; m->max_pre_len = B.max_pre_len; m->total_chunks = total_chunks;
  cudaStream_t s = m->stream;
  LG_TRY(cudaMemsetAsync(m->status.p, 0, 4, s), "clear status");  // the status word describes this step only
  LG_TRY(cudaMemcpyAsync(m->ids.p, B.ids, (size_t)total * 4, cudaMemcpyHostToDevice, s), "H2D ids");
  LG_TRY(cudaMemcpyAsync(m->pos.p, B.pos, (size_t)total * 4, cudaMemcpyHostToDevice, s), "H2D positions");
  LG_TRY(cudaMemcpyAsync(m->slots.p, B.slots, (size_t)total * 8, cudaMemcpyHostToDevice, s), "H2D slots");
  LG_TRY(cudaMemcpyAsync(m->cu_prefill.p, B.cu_pre, (size_t)(B.run_count + 1) * 4, cudaMemcpyHostToDevice, s), "H2D cu_seqlens");
  LG_TRY(cudaMemcpyAsync(m->last_idx.p, B.last, (size_t)n_seqs * 4, cudaMemcpyHostToDevice, s), "H2D last rows");
  if (n_dec > 0) {
    LG_TRY(cudaMemcpyAsync(m->dec_ctx.p, B.ctx, (size_t)n_dec * 4, cudaMemcpyHostToDevice, s), "H2D context lens");
    LG_TRY(cudaMemcpyAsync(m->dec_chunks.p, B.chunks, (size_t)(n_dec + 1) * 4, cudaMemcpyHostToDevice, s), "H2D chunk offsets");
  }
  if (n_dec > 0 || has_prefix)  // block tables in packed order: decode rows first, prefill rows after them
    LG_TRY(cudaMemcpyAsync(m->dec_tables.p, B.tables, (size_t)(has_prefix ? n_seqs : n_dec) * MB * 4, cudaMemcpyHostToDevice, s), "H2D block tables");
  if (has_prefix) LG_TRY(cudaMemcpyAsync(m->pre_kv.p, B.pre_kv, (size_t)B.run_count * 4, cudaMemcpyHostToDevice, s), "H2D prefill key counts");
  if (uint32_t rc = run_device(m, s)) { m->acc_dirty = true; return rc; }
  std::vector<uint32_t> toks(n_seqs);
  LG_TRY(cudaMemcpyAsync(toks.data(), m->tokens.p, (size_t)n_seqs * 4, cudaMemcpyDeviceToHost, s), "D2H tokens");
  LG_TRY(cudaStreamSynchronize(s), "stream synchronize");
  for (int k = 0; k < n_seqs; ++k) next_tokens[B.order[k]] = toks[k];
  if (const int dev_status = lg_decoder_device_status(m)) {
    m->acc_dirty = true;
    char buf[256];
    std::snprintf(buf, sizeof(buf), "device status 0x%x after a step of %d tokens in %d sequences (low byte 1: a range check failed, 2: a bounded wait expired in kernel family <next byte>, 3: a peer did not arrive)",
                  dev_status, (int)total, n_seqs);
    set_error(buf);
    return LG_EMB_COMPUTE;
  }
  return LG_EMB_OK;
}

uint32_t lg_decoder_replay_device(void* model, void* stream) {
  Decoder* m = static_cast<Decoder*>(model);
  if (m->T <= 0) { set_error("lg_decoder_replay_device: no step has run"); return LG_EMB_COMPUTE; }
  if (cudaSetDevice(m->device) != cudaSuccess) { set_error("cudaSetDevice failed"); return LG_EMB_COMPUTE; }
  return run_device(m, (cudaStream_t)stream);
}

uint32_t lg_decoder_last_hidden(void* model, int32_t n_seqs, float* host_out) {
  Decoder* m = static_cast<Decoder*>(model);
  if (n_seqs != m->n_seqs) { set_error("lg_decoder_last_hidden: n_seqs differs from the last step"); return LG_EMB_COMPUTE; }
  cudaSetDevice(m->device);
  const size_t H = m->cfg.hidden;
  std::vector<uint16_t> tmp((size_t)n_seqs * H);
  LG_TRY(cudaDeviceSynchronize(), "device synchronize");
  LG_TRY(cudaMemcpy(tmp.data(), m->last_bf16.p, tmp.size() * 2, cudaMemcpyDeviceToHost), "D2H hidden");
  for (int k = 0; k < n_seqs; ++k)
    for (size_t j = 0; j < H; ++j) {
      const uint32_t u = (uint32_t)tmp[(size_t)k * H + j] << 16;
      std::memcpy(&host_out[(size_t)m->batch.order[k] * H + j], &u, 4);
    }
  return LG_EMB_OK;
}

uint32_t lg_decoder_last_logits(void* model, int32_t n_seqs, float* host_out) {
  Decoder* m = static_cast<Decoder*>(model);
  if (n_seqs != m->n_seqs) { set_error("lg_decoder_last_logits: n_seqs differs from the last step"); return LG_EMB_COMPUTE; }
  cudaSetDevice(m->device);
  const size_t V = m->cfg.vocab;
  LG_TRY(cudaDeviceSynchronize(), "device synchronize");
  if (m->logits_f32) {
    std::vector<float> tmp((size_t)n_seqs * V);
    LG_TRY(cudaMemcpy(tmp.data(), m->logits.p, tmp.size() * 4, cudaMemcpyDeviceToHost), "D2H logits");
    for (int k = 0; k < n_seqs; ++k) std::memcpy(host_out + (size_t)m->batch.order[k] * V, tmp.data() + (size_t)k * V, V * 4);
    return LG_EMB_OK;
  }
  std::vector<uint16_t> tmp((size_t)n_seqs * V);
  LG_TRY(cudaMemcpy(tmp.data(), m->logits.p, tmp.size() * 2, cudaMemcpyDeviceToHost), "D2H logits");
  for (int k = 0; k < n_seqs; ++k)
    for (size_t j = 0; j < V; ++j) {
      const uint32_t u = (uint32_t)tmp[(size_t)k * V + j] << 16;
      std::memcpy(&host_out[(size_t)m->batch.order[k] * V + j], &u, 4);
    }
  return LG_EMB_OK;
}

int32_t lg_decoder_launches_last_step(const void* model) { return static_cast<const Decoder*>(model)->launches; }

int32_t lg_decoder_device_status(void* model) {
  Decoder* m = static_cast<Decoder*>(model);
  int32_t v = -1;
  cudaSetDevice(m->device);
  if (cudaMemcpy(&v, m->status.p, 4, cudaMemcpyDeviceToHost) != cudaSuccess) return -1;
  return v;
}

}  // extern "C"
