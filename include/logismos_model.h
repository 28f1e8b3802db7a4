/*
 * logismos_model.h - C ABI of the host-side executors above the kernel launchers.
 *
 * lg_stella_* is the GPU form of the reference's Stella embedding model:
 *   StellaEncoder::forward        crates/encoders/src/stella.rs:278-313 (layer body :190-206)
 *   StellaModel::encode_raw       crates/embed/src/stella.rs:221-248
 *   StellaModel::encode_batch     crates/embed/src/stella.rs:264-294
 * behind the consumer contract core::EmbeddingModel (crates/core/src/lib.rs:139-163). Text
 * handling (prompt, tokenizer) stays on the caller's side of this boundary: the entry points
 * take token ids, which is what `encode_raw(ids, mask, dim)` takes in the reference. There is no
 * padding in this path (the reference builds an all-ones mask, crates/embed/src/stella.rs:318),
 * so a batch is a ragged concatenation of id runs delimited by cu_seqlens.
 *
 * Results are EmbeddingError-shaped status codes; 0 is success.
 */
#ifndef LOGISMOS_MODEL_H
#define LOGISMOS_MODEL_H
#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* EmbeddingError (crates/core/src/lib.rs:75-133) as status codes */
enum lg_embedding_status {
  LG_EMB_OK = 0,
  LG_EMB_INPUT_TOO_LONG = 1,   /* InputTooLong { got, limit }: never truncates (:63-66) */
  LG_EMB_UNSUPPORTED_DIM = 2,  /* UnsupportedDim { dim } */
  LG_EMB_TOKENIZE = 3,         /* unused at id level */
  LG_EMB_COMPUTE = 4,          /* Compute { message }: shape errors, CUDA failures */
  LG_EMB_IO = 5,
  LG_EMB_UNSUPPORTED_PROMPT = 6
};

/* StellaConfig (crates/encoders/src/stella.rs:45-80). head_dim = hidden / n_heads must be 128. */
typedef struct lg_stella_config {
  int32_t vocab, hidden, n_layers, n_heads, n_kv_heads, intermediate, max_pos;
  float rms_eps;
  double rope_theta;
  int32_t max_tokens;        /* default per-input limit (EncodeOpts::max_tokens None -> 512) */
  int32_t n_dims;            /* number of dense heads loaded (supported_dims) */
  int32_t dims[8];           /* output dims, dims[0] is default_dim */
  int32_t max_batch_tokens;  /* workspace capacity in tokens; larger batches are run in pieces */
  int32_t max_batch_seqs;
  int32_t fuse_swiglu;       /* 1: SwiGLU fused into the gate/up GEMM epilogue */
} lg_stella_config_t;

/* The 12 tensors of one layer (crates/encoders/src/stella.rs:326-349), HOST fp32, HF [out, in]. */
typedef struct lg_stella_layer_weights {
  const float *norm1, *norm2;
  const float *wq, *bq, *wk, *bk, *wv, *bv, *wo;
  const float *w_gate, *w_up, *w_down;
} lg_stella_layer_weights_t;

typedef struct lg_stella_weights {
  const float* tok_embed;   /* [vocab, hidden] */
  const float* final_norm;  /* [hidden] */
  const lg_stella_layer_weights_t* layers;
  const float* head_w[8];   /* [dims[i], hidden]  (2_Dense_{dim}/linear.weight) */
  const float* head_b[8];   /* [dims[i]] */
} lg_stella_weights_t;

/* StellaModel::load counterpart for in-memory weights: casts to bf16, uploads, sizes the
 * workspace. All device allocation happens here. Returns LG_EMB_COMPUTE on failure with the
 * reason available from lg_last_error(). */
uint32_t lg_stella_create(int32_t device, const lg_stella_config_t* cfg, const lg_stella_weights_t* w,
                          void** model);
void lg_stella_destroy(void* model);

/* StellaModel::load (crates/embed/src/stella.rs:138-201) from a checkpoint directory: `root`/
 * model.safetensors must hold exactly 2 + 12 n_layers fp32 tensors under the names and shapes of
 * crates/encoders/src/stella.rs:126-127, :326-349 (anything else is LG_EMB_COMPUTE with the reason in
 * lg_last_error(); a missing or malformed file is LG_EMB_IO), and `root`/2_Dense_<dim>/model.safetensors
 * one dense head (linear.weight [dim, hidden], linear.bias [dim]) for every cfg->dims entry. The
 * supported dims are sorted and the default is 1024 when that head is loaded, else the smallest. The
 * files are mapped, not copied; the mapping is released before returning. */
uint32_t lg_stella_load(int32_t device, const char* root, const lg_stella_config_t* cfg, void** model);

/* EmbeddingModel::{default_dim, supported_dims, max_tokens} */
int32_t lg_stella_default_dim(const void* model);
int32_t lg_stella_supported_dims(const void* model, int32_t* out, int32_t cap);
int32_t lg_stella_max_tokens(const void* model);

/* EmbeddingModel::encode_batch at id level. host_ids u32 [cu_seqlens[n_seqs]], host_cu_seqlens
 * i32 [n_seqs + 1], host_out f32 [n_seqs, dim], unit-norm rows. dim == 0 selects default_dim;
 * max_tokens == 0 selects the model default. Copies ids to the device, runs the forward, copies
 * the embeddings back and synchronises. Thread-safe (calls are serialised per model). */
uint32_t lg_stella_encode_ids_batch(void* model, const uint32_t* host_ids, const int32_t* host_cu_seqlens,
                                    int32_t n_seqs, int32_t dim, int32_t max_tokens, float* host_out);

/* The same forward with everything already resident: dev_ids u32 [n_tokens], dev_cu_seqlens i32
 * [n_seqs+1], dev_positions i32 [n_tokens] (position of each token inside its sequence),
 * dev_out f32 [n_seqs, dim]. Enqueues on `stream` and returns without synchronising.
 * n_tokens <= max_batch_tokens and n_seqs <= max_batch_seqs (LG_EMB_COMPUTE otherwise); max_seqlen
 * must be >= the longest sequence of the batch (it sizes the attention grid: queries beyond it are
 * not computed) and <= max_pos. causal != 0 runs the decoder-style (causal) variant. */
uint32_t lg_stella_forward_device(void* model, const void* dev_ids, const void* dev_cu_seqlens,
                                  const void* dev_positions, int32_t n_tokens, int32_t n_seqs,
                                  int32_t max_seqlen, int32_t dim, int32_t causal, void* dev_out, void* stream);

/* StellaEncoder::forward output of the last forward: f32 [n_tokens, hidden] copied to host. */
uint32_t lg_stella_last_hidden(void* model, int32_t n_tokens, float* host_out);
/* Number of kernel launches one forward of n_layers issues (for launch accounting). */
int32_t lg_stella_launches_per_forward(const void* model);
/* Status word written by kernels with bounded waits / range checks during the last forward. */
int32_t lg_stella_device_status(void* model);

/* ====================================================================================
 * Continuous-batching decoder step over a Qwen2-style layer stack with int4 group-32 weights and
 * a paged KV cache. The reference has no decoder executor (crates/decoders is an empty scaffold,
 * src/lib.rs:1-15) and no scheduler (crates/sched/src/lib.rs:1-30); the contract kept is the
 * reference's only execution semantics, one sequence per call
 * (crates/transformers/src/attention.rs:13-14): a packed step must equal running every sequence
 * alone through the causal variant of StellaEncoder::forward, followed by lm_head + decode::greedy
 * (crates/decode/src/lib.rs:73-83) on its last token.
 * ==================================================================================== */
typedef struct lg_decoder_config {
  int32_t vocab, hidden, n_layers, n_heads, n_kv_heads, intermediate, max_pos;
  float rms_eps;
  double rope_theta;
  int32_t n_pool_blocks;       /* KV blocks of 16 tokens per layer */
  int32_t max_blocks_per_seq;  /* width of a block-table row */
  int32_t max_step_tokens;     /* capacity of one packed step */
  int32_t max_step_seqs;
  int32_t keep_bf16_copy;      /* != 0: also keep a bf16 expansion of every layer matrix (2 B per weight) for
                                  steps of more than 128 rows, instead of expanding per layer per step */
  int32_t kv_turbo3;           /* != 0: the paged cache holds TurboQuant 3-bit rows (56 bytes per 128-value head
                                  chunk instead of 256: crates/quant/src/lib.rs:316-413); every sequence of a step,
                                  decode tokens included, then attends through the decoding gather of
                                  logismos_launch_paged_prefix_attention_turbo3_bf16. A capacity mode: 4.57 times
                                  more context per byte of pool, at the codec's accuracy */
} lg_decoder_config_t;

/* int4 group-32 matrix on the HOST: codes u8 [n, k/2], scales fp16 bits [n, k/32]
 * (storage contract of logismos_launch_gemv_int4_g32_bf16). */
typedef struct lg_int4_matrix { const uint8_t* codes; const uint16_t* scales; } lg_int4_matrix_t;
typedef struct lg_decoder_layer_weights {
  const float *norm1, *norm2, *bq, *bk, *bv;            /* fp32 */
  lg_int4_matrix_t wq, wk, wv, wo, w_gate, w_up, w_down;  /* HF [out, in] */
} lg_decoder_layer_weights_t;
typedef struct lg_decoder_weights {
  const float* tok_embed;  /* fp32 [vocab, hidden], stored bf16 on the device */
  const float* final_norm;
  const lg_decoder_layer_weights_t* layers;
  lg_int4_matrix_t lm_head;  /* [vocab, hidden] */
} lg_decoder_weights_t;

uint32_t lg_decoder_create(int32_t device, const lg_decoder_config_t* cfg, const lg_decoder_weights_t* w, void** model);
/* The decoder from a Qwen2-style fp32 safetensors file (the tensor names of crates/encoders/src/
 * stella.rs:326-349, plus lm_head.weight [vocab, hidden]; without it the head is tied to the
 * embedding): exact tensor accounting as lg_stella_load, every matrix quantised to int4 group-32 on
 * the device (logismos_launch_quantize_int4_g32). */
uint32_t lg_decoder_load(int32_t device, const char* path, const lg_decoder_config_t* cfg, void** model);
void lg_decoder_destroy(void* model);

/* One packed step. Sequence i brings new_lens[i] new tokens (ids packed in sequence order in
 * host_ids) on top of cached_lens[i] tokens already in the paged cache; its block-table row
 * host_block_tables[i, :] must cover cached + new tokens. new_lens[i] == 1 is a decode token,
 * > 1 a prefill chunk, which may start its sequence (cached_lens[i] == 0) or continue it: positions
 * and cache slots carry on from the cached length and the chunk attends to the cached prefix through
 * the block table, so a prompt fed in chunks gives the result of the whole prompt fed at once. All
 * K/V rows of the new tokens are written to the cache; host_next_tokens[i] receives the greedy token after the last
 * new token of sequence i. Synchronises before returning. Status codes as lg_embedding_status. */
uint32_t lg_decoder_step(void* model, const uint32_t* host_ids, const int32_t* host_cached_lens,
                         const int32_t* host_new_lens, int32_t n_seqs, const int32_t* host_block_tables,
                         uint32_t* host_next_tokens);
/* Re-runs the device work of the last lg_decoder_step (same indices, same ids; the cache rows are
 * rewritten with the same values) on `stream` without host transfers or synchronisation: for
 * kernel-only timing. */
uint32_t lg_decoder_replay_device(void* model, void* stream);
/* fp32 [n_seqs, hidden]: final-norm output of each sequence's last new token in the last step. */
uint32_t lg_decoder_last_hidden(void* model, int32_t n_seqs, float* host_out);
/* fp32 logits of the last step [n_seqs, vocab] (the values decode::greedy ran on). */
uint32_t lg_decoder_last_logits(void* model, int32_t n_seqs, float* host_out);
int32_t lg_decoder_launches_last_step(const void* model);
int32_t lg_decoder_device_status(void* model);

/* ====================================================================================
 * Hybrid decoder step: a stack that mixes gated-delta-rule linear-attention layers (fp32 recurrent
 * state per sequence, crates/kernels/src/gated_delta_rule/cpu.rs:92-182) with gated full-attention
 * layers (paged KV cache, head_dim 128 or 256), SwiGLU MLPs, int4 group-32 weights. No reference
 * counterpart (crates/decoders/src/lib.rs:1-15 is an empty scaffold); the layer formulas are those
 * of research/14-gdn-aiter-preflight.md:190-198, :209-219 and the contract is the same as
 * lg_decoder_step: a packed step equals running every sequence alone.
 *   block:  x += mixer(rms_norm(x, norm1));  x += swiglu(rms_norm(x, norm2))
 *   full attention (layer l with (l + 1) % full_attn_interval == 0), no biases:
 *     q, gate [n_heads * d], k, v [n_kv_heads * d] = h W^T; RoPE(halves) on q, k; causal attention;
 *     out *= sigmoid(gate); o_proj
 *   linear attention (all other layers), gdn_heads heads of key = value dim 128:
 *     q, k, v, z [gdn_heads * 128] = h W^T; a, b [gdn_heads] = h W^T (fp32 outputs);
 *     q, k L2-normalised per head; g = -exp(A_log) softplus(a + dt_bias); beta = sigmoid(b);
 *     o = gated delta rule (scale 1/sqrt(128)); o *= silu(z); out_proj
 * ==================================================================================== */
typedef struct lg_hybrid_config {
  int32_t vocab, hidden, n_layers, n_heads, n_kv_heads, attn_head_dim, gdn_heads, intermediate, max_pos;
  int32_t full_attn_interval;  /* 4 = three linear-attention layers, then one full-attention layer */
  float rms_eps;
  double rope_theta;
  int32_t n_pool_blocks;       /* KV blocks of 16 tokens per full-attention layer */
  int32_t max_blocks_per_seq;
  int32_t max_step_tokens;
  int32_t max_step_seqs;
  int32_t n_state_slots;       /* recurrent-state slots per linear-attention layer */
  int32_t keep_bf16_copy;      /* as in lg_decoder_config_t */
} lg_hybrid_config_t;

typedef struct lg_hybrid_layer_weights {
  const float *norm1, *norm2;
  /* full attention: wq, wgate [n_heads*d, hidden], wk, wv [n_kv_heads*d, hidden], wo [hidden, n_heads*d]
   * linear attention: wq, wk, wv, wgate(= z) [gdn_heads*128, hidden], wo [hidden, gdn_heads*128],
   *                   wa, wb [gdn_heads, hidden], A_log, dt_bias fp32 [gdn_heads] */
  lg_int4_matrix_t wq, wk, wv, wgate, wo, wa, wb;
  const float *A_log, *dt_bias;
  lg_int4_matrix_t w_gate, w_up, w_down;
} lg_hybrid_layer_weights_t;
typedef struct lg_hybrid_weights {
  const float* tok_embed;
  const float* final_norm;
  const lg_hybrid_layer_weights_t* layers;
  lg_int4_matrix_t lm_head;
} lg_hybrid_weights_t;

uint32_t lg_hybrid_create(int32_t device, const lg_hybrid_config_t* cfg, const lg_hybrid_weights_t* w, void** model);
void lg_hybrid_destroy(void* model);
/* As lg_decoder_step, plus host_state_slots i32 [n_seqs]: the recurrent-state slot of each
 * sequence (distinct within a step, < n_state_slots). A sequence with cached_lens[i] == 0 starts
 * from the zero state; otherwise its slot must hold the state its previous step left (decode tokens
 * and continuing prefill chunks alike). */
uint32_t lg_hybrid_step(void* model, const uint32_t* host_ids, const int32_t* host_cached_lens,
                        const int32_t* host_new_lens, int32_t n_seqs, const int32_t* host_block_tables,
                        const int32_t* host_state_slots, uint32_t* host_next_tokens);
/* Tensor-parallel form. A model created from a 1/tp slice of the heads and of the MLP (n_heads,
 * n_kv_heads, gdn_heads, intermediate divided by tp; input projections sliced by rows, output
 * projections by columns; embeddings, norms and lm_head replicated) produces partial sums in its
 * output projections. With a reduction installed, each partial sum [tokens, hidden] is computed into
 * a zeroed fp32 buffer, handed to `fn`, which must leave the sum over all ranks in place, ordered on
 * `stream` (an NCCL all-reduce enqueued on it; it need not synchronise), and is then added to the
 * residual stream. fn returns 0 on success. fn == NULL removes the reduction. No reference
 * counterpart (the reference has no tensor parallelism). */
typedef uint32_t (*lg_allreduce_f32_fn)(void* user, void* dev_buf_f32, uint64_t count, void* stream);
uint32_t lg_hybrid_set_allreduce(void* model, lg_allreduce_f32_fn fn, void* user);
/* The same slot for a reduction fused with the residual add: each partial sum is computed into a zeroed
 * fp32 buffer `delta` and fn(user, x, delta, count, status, stream) must leave x += sum over all ranks
 * of delta, ordered on `stream`, without synchronising; status_i32 is the model's device status word
 * (a bounded wait that expires raises it). lg_tp_reduce_add_f32 below has this signature. Installing
 * one kind of reduction removes the other. */
typedef uint32_t (*lg_reduce_add_f32_fn)(void* user, void* x_f32, void* delta_f32, uint64_t count, void* status_i32, void* stream);
uint32_t lg_hybrid_set_reduce_add(void* model, lg_reduce_add_f32_fn fn, void* user);
uint32_t lg_hybrid_replay_device(void* model, void* stream);
uint32_t lg_hybrid_last_hidden(void* model, int32_t n_seqs, float* host_out);
uint32_t lg_hybrid_last_logits(void* model, int32_t n_seqs, float* host_out);
int32_t lg_hybrid_launches_last_step(const void* model);
int32_t lg_hybrid_device_status(void* model);

/* ====================================================================================
 * Latent-attention decoder step: a stack of parallel blocks over a paged cache of latents. No reference
 * counterpart; the contract is that of lg_decoder_step. Weights are bf16, dense.
 *   h = rms_norm(x) * (norm_offset + w);  h1 = h + conv1(h), h2 = h + conv2(h)  (causal, depthwise, conv_taps)
 *   X_(i+1) = x + attention(h1) + ff(h2);  x = sum_{j <= i+1} dwa_i[j] X_j  (X_0 = embedding)
 *   attention: q = W_uq (rms_norm(W_dq h1) * g_q); c = rms_norm(W_dkv h1) * g_c (the cached latent);
 *     per head k = W_uk c, v = W_uv c, scores (q . k) * scale, causal softmax; W_o over the heads
 *   ff: g = min(W_gate h2 + b, limit), u = clamp(W_up h2 + b, +-limit); W_down (g sigmoid(alpha g) (u + shift)) + b
 *   logits = cap tanh(head (rms_norm(x) * (norm_offset + w)) / cap)
 * Sizes may differ from layer to layer. is_f32 != 0 computes everything in fp32 (activations, cache, products,
 * sums; the bf16 weights are exact in fp32); otherwise activations and the cache are bf16 and the residual
 * stream, norms, scores, softmax and convolution state fp32.
 * ==================================================================================== */
typedef struct lg_latent_layer_config {
  int32_t heads, dim, vdim;     /* query/key and value dimensions per head, <= 256 */
  int32_t q_rank, kv_rank;      /* latent sizes; kv_rank <= 1024 */
  int32_t ff;                   /* 0: no feed-forward */
  float scale, glu_limit;
} lg_latent_layer_config_t;
typedef struct lg_latent_config {
  int32_t vocab, width, n_layers, conv_taps;
  float rms_eps, norm_offset, glu_alpha, glu_shift;
  float logit_softcap;          /* 0: none */
  int32_t is_f32;
  int32_t n_pool_blocks;        /* cache blocks of 16 tokens per layer */
  int32_t max_blocks_per_seq, max_step_tokens, max_step_seqs;
  int32_t n_state_slots;        /* convolution-state slots */
  int32_t max_out_rows;         /* rows of logits per step (>= max_step_seqs for generation) */
  const lg_latent_layer_config_t* layers;
} lg_latent_config_t;
/* bf16 values on the host, [out, in]; the feed-forward entries are NULL when ff == 0 */
typedef struct lg_latent_layer_weights {
  const void *norm1, *dq, *dq_norm, *uq, *dkv, *dkv_norm, *uk, *uv, *o;
  const void *gate, *gate_b, *up, *up_b, *down, *down_b;
  const void *conv1, *conv2;    /* [width, taps] */
  const void *dwa;              /* [layer index + 2] */
} lg_latent_layer_weights_t;
typedef struct lg_latent_weights {
  const void *embed, *final_norm, *head;
  const lg_latent_layer_weights_t* layers;
} lg_latent_weights_t;

uint32_t lg_latent_create(int32_t device, const lg_latent_config_t* cfg, const lg_latent_weights_t* w, void** model);
/* The same from a bf16 safetensors file with exactly these tensors: embed, final.norm, head and per layer i
 * l<i>.norm1, l<i>.canon1, l<i>.dwa, l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o} and with a feed-forward
 * l<i>.canon2, l<i>.mlp.{gate,up,down} and their .b. */
uint32_t lg_latent_load(int32_t device, const char* path, const lg_latent_config_t* cfg, void** model);
void lg_latent_destroy(void* model);
/* As lg_hybrid_step (cached_lens[i] == 0 starts a sequence, otherwise its slot and blocks must hold what its
 * previous step left). host_out_rows i32 [n_out]: the tokens of the step (indices into host_ids) whose logits
 * are computed; NULL: the last token of every sequence (n_out is then n_seqs). host_next_tokens u32 [n_out]
 * receives the greedy tokens. n_out may be 0. */
uint32_t lg_latent_step(void* model, const uint32_t* host_ids, const int32_t* host_cached_lens,
                        const int32_t* host_new_lens, int32_t n_seqs, const int32_t* host_block_tables,
                        const int32_t* host_state_slots, const int32_t* host_out_rows, int32_t n_out,
                        uint32_t* host_next_tokens);
uint32_t lg_latent_replay_device(void* model, void* stream);
/* fp32 logits of the last step [n_out, vocab], in the order asked for: copied to the host, or the device
 * buffer itself (valid until the next step; for the sampling chain). */
uint32_t lg_latent_last_logits(void* model, int32_t n_out, float* host_out);
void* lg_latent_logits_device(void* model);
/* X_j of the last step, fp32 [tokens, width], rows in the order of host_ids (diagnostics). */
uint32_t lg_latent_snapshot(void* model, int32_t j, int32_t n_tokens, float* host_out);
int32_t lg_latent_launches_last_step(const void* model);
int32_t lg_latent_device_status(void* model);

/* ====================================================================================
 * Decoder step over a stack of layers, each a mixer and a feed-forward of its own kind. No reference counterpart; the
 * contract is that of lg_decoder_step. Weights are bf16, dense. Sizes may differ from layer to layer; a layer may use the
 * tensors of another one (weights_of), with a cache and states of its own. is_f32 as for lg_latent_config_t; in both
 * formats the residual stream, norms, scores, routers, decays, step sizes and states are fp32.
 *   x = embed[id];  per layer x += mixer, x += feed-forward, normed as the stack's `norm` says:
 *   LG_NORM_LAYER_POST (Katadra)  x += norm(f(x)), layer norms (gain and offset); logits = head norm(x)
 *   LG_NORM_TANH_AROUND (Vugedra) x += norm_b(f(norm_a(x))), norms tanh(alpha x) w + b; logits = head norm(x)
 *   LG_NORM_RMS_GATED (Zetalorn)  h = norm(x); x += f(h) sigmoid(W_rg h + b), norms x / rms(x) * g with one gain g; logits =
 *     logit_scale head norm(x)
 * Mixers:
 *   LG_MIXER_SSD: [z | x | B | C | dt] = W_in h, convolution, scalar-decay recurrence, gate, norm in parts, W_o
 *     (lg_ssd_t, logismos_launch_gated_group_norm)
 *   LG_MIXER_PARALLEL (in a post-norm stack): left_scale * attention(h) + right_scale * time_mixing(h); attention without
 *     positions, unit queries and keys, capped scores, a learned bias by distance bucket, a query temperature and an output
 *     gate (lg_score_bias_t); time mixing with token shift and a low-rank data-dependent decay (lg_time_mix_t)
 *   LG_MIXER_ATTENTION: q, k, v with biases, q and k normed over the whole projection and rotated; a window with kept first
 *     keys, one added to the softmax denominator, an output gate per head (lg_window_t); W_o
 *   LG_MIXER_GLA: gated linear attention, a decay per key channel (lg_time_mix_t, LG_DECAY_GATED); W_o
 *   LG_MIXER_DIFF (in a gated RMS stack): differential attention over chunks. Every head has two maps of queries and keys, q
 *     and k normed per head and map and rotated, over one set of values; out = (a1 - lambda a2) / rms * (1 - diff) with lambda =
 *     exp(lq1 . lk1) - exp(lq2 . lk2) + diff; W_o
 *   LG_MIXER_PAIR (in a gated RMS stack): half the sum of two branches, each with its W_o, then normed over the width with a
 *     gain. Left: attention over a sliding window and, before it, pooled blocks (lg_window_t), q and k normed per head and
 *     rotated. Right: linear attention with a fixed decay per head, q, k, v with silu; normed over all heads, times sigmoid(W_g h)
 *   LG_MIXER_LATENT: queries W_uq rms(W_dq h), per head dim unrotated and rot_dims rotated channels; W_dkv h is the latent
 *     (normed, cached) and one rotated key part for all heads; keys W_uk c, values W_uv c; causal, a gate per head; W_o
 * Feed-forwards:
 *   LG_FF_RELU2: W_down max(W_up h, 0)^2
 *   LG_FF_GATED: W_down (silu(W_gate h) * (W_up h))
 *   LG_FF_MIXTURE: `top` of experts + identity experts of the latter form by a softmax router with a correction for the
 *     choice alone (lg_moe_route_t); identity experts return h; a shared expert is added (shared_ff 0: none). Also with sigmoid
 *     scores, a choice among the best groups, and clamped gated units (LG_EPI_GLU_CLAMP)
 * Layers may be repeated: a run of them is listed once per pass, those of later passes with weights_of, and the first of each
 * pass names it: x += embed[id] (not in the first), x += loop_step[pass], before its norm.
 * ==================================================================================== */
enum { LG_MIXER_SSD = 0, LG_MIXER_PARALLEL = 1, LG_MIXER_ATTENTION = 2, LG_MIXER_GLA = 3, LG_MIXER_LATENT = 4,
       LG_MIXER_DIFF = 5, LG_MIXER_PAIR = 6 };
enum { LG_FF_RELU2 = 0, LG_FF_GATED = 1, LG_FF_MIXTURE = 2 };
enum { LG_NORM_LAYER_POST = 0, LG_NORM_TANH_AROUND = 1, LG_NORM_RMS_GATED = 2 };
typedef struct lg_mixer_layer_config {
  int32_t kind;
  int32_t weights_of;           /* layer whose tensors are used; its own index: its own */
  int32_t ff;                   /* 0: no feed-forward; a mixture: of one expert */
  /* state-space */
  int32_t ssd_heads, ssd_vdim, ssd_state, ssd_groups, ssd_norm_groups, ssd_taps;
  /* attention of any kind and gated linear attention: sizes <= 256. Parallel layers: bias_rows rows of the bias table,
   * distances from bias_max on share the last one */
  int32_t heads, kv_heads, dim, vdim, bias_rows, bias_max;
  float scale, softcap, temp_coef, temp_every;
  /* time mixing; tm_rank (of the decay) also for gated linear attention */
  int32_t tm_heads, tm_dim, tm_rank;
  float left_scale, right_scale;
  int32_t ff_kind;
  int32_t experts, identity, top, shared_ff;   /* a mixture */
  int32_t window, keep_first;   /* attention; window 0: all keys */
  int32_t q_rank, kv_rank;      /* latent attention: kv_rank + rot_dims <= 1024 */
  int32_t rot_dims;             /* rotated channels per head, interleaved pairs */
  float tau;                    /* gated linear attention */
  double rot_base, rot_factor, rot_original, rot_fast, rot_slow;   /* YaRN interpolation; rot_factor 0: none, rot_original 0: linear */
  int32_t rot_halves;           /* pairs (i, i + rot_dims / 2) instead; differential and paired attention */
  int32_t chunked, pool;        /* the window is a chunk; pooled blocks before it */
  float diff;
  int32_t lin_heads, lin_dim, lin_vdim;        /* linear attention of a pair: sizes <= 256 */
  const double* decay;          /* [lin_heads], in (0, 1]; read while the model is made */
  float glu_alpha, glu_limit, glu_shift;       /* of the experts; glu_limit 0: silu(gate) * up */
  int32_t scoring, route_groups, keep_groups;  /* LG_ROUTE_*; route_groups 0: none */
  int32_t no_correction;
  int32_t file_layer;           /* 1 + the layer's number in tensor names, 0: its own index */
  int32_t pass;                 /* 1 + the pass that begins with this layer, 0: none */
} lg_mixer_layer_config_t;
typedef struct lg_mixer_config {
  int32_t vocab, width, n_layers;
  float norm_eps;
  int32_t is_f32;
  int32_t n_pool_blocks;        /* cache blocks of 16 tokens per attention layer */
  int32_t max_blocks_per_seq, max_step_tokens, max_step_seqs;
  int32_t n_state_slots;        /* recurrent, convolution and shift states */
  int32_t max_out_rows;
  int32_t keep_layers;          /* != 0: the stream after every layer is kept (lg_mixer_snapshot) */
  const lg_mixer_layer_config_t* layers;
  int32_t norm;
  int32_t passes;               /* over repeated layers, 0: none are */
  float logit_scale;            /* gated RMS stack */
} lg_mixer_config_t;
/* bf16 values on the host, [out, in]; entries of other kinds of mixer, of a missing feed-forward and of a layer
 * with weights_of are NULL. mu [5] in the order r, k, v, g, w. experts [3 * experts]: gate, up, down of each. */
typedef struct lg_mixer_layer_weights {
  const void *norm1, *norm1_b, *norm2, *norm2_b, *up, *down;
  const void *in, *conv, *conv_b, *dt_bias, *A_log, *D, *norm, *o;
  const void *left_q, *left_k, *left_v, *left_rel, *left_g, *left_o;
  const void* mu[5];
  const void *right_r, *right_k, *right_v, *right_g, *right_w1, *right_w2, *right_w0, *right_u, *right_norm, *right_o;
  const void *norm1_alpha, *norm1b, *norm1b_b, *norm1b_alpha, *norm2_alpha, *norm2b, *norm2b_b, *norm2b_alpha;
  const void *q, *q_b, *q_norm, *k, *k_b, *k_norm, *v, *v_b, *g, *a1, *a2, *a2_b;
  const void *dq, *dq_norm, *uq, *dkv, *dkv_norm, *uk, *uv;
  const void *gate, *router, *correction, *shared_gate, *shared_up, *shared_down;
  const void* const* experts;
  const void *rg1, *rg1_b, *rg2, *rg2_b;        /* gated residual; norm1 and norm2 are then single values */
  const void *lq1, *lk1, *lq2, *lk2;            /* differential attention: also q, k, v, o, q_norm and k_norm [dim] */
  const void *left_q_norm, *left_k_norm, *left_out, *right_q, *right_out;   /* a pair: also left_* q, k, v, o, right_* k, v, g, norm, o */
} lg_mixer_layer_weights_t;
typedef struct lg_mixer_weights {
  const void *embed, *final_norm, *final_norm_b, *head;
  const lg_mixer_layer_weights_t* layers;
  const void* final_norm_alpha; /* tanh norms */
  const void* loop_step;        /* [passes, width] */
} lg_mixer_weights_t;

uint32_t lg_mixer_create(int32_t device, const lg_mixer_config_t* cfg, const lg_mixer_weights_t* w, void** model);
/* The same from a bf16 safetensors file with exactly these tensors: embed, final.norm, head and, per layer i that owns
 * tensors, l<i>.norm1 and with a feed-forward l<i>.norm2 (tanh norms: also l<i>.norm1b, l<i>.norm2b), every one of them with
 * .b (and .alpha); under l<i>.mix.: {in,conv,conv.b,dt_bias,A_log,D,norm,o}, left.{q,k,v,rel,g,o} and right.{mu.r,mu.k,mu.v,
 * mu.g,mu.w,r,k,v,g,w1,w2,w0,u,norm,o}, {q,k,v,g,o} with {q,k,v}.b and {q,k}.norm, {q,k,v,g,o,norm,a1,a2,a2.b}, or {dq,
 * dq.norm,uq,dkv,dkv.norm,uk,uv,g,o}; under l<i>.mlp.: {up,down}, {gate,up,down}, or {router,correction} with {e<j>,shared}.
 * {gate,up,down}. bias_rows and tm_rank are taken from the tensors. A gated RMS stack: norms of one value without .b, l<i>.rg1,
 * l<i>.rg2 with .b, l<i>.mix.{q,k,v,q.norm,k.norm,lq1,lk1,lq2,lk2,o}, or left.{q,k,v,q.norm,k.norm,o,out} and right.{q,k,v,g,
 * norm,o,out}, no mlp.correction, and loop.step when layers are repeated. */
uint32_t lg_mixer_load(int32_t device, const char* path, const lg_mixer_config_t* cfg, void** model);
void lg_mixer_destroy(void* model);
/* Step, logits and diagnostics as for lg_latent_*. Recurrent states are updated in place: a step that failed part-way
 * leaves those of its sequences undefined, and lg_mixer_replay_device (timing) moves them on. */
uint32_t lg_mixer_step(void* model, const uint32_t* host_ids, const int32_t* host_cached_lens, const int32_t* host_new_lens,
                       int32_t n_seqs, const int32_t* host_block_tables, const int32_t* host_state_slots,
                       const int32_t* host_out_rows, int32_t n_out, uint32_t* host_next_tokens);
uint32_t lg_mixer_replay_device(void* model, void* stream);
uint32_t lg_mixer_last_logits(void* model, int32_t n_out, float* host_out);
void* lg_mixer_logits_device(void* model);
/* The stream of the last step before the first layer (j = 0) and after layer j - 1, fp32 [tokens, width], rows in the
 * order of host_ids; needs keep_layers. */
uint32_t lg_mixer_snapshot(void* model, int32_t j, int32_t n_tokens, float* host_out);
int32_t lg_mixer_launches_last_step(const void* model);
int32_t lg_mixer_device_status(void* model);

/* ====================================================================================
 * Tensor-parallel exchange over NVLink peer memory (ranks = processes on different GPUs of one node).
 * No reference counterpart (the reference is single-device, README.md:19-21). One kernel per rank
 * writes the local partial sum into every peer's receive buffer with plain peer stores, raises a
 * flag there, waits (bounded: status 3 on expiry, the add is then skipped) for the peers' flags and adds all partial
 * sums, in rank order, into the residual stream.
 *   lg_tp_comm_alloc   allocates this rank's region (flags + two receive sets of tp * max_elems floats,
 *                      zeroed) on `device` and returns its 64-byte cudaIpc handle
 *   lg_tp_comm_open    given the handles of all ranks [tp][64] (exchanged by the host, e.g. an
 *                      all-gather over the process group), maps the peers' regions
 *   lg_tp_reduce_add_f32  x += sum over ranks of delta for count floats (count % 4 == 0, count <=
 *                      max_elems); every rank makes the same sequence of calls; signature of
 *                      lg_reduce_add_f32_fn with user = the communicator
 * ==================================================================================== */
size_t lg_tp_comm_region_bytes(int32_t tp, uint64_t max_elems);
uint32_t lg_tp_comm_alloc(int32_t device, int32_t tp, uint64_t max_elems, void** region, uint8_t* handle_out64);
uint32_t lg_tp_comm_open(int32_t device, void* region, int32_t rank, int32_t tp, uint64_t max_elems,
                         const uint8_t* all_handles, void** comm);
void lg_tp_comm_destroy(void* comm, int32_t free_region);
uint32_t lg_tp_reduce_add_f32(void* comm, void* x_f32, void* delta_f32, uint64_t count, void* status_i32, void* stream);

/* ====================================================================================
 * safetensors reader: crates/loader/src/safetensors.rs:44-197 (Reader::open / get / names / len) with
 * the dtype map of :199-217 and the truncation guard of crates/loader/src/lib.rs:229-246 (every get
 * re-stats the file and fails if its length changed since it was mapped). Status codes as
 * lg_embedding_status: LG_EMB_IO for I/O and format errors, with the reason in lg_last_error().
 * ==================================================================================== */
enum lg_dtype { LG_DT_F32 = 0, LG_DT_F16 = 1, LG_DT_BF16 = 2, LG_DT_F8E4M3 = 3, LG_DT_F8E5M2 = 4, LG_DT_I32 = 5, LG_DT_I8 = 6,
                LG_DT_I4 = 7, LG_DT_U8 = 8 };  /* order of taxis::DType, crates/taxis/src/dtype.rs:16-26 */
typedef struct lg_tensor_view {
  int32_t dtype;       /* lg_dtype */
  int32_t rank;
  int64_t shape[8];
  const void* data;    /* into the mapping; valid until lg_safetensors_close */
  uint64_t nbytes;
} lg_tensor_view_t;
uint32_t lg_safetensors_open(const char* path, void** reader);
void lg_safetensors_close(void* reader);
int32_t lg_safetensors_len(const void* reader);
/* name of tensor i in archive order (by on-disk offset); NULL when i is out of range */
const char* lg_safetensors_name(const void* reader, int32_t i);
uint64_t lg_safetensors_data_region_start(const void* reader);
uint32_t lg_safetensors_get(const void* reader, const char* name, lg_tensor_view_t* out);

/* Message of the last failure on the calling thread ("" if none). */
const char* lg_last_error(void);

#ifdef __cplusplus
}
#endif
#endif
