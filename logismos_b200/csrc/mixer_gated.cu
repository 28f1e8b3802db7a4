// Windowed attention, gated linear attention, latent attention and the gated feed-forwards of the stack of mixers: layout
// and upload of their weights, buffers, and their part of a step (the output projection and the norms follow in
// mixer_model.cu).
//   attention: one GEMM to q | k | v (biases) and the fp32 gates -> norm over the whole projections, rotation, cache store ->
//     attention over the window, with the sink and the gate
//   gated linear attention: one GEMM to q | k | v | gate and the fp32 low-rank activations of the decay -> recurrence with norm
//     and gate, token by token for decode rows, chunk-parallel for prefill rows (their decays by a GEMM of their own)
//   latent: one GEMM to the query latent, the key/value latent with the rotated key part, and the gates (fp32) -> norms,
//     rotation, cache store -> queries, rotation -> as in latent_model.cu: decode rows in the latent space, prefill rows over
//     expanded keys. The rotated part is more columns of a cache row: identity blocks in W_uk carry it through both forms
//   mixture: router (fp32) -> choice -> rows by expert -> gate/up and down of all experts, the shared one among them: it is cut
//     in experts of the routed ones' size that every token takes
#include "mixer_stack.h"

namespace lgm {

namespace {

constexpr uint16_t kOne = 0x3f80;  // 1.0 in bf16

uint32_t attention(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int T = B.T, P = L.groups.n_main, f32 = c.is_f32;
  void *st = m->status.p, *proj = m->proj.p;
  LG_TRY(projections(m, L, W, false, s), "input projections");
  LG_TRY(logismos_launch_qk_norm_rotary_store(proj, P, L.kpool.p, L.vpool.p, m->dev(B.slots), m->dev(B.pos), T, L.c.heads, L.c.kv_heads, L.Dh, L.c.dim, W.gain_q.p,
                                              W.gain_k.p, c.norm_eps, L.table < 0 ? nullptr : m->tables[(size_t)L.table].angles.p, L.c.rot_dims,
                                              (int64_t)c.n_pool_blocks * kKvBlock, f32, st, s), "queries, keys and cache store");
  m->launches += 1;
  lg_window_t w = m->views[(size_t)L.view].shape;
  w.scale = L.c.scale; w.sink = 1; w.gate = m->tail.p; w.ld_gate = L.groups.ld_tail;
  return window_attention(m, L, w, proj, P, L.c.heads, L.c.kv_heads, L.Dh, m->act.p, L.Kout, s);
}

uint32_t gated_linear_attention(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  StepBatch& B = m->batch;
  const int f32 = m->cfg.is_f32;
  const bool chunked = !f32 && B.n_pre > 0 && logismos_time_mix_has_chunked(L.Dp, L.Vp);
  LG_TRY(projections(m, L, W, chunked, s), "input projections");
  const int kw = L.c.heads * L.Dp, vw = L.c.heads * L.Vp;
  lg_time_mix_t a{};
  a.proj = m->proj.p; a.ld = L.groups.n_main; a.off_r = 0; a.off_k = kw; a.off_v = 2 * kw; a.off_g = 2 * kw + vw;
  a.low = m->tail.p; a.ld_low = L.groups.ld_tail; a.w2 = W.w2.p; a.ld_w2 = 2 * L.Lr; a.rank = L.Lr; a.w0 = W.w0.p; a.gain = W.gain.p;
  a.state = L.state.p; a.state_slots = m->dev(B.state); a.fresh = m->dev(B.fresh); a.cu = m->dev(B.cu);
  a.out = m->act.p; a.ld_out = L.Kout; a.heads = L.c.heads; a.d = L.c.vdim; a.dp = L.Dp; a.vp = L.Vp;
  a.scale = 1.0f; a.eps = m->cfg.norm_eps; a.mode = LG_DECAY_GATED; a.tau = L.c.tau; a.q_scale = 1.0f / std::sqrt((float)L.c.dim);
  const int serial = chunked ? B.n_dec : B.n_seqs;  // sequences that go token by token
  if (serial > 0) {
    LG_TRY(logismos_launch_time_mix_step(&a, serial, f32, s), "gated linear attention");
    m->launches += 1;
  }
  if (chunked) {
    const int rows = B.T - B.n_dec, w = L.Lr;
    LG_TRY(logismos_launch_linear_t_act_bf16((const uint16_t*)m->low2.p + (size_t)B.n_dec * 2 * w, W.w2.p, W.w0.p, (float*)m->z.p + (size_t)B.n_dec * L.Rw, rows, L.Rw, 2 * w, 2 * w, L.Rw,
                                             LG_EPI_F32 | LG_EPI_STATIC_W, 0, 0, 0, m->status.p, s), "decay");
    a.z = m->z.p; a.ld_z = L.Rw;
    a.state_slots = m->dev(B.state) + B.n_dec; a.fresh = m->dev(B.fresh) + B.n_dec; a.cu = m->dev(B.cu) + B.n_dec;
    LG_TRY(logismos_launch_time_mix_chunked_bf16(&a, B.n_pre, s), "gated linear attention (prompts)");
    m->launches += 2;
  }
  return 0;
}

uint32_t latent_attention(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const DecodeView& V = m->views[(size_t)L.view];
  const int T = B.T, MB = c.max_blocks_per_seq, heads = L.c.heads, HD = heads * L.Dh, HR = heads * L.Rp, f32 = c.is_f32, LG = round_up(heads, 16);
  void* st = m->status.p;
  // a few dozen rows: the narrow projection is accumulated, so that the tiles split its reduction over the idle SMs
  const bool acc = T > 32 && m->accumulates(T);
  void* raw = acc ? m->raw_acc.p : m->tail.p;
  LG_TRY(linear(m, m->h.p, m->Hp, W.w_in, L.N, m->Hp, raw, L.N, acc ? LG_EPI_RESID_F32 : LG_EPI_F32, T, s), "latent projections");
  const void* angles = m->tables[(size_t)L.table].angles.p;
  const lg_latent_rotary_t rot{angles, m->dev(B.pos), L.Rc, L.c.rot_dims, m->gate.p, heads, LG};
  LG_TRY(logismos_launch_latent_norm_store(raw, L.N, W.gain_q.p, W.gain_k.p, m->cq.p, L.kpool.p, m->dev(B.slots), T, L.Qp, L.c.q_rank, L.Rp, L.c.kv_rank, c.norm_eps,
                                           (int64_t)c.n_pool_blocks * kKvBlock, f32, acc, &rot, st, s), "latent norm and store");
  LG_TRY(linear(m, m->cq.p, L.Qp, W.w_uq, HD, L.Qp, m->proj.p, HD, LG_EPI_BF16, T, s), "queries");
  m->launches += 1;
  const int turned = f32 ? 0 : B.n_dec;  // decode rows are turned by the decode kernel, in the latent space
  if (T > turned) {
    LG_TRY(logismos_launch_rotary_heads((uint8_t*)m->proj.p + (size_t)turned * HD * (f32 ? 4 : 2), HD, m->dev(B.pos) + turned, T - turned, heads, L.Dh, L.Dn, angles, L.c.rot_dims, f32, s),
           "rotation of the queries");
    m->launches += 1;
  }
  const float* gate = (const float*)m->gate.p;
  if (f32) {
    LG_TRY(head_linear(m, m->proj.p, HD, W.w_ukt, heads, L.Rp, L.Dh, m->qlat.p, HR, T, s), "latent queries");
    LG_TRY(logismos_launch_latent_attention_f32(m->qlat.p, L.kpool.p, m->dev(B.tables), m->dev(B.seq_ids), m->dev(B.pos), m->olat.p, T, MB, c.n_pool_blocks, heads,
                                                L.Rp, L.c.scale, gate, LG, st, s), "latent attention");
    m->launches += 1;
    LG_TRY(head_linear(m, m->olat.p, HR, W.w_uv, heads, L.Dh, L.Rp, m->act.p, L.Kout, T, s), "latent values");
    return 0;
  }
  if (B.n_dec > 0) {
    LG_TRY(head_linear(m, m->proj.p, HD, W.w_ukt, heads, L.Rp, L.Dh, m->qlat.p, HR, B.n_dec, s), "latent queries");
    LG_TRY(logismos_launch_latent_decode_bf16(m->qlat.p, L.kpool.p, m->dev(B.tables), m->dev(B.ctx), m->dev(V.chunks), m->olat.p, m->dec_scratch.p, B.n_dec, V.total,
                                              V.chunk_tokens, MB, c.n_pool_blocks, heads, L.Rp, L.c.scale, gate, LG, angles, L.Rc, L.c.rot_dims, st, s), "latent decode");
    m->launches += V.total > B.n_dec ? 2 : 1;
    LG_TRY(head_linear(m, m->olat.p, HR, W.w_uv, heads, L.Dh, L.Rp, m->act.p, L.Kout, B.n_dec, s), "latent values");
  }
  const uint16_t* q = (const uint16_t*)m->proj.p + (size_t)B.n_dec * HD;
  uint16_t* out = (uint16_t*)m->act.p + (size_t)B.n_dec * L.Kout;
  for (const PrefixRun& r : B.runs) {
    const int ns = r.s1 - r.s0, tp = logismos_latent_gather_rows(r.total_kv, ns);
    const int32_t* kv_lens = m->dev(B.pre_kv) + r.s0;
    LG_TRY(logismos_launch_latent_gather_bf16(L.kpool.p, m->dev(B.tables) + (size_t)(B.n_dec + r.s0) * MB, MB, c.n_pool_blocks, kv_lens, m->lat.p, m->kv_start.p,
                                              r.total_kv, ns, r.max_kv, L.Rp, st, s), "latent gather");
    LG_TRY(logismos_launch_linear_t_act_bf16(m->lat.p, W.w_uk.p, nullptr, m->kbuf.p, tp, HD, L.Rp, L.Rp, HD, LG_EPI_BF16 | LG_EPI_STATIC_W, 0, 0, 0, st, s), "keys");
    LG_TRY(logismos_launch_linear_t_act_bf16(W.w_uv.p, m->lat.p, nullptr, m->vt.p, HD, tp, L.Rp, L.Rp, tp, LG_EPI_BF16, 0, 0, 0, st, s), "values");
    LG_TRY(logismos_launch_varlen_attention_kv_tc_bf16(q, HD, m->dev(B.cu_pre) + r.s0, kv_lens, m->kv_start.p, m->kbuf.p, m->vt.p, tp, out, L.Kout, T - B.n_dec, ns,
                                                       r.max_q, heads, heads, L.Dh, L.c.scale, gate + (size_t)B.n_dec * LG, LG, st, s), "attention");
    m->launches += 4;
  }
  return 0;
}

// rows [0, ff) of gate and up, interleaved in blocks of 32 from row0 of dst on, as the gated epilogue reads them
void gate_up_rows(Mat& dst, int row0, const void* gate, const void* up, int first, int ff, int k) {
  for (int i = 0; i < ff; ++i) {
    const int at = row0 + (i / 32) * 64 + i % 32;
    dst.row(at, 0, gate, (size_t)(first + i) * k, k);
    dst.row(at + 32, 0, up, (size_t)(first + i) * k, k);
  }
}

}  // namespace

void gathered_keys(const StepBatch& B, const lg_window_t& w, const PrefixRun& r, int* total, int* longest) {
  *total = *longest = 0;
  for (int k = r.s0; k < r.s1; ++k) {
    const int n = logismos_window_view_keys(&w, B.pre_kv[k], B.newl[(size_t)(B.n_dec + k)]);
    *total += n;
    *longest = std::max(*longest, n);
  }
}

uint32_t window_attention(Mixer* m, MLayer& L, lg_window_t w, const void* q, int ld_q, int heads, int kv, int hd, void* out, int ld_out, cudaStream_t s, bool prompts_only) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const DecodeView& V = m->views[(size_t)L.view];
  const int T = B.T, MB = c.max_blocks_per_seq;
  void* st = m->status.p;
  if (c.is_f32) {
    LG_TRY(logismos_launch_window_attention_f32(q, ld_q, L.kpool.p, L.vpool.p, m->dev(B.tables), m->dev(B.seq_ids), m->dev(B.pos), out, ld_out, T, MB, c.n_pool_blocks,
                                                heads, kv, hd, &w, st, s), "attention");
    m->launches += 1;
    return 0;
  }
  if (B.n_dec > 0 && !prompts_only) {
    LG_TRY(logismos_launch_window_attention_decode_bf16(q, ld_q, L.kpool.p, L.vpool.p, m->dev(B.tables), m->dev(B.ctx), m->dev(V.chunks), out, ld_out, m->dec_scratch.p,
                                                        B.n_dec, V.total, V.chunk_tokens, MB, c.n_pool_blocks, heads, kv, hd, &w, st, s), "decode attention");
    m->launches += V.total > B.n_dec ? 2 : 1;
  }
  const size_t row0 = (size_t)B.n_dec;
  if (w.gate) w.gate = (const float*)w.gate + row0 * w.ld_gate;
  for (const PrefixRun& r : B.runs) {
    int total, longest;
    gathered_keys(B, w, r, &total, &longest);
    LG_TRY(logismos_launch_window_attention_prefix_bf16((const uint16_t*)q + row0 * ld_q, ld_q, m->dev(B.cu_pre) + r.s0, m->dev(B.pre_kv) + r.s0, L.kpool.p, L.vpool.p,
                                                        m->dev(B.tables) + (row0 + r.s0) * MB, MB, c.n_pool_blocks, (uint8_t*)out + row0 * ld_out * (w.out_f32 ? 4 : 2),
                                                        ld_out, m->attn_ws.p, T - B.n_dec, total, r.s1 - r.s0, r.max_q, longest, heads, kv, hd, &w, st, s), "attention");
    m->launches += 2;
  }
  return 0;
}

uint32_t run_gated_kinds(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  return L.c.kind == LG_MIXER_ATTENTION ? attention(m, L, W, s) : L.c.kind == LG_MIXER_GLA ? gated_linear_attention(m, L, W, s) : latent_attention(m, L, W, s);
}

uint32_t run_mixture(Mixer* m, const MLayer& L, const MWeights& W, lg_mixture_out_t* out, cudaStream_t s) {
  const lg_mixer_layer_config_t& y = L.c;
  const int T = m->batch.T, Hp = m->Hp, n_routed = y.experts + y.identity, groups = y.experts + L.always, pairs = y.top + L.always, f32 = m->cfg.is_f32;
  const bool few = f32 || logismos_moe_streams(T, y.top, y.experts, y.identity, L.always, Hp, L.Fp);
  const bool acc = T > 32 && !f32 && !logismos_get_deterministic();  // the narrow product is split over k whatever the rows
  void *logits = acc ? m->route_acc.p : m->route.p, *st = m->status.p;
  // a step of a few tokens with a small router: the product rides on the choice; in a gated stack on the gate's
  const bool gated = m->cfg.norm == LG_NORM_RMS_GATED, fused = !gated && few && !f32 && (int64_t)T * n_routed * Hp <= 1 << 22;
  if (gated) logits = m->route.p;
  else if (!fused) LG_TRY(linear(m, m->h.p, Hp, W.w_router, L.route_ld, Hp, logits, L.route_ld, acc ? LG_EPI_RESID_F32 : LG_EPI_F32, T, s), "router");
  lg_moe_route_t r{};
  if (fused) { r.h = m->h.p; r.w = W.w_router.p; r.width = Hp; r.arrived = (uint8_t*)m->counts.p + m->counts_bytes - 4; }
  r.logits = logits; r.ld = L.route_ld; r.zero_logits = acc && !gated; r.correction = W.correction.p;
  r.scoring = y.scoring; r.groups = y.route_groups; r.keep_groups = y.keep_groups;
  const bool clamped = y.glu_limit > 0.0f;
  const int glu = clamped ? LG_EPI_GLU_CLAMP : LG_EPI_SWIGLU;
  r.n_experts = y.experts; r.n_identity = n_routed - y.experts; r.top = y.top; r.n_always = L.always;
  r.weights = m->pair_w.p; r.pair_row = m->pair_row.p; r.identity = m->identity.p;
  *out = lg_mixture_out_t{m->expert_rows.p, m->pair_row.p, m->pair_w.p, m->identity.p, pairs, y.top, nullptr, 0};
  if (few) {
    r.offsets = m->offsets.p; r.row_token = m->row_token.p;
    LG_TRY(logismos_launch_moe_route(&r, T, s), "choice of experts");
    const int expected = T <= 8 ? 8 : 16;
    if (f32) {
      LG_TRY(logismos_launch_linear_experts_f32(m->h.p, W.w_up.p, m->ffb.p, r.offsets, r.row_token, groups, T, 2 * L.Fp, Hp, Hp, L.Fp, LG_EPI_GLU_CLAMP,
                                                clamped ? y.glu_alpha : 1.0f, clamped ? y.glu_limit : INFINITY, clamped ? y.glu_shift : 0.0f, s), "experts, gate and up");
      LG_TRY(logismos_launch_linear_experts_f32(m->ffb.p, W.w_down.p, m->expert_rows.p, r.offsets, nullptr, groups, T, Hp, L.Fp, L.Fp, Hp, LG_EPI_F32, 0, 0, 0, s), "experts, down");
    } else {
      LG_TRY(logismos_launch_linear_experts_small_bf16(m->h.p, W.w_up.p, m->ffb.p, r.offsets, r.row_token, groups, T, expected, 2 * L.Fp, Hp, Hp, L.Fp, glu, y.glu_alpha,
                                                       y.glu_limit, y.glu_shift, s),
             "experts, gate and up");
      LG_TRY(logismos_launch_linear_experts_small_bf16(m->ffb.p, W.w_down.p, m->expert_rows.p, r.offsets, nullptr, groups, T, expected, Hp, L.Fp, L.Fp, Hp, LG_EPI_BF16, 0, 0, 0, s),
             "experts, down");
    }
    m->launches += 3;
    return 0;
  }
  const int max_tiles = logismos_moe_max_tiles(T, y.top, y.experts, L.always), rows = T * pairs;
  r.counts = m->counts.p; r.pair_expert = m->pair_expert.p;
  r.n_tiles = m->tiles.p; r.tiles = (int32_t*)m->tiles.p + 4;
  LG_TRY(logismos_launch_moe_route(&r, T, s), "choice of experts");
  LG_TRY(logismos_launch_moe_place(&r, m->h.p, m->gathered.p, Hp, T, s), "rows by expert");
  LG_TRY(logismos_launch_linear_experts_tc_bf16(m->gathered.p, rows, m->h.p, T, W.w_up.p, m->ffb.p, r.tiles, r.n_tiles, max_tiles, groups, 2 * L.Fp, Hp, Hp, L.Fp,
                                                glu, y.glu_alpha, y.glu_limit, y.glu_shift, st, s), "experts, gate and up");
  LG_TRY(logismos_launch_linear_experts_tc_bf16(m->ffb.p, rows, nullptr, 0, W.w_down.p, m->expert_rows.p, r.tiles, r.n_tiles, max_tiles, groups, Hp, L.Fp, L.Fp, Hp,
                                                LG_EPI_BF16, 0, 0, 0, st, s), "experts, down");
  m->launches += 4;
  out->counts = r.counts;
  out->n_counts = y.experts;
  return 0;
}

// ---- what a layer needs --------------------------------------------------------------------------------

const char* check_gated_kinds(const lg_mixer_layer_config_t& y) {
  if (y.heads <= 0 || y.dim <= 0 || y.dim > 256 || y.vdim <= 0 || y.vdim > 256) return "heads, or head dimensions above 256";
  if (y.kind == LG_MIXER_GLA) return y.tau > 0.0f ? nullptr : "a decay exponent that is not positive";
  if (!(y.scale > 0.0f)) return "a score scale that is not positive";
  if (y.rot_dims < 0 || y.rot_dims % 2 || (y.rot_dims > 0 && !(y.rot_base > 1.0))) return "rotated dimensions that are not pairs, or a base that is not above 1";
  if (y.rot_factor != 0.0 && (!(y.rot_factor > 0.0) || !(y.rot_original > 0.0) || !(y.rot_fast > 0.0) || !(y.rot_slow > 0.0))) return "scaling of the rotation";
  if (y.kind == LG_MIXER_ATTENTION) {
    if (y.kv_heads <= 0 || y.heads % y.kv_heads) return "attention heads";
    if (y.rot_dims > y.dim) return "more rotated dimensions than a head has";
    if (y.window < 0 || y.keep_first < 0 || y.keep_first > 1 << 24) return "window";
    return nullptr;
  }
  if (y.kind != LG_MIXER_LATENT) return "kind of mixer";
  if (y.q_rank <= 0 || y.kv_rank <= 0 || y.rot_dims <= 0) return "latent sizes, or no rotated part";
  if (r64(round_up(y.kv_rank, 8) + y.rot_dims) > 1024) return "a latent above 1024 with its rotated part";
  if (round_up(y.dim, 8) + round_up(y.rot_dims, 8) > 256) return "head dimensions above 256 with the rotated part";
  return nullptr;
}

void layout_gated_kinds(MLayer& L) {
  const lg_mixer_layer_config_t& c = L.c;
  lg_linear_groups_t& g = L.groups;
  if (c.kind == LG_MIXER_LATENT) {
    L.Dn = round_up(c.dim, 8);
    L.Dh = pow2_at_least(std::max(L.Dn + round_up(c.rot_dims, 8), c.vdim), 64);
    L.Rc = round_up(c.kv_rank, 8);
    L.Rp = r64(L.Rc + c.rot_dims);
    L.Qp = r64(c.q_rank);
    L.N = L.Qp + L.Rp + round_up(c.heads, 16);
    L.Kout = c.heads * L.Dh;
    return;
  }
  g.n_groups = 1;
  if (c.kind == LG_MIXER_ATTENTION) {
    L.Dh = pow2_at_least(std::max(c.dim, c.vdim), 64);
    L.Kout = c.heads * L.Dh;
    g.n_main = round_up((c.heads + 2 * c.kv_heads) * L.Dh, 128);
    g.ld_tail = round_up(c.heads, 16);
  } else {
    L.Dp = pow2_at_least(c.dim, 32);
    L.Vp = pow2_at_least(c.vdim, 32);
    L.Rw = round_up(c.heads * L.Dp, 128);
    L.Lr = round_up(c.tm_rank, 32);
    L.Kout = r64(c.heads * L.Vp);
    g.n_main = round_up(2 * c.heads * (L.Dp + L.Vp), 128);
    g.ld_tail = L.Lr;
  }
  L.N = g.end[0] = g.n_main + g.ld_tail;
}

bool upload_gated_kinds(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w, Mat& out) {
  const int H = m->cfg.width, Hp = m->Hp, heads = L.c.heads, dim = L.c.dim, vdim = L.c.vdim;
  const lg_mixer_layer_config_t& c = L.c;
  Mat in(L.N, Hp);
  if (c.kind == LG_MIXER_ATTENTION) {
    const int G = c.kv_heads, D = L.Dh;
    head_rows(in, 0, w.q, heads, dim, D, H);
    head_rows(in, heads * D, w.k, G, dim, D, H);
    head_rows(in, (heads + G) * D, w.v, G, vdim, D, H);
    for (int h = 0; h < heads; ++h) in.row(L.groups.n_main + h, 0, w.g, (size_t)h * H, H);
    std::vector<float> b((size_t)L.groups.n_main, 0.0f);
    auto bias = [&](int at, const void* src, int n, int d) {
      for (int h = 0; h < n; ++h)
        for (int i = 0; i < d; ++i) b[(size_t)at + h * D + i] = f_at(src, (size_t)h * d + i);
    };
    bias(0, w.q_b, heads, dim);
    bias(heads * D, w.k_b, G, dim);
    bias((heads + G) * D, w.v_b, G, vdim);
    head_cols(out, 0, w.o, H, heads, vdim, D);
    return in.up(W.w_in) && W.b_in.upload(b.data(), b.size() * 4) && upload_heads(W.gain_q, w.q_norm, heads, dim, D) && upload_heads(W.gain_k, w.k_norm, G, dim, D);
  }
  if (c.kind == LG_MIXER_GLA) {
    const int R = c.tm_rank, kw = heads * L.Dp, vw = heads * L.Vp;
    head_rows(in, 0, w.q, heads, dim, L.Dp, H);
    head_rows(in, kw, w.k, heads, dim, L.Dp, H);
    head_rows(in, 2 * kw, w.v, heads, vdim, L.Vp, H);
    head_rows(in, 2 * kw + vw, w.g, heads, vdim, L.Vp, H);
    for (int i = 0; i < R; ++i) in.row(L.groups.n_main + i, 0, w.a1, (size_t)i * H, H);
    head_cols(out, 0, w.o, H, heads, vdim, L.Vp);
    // the low-rank matrix twice over: the chunked form multiplies rounded activations and what rounding dropped
    Mat w2(L.Rw, 2 * L.Lr);
    std::vector<float> b((size_t)L.Rw, 0.0f), gain((size_t)vw, 0.0f);
    for (int h = 0; h < heads; ++h) {
      for (int d = 0; d < dim; ++d) {
        for (int half = 0; half < 2; ++half) w2.row(h * L.Dp + d, half * L.Lr, w.a2, ((size_t)h * dim + d) * R, R);
        b[(size_t)h * L.Dp + d] = f_at(w.a2_b, (size_t)h * dim + d);
      }
      for (int d = 0; d < vdim; ++d) gain[(size_t)h * L.Vp + d] = f_at(w.norm, (size_t)d);
    }
    return in.up(W.w_in) && w2.up(W.w2) && W.w0.upload(b.data(), b.size() * 4) && W.gain.upload(gain.data(), gain.size() * 4);
  }
  const int Q = c.q_rank, R = c.kv_rank, rot = c.rot_dims, D = L.Dh, HD = heads * D;
  for (int i = 0; i < Q; ++i) in.row(i, 0, w.dq, (size_t)i * H, H);
  for (int i = 0; i < R; ++i) in.row(L.Qp + i, 0, w.dkv, (size_t)i * H, H);
  for (int i = 0; i < rot; ++i) in.row(L.Qp + L.Rc + i, 0, w.dkv, (size_t)(R + i) * H, H);
  for (int h = 0; h < heads; ++h) in.row(L.Qp + L.Rp + h, 0, w.g, (size_t)h * H, H);
  Mat uq(HD, L.Qp), k(HD, L.Rp), kt(heads * L.Rp, D), v(HD, L.Rp);
  for (int h = 0; h < heads; ++h) {
    for (int d = 0; d < dim; ++d) {
      uq.row(h * D + d, 0, w.uq, ((size_t)h * (dim + rot) + d) * Q, Q);
      k.row(h * D + d, 0, w.uk, ((size_t)h * dim + d) * R, R);
      for (int r = 0; r < R; ++r) kt.v[((size_t)h * L.Rp + r) * D + d] = bf_at(w.uk, ((size_t)h * dim + d) * R + r);
    }
    for (int j = 0; j < rot; ++j) {
      uq.row(h * D + L.Dn + j, 0, w.uq, ((size_t)h * (dim + rot) + dim + j) * Q, Q);
      k.v[((size_t)h * D + L.Dn + j) * L.Rp + L.Rc + j] = kOne;
      kt.v[((size_t)h * L.Rp + L.Rc + j) * D + L.Dn + j] = kOne;
    }
    for (int d = 0; d < vdim; ++d) v.row(h * D + d, 0, w.uv, ((size_t)h * vdim + d) * R, R);
  }
  head_cols(out, 0, w.o, H, heads, vdim, D);
  return in.up(W.w_in) && uq.up(W.w_uq) && (m->cfg.is_f32 || k.up(W.w_uk)) && kt.up(W.w_ukt) && v.up(W.w_uv) && upload_vec(W.gain_q, w.dq_norm, Q, L.Qp, 0.0f) &&
         upload_vec(W.gain_k, w.dkv_norm, R, L.Rp, 0.0f);
}

bool alloc_gated_kinds(Mixer* m, MLayer& L, Sizes& z) {
  const lg_mixer_config_t& c = m->cfg;
  const size_t esz = c.is_f32 ? 4 : 2, tokens = (size_t)c.n_pool_blocks * kKvBlock, cap_tokens = std::max((size_t)c.max_blocks_per_seq * kKvBlock, (size_t)c.max_step_tokens);
  if (L.c.kind == LG_MIXER_GLA) {
    grow(z.z, (size_t)L.Rw);
    grow(z.low, (size_t)2 * L.Lr);
    return zeroed(L.state, (size_t)c.n_state_slots * L.c.heads * L.Dp * L.Vp * 4);
  }
  const int max_chunks = m->views[(size_t)L.view].max_chunks;
  if (L.c.kind == LG_MIXER_ATTENTION) {
    if (!c.is_f32) {
      grow(z.attn_ws, logismos_paged_prefix_attention_scratch_bytes((int32_t)cap_tokens, c.max_step_seqs, L.c.kv_heads, L.Dh));
      grow(z.scratch, logismos_paged_decode_scratch_bytes(max_chunks, L.c.heads, L.Dh));
    }
    const size_t pool = tokens * L.c.kv_heads * L.Dh * esz;
    return zeroed(L.kpool, pool) && zeroed(L.vpool, pool);
  }
  grow(z.raw, (size_t)L.N);
  grow(z.tail, (size_t)L.N);
  grow(z.cq, (size_t)L.Qp);
  grow(z.proj, (size_t)L.c.heads * L.Dh);
  grow(z.heads, (size_t)round_up(L.c.heads, 16));
  grow(z.lat_q, (size_t)L.c.heads * L.Rp);
  grow(z.lat, (size_t)L.Rp);
  grow(z.lat_heads, (size_t)L.c.heads * L.Dh);
  if (!c.is_f32) grow(z.scratch, logismos_latent_decode_scratch_bytes(max_chunks, L.c.heads, L.Rp));
  return zeroed(L.kpool, tokens * L.Rp * esz);
}

bool want_gated_kinds(Wanted& t, const std::string& mix, int64_t H, lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L) {
  const int64_t heads = y.heads, QD = heads * y.dim, HV = heads * y.vdim;
  if (!t.get(mix + "o", {H, HV}, &L.o)) return false;
  if (y.kind == LG_MIXER_ATTENTION) {
    const int64_t KD = (int64_t)y.kv_heads * y.dim, KV = (int64_t)y.kv_heads * y.vdim;
    return t.get(mix + "q", {QD, H}, &L.q) && t.get(mix + "q.b", {QD}, &L.q_b) && t.get(mix + "q.norm", {QD}, &L.q_norm) && t.get(mix + "k", {KD, H}, &L.k) &&
           t.get(mix + "k.b", {KD}, &L.k_b) && t.get(mix + "k.norm", {KD}, &L.k_norm) && t.get(mix + "v", {KV, H}, &L.v) && t.get(mix + "v.b", {KV}, &L.v_b) &&
           t.get(mix + "g", {heads, H}, &L.g);
  }
  if (y.kind == LG_MIXER_GLA) {
    if (!t.rows(mix + "a1", &y.tm_rank)) return false;
    return t.get(mix + "q", {QD, H}, &L.q) && t.get(mix + "k", {QD, H}, &L.k) && t.get(mix + "v", {HV, H}, &L.v) && t.get(mix + "g", {HV, H}, &L.g) &&
           t.get(mix + "norm", {y.vdim}, &L.norm) && t.get(mix + "a1", {y.tm_rank, H}, &L.a1) && t.get(mix + "a2", {QD, y.tm_rank}, &L.a2) && t.get(mix + "a2.b", {QD}, &L.a2_b);
  }
  const int64_t Q = y.q_rank, R = y.kv_rank;
  return t.get(mix + "dq", {Q, H}, &L.dq) && t.get(mix + "dq.norm", {Q}, &L.dq_norm) && t.get(mix + "uq", {heads * (y.dim + y.rot_dims), Q}, &L.uq) &&
         t.get(mix + "dkv", {R + y.rot_dims, H}, &L.dkv) && t.get(mix + "dkv.norm", {R}, &L.dkv_norm) && t.get(mix + "uk", {QD, R}, &L.uk) &&
         t.get(mix + "uv", {HV, R}, &L.uv) && t.get(mix + "g", {heads, H}, &L.g);
}

// ---- feed-forwards ----------------------------------------------------------------------------------

const char* check_feed_forward(const lg_mixer_layer_config_t& y) {
  if (y.ff < 0) return "feed-forward size";
  if (y.ff == 0 || y.ff_kind == LG_FF_RELU2 || y.ff_kind == LG_FF_GATED) return nullptr;
  if (y.ff_kind != LG_FF_MIXTURE) return "kind of feed-forward";
  if (y.experts <= 0 || y.identity < 0 || y.experts + y.identity > 512) return "experts (at most 512 with the identity experts)";
  if (y.top <= 0 || y.top > 32 || y.top > y.experts + y.identity) return "experts per token (at most 32)";
  if (y.scoring != LG_ROUTE_SOFTMAX && y.scoring != LG_ROUTE_SIGMOID) return "scores of the router";
  if (y.route_groups < 0 || (y.route_groups > 0 && ((y.experts + y.identity) % y.route_groups || y.keep_groups <= 0 || y.keep_groups > y.route_groups ||
                                                    y.top > (y.experts + y.identity) / y.route_groups * y.keep_groups)))
    return "groups of experts";
  if (!(y.glu_limit >= 0.0f)) return "a limit of the gated units that is negative";
  if (y.shared_ff < 0 || (y.shared_ff + y.ff - 1) / y.ff > 64) return "a shared expert of more than 64 times an expert's size";
  return nullptr;
}

bool upload_feed_forward(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w) {
  const int H = m->cfg.width, Hp = m->Hp;
  const lg_mixer_layer_config_t& c = L.c;
  if (c.ff_kind == LG_FF_RELU2) {
    Mat up(L.Fp, Hp), down(Hp, L.Fp);
    for (int i = 0; i < c.ff; ++i) up.row(i, 0, w.up, (size_t)i * H, H);
    for (int i = 0; i < H; ++i) down.row(i, 0, w.down, (size_t)i * c.ff, c.ff);
    return up.up(W.w_up) && down.up(W.w_down);
  }
  if (c.ff_kind == LG_FF_GATED) {
    Mat up(2 * L.Fp, Hp), down(Hp, L.Fp);
    gate_up_rows(up, 0, w.gate, w.up, 0, c.ff, H);
    for (int i = 0; i < H; ++i) down.row(i, 0, w.down, (size_t)i * c.ff, c.ff);
    return up.up(W.w_up) && down.up(W.w_down);
  }
  const int groups = c.experts + L.always, n = c.experts + c.identity;
  const size_t up_bytes = (size_t)2 * L.Fp * Hp * 2, down_bytes = (size_t)Hp * L.Fp * 2;
  if (!W.w_up.alloc(groups * up_bytes) || !W.w_down.alloc(groups * down_bytes)) return false;
  for (int e = 0; e < groups; ++e) {
    const bool routed = e < c.experts;
    const int first = routed ? 0 : (e - c.experts) * c.ff, ff = routed ? c.ff : std::min(c.ff, c.shared_ff - first), ld = routed ? c.ff : c.shared_ff;
    const void *gate = routed ? w.experts[3 * e] : w.shared_gate, *up = routed ? w.experts[3 * e + 1] : w.shared_up, *down = routed ? w.experts[3 * e + 2] : w.shared_down;
    Mat gu(2 * L.Fp, Hp), d(Hp, L.Fp);
    gate_up_rows(gu, 0, gate, up, first, ff, H);
    for (int i = 0; i < H; ++i) d.row(i, 0, down, (size_t)i * ld + first, ff);
    if (cudaMemcpy((uint8_t*)W.w_up.p + e * up_bytes, gu.v.data(), up_bytes, cudaMemcpyHostToDevice) != cudaSuccess ||
        cudaMemcpy((uint8_t*)W.w_down.p + e * down_bytes, d.v.data(), down_bytes, cudaMemcpyHostToDevice) != cudaSuccess)
      return false;
  }
  if (!c.no_correction && !upload_vec(W.correction, w.correction, n, n, 0.0f)) return false;
  if (m->cfg.norm == LG_NORM_RMS_GATED) return true;  // the router's rows follow those of the gate
  Mat router(L.route_ld, Hp);
  for (int i = 0; i < n; ++i) router.row(i, 0, w.router, (size_t)i * H, H);
  return router.up(W.w_router);
}

void size_feed_forward(const MLayer& L, Sizes& z) {
  if (!L.c.ff) return;
  if (L.c.ff_kind != LG_FF_MIXTURE) { grow(z.ff, (size_t)L.Fp); return; }
  const size_t pairs = (size_t)(L.c.top + L.always);
  grow(z.ff, pairs * L.Fp);
  grow(z.route, (size_t)L.route_ld);
  grow(z.pairs, pairs);
  grow(z.top, (size_t)L.c.top);
  grow(z.groups, (size_t)(L.c.experts + L.always));
}

bool want_feed_forward(Wanted& t, const std::string& mlp, int64_t H, const lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L, std::vector<const void*>& experts) {
  auto unit = [&](const std::string& p, int64_t F, const void** gate, const void** up, const void** down) {
    return t.get(p + "gate", {F, H}, gate) && t.get(p + "up", {F, H}, up) && t.get(p + "down", {H, F}, down);
  };
  if (y.ff_kind == LG_FF_RELU2) return t.get(mlp + "up", {y.ff, H}, &L.up) && t.get(mlp + "down", {H, y.ff}, &L.down);
  if (y.ff_kind == LG_FF_GATED) return unit(mlp, y.ff, &L.gate, &L.up, &L.down);
  experts.assign((size_t)3 * y.experts, nullptr);
  L.experts = experts.data();
  for (int e = 0; e < y.experts; ++e)
    if (!unit(mlp + "e" + std::to_string(e) + ".", y.ff, &experts[(size_t)3 * e], &experts[(size_t)3 * e + 1], &experts[(size_t)3 * e + 2])) return false;
  const int64_t n = y.experts + y.identity;
  return t.get(mlp + "router", {n, H}, &L.router) && (y.no_correction || t.get(mlp + "correction", {n}, &L.correction)) &&
         (!y.shared_ff || unit(mlp + "shared.", y.shared_ff, &L.shared_gate, &L.shared_up, &L.shared_down));
}

}  // namespace lgm
