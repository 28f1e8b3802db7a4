// Differential attention and pooled-window attention beside linear attention, the mixers of a stack with gated residuals:
// layout and upload of their weights, buffers, and their part of a step (the output projections and the residual follow in
// mixer_model.cu).
//   differential: one GEMM to q | k | v | gate of the residual -> norm per head and map, rotation, cache store. A cache row holds
//     both maps' keys side by side, a query fills the half of its map: one attention over twice the heads, in fp32 -> difference,
//     norm
//   pair: one GEMM to q | k | v of the left and v | k | q (silu in its epilogue) | gate of the right branch | gate of the residual.
//     Left: norm per head, rotation, cache store, means of the blocks that end -> attention over pooled blocks and window. Right:
//     recurrence with a fixed decay, token by token for decode rows, chunk-parallel for prompt rows -> norm and gate
// Rotations of halves become rotations of neighbours by an order of the channels that queries and keys share.
#include "mixer_stack.h"

namespace lgm {

namespace {

// where channel i of a head stands, so that rotated pairs are neighbours
int place(const lg_mixer_layer_config_t& c, int i) {
  if (!c.rot_halves || i >= c.rot_dims) return i;
  const int half = c.rot_dims / 2;
  return i < half ? 2 * i : 2 * (i - half) + 1;
}

bool upload_head_gain(Buf& b, const void* src, const lg_mixer_layer_config_t& c, int padded) {
  std::vector<float> v((size_t)padded, 0.0f);
  for (int i = 0; i < c.dim; ++i) v[(size_t)place(c, i)] = f_at(src, (size_t)i);
  return b.upload(v.data(), v.size() * 4);
}

// queries, keys and values of the step: norms, rotation, cache
uint32_t store_heads(Mixer* m, MLayer& L, const MWeights& W, int maps, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  lg_head_norm_t a{};
  a.qkv = m->proj.p; a.ld = L.groups.n_main; a.rows = B.T; a.heads = L.c.heads; a.n_kv = L.c.kv_heads; a.maps = maps; a.hd = L.Dh / maps; a.dim = L.c.dim;
  a.gain_q = W.gain_q.p; a.gain_k = W.gain_k.p; a.eps = c.norm_eps;
  if (L.table >= 0) { a.table = m->tables[(size_t)L.table].angles.p; a.rot_dims = L.c.rot_dims; }
  if (maps == 2) { a.q_out = m->qx.p; a.ld_q = 2 * L.c.heads * L.Dh; }
  a.k_pool = L.kpool.p; a.v_pool = L.vpool.p; a.slots_i64 = m->dev(B.slots); a.positions_i32 = m->dev(B.pos); a.n_pool_slots = (int64_t)c.n_pool_blocks * kKvBlock;
  a.pool = L.c.pool; a.pool_rows = B.n_dec; a.k_mean = L.kmean.p; a.v_mean = L.vmean.p; a.tables_i32 = m->dev(B.tables); a.seq_ids_i32 = m->dev(B.seq_ids);
  a.max_blocks = c.max_blocks_per_seq; a.n_pool_blocks = c.n_pool_blocks;
  LG_TRY(logismos_launch_head_norm_store(&a, c.is_f32, m->status.p, s), "queries, keys and cache store");
  m->launches += 1;
  bool ends = false;  // a block inside the step's prompt rows
  for (int k = B.n_dec; k < B.n_seqs && a.pool; ++k) ends = ends || (B.cached[(size_t)k] + B.newl[(size_t)k]) / a.pool > B.cached[(size_t)k] / a.pool;
  if (ends) {
    LG_TRY(logismos_launch_pool_blocks(&a, c.is_f32, m->status.p, s), "means of blocks");
    m->launches += 1;
  }
  return 0;
}

uint32_t differential(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int heads = 2 * L.c.heads, ld = heads * L.Dh, T = B.T;
  LG_TRY(projections(m, L, W, false, s), "input projections");
  if (uint32_t rc = store_heads(m, L, W, 2, s)) return rc;
  lg_window_t w = m->views[(size_t)L.view].shape;
  w.scale = L.c.scale; w.out_f32 = 1;
  const int alone = c.is_f32 ? 0 : B.n_dec;   // decode rows whose merge takes the difference too
  if (alone > 0) {
    const DecodeView& V = m->views[(size_t)L.view];
    LG_TRY(logismos_launch_differential_decode_bf16(m->qx.p, ld, L.kpool.p, L.vpool.p, m->dev(B.tables), m->dev(B.ctx), m->dev(V.chunks), m->act.p, L.Kout, m->dec_scratch.p, alone,
                                                    V.total, V.chunk_tokens, c.max_blocks_per_seq, c.n_pool_blocks, L.c.heads, L.c.kv_heads, L.Dh, &w, L.c.vdim, W.lambda,
                                                    1.0f - L.c.diff, c.norm_eps, m->status.p, s), "differential decode");
    m->launches += 2;
  }
  if (T == alone) return 0;
  if (!c.is_f32 && logismos_differential_has_prompts(L.Dh)) {
    const size_t row0 = (size_t)alone;
    for (const PrefixRun& r : B.runs) {
      int total, longest;
      gathered_keys(B, w, r, &total, &longest);
      LG_TRY(logismos_launch_differential_prefix_bf16((const uint16_t*)m->qx.p + row0 * ld, ld, m->dev(B.cu_pre) + r.s0, m->dev(B.pre_kv) + r.s0, L.kpool.p, L.vpool.p,
                                                      m->dev(B.tables) + (row0 + r.s0) * c.max_blocks_per_seq, c.max_blocks_per_seq, c.n_pool_blocks,
                                                      (uint16_t*)m->act.p + row0 * L.Kout, L.Kout, m->attn_ws.p, T - alone, total, r.s1 - r.s0, r.max_q, longest, L.c.heads,
                                                      L.c.kv_heads, L.Dh, &w, L.c.vdim, W.lambda, 1.0f - L.c.diff, c.norm_eps, m->status.p, s), "differential attention");
      m->launches += 2;
    }
    return 0;
  }
  if (uint32_t rc = window_attention(m, L, w, m->qx.p, ld, heads, L.c.kv_heads, L.Dh, m->maps_out.p, ld, s, true)) return rc;
  LG_TRY(logismos_launch_attention_difference((const float*)m->maps_out.p + (size_t)alone * ld, ld, (uint8_t*)m->act.p + (size_t)alone * L.Kout * (c.is_f32 ? 4 : 2), L.Kout, c.is_f32,
                                              T - alone, L.c.heads, L.c.kv_heads, L.c.vdim, L.Dh, W.lambda, 1.0f - L.c.diff, c.norm_eps, s), "difference");
  m->launches += 1;
  return 0;
}

uint32_t linear_attention(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const int f32 = c.is_f32, inner = L.c.lin_heads * L.Vp, P = L.groups.n_main;
  const size_t esz = f32 ? 4 : 2;
  lg_ssd_t a{};
  a.xbc = (uint8_t*)m->proj.p + (size_t)L.off_right * esz; a.ld_xbc = P; a.decay = W.decay.p;
  a.state = L.state.p; a.state_slots = m->dev(B.state); a.fresh = m->dev(B.fresh); a.cu = m->dev(B.cu);
  a.y = m->ffb.p; a.ld_y = inner; a.heads = a.groups = L.c.lin_heads; a.np = L.Np; a.vp = L.Vp;
  const bool chunked = !f32 && B.n_pre > 0 && logismos_ssd_has_chunked(L.Np, L.Vp);
  const int serial = chunked ? B.n_dec : B.n_seqs;  // sequences that go token by token
  if (serial > 0) {
    LG_TRY(logismos_launch_ssd_step(&a, serial, f32, s), "linear attention");
    m->launches += 1;
  }
  if (chunked) {
    a.state_slots = m->dev(B.state) + B.n_dec; a.fresh = m->dev(B.fresh) + B.n_dec; a.cu = m->dev(B.cu) + B.n_dec;
    LG_TRY(prompt_recurrence(m, &a, s), "linear attention (prompts)");
  }
  const uint8_t* gate = (const uint8_t*)m->proj.p + (size_t)(L.off_right + L.channels) * esz;
  LG_TRY(logismos_launch_norm_gate(m->ffb.p, inner, gate, P, W.gain.p, (uint8_t*)m->act.p + (size_t)L.Kleft * esz, L.Kout, f32, B.T, L.c.lin_heads, L.c.lin_vdim, L.Vp,
                                   c.norm_eps, s), "norm and gate");
  m->launches += 1;
  return 0;
}

uint32_t pair(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  LG_TRY(projections(m, L, W, false, s), "input projections");
  if (uint32_t rc = store_heads(m, L, W, 1, s)) return rc;
  lg_window_t w = m->views[(size_t)L.view].shape;
  w.scale = L.c.scale; w.k_mean = L.kmean.p; w.v_mean = L.vmean.p;
  if (uint32_t rc = window_attention(m, L, w, m->proj.p, L.groups.n_main, L.c.heads, L.c.kv_heads, L.Dh, m->act.p, L.Kout, s)) return rc;
  return linear_attention(m, L, W, s);
}

}  // namespace

uint32_t run_paired_kinds(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) { return L.c.kind == LG_MIXER_DIFF ? differential(m, L, W, s) : pair(m, L, W, s); }

const char* check_paired_kinds(const lg_mixer_layer_config_t& y) {
  const bool diff = y.kind == LG_MIXER_DIFF;
  if (!diff && y.kind != LG_MIXER_PAIR) return "kind of mixer";
  if (y.heads <= 0 || y.kv_heads <= 0 || y.heads % y.kv_heads) return "attention heads";
  if (y.dim <= 0 || y.dim > (diff ? 128 : 256) || y.vdim <= 0 || y.vdim > 256) return "head dimensions above 256 (queries of differential attention: 128)";
  if (!(y.scale > 0.0f)) return "a score scale that is not positive";
  if (y.rot_dims < 0 || y.rot_dims % 2 || y.rot_dims > y.dim || (y.rot_dims > 0 && !(y.rot_base > 1.0))) return "rotated dimensions that are not pairs of a head's, or a base that is not above 1";
  if (!(y.rot_factor >= 0.0) || (y.rot_factor != 0.0 && y.rot_original != 0.0 && (!(y.rot_original > 0.0) || !(y.rot_fast > 0.0) || !(y.rot_slow > 0.0)))) return "scaling of the rotation";
  if (y.window < 0 || y.keep_first || y.pool < 0 || (y.chunked && y.pool) || ((y.chunked || y.pool) && !y.window)) return "window, chunks or pooled blocks";
  if (diff) return nullptr;
  if (y.lin_heads <= 0 || y.lin_dim <= 0 || y.lin_dim > 256 || y.lin_vdim <= 0 || y.lin_vdim > 256) return "heads of the linear attention, or their dimensions above 256";
  if (!y.decay) return "decays of the linear attention";
  for (int h = 0; h < y.lin_heads; ++h)
    if (!(y.decay[h] >= 0.0) || y.decay[h] > 1.0) return "a decay outside [0, 1]";
  return nullptr;
}

void layout_paired_kinds(const Mixer* m, MLayer& L) {
  const lg_mixer_layer_config_t& c = L.c;
  lg_linear_groups_t& g = L.groups;
  L.Dh = c.kind == LG_MIXER_DIFF ? std::max(2 * pow2_at_least(c.dim, 32), pow2_at_least(c.vdim, 64)) : pow2_at_least(std::max(c.dim, c.vdim), 64);
  L.Kleft = L.Kout = c.heads * L.Dh;
  L.off_right = L.off_gate = (c.heads + 2 * c.kv_heads) * L.Dh;
  if (c.kind == LG_MIXER_PAIR) {
    L.Vp = pow2_at_least(c.lin_vdim, 32);
    L.Np = pow2_at_least(c.lin_dim, 32);
    L.channels = c.lin_heads * (L.Vp + 2 * L.Np);
    g.silu_begin = L.off_right;
    g.silu_end = L.off_right + L.channels;
    L.off_gate = r64(g.silu_end + c.lin_heads * L.Vp);
    L.Kout += r64(c.lin_heads * L.Vp);
  }
  g.n_groups = 1;
  L.N = g.end[0] = g.n_main = L.off_gate + m->Hp;
}

bool upload_paired_kinds(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w) {
  const int H = m->cfg.width, Hp = m->Hp, heads = L.c.heads, G = L.c.kv_heads, rep = heads / G, dim = L.c.dim, vdim = L.c.vdim, D = L.Dh;
  const lg_mixer_layer_config_t& c = L.c;
  const bool diff = c.kind == LG_MIXER_DIFF;
  Mat in(L.N, Hp);
  auto head = [&](int row0, const void* src, int src_head) {  // one head (and map) of queries or keys
    for (int d = 0; d < dim; ++d) in.row(row0 + place(c, d), 0, src, ((size_t)src_head * dim + d) * H, H);
  };
  const int maps = diff ? 2 : 1, piece = D / maps;
  const void *q = diff ? w.q : w.left_q, *k = diff ? w.k : w.left_k, *v = diff ? w.v : w.left_v;
  for (int kv = 0; kv < G; ++kv)
    for (int mp = 0; mp < maps; ++mp) {
      for (int r = 0; r < rep; ++r) head(((kv * maps + mp) * rep + r) * piece, q, (kv * rep + r) * maps + mp);
      head(heads * D + (kv * maps + mp) * piece, k, kv * maps + mp);
    }
  head_rows(in, (heads + G) * D, v, G, vdim, D, H);
  Mat out(Hp, L.Kleft);
  head_cols(out, 0, diff ? w.o : w.left_o, H, heads, vdim, D);
  bool ok = out.up(W.w_out) && upload_head_gain(W.gain_q, diff ? w.q_norm : w.left_q_norm, c, piece) && upload_head_gain(W.gain_k, diff ? w.k_norm : w.left_k_norm, c, piece);
  if (diff) {
    double a = 0.0, b = 0.0;
    for (int i = 0; i < dim; ++i) {
      a += (double)f_at(w.lq1, (size_t)i) * f_at(w.lk1, (size_t)i);
      b += (double)f_at(w.lq2, (size_t)i) * f_at(w.lk2, (size_t)i);
    }
    W.lambda = (float)(std::exp(a) - std::exp(b) + c.diff);
  } else {
    const int lin = c.lin_heads, kr = L.off_right + lin * L.Vp, qr = kr + lin * L.Np;
    head_rows(in, L.off_right, w.right_v, lin, c.lin_vdim, L.Vp, H);
    head_rows(in, kr, w.right_k, lin, c.lin_dim, L.Np, H);
    head_rows(in, qr, w.right_q, lin, c.lin_dim, L.Np, H);
    head_rows(in, qr + lin * L.Np, w.right_g, lin, c.lin_vdim, L.Vp, H);
    Mat out2(Hp, L.Kout - L.Kleft);
    head_cols(out2, 0, w.right_o, H, lin, c.lin_vdim, L.Vp);
    std::vector<float> decay((size_t)lin * 3);
    for (int h = 0; h < lin; ++h) {
      float* d = decay.data() + (size_t)h * 3;
      d[0] = (float)std::max(std::log2(c.decay[h]), -1e4);  // nothing is left of a step further down
      d[1] = (float)c.decay[h];
      d[2] = (float)(c.decay[h] - (double)d[1]);
    }
    if (L.Kout == 2 * L.Kleft) {  // one batch of two products
      Mat both(2 * Hp, L.Kleft);
      std::copy(out.v.begin(), out.v.end(), both.v.begin());
      std::copy(out2.v.begin(), out2.v.end(), both.v.begin() + (std::ptrdiff_t)out.v.size());
      W.w_out.release();
      ok = ok && both.up(W.w_out);
    } else {
      ok = ok && out2.up(W.w_out2);
    }
    ok = ok && W.decay.upload(decay.data(), decay.size() * 4) && upload_heads(W.gain, w.right_norm, lin, c.lin_vdim, L.Vp) &&
         upload_vec(W.branch_gain[0], w.left_out, H, Hp, 0.0f) && upload_vec(W.branch_gain[1], w.right_out, H, Hp, 0.0f);
  }
  std::vector<float> b((size_t)L.N, 0.0f);
  for (int i = 0; i < H; ++i) {
    in.row(L.off_gate + i, 0, w.rg1, (size_t)i * H, H);
    b[(size_t)L.off_gate + i] = f_at(w.rg1_b, (size_t)i);
  }
  return ok && in.up(W.w_in) && W.b_in.upload(b.data(), b.size() * 4);
}

bool alloc_paired_kinds(Mixer* m, MLayer& L, Sizes& z) {
  const lg_mixer_config_t& c = m->cfg;
  const size_t esz = c.is_f32 ? 4 : 2, row = (size_t)L.c.kv_heads * L.Dh, pool = (size_t)c.n_pool_blocks * kKvBlock * row * esz;
  const int maps = L.c.kind == LG_MIXER_DIFF ? 2 : 1;
  if (!c.is_f32) {
    size_t keys = std::max((size_t)c.max_blocks_per_seq * kKvBlock, (size_t)c.max_step_tokens);
    if (L.c.pool) keys += keys / (size_t)L.c.pool + (size_t)128 * c.max_step_seqs;   // leading tiles of pooled blocks
    grow(z.attn_ws, logismos_paged_prefix_attention_scratch_bytes((int32_t)keys, c.max_step_seqs, L.c.kv_heads, L.Dh));
    grow(z.scratch, logismos_paged_decode_scratch_bytes(m->views[(size_t)L.view].max_chunks, maps * L.c.heads, L.Dh));
  }
  if (maps == 2) grow(z.maps, (size_t)2 * L.c.heads * L.Dh);
  bool ok = zeroed(L.kpool, pool) && zeroed(L.vpool, pool);
  if (L.c.pool) {
    const size_t means = (size_t)c.n_pool_blocks * (kKvBlock + L.c.pool - 1) / L.c.pool * row * esz;
    ok = ok && zeroed(L.kmean, means) && zeroed(L.vmean, means);
  }
  if (L.c.kind == LG_MIXER_PAIR) {
    grow(z.ff, (size_t)L.c.lin_heads * L.Vp);
    size_prompt_recurrence(m, L.c.lin_heads, L.Np, L.Vp, z);
    ok = ok && zeroed(L.state, (size_t)c.n_state_slots * L.c.lin_heads * L.Np * L.Vp * 4);
  }
  return ok;
}

bool want_paired_kinds(Wanted& t, const std::string& mix, int64_t H, lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L) {
  const bool diff = y.kind == LG_MIXER_DIFF;
  const int64_t QD = (int64_t)y.heads * y.dim, KD = (int64_t)y.kv_heads * y.dim, KV = (int64_t)y.kv_heads * y.vdim, HV = (int64_t)y.heads * y.vdim;
  if (diff)
    return t.get(mix + "q", {2 * QD, H}, &L.q) && t.get(mix + "k", {2 * KD, H}, &L.k) && t.get(mix + "v", {KV, H}, &L.v) && t.get(mix + "q.norm", {y.dim}, &L.q_norm) &&
           t.get(mix + "k.norm", {y.dim}, &L.k_norm) && t.get(mix + "lq1", {y.dim}, &L.lq1) && t.get(mix + "lk1", {y.dim}, &L.lk1) && t.get(mix + "lq2", {y.dim}, &L.lq2) &&
           t.get(mix + "lk2", {y.dim}, &L.lk2) && t.get(mix + "o", {H, HV}, &L.o);
  const std::string a = mix + "left.", b = mix + "right.";
  const int64_t D = (int64_t)y.lin_heads * y.lin_dim, V = (int64_t)y.lin_heads * y.lin_vdim;
  return t.get(a + "q", {QD, H}, &L.left_q) && t.get(a + "k", {KD, H}, &L.left_k) && t.get(a + "v", {KV, H}, &L.left_v) && t.get(a + "q.norm", {y.dim}, &L.left_q_norm) &&
         t.get(a + "k.norm", {y.dim}, &L.left_k_norm) && t.get(a + "o", {H, HV}, &L.left_o) && t.get(a + "out", {H}, &L.left_out) && t.get(b + "q", {D, H}, &L.right_q) &&
         t.get(b + "k", {D, H}, &L.right_k) && t.get(b + "v", {V, H}, &L.right_v) && t.get(b + "g", {V, H}, &L.right_g) && t.get(b + "norm", {V}, &L.right_norm) &&
         t.get(b + "o", {H, V}, &L.right_o) && t.get(b + "out", {H}, &L.right_out);
}

}  // namespace lgm
