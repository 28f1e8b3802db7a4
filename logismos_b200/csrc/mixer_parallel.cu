// State-space mixers and parallel mixers (attention beside time mixing) of the stack of mixers: layout and upload of their
// weights, buffers, and their part of a step.
//   state-space: convolution -> recurrence, token by token for decode rows, chunk-parallel for prefill rows -> gate + norm
//   parallel: unit q, k + cache store -> attention with its gate into the left columns of one activation row; time mixing
//     with its norm and gate into the right ones; one GEMM over [left W_o | right W_o] follows (the branch scales ride on
//     the gates)
#include "mixer_stack.h"

namespace lgm {

uint32_t run_ssd(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
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
    LG_TRY(prompt_recurrence(m, &a, s), "state-space recurrence (prompts)");
  }
  LG_TRY(logismos_launch_gated_group_norm(m->ffb.p, inner, m->proj.p, L.groups.n_main, W.gain.p, m->act.p, L.Kout, f32, T, L.c.ssd_heads, L.c.ssd_vdim, L.Vp,
                                          L.c.ssd_norm_groups, c.norm_eps, s), "gate and norm");
  m->launches += 1;
  return 0;
}

uint32_t prompt_recurrence(Mixer* m, lg_ssd_t* a, cudaStream_t s) {
  const StepBatch& B = m->batch;
  int entries = logismos_ssd_segments(B.T - B.n_dec, B.n_pre, B.max_pre_len, a->heads);
  if (logismos_ssd_scratch_bytes(entries, a->heads, a->np, a->vp) > m->segment_bytes) entries = 0;
  m->launches += entries > 0 ? 3 : 1;
  return logismos_launch_ssd_segmented_bf16(a, B.n_pre, B.max_pre_len, m->segments.p, entries, s);
}

// room for a step of one long prompt, and of as many as are still cut
void size_prompt_recurrence(const Mixer* m, int heads, int np, int vp, Sizes& z) {
  if (m->cfg.is_f32 || !logismos_ssd_has_chunked(np, vp)) return;
  const int T = m->cfg.max_step_tokens;
  for (int n = 1; n <= m->cfg.max_step_seqs; ++n) grow(z.segments, logismos_ssd_scratch_bytes(logismos_ssd_segments(T, n, T, heads), heads, np, vp));
}

namespace {

uint32_t attention(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  const lg_mixer_config_t& c = m->cfg;
  StepBatch& B = m->batch;
  const DecodeView& V = m->views[(size_t)L.view];
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
    LG_TRY(logismos_launch_bias_attention_decode_bf16(proj, P, L.kpool.p, L.vpool.p, m->dev(B.tables), m->dev(B.ctx), m->dev(V.chunks), out, L.Kout,
                                                      m->dec_scratch.p, B.n_dec, V.total, V.chunk_tokens, MB, c.n_pool_blocks, L.c.heads,
                                                      L.c.kv_heads, L.Dh, &sb, st, s), "decode attention");
    m->launches += V.total > B.n_dec ? 2 : 1;
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
  const bool chunked = !f32 && B.n_pre > 0 && logismos_time_mix_has_chunked(L.Dp, L.Dp);
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

}  // namespace

uint32_t run_parallel(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s) {
  if (uint32_t rc = attention(m, L, W, s)) return rc;
  return time_mixing(m, L, W, s);
}

// ---- weights ---------------------------------------------------------------------------------------

namespace {

// row of the bias table for a distance: one per distance below rows / 2, then logarithmic up to `far`
int distance_bucket(int n, int rows, int far) {
  const int half = rows / 2;
  if (n < half) return n;
  const double at = std::log((double)n / half) / std::log((double)far / half) * (rows - half);
  const int b = half + (int)std::floor(at);
  return b < rows - 1 ? b : rows - 1;
}

}  // namespace

bool upload_parallel_kinds(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w, Mat& in, Mat& out) {
  const int H = m->cfg.width, Hp = m->Hp;
  const lg_mixer_layer_config_t& c = L.c;
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
    return in.up(W.w_in) && W.conv.upload(cw.data(), cw.size() * 4) && W.conv_b.upload(cb.data(), cb.size() * 4) &&
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
  return in.up(W.w_in) && w2.up(W.w2) && W.mu.upload(mu.data(), mu.size() * 4) && W.bias.upload(bias.data(), bias.size() * 4) &&
         W.w0.upload(w0.data(), w0.size() * 4) && upload_heads(W.u, w.right_u, tm, D, L.Dp) && upload_heads(W.gain, w.right_norm, tm, D, L.Dp);
}

const char* check_parallel_kinds(const lg_mixer_layer_config_t& y) {
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
const char* check_parallel_tensors(const lg_mixer_layer_config_t& y) {
  if (y.kind != LG_MIXER_PARALLEL) return nullptr;
  if (y.bias_rows < 2 || y.bias_max <= y.bias_rows / 2) return "bias table: at least two rows, and bias_max above half of them";
  if (y.tm_rank <= 0) return "rank of the decay";
  return nullptr;
}

void layout_parallel_kinds(MLayer& L) {
  const lg_mixer_layer_config_t& c = L.c;
  lg_linear_groups_t& g = L.groups;
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

bool alloc_parallel_kinds(Mixer* m, MLayer& L, Sizes& z) {
  const lg_mixer_config_t& c = m->cfg;
  const size_t slots = (size_t)c.n_state_slots, MB = (size_t)c.max_blocks_per_seq, T = (size_t)c.max_step_tokens;
  if (L.c.kind == LG_MIXER_SSD) {
    grow(z.ff, (size_t)L.c.ssd_heads * L.Vp);
    grow(z.xbc, (size_t)L.channels);
    size_prompt_recurrence(m, L.c.ssd_heads, L.Np, L.Vp, z);
    return zeroed(L.state, slots * L.c.ssd_heads * L.Np * L.Vp * 4) && zeroed(L.conv_state, slots * 2 * (L.c.ssd_taps - 1) * L.channels * 4);
  }
  const size_t pool = (size_t)c.n_pool_blocks * kKvBlock * L.c.kv_heads * L.Dh * (c.is_f32 ? 4 : 2), cap_tokens = std::max(MB * kKvBlock, T);
  grow(z.z, (size_t)L.Rw);
  grow(z.low, (size_t)2 * L.Lr);
  if (!c.is_f32) {
    grow(z.attn_ws, logismos_paged_prefix_attention_scratch_bytes((int32_t)cap_tokens, c.max_step_seqs, L.c.kv_heads, L.Dh));
    grow(z.scratch, logismos_paged_decode_scratch_bytes(m->views[(size_t)L.view].max_chunks, L.c.heads, L.Dh));
  }
  return zeroed(L.kpool, pool) && zeroed(L.vpool, pool) && zeroed(L.shift, slots * 2 * m->Hp * 4) && zeroed(L.state, slots * L.c.tm_heads * L.Dp * L.Dp * 4);
}

bool want_parallel_kinds(Wanted& t, const std::string& mix, int64_t H, lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L) {
  if (y.kind == LG_MIXER_SSD) {
    const int64_t heads = y.ssd_heads, inner = heads * y.ssd_vdim, ch = inner + 2 * (int64_t)y.ssd_groups * y.ssd_state;
    return t.get(mix + "in", {inner + ch + heads, H}, &L.in) && t.get(mix + "conv", {ch, y.ssd_taps}, &L.conv) && t.get(mix + "conv.b", {ch}, &L.conv_b) &&
           t.get(mix + "dt_bias", {heads}, &L.dt_bias) && t.get(mix + "A_log", {heads}, &L.A_log) && t.get(mix + "D", {heads}, &L.D) &&
           t.get(mix + "norm", {inner}, &L.norm) && t.get(mix + "o", {H, inner}, &L.o);
  }
  const std::string a = mix + "left.", b = mix + "right.";
  if (!t.rows(a + "rel", &y.bias_rows) || !t.rows(b + "w1", &y.tm_rank)) return false;
  if (const char* what = check_parallel_tensors(y)) { t.rc = fail(LG_EMB_COMPUTE, std::string("unsupported mixer-stack config: ") + what); return false; }
  const int64_t QD = (int64_t)y.heads * y.dim, HV = (int64_t)y.heads * y.vdim, HD = (int64_t)y.tm_heads * y.tm_dim, R = y.tm_rank;
  if (!(t.get(a + "q", {QD, H}, &L.left_q) && t.get(a + "k", {(int64_t)y.kv_heads * y.dim, H}, &L.left_k) && t.get(a + "v", {(int64_t)y.kv_heads * y.vdim, H}, &L.left_v) &&
        t.get(a + "rel", {y.bias_rows, y.heads}, &L.left_rel) && t.get(a + "g", {HV, H}, &L.left_g) && t.get(a + "o", {H, HV}, &L.left_o)))
    return false;
  const char* order[kMixes] = {"mu.r", "mu.k", "mu.v", "mu.g", "mu.w"};
  for (int s = 0; s < kMixes; ++s)
    if (!t.get(b + order[s], {H}, &L.mu[s])) return false;
  return t.get(b + "r", {HD, H}, &L.right_r) && t.get(b + "k", {HD, H}, &L.right_k) && t.get(b + "v", {HD, H}, &L.right_v) && t.get(b + "g", {HD, H}, &L.right_g) &&
         t.get(b + "w1", {R, H}, &L.right_w1) && t.get(b + "w2", {HD, R}, &L.right_w2) && t.get(b + "w0", {HD}, &L.right_w0) &&
         t.get(b + "u", {y.tm_heads, y.tm_dim}, &L.right_u) && t.get(b + "norm", {HD}, &L.right_norm) && t.get(b + "o", {H, HD}, &L.right_o);
}

}  // namespace lgm
