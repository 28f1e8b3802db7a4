// The executor of a stack of mixers (lg_mixer_*) as its parts see it: mixer_model.cu holds the step, the norms around the
// sublayers, creation and loading; mixer_parallel.cu the state-space and the parallel mixers; mixer_gated.cu windowed
// attention, gated linear attention, latent attention and the gated feed-forwards; mixer_paired.cu differential attention and
// pooled-window attention beside linear attention.
#pragma once
#include <cuda_runtime.h>

#include <algorithm>
#include <cmath>
#include <initializer_list>
#include <mutex>
#include <string>
#include <vector>

#include "logismos_kernels.h"
#include "logismos_model.h"

#include "model_util.h"
#include "safetensors.h"
#include "step_batch.h"
#include "weight_pack.h"

namespace lgm {

constexpr int kAccRows = 512;   // steps up to this size accumulate their narrow projections over slices of k
constexpr int kMixes = 5;       // r, k, v, g, w

inline int pow2_at_least(int v, int lo) {
  int p = lo;
  while (p < v) p *= 2;
  return p;
}

struct TanhNorm {
  float alpha = 0.0f;
  Buf w, b;
  lg_tanh_norm_t view() const { return lg_tanh_norm_t{alpha, w.p, b.p}; }
};

struct MWeights {   // of a layer that owns tensors
  Buf norm1, norm1_b, norm2, norm2_b, w_up, w_down, w_in, w_out;
  TanhNorm pre1, post1, pre2, post2;
  Buf conv, conv_b, dt_bias, A_log, D, gain;              // state-space (gain also: linear attention)
  Buf bias, mu, w2, w0, u;                                // parallel (w2, w0 also: gated linear attention)
  Buf b_in, gain_q, gain_k;                               // windowed attention; latent attention: gains of its latents
  Buf w_uq, w_uk, w_ukt, w_uv;                            // latent attention
  Buf w_router, correction;                               // mixture: w_up, w_down hold its experts one after the other
  Buf w_gate2, b_gate2;                                   // gated residual: the gate of a feed-forward, then the router's rows
  Buf w_out2, branch_gain[2], decay;                 // a pair
  float gain1 = 0.0f, gain2 = 0.0f, lambda = 0.0f;        // norms of one value; differential attention
  float max_bias = 0.0f;
  void release();
};

struct MLayer {
  lg_mixer_layer_config_t c{};
  int owner = 0;
  lg_linear_groups_t groups{};
  int N = 0, Fp = 0, Kout = 0;          // projection width, feed-forward and output-projection inputs
  int Vp = 0, Np = 0, channels = 0;     // state-space; gated linear attention: value head Vp
  int Dh = 0, Dp = 0, Rw = 0, Lr = 0;   // attention head, linear-attention key head, padded block of its heads, padded rank
  int Qp = 0, Rp = 0, Rc = 0, Dn = 0;   // latent attention: padded latents, first rotated column of a cache row and of a head
  int always = 0, route_ld = 0;         // mixture: experts that every token takes, columns of the router
  int off_right = 0, off_gate = 0, Kleft = 0;   // first columns of the right branch and of the residual's gate, inputs of the left W_o
  lg_linear_groups_t gate2{};           // gated residual: the feed-forward's gate and router
  int view = -1, table = -1;            // decode view, rotation table
  Buf kpool, vpool, kmean, vmean, shift, conv_state, state;
};

// How decode launches split the contexts of a kind of attention: the same for all layers with one window
struct DecodeView {
  bool latent = false;
  lg_window_t shape{};                  // window, kept keys, chunks, pooled blocks
  int kv = 1, hd = 64, heads = 1;       // of the widest layer
  int chunk_tokens = 512, total = 0, max_chunks = 0;
  int32_t* chunks = nullptr;            // host, in the step's index block
};

struct RotationTable {
  int dims = 0;
  double base = 0, factor = 0, original = 0, fast = 0, slow = 0;
  Buf angles;                           // f32 [positions][dims / 2][2]
};

struct Mixer {
  lg_mixer_config_t cfg{};
  std::vector<lg_mixer_layer_config_t> layer_cfg;
  int device = 0, Hp = 0;
  Buf embed, head, final_norm, final_norm_b, loop_step;
  TanhNorm final_tanh;
  float final_gain = 0.0f;
  std::vector<MWeights> weights;
  std::vector<MLayer> layers;
  std::vector<DecodeView> views;
  std::vector<RotationTable> tables;
  Buf x, h, proj, tail, low2, z, xbc, act, ffb, y, y_acc, hist, last, logits, tokens, status, attn_ws, dec_scratch, dev_batch;
  Buf raw_acc;                          // sums of input projections over slices of k
  Buf cq, gate, qlat, olat, lat, kbuf, vt, kv_start;                                                      // latent attention
  Buf segments;                         // scalar-decay recurrences of long prompts
  Buf qx, maps_out;                     // differential attention: queries of both maps, outputs of both (fp32)
  Buf route, route_acc, pair_w, pair_row, pair_expert, identity, offsets, row_token, counts, tiles, gathered, expert_rows;  // mixture
  StepBatch batch;
  std::vector<uint8_t> slot_phase;      // per state slot: the copy that holds its convolution and shift states
  cudaStream_t stream = nullptr;
  std::mutex mu;
  int n_out = 0, launches = 0;
  // `y_acc`, `raw_acc`, `route_acc` and `counts` are all zero between their uses (the kernel that reads them zeroes them); a
  // step that failed part-way may have left sums there, so the next one clears them
  bool acc_dirty = true, ready = false;
  size_t acc_bytes = 0, raw_acc_bytes = 0, route_acc_bytes = 0, counts_bytes = 0, segment_bytes = 0;
  template <typename T> T* dev(T* host) const { return (T*)((uint8_t*)dev_batch.p + ((uint8_t*)host - batch.pinned)); }
  bool accumulates(int rows) const { return !cfg.is_f32 && rows <= kAccRows && !logismos_get_deterministic(); }
};

// largest sizes over the layers, per token unless said otherwise (elements)
struct Sizes {
  size_t proj = 0, tail = 0, act = 0, ff = 0, z = 0, low = 0, xbc = 0, attn_ws = 0, scratch = 0;   // the last two in bytes
  size_t raw = 0;                                                                                    // of summed input projections
  size_t cq = 0, heads = 0, lat_q = 0, lat = 0, lat_heads = 0;                             // latent attention
  size_t route = 0, pairs = 0, top = 0, groups = 0, expert_ff = 0;                                  // mixture
  size_t segments = 0;                                                                               // bytes
  size_t maps = 0;                                                                                   // differential attention
};
inline void grow(size_t& a, size_t b) { if (b > a) a = b; }

// tensors of an archive by name, counted
struct Wanted {
  const Archive* r;
  uint32_t rc = 0;
  size_t count = 0;
  bool has(const std::string& name) const { return r->index.count(name) != 0; }
  bool get(const std::string& name, std::initializer_list<int64_t> shape, const void** out) {
    ++count;
    return (rc = want_tensor(r, name, LG_DT_BF16, shape, out)) == 0;
  }
  // the rows of a matrix, where the file's tensor sets a size
  bool rows(const std::string& name, int32_t* out) {
    lg_tensor_view_t v;
    if ((rc = get_view(r, name.c_str(), &v))) return false;
    if (v.rank != 2 || v.shape[0] <= 0 || v.shape[0] > 1 << 20) { rc = fail(LG_EMB_COMPUTE, name + ": expected a matrix"); return false; }
    *out = (int32_t)v.shape[0];
    return true;
  }
};

// ---- products (mixer_model.cu) ----------------------------------------------------------------------
uint32_t linear(Mixer* m, const void* a, int lda, const Buf& w, int n, int k, void* out, int ldc, int epi, int rows, cudaStream_t s, const Buf* bias = nullptr);
// one small matrix per head: out[r, h, :n] = W_h a[r, h, :k]
uint32_t head_linear(Mixer* m, const void* a, int lda, const Buf& w, int heads, int n, int k, void* out, int ldc, int rows, cudaStream_t s);
// input projections of a layer: main columns to proj, fp32 tail to `tail` (and rounded with remainders to low2)
uint32_t projections(Mixer* m, const MLayer& L, const MWeights& W, bool tail_parts, cudaStream_t s);
// one grouped projection of the step's rows of h (n columns in all) to m->proj
uint32_t grouped_projection(Mixer* m, const Buf& w, int n, const lg_linear_groups_t& g, cudaStream_t s);
// a scalar-decay recurrence over the step's prompt sequences (args: theirs), cut in segments where that pays
uint32_t prompt_recurrence(Mixer* m, lg_ssd_t* args, cudaStream_t s);
void size_prompt_recurrence(const Mixer* m, int heads, int np, int vp, Sizes& z);
// whether a grouped projection is summed over slices of k at this number of rows
bool splits_projections(const lg_linear_groups_t& g, int n, int rows);
bool zeroed(Buf& b, size_t bytes);

// rows of head h of src [heads * d, k] -> rows of dst at row0 + h * dp
void head_rows(Mat& dst, int row0, const void* src, int heads, int d, int dp, int k);
// columns of head h of src [n, heads * d] -> columns of dst at col0 + h * dp
void head_cols(Mat& dst, int col0, const void* src, int n, int heads, int d, int dp);

// ---- kinds of mixers: what a layer needs (NULL or 0: fine), its layout, weights, buffers and step ----
inline bool is_gated_kind(int kind) { return kind >= LG_MIXER_ATTENTION && kind <= LG_MIXER_LATENT; }
inline bool is_paired_kind(int kind) { return kind >= LG_MIXER_DIFF; }

const char* check_parallel_kinds(const lg_mixer_layer_config_t& y);
const char* check_parallel_tensors(const lg_mixer_layer_config_t& y);   // sizes that a file's tensors give
void layout_parallel_kinds(MLayer& L);
bool upload_parallel_kinds(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w, Mat& in, Mat& out);
bool alloc_parallel_kinds(Mixer* m, MLayer& L, Sizes& z);
bool want_parallel_kinds(Wanted& t, const std::string& mix, int64_t width, lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L);
uint32_t run_ssd(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s);
uint32_t run_parallel(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s);

const char* check_gated_kinds(const lg_mixer_layer_config_t& y);
void layout_gated_kinds(MLayer& L);
bool upload_gated_kinds(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w, Mat& out);
bool alloc_gated_kinds(Mixer* m, MLayer& L, Sizes& z);
bool want_gated_kinds(Wanted& t, const std::string& mix, int64_t width, lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L);
uint32_t run_gated_kinds(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s);

// attention over a window from queries and the layer's cache: `heads` query heads of hd channels, kv key heads (bf16: prompt rows
// alone, where decode rows have a launch of their own)
uint32_t window_attention(Mixer* m, MLayer& L, lg_window_t w, const void* q, int ld_q, int heads, int kv, int hd, void* out, int ld_out, cudaStream_t s,
                          bool prompts_only = false);
// keys that a launch over a run of prompt sequences gathers: of all, and of the longest
void gathered_keys(const StepBatch& B, const lg_window_t& w, const PrefixRun& r, int* total, int* longest);

const char* check_paired_kinds(const lg_mixer_layer_config_t& y);
void layout_paired_kinds(const Mixer* m, MLayer& L);
bool upload_paired_kinds(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w);   // the output projections too
bool alloc_paired_kinds(Mixer* m, MLayer& L, Sizes& z);
bool want_paired_kinds(Wanted& t, const std::string& mix, int64_t width, lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L);
uint32_t run_paired_kinds(Mixer* m, MLayer& L, const MWeights& W, cudaStream_t s);

// ---- feed-forwards -----------------------------------------------------------------------------------
const char* check_feed_forward(const lg_mixer_layer_config_t& y);
bool upload_feed_forward(Mixer* m, const MLayer& L, MWeights& W, const lg_mixer_layer_weights_t& w);
void size_feed_forward(const MLayer& L, Sizes& z);
bool want_feed_forward(Wanted& t, const std::string& mlp, int64_t width, const lg_mixer_layer_config_t& y, lg_mixer_layer_weights_t& L, std::vector<const void*>& experts);
// up to the rows of the experts; their sum (the description `out`) is left to the norm that follows
uint32_t run_mixture(Mixer* m, const MLayer& L, const MWeights& W, lg_mixture_out_t* out, cudaStream_t s);

}  // namespace lgm
