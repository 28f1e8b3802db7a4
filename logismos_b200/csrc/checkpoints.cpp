// Checkpoint loaders of the executors over the safetensors reader. Counterparts in the reference:
//   StellaWeights::load, load_layer     crates/encoders/src/stella.rs:123-166, :320-400 (exact tensor
//                                       count, per-name F32 + shape checks)
//   StellaModel::load, load_dense_head  crates/embed/src/stella.rs:138-201, :380-443
#include <cuda_runtime.h>

#include <algorithm>
#include <cstdint>
#include <string>
#include <vector>

#include "logismos_kernels.h"
#include "logismos_model.h"
#include "safetensors.h"

using namespace lgm;

extern "C" {

uint32_t lg_stella_load(int32_t device, const char* root, const lg_stella_config_t* cfg, void** model) {
  if (!root || !cfg || !model) return fail(LG_EMB_COMPUTE, "null argument");
  *model = nullptr;
  const lg_stella_config_t& c = *cfg;
  if (c.n_heads <= 0 || c.n_layers < 0 || c.n_dims <= 0 || c.n_dims > 8) return fail(LG_EMB_COMPUTE, "lg_stella_load: bad config");
  const std::string dir(root);
  Archive* r = nullptr;
  if (uint32_t rc = open_archive((dir + "/model.safetensors").c_str(), &r)) return rc;
  struct Guard { std::vector<Archive*> rs; ~Guard() { for (Archive* x : rs) delete x; } } guard;
  guard.rs.push_back(r);
  // the archive must hold exactly the tensors this model reads (crates/encoders/src/stella.rs:126-145)
  const size_t expected = 2 + (size_t)c.n_layers * 12;
  if (r->ordering.size() != expected)
    return fail(LG_EMB_COMPUTE, "expected " + std::to_string(expected) + " tensors in stella archive, got " + std::to_string(r->ordering.size()));
  const int64_t H = c.hidden, I = c.intermediate, KV = (int64_t)c.n_kv_heads * (c.hidden / c.n_heads);
  lg_stella_weights_t w{};
  std::vector<lg_stella_layer_weights_t> layers((size_t)c.n_layers);
  if (uint32_t rc = want_f32(r, "model.embed_tokens.weight", {c.vocab, H}, &w.tok_embed)) return rc;
  if (uint32_t rc = want_f32(r, "model.norm.weight", {H}, &w.final_norm)) return rc;
  for (int i = 0; i < c.n_layers; ++i) {
    const std::string p = "model.layers." + std::to_string(i) + ".";
    lg_stella_layer_weights_t& L = layers[(size_t)i];
    uint32_t rc = 0;
    (rc = want_f32(r, p + "input_layernorm.weight", {H}, &L.norm1)) || (rc = want_f32(r, p + "post_attention_layernorm.weight", {H}, &L.norm2)) ||
        (rc = want_f32(r, p + "self_attn.q_proj.weight", {H, H}, &L.wq)) || (rc = want_f32(r, p + "self_attn.q_proj.bias", {H}, &L.bq)) ||
        (rc = want_f32(r, p + "self_attn.k_proj.weight", {KV, H}, &L.wk)) || (rc = want_f32(r, p + "self_attn.k_proj.bias", {KV}, &L.bk)) ||
        (rc = want_f32(r, p + "self_attn.v_proj.weight", {KV, H}, &L.wv)) || (rc = want_f32(r, p + "self_attn.v_proj.bias", {KV}, &L.bv)) ||
        (rc = want_f32(r, p + "self_attn.o_proj.weight", {H, H}, &L.wo)) || (rc = want_f32(r, p + "mlp.gate_proj.weight", {I, H}, &L.w_gate)) ||
        (rc = want_f32(r, p + "mlp.up_proj.weight", {I, H}, &L.w_up)) || (rc = want_f32(r, p + "mlp.down_proj.weight", {H, I}, &L.w_down));
    if (rc) return rc;
  }
  w.layers = layers.data();
  // supported dims sorted, the default is 1024 when that head is loaded, else the smallest
  // (crates/embed/src/stella.rs:143-163); the model takes its default from dims[0]
  lg_stella_config_t cc = c;
  std::sort(cc.dims, cc.dims + cc.n_dims);
  for (int d = 0; d < cc.n_dims; ++d)
    if (cc.dims[d] == 1024) std::rotate(cc.dims, cc.dims + d, cc.dims + d + 1);
  // dense heads: <root>/2_Dense_<dim>/model.safetensors with linear.weight [dim, hidden], linear.bias [dim]
  // (crates/embed/src/stella.rs:380-443)
  for (int d = 0; d < cc.n_dims; ++d) {
    Archive* hr = nullptr;
    const std::string folder = "2_Dense_" + std::to_string(cc.dims[d]);
    if (uint32_t rc = open_archive((dir + "/" + folder + "/model.safetensors").c_str(), &hr)) return rc;
    guard.rs.push_back(hr);
    lg_tensor_view_t wv, bv;
    if (uint32_t rc = get_view(hr, "linear.weight", &wv)) return rc;
    if (uint32_t rc = get_view(hr, "linear.bias", &bv)) return rc;
    if (wv.dtype != LG_DT_F32 || bv.dtype != LG_DT_F32) return fail(LG_EMB_IO, "dense head " + folder + ": expected F32");
    if (wv.rank != 2 || wv.shape[0] != cc.dims[d] || wv.shape[1] != H)
      return fail(LG_EMB_IO, "dense head " + folder + ": expected weight shape [" + std::to_string(cc.dims[d]) + ", " + std::to_string(H) + "]");
    if (bv.rank != 1 || bv.shape[0] != cc.dims[d]) return fail(LG_EMB_IO, "dense head " + folder + ": expected bias shape [" + std::to_string(cc.dims[d]) + "]");
    w.head_w[d] = (const float*)wv.data;
    w.head_b[d] = (const float*)bv.data;
  }
  return lg_stella_create(device, &cc, &w, model);
}

// The int4 decoder from a Qwen2-style checkpoint (fp32 tensors under the names of
// crates/encoders/src/stella.rs:326-349 plus lm_head.weight [vocab, hidden]; when that tensor is absent
// the head is tied to the embedding): every matrix is quantised to int4 group-32 ON THE DEVICE
// (logismos_launch_quantize_int4_g32) and handed to lg_decoder_create. No reference counterpart beyond
// the tensor accounting: the reference has no quantiser and no decoder.
uint32_t lg_decoder_load(int32_t device, const char* path, const lg_decoder_config_t* cfg, void** model) {
  if (!path || !cfg || !model) return fail(LG_EMB_COMPUTE, "null argument");
  *model = nullptr;
  const lg_decoder_config_t& c = *cfg;
  if (c.n_heads <= 0 || c.n_layers < 0 || c.hidden % 32 || c.intermediate % 32) return fail(LG_EMB_COMPUTE, "lg_decoder_load: bad config");
  Archive* r = nullptr;
  if (uint32_t rc = open_archive(path, &r)) return rc;
  struct Guard { Archive* r; ~Guard() { delete r; } } guard{r};
  const bool tied = r->index.find("lm_head.weight") == r->index.end();
  const size_t expected = 2 + (tied ? 0 : 1) + (size_t)c.n_layers * 12;
  if (r->ordering.size() != expected)
    return fail(LG_EMB_COMPUTE, "expected " + std::to_string(expected) + " tensors in decoder archive, got " + std::to_string(r->ordering.size()));
  if (cudaSetDevice(device) != cudaSuccess) return fail(LG_EMB_COMPUTE, "cudaSetDevice failed");
  const int64_t H = c.hidden, I = c.intermediate, KV = (int64_t)c.n_kv_heads * (c.hidden / c.n_heads);
  struct QHost { std::vector<uint8_t> codes; std::vector<uint16_t> scales; };
  std::vector<QHost> store;
  store.reserve((size_t)c.n_layers * 7 + 1);
  size_t scratch_elems = (size_t)c.vocab * H;
  if ((size_t)I * H > scratch_elems) scratch_elems = (size_t)I * H;
  float* d_w = nullptr;
  uint8_t* d_codes = nullptr;
  uint16_t* d_scales = nullptr;
  struct DevGuard { float** a; uint8_t** b; uint16_t** c; ~DevGuard() { if (*a) cudaFree(*a); if (*b) cudaFree(*b); if (*c) cudaFree(*c); } } dg{&d_w, &d_codes, &d_scales};
  if (cudaMalloc(&d_w, scratch_elems * 4) != cudaSuccess || cudaMalloc(&d_codes, scratch_elems / 2) != cudaSuccess ||
      cudaMalloc(&d_scales, scratch_elems / 32 * 2) != cudaSuccess)
    return fail(LG_EMB_COMPUTE, "lg_decoder_load: device scratch allocation failed");
  auto quant = [&](const std::string& name, int64_t n, int64_t k, lg_int4_matrix_t* out) -> uint32_t {
    const float* src = nullptr;
    if (uint32_t rc = want_f32(r, name, {n, k}, &src)) return rc;
    store.emplace_back();
    QHost& q = store.back();
    q.codes.resize((size_t)n * k / 2);
    q.scales.resize((size_t)n * k / 32);
    if (cudaMemcpy(d_w, src, (size_t)n * k * 4, cudaMemcpyHostToDevice) != cudaSuccess ||
        logismos_launch_quantize_int4_g32(d_w, d_codes, d_scales, (int32_t)n, (int32_t)k, nullptr) != 0 ||
        cudaMemcpy(q.codes.data(), d_codes, q.codes.size(), cudaMemcpyDeviceToHost) != cudaSuccess ||
        cudaMemcpy(q.scales.data(), d_scales, q.scales.size() * 2, cudaMemcpyDeviceToHost) != cudaSuccess)
      return fail(LG_EMB_COMPUTE, name + ": quantisation on the device failed");
    out->codes = q.codes.data();
    out->scales = q.scales.data();
    return LG_EMB_OK;
  };
  lg_decoder_weights_t w{};
  std::vector<lg_decoder_layer_weights_t> layers((size_t)c.n_layers);
  if (uint32_t rc = want_f32(r, "model.embed_tokens.weight", {c.vocab, H}, &w.tok_embed)) return rc;
  if (uint32_t rc = want_f32(r, "model.norm.weight", {H}, &w.final_norm)) return rc;
  if (uint32_t rc = quant(tied ? "model.embed_tokens.weight" : "lm_head.weight", c.vocab, H, &w.lm_head)) return rc;
  for (int i = 0; i < c.n_layers; ++i) {
    const std::string p = "model.layers." + std::to_string(i) + ".";
    lg_decoder_layer_weights_t& L = layers[(size_t)i];
    uint32_t rc = 0;
    (rc = want_f32(r, p + "input_layernorm.weight", {H}, &L.norm1)) || (rc = want_f32(r, p + "post_attention_layernorm.weight", {H}, &L.norm2)) ||
        (rc = want_f32(r, p + "self_attn.q_proj.bias", {H}, &L.bq)) || (rc = want_f32(r, p + "self_attn.k_proj.bias", {KV}, &L.bk)) ||
        (rc = want_f32(r, p + "self_attn.v_proj.bias", {KV}, &L.bv)) || (rc = quant(p + "self_attn.q_proj.weight", H, H, &L.wq)) ||
        (rc = quant(p + "self_attn.k_proj.weight", KV, H, &L.wk)) || (rc = quant(p + "self_attn.v_proj.weight", KV, H, &L.wv)) ||
        (rc = quant(p + "self_attn.o_proj.weight", H, H, &L.wo)) || (rc = quant(p + "mlp.gate_proj.weight", I, H, &L.w_gate)) ||
        (rc = quant(p + "mlp.up_proj.weight", I, H, &L.w_up)) || (rc = quant(p + "mlp.down_proj.weight", H, I, &L.w_down));
    if (rc) return rc;
  }
  w.layers = layers.data();
  return lg_decoder_create(device, cfg, &w, model);
}

}  // extern "C"
