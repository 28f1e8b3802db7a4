// One packed continuous-batching step on the host, shared by the decoder executors: validation, the
// internal order (decode sequences first, then prefill chunks), the index arrays in pinned memory, the
// split of the decode contexts into chunks and the runs of prefill sequences whose keys fit a gather
// workspace together. The reference has no scheduler (crates/sched/src/lib.rs:1-30).
#pragma once
#include <cuda_runtime.h>

#include <cstdint>
#include <cstring>
#include <string>
#include <vector>

#include "logismos_kernels.h"
#include "logismos_model.h"
#include "model_util.h"

namespace lgm {

constexpr int kKvBlock = 16;  // tokens per paged-cache block

// a run of prefill sequences [s0, s1) that one gather + attention launch pair serves
struct PrefixRun { int s0, s1, total_kv, max_q, max_kv; };

struct StepLimits {
  int64_t max_pos = 0;         // tokens per sequence
  int max_blocks_per_seq = 0, n_pool_blocks = 0, max_step_tokens = 0, max_step_seqs = 0;
  int n_state_slots = 0;       // 0: the executor keeps no per-sequence state
  size_t prefix_cap_tokens = 0;  // keys one gather may hold
  size_t extra_bytes = 0;      // room at the end of the block for arrays of the executor's own
};

struct StepBatch {
  StepLimits lim;
  uint8_t* pinned = nullptr;
  size_t capacity = 0;          // bytes of `pinned`
  // packed order: decode rows first, prefill rows after them (host views into `pinned`)
  uint32_t* ids = nullptr;      // [T]
  int32_t* pos = nullptr;       // [T]
  int64_t* slots = nullptr;     // [T] cache slot of every token
  int32_t* seq_ids = nullptr;   // [T] packed sequence index
  int32_t* cu = nullptr;        // [n_seqs + 1]
  int32_t* cu_pre = nullptr;    // [runs' sequences + 1], relative to the first prefill row
  int32_t* last = nullptr;      // [n_seqs] last row of every sequence
  int32_t* chunks = nullptr;    // [n_dec + 1] decode chunk offsets (build_decode_chunks)
  int32_t* tables = nullptr;    // [n_seqs, max_blocks_per_seq]
  int32_t* ctx = nullptr;       // [n_dec] decode context lengths, the new token included
  int32_t* pre_kv = nullptr;    // [prefill sequences] keys of each
  int32_t* state = nullptr;     // [n_seqs] state slots
  uint8_t* fresh = nullptr;     // [n_seqs] 1: the sequence starts here
  uint8_t* phase = nullptr;     // [n_seqs] filled by executors whose states alternate between two copies
  uint8_t* extra = nullptr;     // [extra_bytes], 8-byte aligned
  int T = 0, n_dec = 0, n_pre = 0, n_seqs = 0, max_pre_len = 0, run_count = 0;
  bool has_prefix = false;      // some prefill chunk continues a cached sequence
  std::vector<int> order;       // packed sequence -> caller's sequence
  std::vector<int32_t> cached, newl;  // packed order
  std::vector<PrefixRun> runs;

  bool alloc(const StepLimits& l) {
    lim = l;
    const size_t T_ = (size_t)l.max_step_tokens, S = (size_t)l.max_step_seqs, MB = (size_t)l.max_blocks_per_seq;
    capacity = T_ * 20 + (S + 1) * 4 * 4 + S * MB * 4 + S * 4 * 3 + S * 2 + l.extra_bytes + 64;
    return cudaMallocHost((void**)&pinned, capacity) == cudaSuccess;
  }
  void release() {
    if (pinned) cudaFreeHost(pinned);
    pinned = nullptr;
  }

  // Packs one step; 0 or an lg_embedding_status code with the reason in lg_last_error(). `gather_all`: every
  // sequence, decode tokens included, attends through the gather (runs then cover all sequences).
  uint32_t build(const char* who, const uint32_t* host_ids, const int32_t* host_cached, const int32_t* host_new, int32_t n,
                 const int32_t* host_tables, const int32_t* host_slots, bool gather_all) {
    const int MB = lim.max_blocks_per_seq;
    auto fail = [&](uint32_t code, const char* what) { set_error(std::string(who) + ": " + what); return code; };
    if (n <= 0 || n > lim.max_step_seqs || !host_ids || !host_cached || !host_new || !host_tables || (lim.n_state_slots > 0 && !host_slots))
      return fail(LG_EMB_COMPUTE, "bad arguments or too many sequences for the workspace");
    std::vector<int64_t> src_off((size_t)n);
    std::vector<uint8_t> slot_used((size_t)(lim.n_state_slots > 0 ? lim.n_state_slots : 0), 0);
    int64_t total = 0;
    for (int i = 0; i < n; ++i) {
      if (host_new[i] <= 0 || host_cached[i] < 0) return fail(LG_EMB_COMPUTE, "every sequence needs >= 1 new token");
      const int64_t end = (int64_t)host_cached[i] + host_new[i];
      if (end > lim.max_pos || end > (int64_t)MB * kKvBlock) return fail(LG_EMB_INPUT_TOO_LONG, "sequence exceeds max_pos or its block table");
      if (lim.n_state_slots > 0) {
        const int sl = host_slots[i];
        if (sl < 0 || sl >= lim.n_state_slots || slot_used[(size_t)sl]) return fail(LG_EMB_COMPUTE, "state slot out of range or used twice in one step");
        slot_used[(size_t)sl] = 1;
      }
      src_off[(size_t)i] = total;
      total += host_new[i];
    }
    if (total > lim.max_step_tokens) return fail(LG_EMB_COMPUTE, "step exceeds max_step_tokens");
    order.clear();
    for (int i = 0; i < n; ++i) if (host_new[i] == 1) order.push_back(i);
    n_dec = (int)order.size();
    for (int i = 0; i < n; ++i) if (host_new[i] > 1) order.push_back(i);
    n_pre = n - n_dec;
    n_seqs = n;
    T = (int)total;
    uint8_t* pp = pinned;  // 8-byte slots first
    auto carve = [&](size_t b) { uint8_t* p = pp; pp += b; return p; };
    slots = (int64_t*)carve((size_t)total * 8);
    ids = (uint32_t*)carve((size_t)total * 4);
    pos = (int32_t*)carve((size_t)total * 4);
    seq_ids = (int32_t*)carve((size_t)total * 4);
    cu = (int32_t*)carve((size_t)(n + 1) * 4);
    cu_pre = (int32_t*)carve((size_t)(n + 1) * 4);
    last = (int32_t*)carve((size_t)(n + 1) * 4);
    chunks = (int32_t*)carve((size_t)(n + 1) * 4);
    tables = (int32_t*)carve((size_t)n * MB * 4);
    ctx = (int32_t*)carve((size_t)n * 4);
    pre_kv = (int32_t*)carve((size_t)n * 4);
    state = (int32_t*)carve((size_t)n * 4);
    fresh = carve((size_t)n);
    phase = carve((size_t)n);
    extra = carve(0) + ((8 - ((uintptr_t)pp & 7)) & 7);
    std::memset(phase, 0, (size_t)n);
    cached.assign((size_t)n, 0);
    newl.assign((size_t)n, 0);
    int64_t t = 0;
    for (int s = 0; s < n; ++s) {
      const int i = order[(size_t)s];
      cached[(size_t)s] = host_cached[i];
      newl[(size_t)s] = host_new[i];
      state[s] = host_slots && lim.n_state_slots > 0 ? host_slots[i] : 0;
      fresh[s] = host_cached[i] == 0 ? 1 : 0;
      std::memcpy(tables + (size_t)s * MB, host_tables + (size_t)i * MB, (size_t)MB * 4);
      std::memcpy(ids + t, host_ids + src_off[(size_t)i], (size_t)host_new[i] * 4);
      t += host_new[i];
    }
    const int64_t built = logismos_build_packing(cached.data(), newl.data(), n, tables, MB, kKvBlock, lim.n_pool_blocks, cu, pos, slots, seq_ids);
    if (built != total) return fail(LG_EMB_COMPUTE, "a block table entry is missing or outside the pool");
    max_pre_len = 0;
    has_prefix = false;
    cu_pre[0] = 0;
    for (int s = 0; s < n; ++s) {
      last[s] = cu[s + 1] - 1;
      if (s < n_dec) { ctx[s] = cached[(size_t)s] + 1; continue; }
      cu_pre[s - n_dec + 1] = cu[s + 1] - n_dec;
      pre_kv[s - n_dec] = cached[(size_t)s] + newl[(size_t)s];
      if (cached[(size_t)s] > 0) has_prefix = true;
      if (newl[(size_t)s] > max_pre_len) max_pre_len = newl[(size_t)s];
    }
    if (gather_all) {  // all sequences, packed order: key counts and query offsets of the whole step
      has_prefix = true;
      for (int k = 0; k < n; ++k) pre_kv[k] = cached[(size_t)k] + newl[(size_t)k];
      std::memcpy(cu_pre, cu, (size_t)(n + 1) * 4);
    }
    const int first = gather_all ? 0 : n_dec;
    run_count = gather_all ? n : n_pre;
    runs.clear();
    if (run_count > 0) {
      PrefixRun r{0, 0, 0, 0, 0};
      for (int k = 0; k < run_count; ++k) {
        const int kv = pre_kv[k], q = newl[(size_t)(first + k)];
        if (r.s1 > r.s0 && (size_t)r.total_kv + (size_t)kv > lim.prefix_cap_tokens) { runs.push_back(r); r = PrefixRun{k, k, 0, 0, 0}; }
        r.s1 = k + 1;
        r.total_kv += kv;
        if (q > r.max_q) r.max_q = q;
        if (kv > r.max_kv) r.max_kv = kv;
      }
      runs.push_back(r);
    }
    return LG_EMB_OK;
  }

  // rows[i] = packed row of the caller's token i, for all T tokens of the step
  void caller_rows(int32_t* rows) const {
    std::vector<int> at((size_t)n_seqs);  // caller's sequence -> packed sequence
    for (int s = 0; s < n_seqs; ++s) at[(size_t)order[(size_t)s]] = s;
    int32_t t = 0;
    for (int i = 0; i < n_seqs; ++i) {
      const int s = at[(size_t)i];
      for (int r = cu[s]; r < cu[s + 1]; ++r) rows[t++] = r;
    }
  }

  // packed rows of the wanted tokens: out_rows [n_out] index the caller's tokens; NULL: the last token of every
  // sequence. False: an index lies outside the step.
  bool select_rows(const int32_t* out_rows, int32_t n_out, const int32_t* host_new, int32_t* rows) const {
    std::vector<int32_t> packed_row((size_t)T);
    caller_rows(packed_row.data());
    int64_t off = 0;
    for (int i = 0; i < n_out; ++i) {
      int64_t t;
      if (out_rows) t = out_rows[i];
      else { off += host_new[i]; t = off - 1; }
      if (t < 0 || t >= T) return false;
      rows[i] = packed_row[(size_t)t];
    }
    return true;
  }

  // fp32 rows of the step on the device (row stride ld), in the caller's order, to host_out [T, width]
  cudaError_t rows_to_host(const float* dev_rows, int ld, int width, float* host_out) const {
    std::vector<float> tmp((size_t)T * ld);
    std::vector<int32_t> packed_row((size_t)T);
    caller_rows(packed_row.data());
    const cudaError_t e = cudaMemcpy(tmp.data(), dev_rows, tmp.size() * 4, cudaMemcpyDeviceToHost);
    if (e != cudaSuccess) return e;
    for (int t = 0; t < T; ++t) std::memcpy(host_out + (size_t)t * width, tmp.data() + (size_t)packed_row[(size_t)t] * ld, (size_t)width * 4);
    return cudaSuccess;
  }
};

}  // namespace lgm
