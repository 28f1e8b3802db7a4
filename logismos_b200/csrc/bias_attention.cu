// What the extended forms of attention (score_bias.cuh) need around the shared attention kernels: unit queries and keys
// with the cache store, and the fp32 attention, capped and biased by distance or over a window.
#include "common.cuh"
#include "logismos_kernels.h"
#include "recurrent.cuh"
#include "score_bias.cuh"

namespace {

using namespace lg;

constexpr int kBlockTokens = 16, kThreads = 256;

template <typename T, int HD> struct UnitGeometry {
  static constexpr int E = HD * sizeof(T) / 16 > 32 ? HD / 32 : 16 / (int)sizeof(T), LANES = HD / E;
};

struct QkArgs {
  void* qkv;
  int ld;
  void* kpool;
  void* vpool;
  const int64_t* slots;
  const int* pos;
  int rows, heads, n_kv, dim;
  float eps, coef, every;
  int64_t n_slots;
  int* status;
};

// A head of a row, q (in place), k or v (to the cache), is held by LANES lanes, sixteen bytes each (fp32 heads of 256:
// thirty-two); a group of lanes takes ITEMS heads, all requested at once.
template <typename T, int HD, int ITEMS>
__global__ void __launch_bounds__(kThreads)
unit_qk_store_kernel(QkArgs p) {
  lg::pdl_prologue();
  using G = UnitGeometry<T, HD>;
  constexpr int E = G::E, LANES = G::LANES;
  struct alignas(E * sizeof(T)) Vec { T v[E]; };
  const uint32_t per_row = p.heads + 2 * p.n_kv, lane = threadIdx.x % LANES;
  const uint32_t total = p.rows * per_row, first = (blockIdx.x * kThreads + threadIdx.x) / LANES * ITEMS;
  const int row0 = (int)(first / per_row), head0 = (int)(first % per_row);
  Vec x[ITEMS];
#pragma unroll
  for (int k = 0; k < ITEMS; ++k) {
    if (first + k >= total) continue;
    const bool wrap = head0 + k >= (int)per_row;  // ITEMS <= per_row or ITEMS == 1: at most one row further
    const int row = row0 + wrap, h = head0 + k - (wrap ? (int)per_row : 0);
    x[k] = *reinterpret_cast<const Vec*>(reinterpret_cast<const T*>(p.qkv) + (size_t)row * p.ld + h * HD + lane * E);
  }
#pragma unroll
  for (int k = 0; k < ITEMS; ++k) {
    const bool in = first + k < total;
    const bool wrap = head0 + k >= (int)per_row;
    const int row = in ? row0 + wrap : 0, h = in ? head0 + k - (wrap ? (int)per_row : 0) : 0;
    const bool is_v = h >= p.heads + p.n_kv;
    float f[E], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < E; ++i) { f[i] = in ? rec::Io<T>::load(&x[k].v[i]) : 0.0f; ss += f[i] * f[i]; }
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!in) continue;
    if (!is_v) {
      float m = 1.0f / sqrtf(ss / (float)p.dim + p.eps);
      if (h < p.heads && p.coef != 0.0f) m *= 1.0f + p.coef * logf(floorf(__fdiv_rn((float)(p.pos[row] + 1), p.every)) + 1.0f);
#pragma unroll
      for (int i = 0; i < E; ++i) rec::Io<T>::store(&x[k].v[i], f[i] * m);
    }
    if (h < p.heads) {
      *reinterpret_cast<Vec*>(reinterpret_cast<T*>(p.qkv) + (size_t)row * p.ld + h * HD + lane * E) = x[k];
      continue;
    }
    const int64_t slot = p.slots[row];
    if (slot < 0 || slot >= p.n_slots) {
      if (lane == 0 && p.status) atomicExch(p.status, 1);
      continue;
    }
    const int kvh = h - p.heads - (is_v ? p.n_kv : 0);
    T* pool = reinterpret_cast<T*>(is_v ? p.vpool : p.kpool);
    *reinterpret_cast<Vec*>(pool + (size_t)slot * p.n_kv * HD + kvh * HD + lane * E) = x[k];
  }
}

// CTA = (row, head), keys in tiles of 64
constexpr int kTile = 64, kAttnThreads = 128;
template <bool WINDOW>
__global__ void __launch_bounds__(kAttnThreads)
attention_f32_kernel(const float* __restrict__ q, const float* __restrict__ kpool, const float* __restrict__ vpool, const int* __restrict__ tables,
                     int max_blocks, int n_pool_blocks, const int* __restrict__ seq_ids, const int* __restrict__ pos, float* __restrict__ out,
                     int n_kv, int hd, float scale, float cap, const float* __restrict__ gate, ScoreExt ext, WindowExt win, int* __restrict__ status) {
  lg::pdl_prologue();
  __shared__ float sq[256], ss[kTile], red[32];
  __shared__ int64_t row_s[kTile];  // cache row of every key of the tile, -1: not seen; pooled rows lie in pools of their own
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int kvh = h / (gridDim.y / n_kv), n_keys = pos[r] + 1;
  const int* table = tables + (size_t)seq_ids[r] * max_blocks;
  const float* bias = WINDOW ? nullptr : ext.bias + (size_t)h * (ext.far + 1);
  const size_t row_w = (size_t)n_kv * hd;
  for (int i = tid; i < hd; i += kAttnThreads) sq[i] = q[(size_t)r * (WINDOW ? win.ld_q : ext.ld_q) + h * hd + i];
  const bool sink = WINDOW && win.sink;  // a further score of 0
  float m = sink ? 0.0f : -1e30f, l = sink ? 1.0f : 0.0f, acc[2] = {0.f, 0.f};
  const int n_means = WINDOW ? win.pooled(n_keys - 1) : 0, mean_tiles = (n_means + kTile - 1) / kTile * kTile;
  for (int at = 0; at < mean_tiles + n_keys; at += kTile) {
    const bool means = WINDOW && at < mean_tiles;
    const int k0 = means ? at : at - mean_tiles, n = min(kTile, (means ? n_means : n_keys) - k0);
    if (WINDOW && !means && k0 >= win.keep && k0 + kTile - 1 < win.first(n_keys - 1)) continue;  // a tile that is not seen
    __syncthreads();
    if (tid < kTile) {
      const int k = k0 + tid, bi = means ? win.mean_block(k) : k / kBlockTokens;
      int64_t row = -1;
      if (tid < n && (!WINDOW || means || win.sees(n_keys - 1, k))) {
        const int b = bi < max_blocks ? __ldg(table + bi) : -1;
        if (b < 0 || b >= n_pool_blocks) {
          if (status) atomicExch(status, 1);
        } else {
          row = means ? (int64_t)b * win.mean_rows() + win.mean_row(k) : (int64_t)b * kBlockTokens + k % kBlockTokens;
        }
      }
      row_s[tid] = row;
    }
    __syncthreads();
    const float *keys = means ? (const float*)win.kmean : kpool, *values = means ? (const float*)win.vmean : vpool;
    for (int k = warp; k < kTile; k += kAttnThreads / 32) {
      const int64_t row = row_s[k];
      float s = 0.0f;
      if (row >= 0) {
        const float* c = keys + row * row_w + kvh * hd;
        for (int i = lane; i < hd; i += 32) s = fmaf(sq[i], c[i], s);
      }
      s = warp_sum(s) * scale;
      if (WINDOW) {
        if (lane == 0) ss[k] = row >= 0 ? s * 1.4426950408889634f : -INFINITY;
        continue;
      }
      if (cap > 0.0f) s = cap * tanhf(s / cap);
      if (lane == 0) ss[k] = row >= 0 ? s * 1.4426950408889634f + bias[min(n_keys - 1 - (k0 + k), ext.far)] : -1e30f;
    }
    __syncthreads();
    const float mine = tid < kTile ? ss[tid] : -1e30f;
    const float m_new = fmaxf(m, block_max(mine, red));
    const float alpha = exp2f(m - m_new), e = tid < n ? exp2f(mine - m_new) : 0.0f;
    l = l * alpha + block_sum(e, red);
    m = m_new;
    if (tid < kTile) ss[tid] = e;
    __syncthreads();
    acc[0] *= alpha;
    acc[1] *= alpha;
    for (int k = 0; k < n; ++k) {
      if (row_s[k] < 0) continue;
      const float* c = values + row_s[k] * row_w + kvh * hd;
      if (tid < hd) acc[0] = fmaf(ss[k], c[tid], acc[0]);
      if (tid + kAttnThreads < hd) acc[1] = fmaf(ss[k], c[tid + kAttnThreads], acc[1]);
    }
  }
  if constexpr (WINDOW) {
    const float g = win.gate ? rec::sigmoid_f(win.gate[(size_t)r * win.ld_gate + h]) : 1.0f;
    if (tid < hd) out[(size_t)r * win.ld_out + h * hd + tid] = acc[0] / l * g;
    if (tid + kAttnThreads < hd) out[(size_t)r * win.ld_out + h * hd + tid + kAttnThreads] = acc[1] / l * g;
  } else {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int d = tid + i * kAttnThreads;
      if (d < hd) out[(size_t)r * ext.ld_out + h * hd + d] = acc[i] / l * (ext.gate_scale * rec::sigmoid_f(gate[(size_t)r * ext.ld_gate + h * hd + d]));
    }
  }
}

}  // namespace

extern "C" {

uint32_t logismos_launch_unit_qk_store(void* qkv, int32_t ld, void* k_pool, void* v_pool, const void* slot_mapping_i64, const void* positions_i32,
                                       int32_t rows, int32_t n_heads, int32_t n_kv_heads, int32_t head_dim, int32_t dim, float eps, float coef,
                                       float every, int64_t n_pool_slots, int32_t is_f32, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!qkv || !k_pool || !v_pool || !slot_mapping_i64 || !positions_i32 || rows <= 0 || n_heads <= 0 || n_kv_heads <= 0 || dim <= 0 || dim > head_dim ||
      (head_dim != 64 && head_dim != 128 && head_dim != 256) || ld < (n_heads + 2 * n_kv_heads) * head_dim || (ld % 8) ||
      (((uintptr_t)qkv | (uintptr_t)k_pool | (uintptr_t)v_pool) & 15) || (coef != 0.0f && !(every > 0.0f)))
    return lg::kInvalidValue;
  const QkArgs p{qkv, ld, k_pool, v_pool, (const int64_t*)slot_mapping_i64, (const int*)positions_i32, rows, n_heads, n_kv_heads, dim, eps, coef, every,
                 n_pool_slots, (int*)status_i32};
  const int64_t items = (int64_t)rows * (n_heads + 2 * n_kv_heads);
  if (items > 0x3fffffff) return lg::kInvalidValue;
  auto go = [&](auto kern, int per_block) -> uint32_t {
    const int64_t blocks = (items + per_block - 1) / per_block;
    if (blocks > 0x7fffffff) return lg::kInvalidValue;
    lg::launch(kern, dim3((unsigned)blocks), dim3(kThreads), 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
#define LG_UNIT(T, HD)                                                                             \
  (items < 20000 || n_heads + 2 * n_kv_heads < 4 ? go(unit_qk_store_kernel<T, HD, 1>, kThreads / UnitGeometry<T, HD>::LANES)       \
                 : go(unit_qk_store_kernel<T, HD, 4>, kThreads / UnitGeometry<T, HD>::LANES * 4))
  if (is_f32) return head_dim == 64 ? LG_UNIT(float, 64) : head_dim == 128 ? LG_UNIT(float, 128) : LG_UNIT(float, 256);
  return head_dim == 64 ? LG_UNIT(__nv_bfloat16, 64) : head_dim == 128 ? LG_UNIT(__nv_bfloat16, 128) : LG_UNIT(__nv_bfloat16, 256);
#undef LG_UNIT
}

uint32_t logismos_launch_bias_attention_f32(const void* q, int32_t ld_q, const void* k_pool, const void* v_pool, const void* block_tables,
                                            const void* seq_ids_i32, const void* positions_i32, void* out, int32_t ld_out, int32_t rows,
                                            int32_t max_blocks, int32_t n_pool_blocks, int32_t n_heads, int32_t n_kv_heads, int32_t head_dim,
                                            const lg_score_bias_t* score, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!q || !k_pool || !v_pool || !block_tables || !seq_ids_i32 || !positions_i32 || !out || rows <= 0 || max_blocks <= 0 || n_pool_blocks <= 0 || n_heads <= 0 ||
      n_heads > 65535 || n_kv_heads <= 0 || n_heads % n_kv_heads || head_dim <= 0 || head_dim > 256 || ld_q < n_heads * head_dim || ld_out < n_heads * head_dim ||
      !score_ok(score, n_heads * head_dim))
    return lg::kInvalidValue;
  const ScoreExt ext = score_ext(score, ld_q, ld_out);
  lg::launch(attention_f32_kernel<false>, dim3((unsigned)rows, (unsigned)n_heads), dim3(kAttnThreads), 0, (cudaStream_t)stream, (const float*)q, (const float*)k_pool,
             (const float*)v_pool, (const int*)block_tables, max_blocks, n_pool_blocks, (const int*)seq_ids_i32, (const int*)positions_i32, (float*)out, n_kv_heads,
             head_dim, score->scale, score->cap, (const float*)score->gate, ext, WindowExt{}, (int*)status_i32);
  return lg::launch_status();
}

uint32_t logismos_launch_window_attention_f32(const void* q, int32_t ld_q, const void* k_pool, const void* v_pool, const void* block_tables,
                                              const void* seq_ids_i32, const void* positions_i32, void* out, int32_t ld_out, int32_t rows,
                                              int32_t max_blocks, int32_t n_pool_blocks, int32_t n_heads, int32_t n_kv_heads, int32_t head_dim,
                                              const lg_window_t* window, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!q || !k_pool || !v_pool || !block_tables || !seq_ids_i32 || !positions_i32 || !out || rows <= 0 || max_blocks <= 0 || n_pool_blocks <= 0 || n_heads <= 0 ||
      n_heads > 65535 || n_kv_heads <= 0 || n_heads % n_kv_heads || head_dim <= 0 || head_dim > 256 || ld_q < n_heads * head_dim || ld_out < n_heads * head_dim ||
      !window_ok(window, n_heads))
    return lg::kInvalidValue;
  lg::launch(attention_f32_kernel<true>, dim3((unsigned)rows, (unsigned)n_heads), dim3(kAttnThreads), 0, (cudaStream_t)stream, (const float*)q, (const float*)k_pool,
             (const float*)v_pool, (const int*)block_tables, max_blocks, n_pool_blocks, (const int*)seq_ids_i32, (const int*)positions_i32, (float*)out, n_kv_heads,
             head_dim, window->scale, 0.0f, (const float*)nullptr, ScoreExt{}, window_ext(window, ld_q, ld_out), (int*)status_i32);
  return lg::launch_status();
}

}  // extern "C"
