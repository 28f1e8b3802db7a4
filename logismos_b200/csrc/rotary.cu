// Rotary positions in the interleaved layout, fused with what surrounds them: norms of whole query and key projections, or of
// every head, and the cache store of a packed q | k | v row, or the rotated part of every query head in place. Angles come
// from a table of (cos, sin) per position and pair, amplitude included; norms and rotations are fp32. The means of blocks of
// cached keys and values are made where the last token of a block is stored, or by a launch after it.
#include "common.cuh"
#include "logismos_kernels.h"
#include "recurrent.cuh"

namespace {

using namespace lg;

constexpr int kThreads = 256;

template <typename T> struct alignas(8 * sizeof(T)) Vec8 { T v[8]; };

template <typename T> LG_DEVINL void unpack(const Vec8<T>& x, float (&f)[8]) {
#pragma unroll
  for (int i = 0; i < 8; ++i) f[i] = rec::Io<T>::load(&x.v[i]);
}
template <typename T> LG_DEVINL Vec8<T> pack(const float (&f)[8]) {
  Vec8<T> x;
#pragma unroll
  for (int i = 0; i < 8; ++i) rec::Io<T>::store(&x.v[i], f[i]);
  return x;
}

// channels d0 .. d0 + 7 of a vector whose first 2 * pairs channels turn
LG_DEVINL void rotate8(float (&f)[8], int d0, int pairs, const float2* __restrict__ row) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int pr = (d0 >> 1) + i;
    if (pr >= pairs) continue;
    const float2 cs = __ldg(row + pr);
    const float u = f[2 * i], v = f[2 * i + 1];
    f[2 * i] = u * cs.x - v * cs.y;
    f[2 * i + 1] = v * cs.x + u * cs.y;
  }
}

struct QkvArgs {
  void* qkv;
  int ld;
  void *kpool, *vpool;
  const int64_t* slots;
  const int* pos;
  int heads, n_kv, hd, dim;
  const float *gain_q, *gain_k;
  float eps;
  const float2* table;
  int pairs;
  int64_t n_slots;
  int* status;
};

// CTA = row; eight channels per thread and turn. The row is read twice, the second time from L1.
template <typename T>
__global__ void __launch_bounds__(kThreads)
qk_norm_rotary_store_kernel(QkvArgs p) {
  lg::pdl_prologue();
  __shared__ float part[2][kThreads / 32];
  const int r = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  Vec8<T>* row = reinterpret_cast<Vec8<T>*>(reinterpret_cast<T*>(p.qkv) + (size_t)r * p.ld);
  const int nq = p.heads * p.hd >> 3, nk = p.n_kv * p.hd >> 3, octs = p.hd >> 3;
  float sq = 0.0f, sk = 0.0f;
  for (int v = tid; v < nq + nk; v += kThreads) {
    float f[8], s = 0.0f;
    unpack<T>(row[v], f);
#pragma unroll
    for (int i = 0; i < 8; ++i) s = fmaf(f[i], f[i], s);
    if (v < nq) sq += s;
    else sk += s;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { part[0][warp] = sq; part[1][warp] = sk; }
  __syncthreads();
  sq = sk = 0.0f;
#pragma unroll
  for (int w = 0; w < kThreads / 32; ++w) { sq += part[0][w]; sk += part[1][w]; }
  const float iq = 1.0f / sqrtf(sq / (float)(p.heads * p.dim) + p.eps), ik = 1.0f / sqrtf(sk / (float)(p.n_kv * p.dim) + p.eps);
  const int64_t slot = p.slots[r];
  const bool ok = slot >= 0 && slot < p.n_slots;
  if (!ok && tid == 0 && p.status) atomicExch(p.status, 1);
  const float2* angles = p.table + (size_t)p.pos[r] * p.pairs;
  for (int v = tid; v < nq + 2 * nk; v += kThreads) {
    if (v >= nq + nk) {
      if (ok) reinterpret_cast<Vec8<T>*>(reinterpret_cast<T*>(p.vpool) + (size_t)slot * p.n_kv * p.hd)[v - nq - nk] = row[v];
      continue;
    }
    const bool is_q = v < nq;
    const int u = is_q ? v : v - nq;
    const float4* gain = reinterpret_cast<const float4*>(is_q ? p.gain_q : p.gain_k) + 2 * u;
    const float4 g0 = __ldg(gain), g1 = __ldg(gain + 1);
    const float g[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w}, m = is_q ? iq : ik;
    float f[8];
    unpack<T>(row[v], f);
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] *= m * g[i];
    rotate8(f, 8 * (u % octs), p.pairs, angles);
    const Vec8<T> o = pack<T>(f);
    if (is_q) row[v] = o;
    else if (ok) reinterpret_cast<Vec8<T>*>(reinterpret_cast<T*>(p.kpool) + (size_t)slot * p.n_kv * p.hd)[u] = o;
  }
}

// thread = eight channels of the rotated part of one head
template <typename T>
__global__ void __launch_bounds__(kThreads)
rotary_heads_kernel(T* __restrict__ q, int ld, const int* __restrict__ pos, int rows, int heads, int hd, int at, const float2* __restrict__ table, int pairs) {
  lg::pdl_prologue();
  const int octs = (2 * pairs + 7) >> 3;
  const int64_t i = (int64_t)blockIdx.x * kThreads + threadIdx.x;
  if (i >= (int64_t)rows * heads * octs) return;
  const int o = (int)(i % octs), h = (int)(i / octs % heads), r = (int)(i / ((int64_t)octs * heads));
  Vec8<T>* x = reinterpret_cast<Vec8<T>*>(q + (size_t)r * ld + h * hd + at) + o;
  float f[8];
  unpack<T>(*x, f);
  rotate8(f, 8 * o, pairs, table + (size_t)pos[r] * pairs);
  *x = pack<T>(f);
}

struct HeadArgs {
  void* qkv;
  int ld, rows, heads, n_kv, maps, dim;
  const float *gain_q, *gain_k;
  float eps;
  const float2* table;
  int pairs;
  void* q_out;
  int ld_q;
  void *kpool, *vpool;
  const int64_t* slots;
  const int* pos;
  int64_t n_slots;
  int pool, pool_rows;
  void *kmean, *vmean;
  const int *tables, *seq_ids;
  int max_blocks, n_pool_blocks;
  int* status;
};

// The mean of the block of tokens that ends at position `at`, eight channels of a cache row from channel c0 on
template <typename T>
LG_DEVINL void pool_piece(const HeadArgs& p, const T* pool, T* mean, int seq, int at, int row_w, int c0) {
  const int* table = p.tables + (size_t)seq * p.max_blocks;
  float sum[8] = {};
  int page = -1, block = -1;
#pragma unroll 4
  for (int j = at + 1 - p.pool; j <= at; ++j) {
    if (j >> 4 != page) {
      page = j >> 4;
      block = page < p.max_blocks ? table[page] : -1;
      if (block < 0 || block >= p.n_pool_blocks) {
        if (p.status) atomicExch(p.status, 1);
        return;
      }
    }
    float f[8];
    unpack<T>(*reinterpret_cast<const Vec8<T>*>(pool + ((size_t)block * 16 + (j & 15)) * row_w + c0), f);
#pragma unroll
    for (int i = 0; i < 8; ++i) sum[i] += f[i];
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) sum[i] /= (float)p.pool;
  const int b = at / p.pool, rows = (15 + p.pool) / p.pool;
  *reinterpret_cast<Vec8<T>*>(mean + ((size_t)block * rows + b - (page << 4) / p.pool) * row_w + c0) = pack<T>(sum);
}

// LANES lanes hold a piece of HD channels, eight each; a group of lanes takes ITEMS pieces, all requested at once
template <typename T, int LANES, int ITEMS>
__global__ void __launch_bounds__(kThreads)
head_norm_store_kernel(HeadArgs p) {
  lg::pdl_prologue();
  constexpr int HD = LANES * 8;
  const uint32_t nq = p.heads * p.maps, nk = p.n_kv * p.maps, per_row = nq + 2 * nk, lane = threadIdx.x % LANES;
  const uint32_t total = p.rows * per_row, first = (blockIdx.x * kThreads + threadIdx.x) / LANES * ITEMS;
  const int row_w = (int)nk * HD, c = (int)lane * 8;
  Vec8<T> x[ITEMS];
  int row[ITEMS], unit[ITEMS];
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const uint32_t at = min(first + i, total - 1);
    row[i] = (int)(at / per_row);
    unit[i] = (int)(at % per_row);
    x[i] = *reinterpret_cast<const Vec8<T>*>(reinterpret_cast<const T*>(p.qkv) + (size_t)row[i] * p.ld + unit[i] * HD + c);
  }
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const bool in = first + i < total;
    const uint32_t u = (uint32_t)unit[i];
    const int r = row[i], pos = p.pos[r];
    if (u < nq + nk) {   // the same for all lanes of a piece
      float f[8], ss = 0.0f;
      unpack<T>(x[i], f);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(f[j], f[j], ss);
      constexpr int kWidth = LANES;
      const uint32_t mask = kWidth == 32 ? 0xffffffffu : ((1u << (kWidth & 31)) - 1u) << ((threadIdx.x & 31) / kWidth * kWidth);
#pragma unroll
      for (int o = 1; o < LANES; o <<= 1) ss += __shfl_xor_sync(mask, ss, o);
      const float m = 1.0f / sqrtf(ss / (float)p.dim + p.eps);
      const float4* gain = reinterpret_cast<const float4*>((u < nq ? p.gain_q : p.gain_k) + c);
      const float4 g0 = __ldg(gain), g1 = __ldg(gain + 1);
      const float g[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] *= m * g[j];
      rotate8(f, c, p.pairs, p.table + (size_t)pos * p.pairs);
      x[i] = pack<T>(f);
    }
    if (!in) continue;
    if (u < nq) {
      T* q = reinterpret_cast<T*>(p.q_out) + (size_t)r * p.ld_q + u * p.maps * HD + c;
      if (p.maps == 1) { *reinterpret_cast<Vec8<T>*>(q) = x[i]; continue; }
      const int map = (int)(u / (p.heads / p.n_kv)) & 1;
      const float zero[8] = {};
      *reinterpret_cast<Vec8<T>*>(q + map * HD) = x[i];
      *reinterpret_cast<Vec8<T>*>(q + (1 - map) * HD) = pack<T>(zero);
      continue;
    }
    const int64_t slot = p.slots[r];
    if (slot < 0 || slot >= p.n_slots) {
      if (lane == 0 && p.status) atomicExch(p.status, 1);
      continue;
    }
    const bool is_v = u >= nq + nk;
    const int at = (int)(u - nq - (is_v ? nk : 0)) * HD + c;
    T* pool = reinterpret_cast<T*>(is_v ? p.vpool : p.kpool);
    *reinterpret_cast<Vec8<T>*>(pool + (size_t)slot * row_w + at) = x[i];
    if (p.pool && r < p.pool_rows && (pos + 1) % p.pool == 0) pool_piece<T>(p, pool, reinterpret_cast<T*>(is_v ? p.vmean : p.kmean), r, pos, row_w, at);
  }
}

// A thread owns eight channels of all blocks that end in `pool` consecutive rows: one, unless a sequence ends among them
template <typename T>
__global__ void __launch_bounds__(kThreads)
pool_blocks_kernel(HeadArgs p, int octs) {
  lg::pdl_prologue();
  const uint32_t at = blockIdx.x * kThreads + threadIdx.x;
  const int r0 = p.pool_rows + (int)(at / (2 * octs)) * p.pool, piece = (int)(at % (2 * octs));
  const bool is_v = piece >= octs;
  const int end = min(r0 + p.pool, p.rows);
  for (int r = r0; r < end;) {
    const int seq = p.seq_ids[r], pos = p.pos[r], last = r + p.pool - 1 - pos % p.pool;   // where the block of row r ends
    if (last < end && p.seq_ids[last] == seq) {
      pool_piece<T>(p, reinterpret_cast<const T*>(is_v ? p.vpool : p.kpool), reinterpret_cast<T*>(is_v ? p.vmean : p.kmean), seq, pos + last - r, octs * 8,
                    8 * (is_v ? piece - octs : piece));
      r = last + 1;
    } else {
      do ++r;
      while (r < end && p.seq_ids[r] == seq);
    }
  }
}

bool head_args(const lg_head_norm_t* a, int is_f32, void* status, HeadArgs* p) {
  if (!a || !a->qkv || !a->gain_q || !a->gain_k || !a->k_pool || !a->v_pool || !a->slots_i64 || !a->positions_i32 || a->rows <= 0 || a->heads <= 0 || a->n_kv <= 0 ||
      a->heads % a->n_kv || (a->maps != 1 && a->maps != 2) || (a->hd != 32 && a->hd != 64 && a->hd != 128 && a->hd != 256) || a->dim <= 0 || a->dim > a->hd ||
      a->rot_dims < 0 || a->rot_dims % 2 || a->rot_dims > a->dim || (a->rot_dims && !a->table) || a->ld % 8 || a->ld < a->maps * (a->heads + 2 * a->n_kv) * a->hd ||
      (a->maps == 2 && (!a->q_out || a->ld_q < 4 * a->heads * a->hd || a->ld_q % 8)) ||
      (((uintptr_t)a->qkv | (uintptr_t)a->k_pool | (uintptr_t)a->v_pool | (uintptr_t)a->q_out | (uintptr_t)a->k_mean | (uintptr_t)a->v_mean) & (is_f32 ? 31 : 15)) ||
      (((uintptr_t)a->gain_q | (uintptr_t)a->gain_k) & 15) || ((uintptr_t)a->table & 7) || (int64_t)a->rows * a->maps * (a->heads + 2 * a->n_kv) > (1 << 26))
    return false;
  if (a->pool < 0 || (a->pool && (!a->k_mean || !a->v_mean || !a->tables_i32 || !a->seq_ids_i32 || a->pool_rows < 0 || a->max_blocks <= 0 || a->n_pool_blocks <= 0))) return false;
  *p = HeadArgs{a->qkv, a->ld, a->rows, a->heads, a->n_kv, a->maps, a->dim, (const float*)a->gain_q, (const float*)a->gain_k, a->eps, (const float2*)a->table, a->rot_dims / 2,
                a->maps == 1 ? a->qkv : a->q_out, a->maps == 1 ? a->ld : a->ld_q, a->k_pool, a->v_pool, (const int64_t*)a->slots_i64, (const int*)a->positions_i32,
                a->n_pool_slots, a->pool, a->pool_rows, a->k_mean, a->v_mean, (const int*)a->tables_i32, (const int*)a->seq_ids_i32, a->max_blocks, a->n_pool_blocks,
                (int*)status};
  return true;
}

}  // namespace

extern "C" {

uint32_t logismos_launch_head_norm_store(const lg_head_norm_t* a, int32_t is_f32, void* status, void* stream) {
  lg::LaunchScope launch_scope_;
  HeadArgs p;
  if (!head_args(a, is_f32, status, &p)) return lg::kInvalidValue;
  const int64_t items = (int64_t)a->rows * a->maps * (a->heads + 2 * a->n_kv);
  auto go = [&](auto kern, int per_block) -> uint32_t {
    lg::launch(kern, dim3((unsigned)((items + per_block - 1) / per_block)), dim3(kThreads), 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
#define LG_HEADS(T, LANES) (items < 20000 ? go(head_norm_store_kernel<T, LANES, 1>, kThreads / LANES) : go(head_norm_store_kernel<T, LANES, 4>, kThreads / LANES * 4))
  if (is_f32) return a->hd == 32 ? LG_HEADS(float, 4) : a->hd == 64 ? LG_HEADS(float, 8) : a->hd == 128 ? LG_HEADS(float, 16) : LG_HEADS(float, 32);
  return a->hd == 32 ? LG_HEADS(__nv_bfloat16, 4) : a->hd == 64 ? LG_HEADS(__nv_bfloat16, 8) : a->hd == 128 ? LG_HEADS(__nv_bfloat16, 16) : LG_HEADS(__nv_bfloat16, 32);
#undef LG_HEADS
}

uint32_t logismos_launch_pool_blocks(const lg_head_norm_t* a, int32_t is_f32, void* status, void* stream) {
  lg::LaunchScope launch_scope_;
  HeadArgs p;
  if (!head_args(a, is_f32, status, &p) || a->pool <= 0 || a->pool_rows >= a->rows) return lg::kInvalidValue;
  const int octs = a->n_kv * a->maps * a->hd / 8;
  const int64_t threads = (int64_t)((a->rows - a->pool_rows + a->pool - 1) / a->pool) * 2 * octs;
  if (threads > 0x7fffff00) return lg::kInvalidValue;
  const dim3 grid((unsigned)((threads + kThreads - 1) / kThreads));
  if (is_f32) lg::launch(pool_blocks_kernel<float>, grid, dim3(kThreads), 0, (cudaStream_t)stream, p, octs);
  else lg::launch(pool_blocks_kernel<__nv_bfloat16>, grid, dim3(kThreads), 0, (cudaStream_t)stream, p, octs);
  return lg::launch_status();
}

uint32_t logismos_launch_qk_norm_rotary_store(void* qkv, int32_t ld, void* k_pool, void* v_pool, const void* slots, const void* positions, int32_t rows,
                                              int32_t n_heads, int32_t n_kv, int32_t head_dim, int32_t dim, const void* gain_q, const void* gain_k, float eps,
                                              const void* table, int32_t rot_dims, int64_t n_pool_slots, int32_t is_f32, void* status, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!qkv || !k_pool || !v_pool || !slots || !positions || !gain_q || !gain_k || rows <= 0 || n_heads <= 0 || n_kv <= 0 || head_dim <= 0 || head_dim % 8 || dim <= 0 ||
      dim > head_dim || rot_dims < 0 || rot_dims % 2 || rot_dims > dim || (rot_dims && !table) || ld < (n_heads + 2 * n_kv) * head_dim || ld % 8 ||
      (((uintptr_t)qkv | (uintptr_t)k_pool | (uintptr_t)v_pool) & (is_f32 ? 31 : 15)) || (((uintptr_t)gain_q | (uintptr_t)gain_k) & 15) || ((uintptr_t)table & 7))
    return lg::kInvalidValue;
  const QkvArgs p{qkv, ld, k_pool, v_pool, (const int64_t*)slots, (const int*)positions, n_heads, n_kv, head_dim, dim, (const float*)gain_q, (const float*)gain_k, eps,
                  (const float2*)table, rot_dims / 2, n_pool_slots, (int*)status};
  auto go = [&](auto kern) -> uint32_t {
    lg::launch(kern, dim3((unsigned)rows), dim3(kThreads), 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
  return is_f32 ? go(qk_norm_rotary_store_kernel<float>) : go(qk_norm_rotary_store_kernel<__nv_bfloat16>);
}

uint32_t logismos_launch_rotary_heads(void* q, int32_t ld, const void* positions, int32_t rows, int32_t n_heads, int32_t head_dim, int32_t at, const void* table,
                                      int32_t dims, int32_t is_f32, void* stream) {
  lg::LaunchScope launch_scope_;
  const int octs = (dims + 7) / 8;
  if (!q || !positions || !table || rows <= 0 || n_heads <= 0 || head_dim <= 0 || head_dim % 8 || at < 0 || at % 8 || dims <= 0 || dims % 2 || at + 8 * octs > head_dim ||
      ld < n_heads * head_dim || ld % 8 || ((uintptr_t)q & (is_f32 ? 31 : 15)) || ((uintptr_t)table & 7))
    return lg::kInvalidValue;
  const int64_t blocks = ((int64_t)rows * n_heads * octs + kThreads - 1) / kThreads;
  if (blocks > 0x7fffffff) return lg::kInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  if (is_f32) lg::launch(rotary_heads_kernel<float>, dim3((unsigned)blocks), dim3(kThreads), 0, s, (float*)q, ld, (const int*)positions, rows, n_heads, head_dim, at, (const float2*)table, dims / 2);
  else lg::launch(rotary_heads_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(kThreads), 0, s, (__nv_bfloat16*)q, ld, (const int*)positions, rows, n_heads, head_dim, at, (const float2*)table, dims / 2);
  return lg::launch_status();
}

}  // extern "C"
