// Rotary positions in the interleaved layout, fused with what surrounds them: norms of whole query and key projections
// and the cache store of a packed q | k | v row, or the rotated part of every query head in place. Angles come from a
// table of (cos, sin) per position and pair, amplitude included; norms and rotations are fp32.
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

}  // namespace

extern "C" {

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
