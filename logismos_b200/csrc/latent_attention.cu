// Latent attention (keys and values are linear images of one cached row c of `rank` values per token, no
// rotated part): the cache side and the decode side.
//   latent_norm_store   RMS norms of the query latent and of the key/value latent from the fp32
//                       projection; the latter goes to its paged-cache slot
//   latent_gather       cached rows of whole sequences made contiguous (prefill expands them to keys and
//                       values with GEMMs and runs the tcgen05 attention kernel)
//   latent_decode       one query token per sequence in the latent space: with q'_h = W_uk,h^T q_h the
//                       score of a key is q'_h . c and the output is W_uv,h (sum_j p_j c_j), so every head
//                       shares the same rank-wide key = value row and a cached row is read once for all
// latent_decode splits the contexts in chunks; CTA = (chunk, group of 16 * MT heads), 8 warps, tiles of
// TK tokens in a two-stage cp.async ring (16-byte chunks XOR-swizzled by row). Per tile: S = Q' C^T
// (mma.sync, a warp per 8 tokens), running maximum and sum in fp32 (exp2 domain), P rounded to bf16,
// O += P C (a warp per rank / 8 columns, C through ldmatrix.trans). Partial results are merged by a
// second kernel; a context that is one chunk is finished in place.
#include "common.cuh"
#include "logismos_kernels.h"

namespace {

using namespace lg;

constexpr float kLog2e = 1.4426950408889634f;
constexpr int kBlockTokens = 16;
constexpr int kThreads = 256;

LG_DEVINL void store4(void* p, size_t i4, float4 v, bool f32) {
  if (f32) reinterpret_cast<float4*>(p)[i4] = v;
  else reinterpret_cast<uint2*>(p)[i4] = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// warp = (row, half): half 0 the query latent (columns 0 .. qw), half 1 the key/value latent (qw .. qw + rw)
__global__ void __launch_bounds__(kThreads)
latent_norm_store_kernel(const float* __restrict__ raw, int ld, const float* __restrict__ gain_q, const float* __restrict__ gain_c,
                         void* __restrict__ cq, void* __restrict__ pool, const int64_t* __restrict__ slots, int rows, int qw, int q_n,
                         int rw, int r_n, float eps, int64_t n_pool_slots, int f32, int* __restrict__ status) {
  lg::pdl_prologue();
  const int id = (blockIdx.x * kThreads + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  const int row = id >> 1, half = id & 1;
  if (row >= rows) return;
  const float4* src = reinterpret_cast<const float4*>(raw + (size_t)row * ld + (half ? qw : 0));
  const int nv = (half ? rw : qw) >> 2;
  float ss = 0.0f;
  for (int v = lane; v < nv; v += 32) {
    const float4 a = src[v];
    ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)(half ? r_n : q_n) + eps);
  size_t dst = (size_t)row * (qw >> 2);
  if (half) {
    const int64_t slot = slots[row];
    if (slot < 0 || slot >= n_pool_slots) {
      if (lane == 0 && status) atomicExch(status, 1);
      return;
    }
    dst = (size_t)slot * (rw >> 2);
  }
  const float4* gain = reinterpret_cast<const float4*>(half ? gain_c : gain_q);
  void* out = half ? pool : cq;
  for (int v = lane; v < nv; v += 32) {
    const float4 a = src[v], g = __ldg(gain + v);
    store4(out, dst + v, make_float4(a.x * inv * g.x, a.y * inv * g.y, a.z * inv * g.z, a.w * inv * g.w), f32 != 0);
  }
}

LG_DEVINL int round8(int v) { return (v + 7) & ~7; }

// rows of sequence s -> out[pstart[s] ..], every sequence starting at a multiple of 8 rows, padding and
// the rows after the last sequence zeroed up to tp. Grid (row blocks of 64, sequences).
__global__ void __launch_bounds__(kThreads)
latent_gather_kernel(const __nv_bfloat16* __restrict__ pool, const int* __restrict__ tables, int max_blocks, int n_pool_blocks,
                     const int* __restrict__ kv_lens, __nv_bfloat16* __restrict__ out, int* __restrict__ pstart, int n_seqs, int tp,
                     int rw, int* __restrict__ status) {
  lg::pdl_prologue();
  __shared__ int p0_s;
  const int tb = blockIdx.x, s = blockIdx.y, tid = threadIdx.x;
  if (tid < 32) {
    int part = 0;
    for (int i = tid; i < s; i += 32) part += round8(max(kv_lens[i], 0));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) part += __shfl_xor_sync(0xffffffffu, part, o);
    if (tid == 0) p0_s = part;
  }
  __syncthreads();
  const int p0 = p0_s, len = max(kv_lens[s], 0), plen = round8(len), cw = rw >> 3;
  if (p0 + plen > tp) {
    if (tid == 0 && status) atomicExch(status, 1);
    return;
  }
  if (tb == 0 && tid == 0) pstart[s] = p0;
  if (tb == 0 && s == n_seqs - 1)
    for (int64_t u = tid; u < (int64_t)(tp - p0 - plen) * cw; u += kThreads)
      reinterpret_cast<uint4*>(out)[(size_t)(p0 + plen) * cw + u] = make_uint4(0u, 0u, 0u, 0u);
  if (tb * 64 >= plen) return;
  for (int u = tid; u < 64 * cw; u += kThreads) {
    const int t = tb * 64 + u / cw, ch = u % cw;
    if (t >= plen) break;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (t < len) {
      const int bi = t / kBlockTokens;
      const int blk = bi < max_blocks ? __ldg(tables + (size_t)s * max_blocks + bi) : -1;
      if (blk < 0 || blk >= n_pool_blocks) {
        if (ch == 0 && status) atomicExch(status, 1);
      } else {
        v = reinterpret_cast<const uint4*>(pool)[((size_t)blk * kBlockTokens + t % kBlockTokens) * cw + ch];
      }
    }
    reinterpret_cast<uint4*>(out)[(size_t)(p0 + t) * cw + ch] = v;
  }
}

struct DecodeArgs {
  const __nv_bfloat16* q;     // [rows, heads, rank]
  const __nv_bfloat16* pool;  // [n_pool_blocks, 16, rank]
  const int* tables;
  const int* ctx;
  const int* chunk_offsets;   // [rows + 1]
  __nv_bfloat16* out;         // [rows, heads, rank]
  float* part_o;              // [chunks, heads, rank]
  float2* part_ml;            // [chunks, heads]
  int rows, heads, rank, chunk_tokens, max_blocks, n_pool_blocks;
  float sl2;
  int* status;
};

// row r with chunk_offsets[r] <= chunk < chunk_offsets[r + 1]
LG_DEVINL int find_row(const int* __restrict__ off, int rows, int chunk) {
  int lo = 0, hi = rows - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (__ldg(off + mid) <= chunk) lo = mid;
    else hi = mid - 1;
  }
  return lo;
}

template <int MT, int TK>
__host__ __device__ constexpr size_t decode_smem(int rank) {
  return (size_t)(16 * MT + 2 * TK) * rank * 2 + (size_t)16 * MT * (TK + 4) * 4 + (size_t)16 * MT * (TK + 8) * 2 + (size_t)16 * MT * 3 * 4;
}

template <int MT, int MAXNT, int TK>
__global__ void __launch_bounds__(kThreads)
latent_decode_kernel(DecodeArgs p) {
  lg::pdl_prologue();
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int kRows = 16 * MT;
  const int R = p.rank, cw = R >> 3, row_bytes = R * 2, nt_n = R >> 6;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  const uint32_t sq = smem_u32(smem), sc = sq + (uint32_t)kRows * row_bytes;
  uint8_t* after = smem + (size_t)(kRows + 2 * TK) * row_bytes;
  float* s_s = reinterpret_cast<float*>(after);                             // [kRows][TK + 4]
  __nv_bfloat16* s_p = reinterpret_cast<__nv_bfloat16*>(s_s + kRows * (TK + 4));  // [kRows][TK + 8]
  float* s_m = reinterpret_cast<float*>(s_p + kRows * (TK + 8));
  float* s_l = s_m + kRows;
  float* s_a = s_l + kRows;
  const uint32_t sp = smem_u32(s_p);
  auto swz = [&](uint32_t base, int row, int chunk) { return base + (uint32_t)row * row_bytes + (uint32_t)((chunk ^ (row & 7)) << 4); };

  const int chunk = blockIdx.x, h0 = blockIdx.y * kRows;
  const int r = find_row(p.chunk_offsets, p.rows, chunk);
  const int c_idx = chunk - __ldg(p.chunk_offsets + r), c_cnt = __ldg(p.chunk_offsets + r + 1) - __ldg(p.chunk_offsets + r);
  const int ctx = p.ctx[r];
  const int k0 = c_idx * p.chunk_tokens, k1 = min(ctx, k0 + p.chunk_tokens);
  const int tiles = (k1 - k0 + TK - 1) / TK;
  const int* table = p.tables + (size_t)r * p.max_blocks;

  // query rows of this head group (heads beyond the last are zero rows)
  for (int u = threadIdx.x; u < kRows * cw; u += kThreads) {
    const int hr = u / cw, ch = u % cw;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h0 + hr < p.heads) v = *reinterpret_cast<const uint4*>(p.q + ((size_t)r * p.heads + h0 + hr) * R + ch * 8);
    *reinterpret_cast<uint4*>(smem + (swz(sq, hr, ch) - sq)) = v;
  }
  for (int i = threadIdx.x; i < kRows; i += kThreads) { s_m[i] = -1e30f; s_l[i] = 0.0f; }

  auto load_tile = [&](int ti) {
    const uint32_t base = sc + (uint32_t)(ti & 1) * TK * row_bytes;
    for (int u = threadIdx.x; u < TK * cw; u += kThreads) {
      const int kr = u / cw, ch = u % cw, key = k0 + ti * TK + kr;
      const uint32_t dst = swz(base, kr, ch);
      int blk = -1;
      if (key < k1) {
        const int bi = key / kBlockTokens;
        blk = bi < p.max_blocks ? __ldg(table + bi) : -1;
        if (blk < 0 || blk >= p.n_pool_blocks) {
          if (ch == 0 && p.status) atomicExch(p.status, 1);
          blk = -1;
        }
      }
      if (blk >= 0) cp_async16(dst, p.pool + ((size_t)blk * kBlockTokens + key % kBlockTokens) * R + ch * 8);
      else *reinterpret_cast<uint4*>(smem + (dst - sq)) = make_uint4(0u, 0u, 0u, 0u);
    }
    cp_async_commit();
  };

  float acc[MT][MAXNT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < MAXNT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.0f;

  load_tile(0);
  for (int ti = 0; ti < tiles; ++ti) {
    if (ti + 1 < tiles) {
      load_tile(ti + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t tile = sc + (uint32_t)(ti & 1) * TK * row_bytes;
    // S = Q' C^T
    if (warp < TK / 8) {
      float s0[MT][4], s1[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) { s0[i][e] = 0.0f; s1[i][e] = 0.0f; }
      for (int ks = 0; ks < (R >> 5); ++ks) {
        uint32_t b[4];
        ldmatrix_x4(b, swz(tile, 8 * warp + (lane & 7), 4 * ks + (lane >> 3)));
        const uint32_t b0[2] = {b[0], b[1]}, b1[2] = {b[2], b[3]};
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          const int mat = lane >> 3, row = 16 * i + (lane & 7) + 8 * (mat & 1);
          uint32_t a0[4], a1[4];
          ldmatrix_x4(a0, swz(sq, row, 4 * ks + (mat >> 1)));
          ldmatrix_x4(a1, swz(sq, row, 4 * ks + 2 + (mat >> 1)));
          mma_bf16_16816(s0[i], a0, b0, s0[i]);
          mma_bf16_16816(s1[i], a1, b1, s1[i]);
        }
      }
      const int col = 8 * warp + 2 * t4, key = k0 + ti * TK + col;
      const bool v0 = key < k1, v1 = key + 1 < k1;
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        float* d0 = s_s + (16 * i + g) * (TK + 4) + col;
        float* d1 = d0 + 8 * (TK + 4);
        d0[0] = v0 ? (s0[i][0] + s1[i][0]) * p.sl2 : -1e30f;
        d0[1] = v1 ? (s0[i][1] + s1[i][1]) * p.sl2 : -1e30f;
        d1[0] = v0 ? (s0[i][2] + s1[i][2]) * p.sl2 : -1e30f;
        d1[1] = v1 ? (s0[i][3] + s1[i][3]) * p.sl2 : -1e30f;
      }
    }
    __syncthreads();
    // running maximum and sum; a tile always holds at least one visible key, so the maximum is a real score
    for (int row = warp; row < kRows; row += kThreads / 32) {
      const float a = s_s[row * (TK + 4) + lane], b = TK > 32 ? s_s[row * (TK + 4) + 32 + lane] : -1e30f;
      const float m_old = s_m[row], m_new = fmaxf(m_old, warp_max(fmaxf(a, b)));
      const float pa = exp2f(a - m_new), pb = TK > 32 ? exp2f(b - m_new) : 0.0f;
      const float sum = warp_sum(pa + pb), alpha = exp2f(m_old - m_new);
      s_p[row * (TK + 8) + lane] = __float2bfloat16_rn(pa);
      if (TK > 32) s_p[row * (TK + 8) + 32 + lane] = __float2bfloat16_rn(pb);
      __syncwarp();
      if (lane == 0) { s_m[row] = m_new; s_l[row] = s_l[row] * alpha + sum; s_a[row] = alpha; }
    }
    __syncthreads();
    // O = O * alpha + P C
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const float a0 = s_a[16 * i + g], a1 = s_a[16 * i + g + 8];
      if (a0 != 1.0f || a1 != 1.0f) {
#pragma unroll
        for (int j = 0; j < MAXNT; ++j) { acc[i][j][0] *= a0; acc[i][j][1] *= a0; acc[i][j][2] *= a1; acc[i][j][3] *= a1; }
      }
    }
#pragma unroll
    for (int ks = 0; ks < TK / 16; ++ks) {
      uint32_t pa[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const int mat = lane >> 3, row = 16 * i + (lane & 7) + 8 * (mat & 1);
        ldmatrix_x4(pa[i], sp + (uint32_t)(row * (TK + 8) + 16 * ks + 8 * (mat >> 1)) * 2);
      }
#pragma unroll
      for (int j = 0; j < MAXNT; j += 2) {
        if (j < nt_n) {
          const int ct = warp * nt_n + j + (lane >> 4);  // column tile; the odd one out is read but not used
          uint32_t b[4];
          ldmatrix_x4_trans(b, swz(tile, 16 * ks + (lane & 7) + 8 * ((lane >> 3) & 1), min(ct, cw - 1)));
          const uint32_t b0[2] = {b[0], b[1]}, b1[2] = {b[2], b[3]};
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            mma_bf16_16816(acc[i][j], pa[i], b0, acc[i][j]);
            if (j + 1 < MAXNT && j + 1 < nt_n) mma_bf16_16816(acc[i][j + 1 < MAXNT ? j + 1 : j], pa[i], b1, acc[i][j + 1 < MAXNT ? j + 1 : j]);
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int hr = 16 * i + g + 8 * half, h = h0 + hr;
      if (h >= p.heads) continue;
      const float inv = 1.0f / s_l[hr];
#pragma unroll
      for (int j = 0; j < MAXNT; ++j) {
        if (j >= nt_n) continue;
        const int col = (warp * nt_n + j) * 8 + 2 * t4;
        const float x = acc[i][j][2 * half], y = acc[i][j][2 * half + 1];
        if (c_cnt == 1)
          *reinterpret_cast<uint32_t*>(p.out + ((size_t)r * p.heads + h) * R + col) = pack_bf16x2(x * inv, y * inv);
        else
          *reinterpret_cast<float2*>(p.part_o + ((size_t)chunk * p.heads + h) * R + col) = make_float2(x, y);
      }
      if (c_cnt > 1 && warp == 0 && t4 == 0) p.part_ml[(size_t)chunk * p.heads + h] = make_float2(s_m[hr], s_l[hr]);
    }
}

// CTA = (row, head): the chunks of a context that was split
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_o, const float2* __restrict__ part_ml, const int* __restrict__ chunk_offsets,
                    __nv_bfloat16* __restrict__ out, int heads, int rank) {
  lg::pdl_prologue();
  const int h = blockIdx.x, r = blockIdx.y;
  const int c0 = chunk_offsets[r], c1 = chunk_offsets[r + 1];
  if (c1 - c0 <= 1) return;
  float m = -1e30f, l = 0.0f;
  for (int c = c0; c < c1; ++c) m = fmaxf(m, part_ml[(size_t)c * heads + h].x);
  for (int c = c0; c < c1; ++c) {
    const float2 ml = part_ml[(size_t)c * heads + h];
    l += ml.y * exp2f(ml.x - m);
  }
  const float inv = 1.0f / l;
  for (int v = threadIdx.x; v < rank / 4; v += 128) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int c = c0; c < c1; ++c) {
      const float w = exp2f(part_ml[(size_t)c * heads + h].x - m) * inv;
      const float4 o = reinterpret_cast<const float4*>(part_o + ((size_t)c * heads + h) * rank)[v];
      a.x += w * o.x; a.y += w * o.y; a.z += w * o.z; a.w += w * o.w;
    }
    store4(out, ((size_t)r * heads + h) * (rank / 4) + v, a, false);
  }
}

// fp32 form: CTA = (query row, head), any row of the step; row t of sequence seq_ids[t] sees keys 0 .. pos[t]
constexpr int kF32Tile = 64;
__global__ void __launch_bounds__(128)
latent_attention_f32_kernel(const float* __restrict__ q, const float* __restrict__ pool, const int* __restrict__ tables, int max_blocks,
                            int n_pool_blocks, const int* __restrict__ seq_ids, const int* __restrict__ pos, float* __restrict__ out,
                            int heads, int rank, float sl2, int* __restrict__ status) {
  lg::pdl_prologue();
  extern __shared__ float fs[];  // q [rank], scores [kF32Tile]
  __shared__ float red[32];
  __shared__ int blk_s[kF32Tile / kBlockTokens];
  float* sq = fs;
  float* ss = fs + rank;
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n_keys = pos[t] + 1;
  const int* table = tables + (size_t)seq_ids[t] * max_blocks;
  const size_t row = ((size_t)t * heads + h) * rank;
  for (int i = tid; i < rank; i += 128) sq[i] = q[row + i];
  float m = -1e30f, l = 0.0f, acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  for (int k0 = 0; k0 < n_keys; k0 += kF32Tile) {
    const int n = min(kF32Tile, n_keys - k0);
    __syncthreads();
    if (tid < kF32Tile / kBlockTokens) {
      const int bi = k0 / kBlockTokens + tid;
      int b = tid * kBlockTokens < n && bi < max_blocks ? __ldg(table + bi) : -1;
      if (tid * kBlockTokens < n && (b < 0 || b >= n_pool_blocks)) {
        if (status) atomicExch(status, 1);
        b = -1;
      }
      blk_s[tid] = b;
    }
    __syncthreads();
    for (int k = warp; k < kF32Tile; k += 4) {
      const int b = blk_s[k / kBlockTokens];
      float s = 0.0f;
      if (k < n && b >= 0) {
        const float* c = pool + ((size_t)b * kBlockTokens + k % kBlockTokens) * rank;
        for (int i = lane; i < rank; i += 32) s = fmaf(sq[i], c[i], s);
      }
      s = warp_sum(s);
      if (lane == 0) ss[k] = k < n && b >= 0 ? s * sl2 : -1e30f;
    }
    __syncthreads();
    const float mine = tid < kF32Tile ? ss[tid] : -1e30f;
    const float m_new = fmaxf(m, block_max(mine, red));
    const float alpha = exp2f(m - m_new), e = tid < n ? exp2f(mine - m_new) : 0.0f;
    l = l * alpha + block_sum(e, red);
    m = m_new;
    if (tid < kF32Tile) ss[tid] = e;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] *= alpha;
    for (int k = 0; k < n; ++k) {
      const int b = blk_s[k / kBlockTokens];
      if (b < 0) continue;
      const float* c = pool + ((size_t)b * kBlockTokens + k % kBlockTokens) * rank;
      const float w = ss[k];
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (tid + i * 128 < rank) acc[i] = fmaf(w, c[tid + i * 128], acc[i]);
    }
  }
  const float inv = 1.0f / l;
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (tid + i * 128 < rank) out[row + tid + i * 128] = acc[i] * inv;
}

}  // namespace

extern "C" {

uint32_t logismos_launch_latent_norm_store(const void* raw_f32, int32_t ld, const void* gain_q_f32, const void* gain_c_f32, void* q_latent,
                                           void* pool, const void* slot_mapping_i64, int32_t rows, int32_t q_width, int32_t q_n,
                                           int32_t c_width, int32_t c_n, float eps, int64_t n_pool_slots, int32_t is_f32,
                                           void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!raw_f32 || rows <= 0 || q_width <= 0 || c_width <= 0 || (q_width % 4) || (c_width % 4) || q_n <= 0 || q_n > q_width || c_n <= 0 ||
      c_n > c_width || ld < q_width + c_width || (ld % 4) || rows > 0x3fffffff)
    return lg::kInvalidValue;
  const int64_t blocks = ((int64_t)rows * 2 + kThreads / 32 - 1) / (kThreads / 32);
  lg::launch(latent_norm_store_kernel, dim3((unsigned)blocks), dim3(kThreads), 0, (cudaStream_t)stream, (const float*)raw_f32, ld,
             (const float*)gain_q_f32, (const float*)gain_c_f32, q_latent, pool, (const int64_t*)slot_mapping_i64, rows, q_width, q_n,
             c_width, c_n, eps, n_pool_slots, is_f32, (int*)status_i32);
  return lg::launch_status();
}

int32_t logismos_latent_gather_rows(int32_t total_kv_tokens, int32_t n_seqs) { return (total_kv_tokens + 8 * n_seqs + 15) & ~15; }

uint32_t logismos_launch_latent_gather_bf16(const void* pool, const void* block_tables_i32, int32_t max_blocks, int32_t n_pool_blocks,
                                            const void* kv_lens_i32, void* out, void* kv_start_i32, int32_t total_kv_tokens,
                                            int32_t n_seqs, int32_t max_kv_len, int32_t width, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!pool || !out || !kv_start_i32 || total_kv_tokens <= 0 || n_seqs <= 0 || n_seqs > 65535 || max_kv_len <= 0 || max_kv_len > total_kv_tokens ||
      width <= 0 || (width % 8) || max_blocks <= 0 || n_pool_blocks <= 0 || (((uintptr_t)pool | (uintptr_t)out) & 15))
    return lg::kInvalidValue;
  lg::launch(latent_gather_kernel, dim3((unsigned)((max_kv_len + 63) / 64), (unsigned)n_seqs), dim3(kThreads), 0, (cudaStream_t)stream,
             (const __nv_bfloat16*)pool, (const int*)block_tables_i32, max_blocks, n_pool_blocks, (const int*)kv_lens_i32, (__nv_bfloat16*)out,
             (int*)kv_start_i32, n_seqs, logismos_latent_gather_rows(total_kv_tokens, n_seqs), width, (int*)status_i32);
  return lg::launch_status();
}

int32_t logismos_pick_latent_chunk(const int32_t* context_lens, int32_t n_seqs, int32_t heads) {
  int64_t total = 0;
  for (int32_t i = 0; i < n_seqs; ++i) total += context_lens[i] > 0 ? context_lens[i] : 0;
  const int32_t groups = (heads + 63) / 64;
  const int64_t per = (total * groups + 295) / 296;  // about two CTAs per SM
  int64_t chunk = (per + 63) / 64 * 64;
  if (chunk < 256) chunk = 256;
  return (int32_t)(chunk > (1 << 20) ? (1 << 20) : chunk);
}

int32_t logismos_latent_max_chunks(int32_t max_rows) { return max_rows + 300; }

size_t logismos_latent_decode_scratch_bytes(int32_t total_chunks, int32_t heads, int32_t rank) {
  if (total_chunks < 0 || heads <= 0 || rank <= 0) return 0;
  return (size_t)total_chunks * heads * ((size_t)rank + 2) * 4;
}

uint32_t logismos_launch_latent_decode_bf16(const void* q, const void* pool, const void* block_tables_i32, const void* context_lens_i32,
                                            const void* chunk_offsets_i32, void* out, void* scratch, int32_t rows, int32_t total_chunks,
                                            int32_t chunk_tokens, int32_t max_blocks, int32_t n_pool_blocks, int32_t heads, int32_t rank,
                                            float scale, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!q || !pool || !out || !scratch || rows <= 0 || rows > 65535 || total_chunks < rows || chunk_tokens <= 0 || (chunk_tokens % 64) || max_blocks <= 0 ||
      n_pool_blocks <= 0 || heads <= 0 || rank <= 0 || (rank % 64) || rank > 1024 ||
      (((uintptr_t)q | (uintptr_t)pool | (uintptr_t)out | (uintptr_t)scratch) & 15))
    return lg::kInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  DecodeArgs p{(const __nv_bfloat16*)q, (const __nv_bfloat16*)pool, (const int*)block_tables_i32, (const int*)context_lens_i32,
               (const int*)chunk_offsets_i32, (__nv_bfloat16*)out, (float*)scratch, nullptr, rows, heads, rank, chunk_tokens, max_blocks,
               n_pool_blocks, scale * kLog2e, (int*)status_i32};
  p.part_ml = (float2*)(p.part_o + (size_t)total_chunks * heads * rank);
  auto go = [&](auto kern, int mt, size_t smem) -> uint32_t {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
    lg::launch(kern, dim3((unsigned)total_chunks, (unsigned)((heads + 16 * mt - 1) / (16 * mt))), dim3(kThreads), smem, s, p);
    return lg::launch_status();
  };
  uint32_t rc;
  if (rank <= 128) {
    if (heads <= 16) rc = go(latent_decode_kernel<1, 2, 64>, 1, decode_smem<1, 64>(rank));
    else if (heads <= 32) rc = go(latent_decode_kernel<2, 2, 64>, 2, decode_smem<2, 64>(rank));
    else rc = go(latent_decode_kernel<4, 2, 64>, 4, decode_smem<4, 64>(rank));
  } else if (rank <= 256) {
    if (heads <= 16) rc = go(latent_decode_kernel<1, 4, 64>, 1, decode_smem<1, 64>(rank));
    else if (heads <= 32) rc = go(latent_decode_kernel<2, 4, 64>, 2, decode_smem<2, 64>(rank));
    else rc = go(latent_decode_kernel<4, 4, 64>, 4, decode_smem<4, 64>(rank));
  } else if (rank <= 512) {
    if (heads <= 16) rc = go(latent_decode_kernel<1, 8, 64>, 1, decode_smem<1, 64>(rank));
    else if (heads <= 32) rc = go(latent_decode_kernel<2, 8, 64>, 2, decode_smem<2, 64>(rank));
    else rc = go(latent_decode_kernel<4, 8, 64>, 4, decode_smem<4, 64>(rank));
  } else {
    if (heads <= 16) rc = go(latent_decode_kernel<1, 16, 32>, 1, decode_smem<1, 32>(rank));
    else rc = go(latent_decode_kernel<2, 16, 32>, 2, decode_smem<2, 32>(rank));
  }
  if (rc || total_chunks == rows) return rc;
  lg::launch(latent_merge_kernel, dim3((unsigned)heads, (unsigned)rows), dim3(128), 0, s, (const float*)p.part_o, (const float2*)p.part_ml,
             p.chunk_offsets, p.out, heads, rank);
  return lg::launch_status();
}

uint32_t logismos_launch_latent_attention_f32(const void* q_f32, const void* pool_f32, const void* block_tables_i32, const void* seq_ids_i32,
                                              const void* positions_i32, void* out_f32, int32_t rows, int32_t max_blocks,
                                              int32_t n_pool_blocks, int32_t heads, int32_t rank, float scale, void* status_i32,
                                              void* stream) {
  lg::LaunchScope launch_scope_;
  if (!q_f32 || !pool_f32 || !out_f32 || rows <= 0 || max_blocks <= 0 || n_pool_blocks <= 0 || heads <= 0 || heads > 65535 || rank <= 0 || rank > 1024)
    return lg::kInvalidValue;
  lg::launch(latent_attention_f32_kernel, dim3((unsigned)rows, (unsigned)heads), dim3(128), (size_t)(rank + kF32Tile) * 4, (cudaStream_t)stream,
             (const float*)q_f32, (const float*)pool_f32, (const int*)block_tables_i32, max_blocks, n_pool_blocks, (const int*)seq_ids_i32,
             (const int*)positions_i32, (float*)out_f32, heads, rank, scale * kLog2e, (int*)status_i32);
  return lg::launch_status();
}

}  // extern "C"
