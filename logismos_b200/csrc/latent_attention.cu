// Latent attention (keys and values are linear images of one cached row c of `rank` values per token; a rotated key part
// that all heads share is more columns of that row): the cache side and the decode side.
//   latent_norm_store   RMS norms of the query latent and of the key/value latent from the fp32
//                       projection; the latter goes to its paged-cache slot, with its rotated columns
//   latent_gather       cached rows of whole sequences made contiguous (prefill expands them to keys and
//                       values with GEMMs and runs the tcgen05 attention kernel)
//   latent_decode       one query token per sequence in the latent space: with q'_h = W_uk,h^T q_h the
//                       score of a key is q'_h . c and the output is W_uv,h (sum_j p_j c_j), so every head
//                       shares the same rank-wide key = value row and a cached row is read once for all
// latent_decode splits the contexts in chunks; CTA = (chunk, group of 16 * MT heads), 8 warps, tiles of TK tokens. A cache block (16 tokens) arrives as rank / 64 TMA boxes of 16 rows
// x 128 bytes (128-byte swizzle) in a ring of stages, so ldmatrix reads are conflict-free and no thread computes
// addresses of cached rows; the stage of the previous tile is refilled once every warp has passed the current
// tile's first barrier. Per tile: partial scores S = Q' C^T (mma.sync; a warp takes half of the tokens and a
// quarter of the rank, its query fragments stay in registers), summed in shared memory in a fixed order; running
// maximum and sum in fp32 (exp2 domain); P rounded to bf16; O += P C (a warp per slice of the rank, C through
// ldmatrix.trans). Partial results are merged by a second kernel; a context that is one chunk is finished in
// place. Every mbarrier wait is bounded: on expiry the status word is raised and the kernel returns.
#include <cuda.h>

#include "common.cuh"
#include "logismos_kernels.h"
#include "tcgen05.cuh"

namespace {

using namespace lg;
using namespace lg::tc;

constexpr float kLog2e = 1.4426950408889634f;

constexpr int kBlockTokens = 16;
constexpr int kThreads = 256;

LG_DEVINL float redux_max(float x) {
  float y;
  asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;\n" : "=f"(y) : "f"(x));
  return y;
}

LG_DEVINL void store4(void* p, size_t i4, float4 v, bool f32) {
  if (f32) reinterpret_cast<float4*>(p)[i4] = v;
  else reinterpret_cast<uint2*>(p)[i4] = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

struct RotaryArgs {
  const float2* table;   // [positions][pairs], NULL: no rotated columns
  const int* pos;
  int at, pairs;         // first rotated column of the key/value row (a multiple of 4)
  float* gate;
  int n_gate, ld_gate;
};

// warp = (row, half): half 0 the query latent (columns 0 .. qw), half 1 the key/value latent (qw .. qw + rw)
__global__ void __launch_bounds__(kThreads)
latent_norm_store_kernel(float* __restrict__ raw, int ld, const float* __restrict__ gain_q, const float* __restrict__ gain_c,
                         void* __restrict__ cq, void* __restrict__ pool, const int64_t* __restrict__ slots, int rows, int qw, int q_n,
                         int rw, int r_n, float eps, int64_t n_pool_slots, int f32, int zero, RotaryArgs rot, int* __restrict__ status) {
  lg::pdl_prologue();
  const int id = (blockIdx.x * kThreads + threadIdx.x) >> 5, lane = threadIdx.x & 31;
  const int row = id >> 1, half = id & 1;
  if (row >= rows) return;
  float4* src = reinterpret_cast<float4*>(raw + (size_t)row * ld + (half ? qw : 0));
  const int all = (half ? rw : qw) >> 2, nv = half && rot.table ? rot.at >> 2 : all;  // float4s, and the normed ones of them
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
  if (half && rot.table) {
    const float2* angles = rot.table + (size_t)rot.pos[row] * rot.pairs;
    for (int v = nv + lane; v < all; v += 32) {
      const int i = 2 * (v - nv);
      const float4 a = src[v];
      const float2 c0 = i < rot.pairs ? __ldg(angles + i) : make_float2(0.f, 0.f), c1 = i + 1 < rot.pairs ? __ldg(angles + i + 1) : make_float2(0.f, 0.f);
      store4(out, dst + v, make_float4(a.x * c0.x - a.y * c0.y, a.y * c0.x + a.x * c0.y, a.z * c1.x - a.w * c1.y, a.w * c1.x + a.z * c1.y), f32 != 0);
      if (zero) src[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float* g = raw + (size_t)row * ld + qw + rw;
    for (int h = lane; h < rot.n_gate; h += 32) {
      rot.gate[(size_t)row * rot.ld_gate + h] = g[h];
      if (zero) g[h] = 0.0f;
    }
  }
  for (int v = lane; v < nv; v += 32) {
    const float4 a = src[v], g = __ldg(gain + v);
    store4(out, dst + v, make_float4(a.x * inv * g.x, a.y * inv * g.y, a.z * inv * g.z, a.w * inv * g.w), f32 != 0);
    if (zero) src[v] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
}

LG_DEVINL int round8(int v) { return (v + 7) & ~7; }

// rows of sequence s -> out[pstart[s] ..], every sequence starting at a multiple of 8 rows, padding and
// the rows after the last sequence zeroed up to tp. Grid (cache blocks, sequences); a warp copies two rows.
__global__ void __launch_bounds__(kThreads)
latent_gather_kernel(const __nv_bfloat16* __restrict__ pool, const int* __restrict__ tables, int max_blocks, int n_pool_blocks,
                     const int* __restrict__ kv_lens, __nv_bfloat16* __restrict__ out, int* __restrict__ pstart, int n_seqs, int tp,
                     int rw, int* __restrict__ status) {
  lg::pdl_prologue();
  const int tb = blockIdx.x, s = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int len = max(kv_lens[s], 0), plen = round8(len), cw = rw >> 3;
  const bool tail = tb == 0 && s == n_seqs - 1;
  if (tb * kBlockTokens >= plen && !tail && tb > 0) return;
  int p0 = 0;
  for (int i = lane; i < s; i += 32) p0 += round8(max(kv_lens[i], 0));
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) p0 += __shfl_xor_sync(0xffffffffu, p0, o);
  if (p0 + plen > tp) {
    if (threadIdx.x == 0 && status) atomicExch(status, 1);
    return;
  }
  if (tb == 0 && threadIdx.x == 0) pstart[s] = p0;
  if (tail)
    for (int64_t u = threadIdx.x; u < (int64_t)(tp - p0 - plen) * cw; u += kThreads)
      reinterpret_cast<uint4*>(out)[(size_t)(p0 + plen) * cw + u] = make_uint4(0u, 0u, 0u, 0u);
  const int blk = tb < max_blocks && tb * kBlockTokens < len ? __ldg(tables + (size_t)s * max_blocks + tb) : -1;
  const bool ok = blk >= 0 && blk < n_pool_blocks;
  if (!ok && tb * kBlockTokens < len && threadIdx.x == 0 && status) atomicExch(status, 1);
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = warp * 2 + h, t = tb * kBlockTokens + r;
    if (t >= plen) break;
    uint4* dst = reinterpret_cast<uint4*>(out) + (size_t)(p0 + t) * cw;
    const uint4* src = reinterpret_cast<const uint4*>(pool) + ((size_t)(ok ? blk : 0) * kBlockTokens + r) * cw;
    for (int c = lane; c < cw; c += 32) dst[c] = ok && t < len ? src[c] : make_uint4(0u, 0u, 0u, 0u);
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
  const float* gate;          // [rows, ld_gate], NULL: none
  int ld_gate;
  const float2* rot;          // [positions][rot_pairs], NULL: none
  int rot_at, rot_pairs;
  int* status;
};

// channels col, col + 1 of a query (col even), turned if they are a rotated pair
LG_DEVINL uint32_t rotate_pair(uint32_t u, int col, const DecodeArgs& p, int pos) {
  const int pr = (col - p.rot_at) >> 1;
  if (!p.rot || col < p.rot_at || pr >= p.rot_pairs) return u;
  const float2 x = unpack_bf16x2(u), cs = __ldg(p.rot + (size_t)pos * p.rot_pairs + pr);
  return pack_bf16x2(x.x * cs.x - x.y * cs.y, x.y * cs.x + x.x * cs.y);
}

LG_DEVINL float head_gate(const float* gate, size_t row, int ld, int head) { return gate ? 1.0f / (1.0f + __expf(-gate[row * ld + head])) : 1.0f; }

constexpr int kMaxStages = 4, kWarps = 8, kDecodeThreads = 32 * kWarps;

// shared memory besides the ring: query rows (when they do not stay in registers), partial scores, P, row state
template <int MT, int TK, bool QREG>
__host__ __device__ constexpr size_t decode_fixed_smem(int rank) {
  return (QREG ? 0 : (size_t)16 * MT * rank * 2) + (size_t)4 * 16 * MT * (TK + 8) * 4 + (size_t)16 * MT * (TK + 8) * 2 + (size_t)16 * MT * 3 * 4 +
         8 * (kMaxStages + 2) + 1024;
}

// MAXKS >= rank / 64: k16 steps of one rank quarter; also the 64-column slabs
template <int MT, int MAXKS, int TK, bool QREG>
__global__ void __launch_bounds__(kDecodeThreads, MT == 1 && MAXKS <= 8 ? 2 : 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap map_pool, DecodeArgs p, int stages) {
  lg::pdl_trigger();
  extern __shared__ uint8_t smem_raw[];
  constexpr int kRows = 16 * MT, NTS = TK / 16, kRowsPerWarp = kRows / kWarps;  // NTS: n8 tiles of a token half
  constexpr int MAXU = (MAXKS * 4 + kWarps - 1) / kWarps;     // 16-column units of the rank per warp
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* gen = smem_raw + (base - smem_u32(smem_raw));
  const int R = p.rank, slabs = R >> 6, tile_bytes = TK * R * 2;
  uint8_t* after = gen + (size_t)stages * tile_bytes;
  const uint32_t sq = smem_u32(after);                        // [kRows][R] swizzled, when !QREG
  float* s_part = reinterpret_cast<float*>(after + (QREG ? 0 : (size_t)kRows * R * 2));  // [4][kRows][TK + 8]
  __nv_bfloat16* s_p = reinterpret_cast<__nv_bfloat16*>(s_part + 4 * kRows * (TK + 8));   // [kRows][TK + 8]
  float* s_m = reinterpret_cast<float*>(s_p + kRows * (TK + 8));
  float* s_l = s_m + kRows;
  float* s_a = s_l + kRows;
  uint8_t* bars_gen = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(s_a + kRows) + 7) & ~(uintptr_t)7);
  const uint32_t bars = smem_u32(bars_gen);
  auto full_bar = [&](int i) { return bars + 8u * i; };
  volatile int* abort_flag = reinterpret_cast<volatile int*>(bars_gen + 8 * kMaxStages);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
  if (threadIdx.x == 0) {
    for (int i = 0; i < stages; ++i) mbar_init(full_bar(i), 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");
  }
  // Index arrays date from before the step's first kernel, and so do all cached rows but this step's new token
  // (the last of each context): both are read ahead of the dependency wait.
  const int chunk = blockIdx.x, h0 = blockIdx.y * kRows;
  int r = 0;  // chunk_offsets[r] <= chunk < chunk_offsets[r + 1]
  for (int i0 = 0; i0 < p.rows; i0 += kDecodeThreads) {
    const int i = i0 + threadIdx.x;
    r += __syncthreads_count(i < p.rows && __ldg(p.chunk_offsets + i + 1) <= chunk);
  }
  const int c0 = __ldg(p.chunk_offsets + r), c_idx = chunk - c0, c_cnt = __ldg(p.chunk_offsets + r + 1) - c0;
  const int ctx = __ldg(p.ctx + r);
  const int k0 = c_idx * p.chunk_tokens, k1 = min(ctx, k0 + p.chunk_tokens);
  const int tiles = (k1 - k0 + TK - 1) / TK;
  // Tile ti of the chunk into its stage (all warps, tiles in order): warp w copies the 64-column slabs w, w + 8, .. of the
  // rank, lane b the boxes of block b (boxes issued by one warp go out one after the other). Lane b holds the id of the
  // tile's block b, read one tile ahead.
  const int* table = p.tables + (size_t)r * p.max_blocks;
  auto block_id = [&](int ti) {
    const int bi = (k0 + ti * TK) / kBlockTokens + lane;
    return lane < TK / kBlockTokens && bi < p.max_blocks && bi * kBlockTokens < k1 ? __ldg(table + bi) : -1;
  };
  int ids = block_id(0);
  auto fetch = [&](int ti) {
    const int st = ti % stages, nb = min(TK, k1 - (k0 + ti * TK) + kBlockTokens - 1) / kBlockTokens;
    if (threadIdx.x == 0) mbar_expect_tx(full_bar(st), (uint32_t)(nb * kBlockTokens * R * 2));
    if (lane < nb) {
      if (ids < 0 || ids >= p.n_pool_blocks) {
        if (p.status) atomicExch(p.status, 1);
        ids = p.n_pool_blocks;  // beyond the pool: the copy fills zeros
      }
      for (int sl = warp; sl < slabs; sl += kWarps)
        tma_load_2d(base + (uint32_t)st * tile_bytes + (uint32_t)sl * (TK * 128) + (uint32_t)lane * (kBlockTokens * 128), &map_pool, full_bar(st), sl * 64,
                    ids * kBlockTokens);
    }
    __syncwarp();
    ids = block_id(ti + 1);
  };
  int fetched = 0;
  auto prefetch = [&](bool all) {
    while (fetched < stages && fetched < tiles && (all || k0 + (fetched + 1) * TK < ctx)) fetch(fetched++);
  };
  prefetch(false);
  lg::pdl_wait();
  prefetch(true);
  if (!QREG) {
    const int cw = R >> 3;
    for (int u = threadIdx.x; u < kRows * cw; u += kDecodeThreads) {
      const int hr = u / cw, ch = u % cw;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (h0 + hr < p.heads) v = *reinterpret_cast<const uint4*>(p.q + ((size_t)r * p.heads + h0 + hr) * R + ch * 8);
      if (p.rot && ch * 8 >= p.rot_at)
        v = make_uint4(rotate_pair(v.x, ch * 8, p, ctx - 1), rotate_pair(v.y, ch * 8 + 2, p, ctx - 1), rotate_pair(v.z, ch * 8 + 4, p, ctx - 1), rotate_pair(v.w, ch * 8 + 6, p, ctx - 1));
      *reinterpret_cast<uint4*>(after + (size_t)hr * R * 2 + ((ch ^ (hr & 7)) << 4)) = v;
    }
  }
  __syncthreads();

  {
    const int half = warp & 1, quarter = warp >> 1;
    // query fragments of this warp's rank quarter
    uint32_t qf[QREG ? MT : 1][QREG ? MAXKS : 1][4];
    if (QREG) {
#pragma unroll
      for (int i = 0; i < (QREG ? MT : 1); ++i)
#pragma unroll
        for (int ks = 0; ks < (QREG ? MAXKS : 1); ++ks) {
          const int col = (quarter * slabs + ks) * 16 + 2 * t4, ha = h0 + 16 * i + g;
          const __nv_bfloat16* q0 = p.q + ((size_t)r * p.heads + ha) * R + col;
          const bool in = ks < slabs;
          qf[i][ks][0] = in && ha < p.heads ? *reinterpret_cast<const uint32_t*>(q0) : 0u;
          qf[i][ks][1] = in && ha + 8 < p.heads ? *reinterpret_cast<const uint32_t*>(q0 + (size_t)8 * R) : 0u;
          qf[i][ks][2] = in && ha < p.heads ? *reinterpret_cast<const uint32_t*>(q0 + 8) : 0u;
          qf[i][ks][3] = in && ha + 8 < p.heads ? *reinterpret_cast<const uint32_t*>(q0 + (size_t)8 * R + 8) : 0u;
          if (p.rot && in && col + 8 >= p.rot_at) {
#pragma unroll
            for (int e = 0; e < 4; ++e) qf[i][ks][e] = rotate_pair(qf[i][ks][e], col + 8 * (e >> 1), p, ctx - 1);
          }
        }
    }
    const int units = slabs * 4, u_per = (units + kWarps - 1) / kWarps, u0 = warp * u_per, u_n = max(0, min(units - u0, u_per));
    float acc[MT][2 * MAXU][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < 2 * MAXU; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.0f;
    // softmax state of the rows warp, warp + 8, ..: the running maximum (the same in every lane) and this lane's share of
    // the sum (lane = token slot of a tile)
    float m_run[kRowsPerWarp], l_run[kRowsPerWarp];
#pragma unroll
    for (int rr = 0; rr < kRowsPerWarp; ++rr) { m_run[rr] = -1e30f; l_run[rr] = 0.0f; }

    // partial S = Q' C^T of tile ti over this warp's quarter of the rank, half of the tokens -> s_part
    auto scores = [&](int ti) {
      const int st = ti % stages;
      mbar_wait_warp(full_bar(st), (uint32_t)((ti / stages) & 1), abort_flag);  // a wait that expires sets the flag
      const uint32_t tile = base + (uint32_t)st * tile_bytes;
      float s[MT][NTS][4];
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NTS; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][j][e] = 0.0f;
#pragma unroll
      for (int ks = 0; ks < MAXKS; ++ks) {
        if (ks < slabs) {
          const int k16 = quarter * slabs + ks;
          uint32_t a[MT][4];
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            if (QREG) {
#pragma unroll
              for (int e = 0; e < 4; ++e) a[i][e] = qf[QREG ? i : 0][QREG ? ks : 0][e];
            } else {
              const int mat = lane >> 3, row = 16 * i + (lane & 7) + 8 * (mat & 1);
              ldmatrix_x4(a[i], sq + (uint32_t)row * R * 2 + (uint32_t)(((2 * k16 + (mat >> 1)) ^ (row & 7)) << 4));
            }
          }
#pragma unroll
          for (int j = 0; j < NTS; j += 2) {
            const int key = half * (TK / 2) + 8 * (j + (lane >> 4)) + (lane & 7);
            const int ch = 2 * (k16 & 3) + ((lane >> 3) & 1);
            uint32_t b[4];
            ldmatrix_x4(b, tile + (uint32_t)(k16 >> 2) * (TK * 128) + (uint32_t)key * 128 + (uint32_t)((ch ^ (key & 7)) << 4));
            const uint32_t b0[2] = {b[0], b[1]}, b1[2] = {b[2], b[3]};
#pragma unroll
            for (int i = 0; i < MT; ++i) {
              mma_bf16_16816(s[i][j], a[i], b0, s[i][j]);
              mma_bf16_16816(s[i][j + 1], a[i], b1, s[i][j + 1]);
            }
          }
        }
      }
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int j = 0; j < NTS; ++j) {
          float* d = s_part + ((size_t)quarter * kRows + 16 * i + g) * (TK + 8) + half * (TK / 2) + 8 * j + 2 * t4;
          *reinterpret_cast<float2*>(d) = make_float2(s[i][j][0], s[i][j][1]);
          *reinterpret_cast<float2*>(d + 8 * (TK + 8)) = make_float2(s[i][j][2], s[i][j][3]);
        }
    };

    bool ok = true;
    scores(0);
    for (int ti = 0; ti < tiles; ++ti) {
      __syncthreads();
      if (*abort_flag) ok = false;  // set before this barrier or not at all until the next one: the same for every warp
      if (ti > 0 && ti - 1 + stages < tiles) fetch(ti - 1 + stages);
      // running maximum and sum; a tile always holds at least one visible key, so the maximum is a real score
      const int first = k0 + ti * TK;
#pragma unroll
      for (int rr = 0; rr < kRowsPerWarp; ++rr) {
        const int row = warp + kWarps * rr;
        float v[TK / 32];
        float mx = -1e30f;
#pragma unroll
        for (int e = 0; e < TK / 32; ++e) {
          const float* d = s_part + (size_t)row * (TK + 8) + 32 * e + lane;
          const float x = (d[0] + d[kRows * (TK + 8)]) + (d[2 * kRows * (TK + 8)] + d[3 * kRows * (TK + 8)]);
          v[e] = first + 32 * e + lane < k1 ? x * p.sl2 : -1e30f;
          mx = fmaxf(mx, v[e]);
        }
        const float m_new = fmaxf(m_run[rr], redux_max(mx)), alpha = fast_exp2(m_run[rr] - m_new);
        m_run[rr] = m_new;
        l_run[rr] *= alpha;
#pragma unroll
        for (int e = 0; e < TK / 32; ++e) {
          const float x = fast_exp2(v[e] - m_new);
          l_run[rr] += x;
          s_p[row * (TK + 8) + 32 * e + lane] = __float2bfloat16_rn(x);
        }
        if (lane == 0) s_a[row] = alpha;
      }
      __syncthreads();
      // the next tile's scores and this tile's O = O * alpha + P C are independent; cache blocks past the end of the
      // chunk were not fetched and are skipped
      if (ti + 1 < tiles) scores(ti + 1);
      const uint32_t tile = base + (uint32_t)(ti % stages) * tile_bytes;
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const float a0 = s_a[16 * i + g], a1 = s_a[16 * i + g + 8];
        if (__any_sync(0xffffffffu, a0 != 1.0f || a1 != 1.0f)) {
#pragma unroll
          for (int j = 0; j < 2 * MAXU; ++j) { acc[i][j][0] *= a0; acc[i][j][1] *= a0; acc[i][j][2] *= a1; acc[i][j][3] *= a1; }
        }
      }
      const int nb = min(TK, k1 - first + kBlockTokens - 1) / kBlockTokens;
#pragma unroll
      for (int ks = 0; ks < TK / 16; ++ks) {
        if (ks < nb) {
          uint32_t pa[MT][4];
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            const int mat = lane >> 3, row = 16 * i + (lane & 7) + 8 * (mat & 1);
            ldmatrix_x4(pa[i], smem_u32(s_p) + (uint32_t)(row * (TK + 8) + 16 * ks + 8 * (mat >> 1)) * 2);
          }
          const int key = 16 * ks + (lane & 7) + 8 * ((lane >> 3) & 1);
#pragma unroll
          for (int j = 0; j < MAXU; ++j) {
            if (j < u_n) {
              const int u = u0 + j, ch = 2 * (u & 3) + (lane >> 4);
              uint32_t b[4];
              ldmatrix_x4_trans(b, tile + (uint32_t)(u >> 2) * (TK * 128) + (uint32_t)key * 128 + (uint32_t)((ch ^ (key & 7)) << 4));
              const uint32_t b0[2] = {b[0], b[1]}, b1[2] = {b[2], b[3]};
#pragma unroll
              for (int i = 0; i < MT; ++i) {
                mma_bf16_16816(acc[i][2 * j], pa[i], b0, acc[i][2 * j]);
                mma_bf16_16816(acc[i][2 * j + 1], pa[i], b1, acc[i][2 * j + 1]);
              }
            }
          }
        }
      }
      if (!ok) break;
    }
#pragma unroll
    for (int rr = 0; rr < kRowsPerWarp; ++rr) {
      const float l = warp_sum(l_run[rr]);
      if (lane == 0) { s_m[warp + kWarps * rr] = m_run[rr]; s_l[warp + kWarps * rr] = l; }
    }
    __syncthreads();
    if (ok) {
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int hr = 16 * i + g + 8 * hh, h = h0 + hr;
          if (h >= p.heads) continue;
          const float inv = c_cnt == 1 ? head_gate(p.gate, r, p.ld_gate, h) / s_l[hr] : 0.0f;
#pragma unroll
          for (int j = 0; j < 2 * MAXU; ++j) {
            if ((j >> 1) >= u_n) continue;
            const int col = (u0 + (j >> 1)) * 16 + (j & 1) * 8 + 2 * t4;
            const float x = acc[i][j][2 * hh], y = acc[i][j][2 * hh + 1];
            if (c_cnt == 1)
              *reinterpret_cast<uint32_t*>(p.out + ((size_t)r * p.heads + h) * R + col) = pack_bf16x2(x * inv, y * inv);
            else
              *reinterpret_cast<float2*>(p.part_o + ((size_t)chunk * p.heads + h) * R + col) = make_float2(x, y);
          }
          if (c_cnt > 1 && warp == 0 && t4 == 0) p.part_ml[(size_t)chunk * p.heads + h] = make_float2(s_m[hr], s_l[hr]);
        }
    }
  }
  __syncthreads();
  if (*abort_flag) {
    // a wait expired: give copies that may still be in flight time to land before the shared memory is released
    for (int i = 0; i < 2000; ++i) __nanosleep(1000);
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, 2 | (4 << 8));
  }
}

// CTA = (row, head): the chunks of a context that was split. Their weights are computed by all threads at once, the rows
// are then summed with several loads in flight.
constexpr int kMergeTile = 256;
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part_o, const float2* __restrict__ part_ml, const int* __restrict__ chunk_offsets,
                    __nv_bfloat16* __restrict__ out, int heads, int rank, const float* __restrict__ gate, int ld_gate) {
  lg::pdl_prologue();
  __shared__ float red[32], w[kMergeTile];
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x;
  const int c0 = chunk_offsets[r], c1 = chunk_offsets[r + 1];
  if (c1 - c0 <= 1) return;
  float m = -1e30f;
  for (int c = c0 + tid; c < c1; c += 128) m = fmaxf(m, part_ml[(size_t)c * heads + h].x);
  m = block_max(m, red);
  float l = 0.0f;
  float4 acc[2] = {make_float4(0.f, 0.f, 0.f, 0.f), make_float4(0.f, 0.f, 0.f, 0.f)};  // rank <= 1024: two float4 per thread
  for (int cb = c0; cb < c1; cb += kMergeTile) {
    const int n = min(kMergeTile, c1 - cb);
    __syncthreads();
    for (int c = tid; c < n; c += 128) {
      const float2 ml = part_ml[(size_t)(cb + c) * heads + h];
      w[c] = exp2f(ml.x - m);
      l += ml.y * w[c];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int v = tid + i * 128;
      if (v >= rank / 4) continue;
      const float4* src = reinterpret_cast<const float4*>(part_o + ((size_t)cb * heads + h) * rank) + v;
      const size_t step = (size_t)heads * rank / 4;
#pragma unroll 8
      for (int c = 0; c < n; ++c) {
        const float4 o = src[c * step];
        acc[i].x = fmaf(w[c], o.x, acc[i].x); acc[i].y = fmaf(w[c], o.y, acc[i].y);
        acc[i].z = fmaf(w[c], o.z, acc[i].z); acc[i].w = fmaf(w[c], o.w, acc[i].w);
      }
    }
  }
  const float inv = head_gate(gate, r, ld_gate, h) / block_sum(l, red);
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int v = tid + i * 128;
    if (v < rank / 4) store4(out, ((size_t)r * heads + h) * (rank / 4) + v, make_float4(acc[i].x * inv, acc[i].y * inv, acc[i].z * inv, acc[i].w * inv), false);
  }
}

// fp32 form: CTA = (query row, head), any row of the step; row t of sequence seq_ids[t] sees keys 0 .. pos[t]
constexpr int kF32Tile = 64;
__global__ void __launch_bounds__(128)
latent_attention_f32_kernel(const float* __restrict__ q, const float* __restrict__ pool, const int* __restrict__ tables, int max_blocks,
                            int n_pool_blocks, const int* __restrict__ seq_ids, const int* __restrict__ pos, float* __restrict__ out,
                            int heads, int rank, float sl2, const float* __restrict__ gate, int ld_gate, int* __restrict__ status) {
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
  const float inv = (gate ? 1.0f / (1.0f + expf(-gate[(size_t)t * ld_gate + h])) : 1.0f) / l;
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (tid + i * 128 < rank) out[row + tid + i * 128] = acc[i] * inv;
}

}  // namespace

extern "C" {

uint32_t logismos_launch_latent_norm_store(void* raw_f32, int32_t ld, const void* gain_q_f32, const void* gain_c_f32, void* q_latent,
                                           void* pool, const void* slot_mapping_i64, int32_t rows, int32_t q_width, int32_t q_n,
                                           int32_t c_width, int32_t c_n, float eps, int64_t n_pool_slots, int32_t is_f32,
                                           int32_t zero_raw, const lg_latent_rotary_t* rotary, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (rotary && (!rotary->table || !rotary->positions || rotary->at <= 0 || rotary->at % 4 || c_n > rotary->at || rotary->dims <= 0 || rotary->dims % 2 ||
                 rotary->at + rotary->dims > c_width || rotary->n_gate < 0 || (rotary->n_gate && (!rotary->gate || rotary->ld_gate < rotary->n_gate)) ||
                 ld < q_width + c_width + rotary->n_gate || ((uintptr_t)rotary->table & 7)))
    return lg::kInvalidValue;
  const RotaryArgs rot = rotary ? RotaryArgs{(const float2*)rotary->table, (const int*)rotary->positions, rotary->at, rotary->dims / 2, (float*)rotary->gate, rotary->n_gate,
                                             rotary->ld_gate}
                                : RotaryArgs{};
  if (!raw_f32 || rows <= 0 || q_width <= 0 || c_width <= 0 || (q_width % 4) || (c_width % 4) || q_n <= 0 || q_n > q_width || c_n <= 0 ||
      c_n > c_width || ld < q_width + c_width || (ld % 4) || rows > 0x3fffffff)
    return lg::kInvalidValue;
  const int64_t blocks = ((int64_t)rows * 2 + kThreads / 32 - 1) / (kThreads / 32);
  lg::launch(latent_norm_store_kernel, dim3((unsigned)blocks), dim3(kThreads), 0, (cudaStream_t)stream, (float*)raw_f32, ld,
             (const float*)gain_q_f32, (const float*)gain_c_f32, q_latent, pool, (const int64_t*)slot_mapping_i64, rows, q_width, q_n,
             c_width, c_n, eps, n_pool_slots, is_f32, zero_raw, rot, (int*)status_i32);
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
  lg::launch(latent_gather_kernel, dim3((unsigned)((max_kv_len + kBlockTokens - 1) / kBlockTokens), (unsigned)n_seqs), dim3(kThreads), 0, (cudaStream_t)stream,
             (const __nv_bfloat16*)pool, (const int*)block_tables_i32, max_blocks, n_pool_blocks, (const int*)kv_lens_i32, (__nv_bfloat16*)out,
             (int*)kv_start_i32, n_seqs, logismos_latent_gather_rows(total_kv_tokens, n_seqs), width, (int*)status_i32);
  return lg::launch_status();
}

// Chunk length by an estimate in token times: full chunks run in waves over the CTA slots (one CTA per SM, two with few
// heads), the remainders of the contexts fit the last wave's idle slots or take further waves; a chunk costs a start and a merge share.
int32_t logismos_pick_latent_chunk(const int32_t* context_lens, int32_t n_seqs, int32_t heads) {
  static const int32_t cands[] = {128, 192, 256, 320, 384, 448, 512, 640, 768, 896, 1024, 1280, 1536, 1792, 2048, 3072, 4096, 8192, 16384, 1 << 20};
  const int64_t groups = (heads + 63) / 64, slots = heads <= 16 ? 296 : 148, start = 96;
  int32_t best = 0;
  int64_t best_cost = 0;
  for (int32_t c : cands) {
    int64_t full = 0, parts = 0, longest = 0;
    for (int32_t i = 0; i < n_seqs; ++i) {
      const int32_t f = context_lens[i] / c, r = context_lens[i] - f * c;
      full += f;
      parts += r > 0;
      if (r > longest) longest = r;
    }
    if (full + parts > logismos_latent_max_chunks(n_seqs)) continue;
    const int64_t waves = (full * groups + slots - 1) / slots, all_waves = ((full + parts) * groups + slots - 1) / slots;
    int64_t cost = waves * (c + start) + (all_waves - waves) * (longest + start);
    cost += (full + parts) * 16 / slots;
    if (best == 0 || cost < best_cost) { best = c; best_cost = cost; }
  }
  return best > 0 ? best : 1 << 20;
}

int32_t logismos_latent_max_chunks(int32_t max_rows) { return max_rows + 1200; }

size_t logismos_latent_decode_scratch_bytes(int32_t total_chunks, int32_t heads, int32_t rank) {
  if (total_chunks < 0 || heads <= 0 || rank <= 0) return 0;
  return (size_t)total_chunks * heads * ((size_t)rank + 2) * 4;
}

uint32_t logismos_launch_latent_decode_bf16(const void* q, const void* pool, const void* block_tables_i32, const void* context_lens_i32,
                                            const void* chunk_offsets_i32, void* out, void* scratch, int32_t rows, int32_t total_chunks,
                                            int32_t chunk_tokens, int32_t max_blocks, int32_t n_pool_blocks, int32_t heads, int32_t rank,
                                            float scale, const void* gate_f32, int32_t ld_gate, const void* rot_table, int32_t rot_at, int32_t rot_dims,
                                            void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if ((gate_f32 && ld_gate < heads) || (rot_table && (rot_at < 0 || rot_at % 8 || rot_dims <= 0 || rot_dims % 2 || rot_at + rot_dims > rank || ((uintptr_t)rot_table & 7))) || !q || !pool || !out || !scratch || rows <= 0 || rows > 65535 || total_chunks < rows || chunk_tokens <= 0 || (chunk_tokens % 64) || max_blocks <= 0 ||
      n_pool_blocks <= 0 || heads <= 0 || rank <= 0 || (rank % 64) || rank > 1024 || (int64_t)n_pool_blocks * kBlockTokens > 0x7fffffff - 64 ||
      (((uintptr_t)q | (uintptr_t)pool | (uintptr_t)out | (uintptr_t)scratch) & 15))
    return lg::kInvalidValue;
  cudaStream_t s = (cudaStream_t)stream;
  DecodeArgs p{(const __nv_bfloat16*)q, (const __nv_bfloat16*)pool, (const int*)block_tables_i32, (const int*)context_lens_i32,
               (const int*)chunk_offsets_i32, (__nv_bfloat16*)out, (float*)scratch, nullptr, rows, heads, rank, chunk_tokens, max_blocks,
               n_pool_blocks, scale * kLog2e, (const float*)gate_f32, ld_gate, (const float2*)rot_table, rot_at, rot_dims / 2, (int*)status_i32};
  p.part_ml = (float2*)(p.part_o + (size_t)total_chunks * heads * rank);
  CUtensorMap map;
  if (!make_map(&map, pool, (uint64_t)n_pool_blocks * kBlockTokens, (uint64_t)rank, (uint64_t)rank, kBlockTokens)) return lg::kInvalidValue;
  // stages: up to four, within what lets the kernel's CTAs share an SM (per_sm)
  auto go = [&](auto kern, int mt, int tk, size_t fixed, int per_sm) -> uint32_t {
    const size_t tile = (size_t)tk * rank * 2, room = (size_t)(227 / per_sm) * 1024 - (per_sm > 1 ? 1024 : 0);
    int stages = kMaxStages;
    while (stages > 2 && fixed + stages * tile > room) --stages;
    const size_t smem = fixed + stages * tile;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
    lg::launch(kern, dim3((unsigned)total_chunks, (unsigned)((heads + 16 * mt - 1) / (16 * mt))), dim3(kDecodeThreads), smem, s, map, p, stages);
    return lg::launch_status();
  };
  uint32_t rc;
#define LG_DECODE(MT, KS, TK, QREG) go(latent_decode_kernel<MT, KS, TK, QREG>, MT, TK, decode_fixed_smem<MT, TK, QREG>(rank), MT == 1 && KS <= 8 ? 2 : 1)
  if (rank <= 128) rc = heads <= 16 ? LG_DECODE(1, 2, 64, true) : heads <= 32 ? LG_DECODE(2, 2, 64, true) : LG_DECODE(4, 2, 64, true);
  else if (rank <= 256) rc = heads <= 16 ? LG_DECODE(1, 4, 64, true) : heads <= 32 ? LG_DECODE(2, 4, 64, true) : LG_DECODE(4, 4, 64, true);
  else if (rank <= 512) rc = heads <= 16 ? LG_DECODE(1, 8, 32, true) : heads <= 32 ? LG_DECODE(2, 8, 64, true) : LG_DECODE(4, 8, 32, false);
  else if (rank <= 640) rc = heads <= 16 ? LG_DECODE(1, 10, 32, true) : heads <= 32 ? LG_DECODE(2, 10, 32, true) : LG_DECODE(4, 10, 32, false);
  else rc = heads <= 16 ? LG_DECODE(1, 16, 32, true) : LG_DECODE(2, 16, 32, false);
#undef LG_DECODE
  if (rc || total_chunks == rows) return rc;
  // an ordinary launch: with the early one the next projection's CTAs moved in ahead of these and a decode step of 8
  // sequences took 1.86 instead of 1.42 ms
  lg::launch_ordered(latent_merge_kernel, dim3((unsigned)heads, (unsigned)rows), dim3(128), 0, s, (const float*)p.part_o, (const float2*)p.part_ml,
             p.chunk_offsets, p.out, heads, rank, p.gate, ld_gate);
  return lg::launch_status();
}

uint32_t logismos_launch_latent_attention_f32(const void* q_f32, const void* pool_f32, const void* block_tables_i32, const void* seq_ids_i32,
                                              const void* positions_i32, void* out_f32, int32_t rows, int32_t max_blocks,
                                              int32_t n_pool_blocks, int32_t heads, int32_t rank, float scale, const void* gate_f32,
                                              int32_t ld_gate, void* status_i32, void* stream) {
  lg::LaunchScope launch_scope_;
  if ((gate_f32 && ld_gate < heads) || !q_f32 || !pool_f32 || !out_f32 || rows <= 0 || max_blocks <= 0 || n_pool_blocks <= 0 || heads <= 0 || heads > 65535 || rank <= 0 || rank > 1024)
    return lg::kInvalidValue;
  lg::launch(latent_attention_f32_kernel, dim3((unsigned)rows, (unsigned)heads), dim3(128), (size_t)(rank + kF32Tile) * 4, (cudaStream_t)stream,
             (const float*)q_f32, (const float*)pool_f32, (const int*)block_tables_i32, max_blocks, n_pool_blocks, (const int*)seq_ids_i32,
             (const int*)positions_i32, (float*)out_f32, heads, rank, scale * kLog2e, (const float*)gate_f32, ld_gate, (int*)status_i32);
  return lg::launch_status();
}

}  // extern "C"
