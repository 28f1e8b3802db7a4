// C = A W^T for few rows and bf16 weights (decode steps): the weights are streamed once, straight from
// global memory into mma.sync fragments. Also the batched form (one small matrix per head) and the
// fp32-activation form of the same contract.
//
// linear_small_kernel: CTA = 16 * MT weight rows x up to 8 * NT activation rows, its warps split k in
// steps of 32. A lane reads 16 consecutive bytes (8 values along k) of weight rows g and g + 8 and of
// activation row g (g = lane / 4): the k order inside a 32-wide step is permuted the same way on both
// sides, so each 16-byte read feeds two m16n8k16 instructions without any shuffle. The partial sums of
// the warps meet in shared memory in a fixed order, so results do not depend on timing.
#include "common.cuh"
#include "logismos_kernels.h"

namespace {

using namespace lg;

struct SmallArgs {
  const __nv_bfloat16* a;
  const __nv_bfloat16* w;
  const float* bias;
  void* out;
  int m, n, k, lda, ldc, epi;
  int64_t a_stride, w_stride, out_stride;  // per batch entry (elements)
  float p0, p1, p2;
  lg_linear_groups_t groups;               // with kEpiGroups
  const int* offsets;                      // EXPERTS: batch entry b has the output rows offsets[b] .. offsets[b + 1]
  const int* row_idx;                      // and reads these input rows (NULL: the same)
  // kEpiTanhNorm: out is the residual stream
  float post_alpha, next_alpha;
  const float *post_w, *post_b, *next_w, *next_b;
  void* h;
};

// internal epilogue of the grouped projections (lg_linear_groups_t): main columns, then an fp32 tail
constexpr int kEpiGroups = 6;
// an output projection with the norms around the residual (lg_tanh_norm_t)
constexpr int kEpiTanhNorm = 7;

// activation copy of a block of columns starting at c
LG_DEVINL int group_of(const lg_linear_groups_t& g, int c) {
  int i = 0;
#pragma unroll
  for (int j = 0; j < LG_MAX_LINEAR_GROUPS - 1; ++j) i += (j + 1 < g.n_groups && c >= g.end[j]) ? 1 : 0;
  return i;
}

LG_DEVINL uint4 ldg16(const void* p) { return __ldg(reinterpret_cast<const uint4*>(p)); }

template <int MT, int NT, bool EXPERTS = false>
__global__ void __launch_bounds__(512)
linear_small_kernel(SmallArgs p) {
  lg::pdl_trigger();
  int first = 0;
  if (EXPERTS) {  // which rows a matrix has is the work of a kernel of this step
    lg::pdl_wait();
    first = p.offsets[blockIdx.z];
    p.m = p.offsets[blockIdx.z + 1] - first;
    if ((int)blockIdx.y * 8 * NT >= p.m) return;
  }
  constexpr int kUnroll = MT * NT >= 8 ? 2 : 4;
  extern __shared__ float red[];  // [warps][16 * MT][8 * NT]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const int g = lane >> 2, t = lane & 3;
  const bool glu = p.epi == LG_EPI_SWIGLU || p.epi == LG_EPI_GLU_CLAMP;
  // first weight row of each m16 tile: gated epilogues take 16 gate rows and the 16 matching up rows
  // (rows interleave in blocks of 32), the others consecutive rows
  int row0[MT];
  if (glu) {
    const int u = blockIdx.x;  // MT == 2
    row0[0] = (u >> 1) * 64 + (u & 1) * 16;
    if (MT == 2) row0[MT - 1] = row0[0] + 32;
  } else {
#pragma unroll
    for (int i = 0; i < MT; ++i) row0[i] = (blockIdx.x * MT + i) * 16;
  }
  const int m0 = blockIdx.y * 8 * NT;
  const __nv_bfloat16* wb = p.w + (size_t)blockIdx.z * p.w_stride;
  const __nv_bfloat16* ab = p.a + (size_t)blockIdx.z * p.a_stride + (p.epi == kEpiGroups ? (size_t)group_of(p.groups, row0[0]) * p.m * p.lda : 0);
  const __nv_bfloat16* wr[MT][2];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int h = 0; h < 2; ++h) wr[i][h] = wb + (size_t)min(row0[i] + g + 8 * h, p.n - 1) * p.k + 8 * t;
  const int steps = p.k >> 5;
  float acc[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.0f;
  uint4 wv[kUnroll][MT][2];
  auto load_w = [&](int s0) {
#pragma unroll
    for (int u = 0; u < kUnroll; ++u) {
      const int s = s0 + u * n_warps;
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) wv[u][i][h] = s < steps ? ldg16(wr[i][h] + (size_t)s * 32) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  load_w(warp);      // the weights are static: requested before the dependency wait
  if (!EXPERTS) lg::pdl_wait();
  int src[NT];       // EXPERTS: input rows of this lane
  if (EXPERTS) {
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int r = m0 + 8 * j + g;
      src[j] = r < p.m ? (p.row_idx ? p.row_idx[first + r] : first + r) : 0;
    }
  }
  for (int s0 = warp; s0 < steps; s0 += kUnroll * n_warps) {
#pragma unroll
    for (int u = 0; u < kUnroll; ++u) {
      const int s = s0 + u * n_warps;
      if (s < steps) {
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int r = m0 + 8 * j + g;
          uint4 x = make_uint4(0u, 0u, 0u, 0u);
          if (r < p.m) x = *reinterpret_cast<const uint4*>(ab + (size_t)(EXPERTS ? src[j] : r) * p.lda + (size_t)s * 32 + 8 * t);
          const uint32_t b0[2] = {x.x, x.y}, b1[2] = {x.z, x.w};
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            const uint4 lo = wv[u][i][0], hi = wv[u][i][1];
            const uint32_t a0[4] = {lo.x, hi.x, lo.y, hi.y}, a1[4] = {lo.z, hi.z, lo.w, hi.w};
            mma_bf16_16816(acc[i][j], a0, b0, acc[i][j]);
            mma_bf16_16816(acc[i][j], a1, b1, acc[i][j]);
          }
        }
      }
    }
    if (s0 + kUnroll * n_warps < steps) load_w(s0 + kUnroll * n_warps);
  }
  // acc[i][j]: weight rows g, g + 8 of tile i; activation rows 8 j + 2 t, + 1
  constexpr int kRows = 16 * MT, kCols = 8 * NT;
  float* mine = red + (size_t)warp * kRows * kCols;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      mine[(8 * j + 2 * t) * kRows + 16 * i + g] = acc[i][j][0];
      mine[(8 * j + 2 * t + 1) * kRows + 16 * i + g] = acc[i][j][1];
      mine[(8 * j + 2 * t) * kRows + 16 * i + g + 8] = acc[i][j][2];
      mine[(8 * j + 2 * t + 1) * kRows + 16 * i + g + 8] = acc[i][j][3];
    }
  __syncthreads();
  const int out_rows = glu ? 16 : kRows;  // output columns this CTA produces
  if (EXPERTS) p.out = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)first * p.ldc;
  for (int e = threadIdx.x; e < out_rows * kCols; e += blockDim.x) {
    const int c = e % out_rows, r = m0 + e / out_rows;
    if (r >= p.m) continue;
    float v = 0.0f, u = 0.0f;
    for (int w = 0; w < n_warps; ++w) {
      const float* q = red + ((size_t)w * kCols + e / out_rows) * kRows;
      v += q[c];
      if (glu) u += q[c + 16];
    }
    const int wrow = row0[0] + c;  // consecutive rows across the MT tiles when not gated
    if (wrow >= p.n) continue;
    if (glu) {
      if (p.bias) { v += p.bias[wrow]; u += p.bias[wrow + 32]; }
      const float y = p.epi == LG_EPI_GLU_CLAMP ? glu_clamp(v, u, p.p0, p.p1, p.p2) : v / (1.0f + __expf(-v)) * u;
      const int oc = (wrow >> 6) * 32 + (wrow & 31);
      reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)blockIdx.z * p.out_stride + (size_t)r * p.ldc + oc] = __float2bfloat16_rn(y);
      continue;
    }
    if (p.bias && (p.epi != kEpiGroups || wrow < p.groups.n_main)) v += p.bias[wrow];
    if (p.epi == LG_EPI_RELU2) { v = fmaxf(v, 0.0f); v *= v; }
    if (p.epi == kEpiGroups && wrow >= p.groups.silu_begin && wrow < p.groups.silu_end) v = silu_fast(v);
    if (p.epi == kEpiGroups && wrow >= p.groups.n_main) {
      const int tc = wrow - p.groups.n_main, width = p.n - p.groups.n_main;
      if (p.groups.tail_cap > 0.0f) v = p.groups.tail_cap * tanhf(v / p.groups.tail_cap);
      reinterpret_cast<float*>(p.groups.tail)[(size_t)r * p.groups.ld_tail + tc] = v;
      if (p.groups.tail_parts) {
        __nv_bfloat16* parts = reinterpret_cast<__nv_bfloat16*>(p.groups.tail_parts) + (size_t)r * 2 * width + tc;
        parts[0] = __float2bfloat16_rn(v);
        parts[width] = __float2bfloat16_rn(v - __bfloat162float(parts[0]));
      }
      continue;
    }
    const size_t o = (size_t)blockIdx.z * p.out_stride + (size_t)r * p.ldc + wrow;
    if (p.epi == kEpiTanhNorm) {
      float* xs = reinterpret_cast<float*>(p.out) + o;
      const float x = *xs + fmaf(tanhf(p.post_alpha * v), __ldg(p.post_w + wrow), __ldg(p.post_b + wrow));
      *xs = x;
      if (p.next_w) reinterpret_cast<__nv_bfloat16*>(p.h)[o] = __float2bfloat16_rn(fmaf(tanhf(p.next_alpha * x), __ldg(p.next_w + wrow), __ldg(p.next_b + wrow)));
      continue;
    }
    if (p.epi == LG_EPI_BF16 || p.epi == LG_EPI_RELU2 || p.epi == kEpiGroups) reinterpret_cast<__nv_bfloat16*>(p.out)[o] = __float2bfloat16_rn(v);
    else if (p.epi == LG_EPI_RESID_F32) reinterpret_cast<float*>(p.out)[o] += v;
    else reinterpret_cast<float*>(p.out)[o] = p.p0 > 0.0f ? p.p0 * tanhf(v / p.p0) : v;
  }
}

template <int MT, int NT>
uint32_t launch_small(const SmallArgs& a, int batch, int warps, cudaStream_t s) {
  const bool glu = a.epi == LG_EPI_SWIGLU || a.epi == LG_EPI_GLU_CLAMP;
  const size_t smem = (size_t)warps * 16 * MT * 8 * NT * 4;
  auto kern = linear_small_kernel<MT, NT>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
  }
  const int tiles = glu ? a.n / 32 : (a.n + 16 * MT - 1) / (16 * MT);
  lg::launch(kern, dim3((unsigned)tiles, (unsigned)((a.m + 8 * NT - 1) / (8 * NT)), (unsigned)batch), dim3(32 * warps), smem, s, a);
  return lg::launch_status();
}

template <int NT>
uint32_t launch_small_experts(const SmallArgs& a, int n_groups, int max_rows, int warps, cudaStream_t s) {
  const bool glu = a.epi == LG_EPI_SWIGLU || a.epi == LG_EPI_GLU_CLAMP;
  const size_t smem = (size_t)warps * 32 * 8 * NT * 4;
  auto kern = linear_small_kernel<2, NT, true>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
  }
  const int tiles = glu ? a.n / 32 : (a.n + 31) / 32;
  lg::launch(kern, dim3((unsigned)tiles, (unsigned)((max_rows + 8 * NT - 1) / (8 * NT)), (unsigned)n_groups), dim3(32 * warps), smem, s, a);
  return lg::launch_status();
}

// ---- fp32 activations -----------------------------------------------------------------------------
// 64 x 64 tile, 256 threads, 4 x 4 outputs per thread: rows 4 ty .. + 3; columns 2 tx, 2 tx + 1 and the
// same + 32, so that a thread holds a gate column and its matching up column. fp32 products and sums.
struct F32Args {
  const float* a;
  const __nv_bfloat16* w;
  const float* bias;
  float* out;
  int m, n, k, lda, ldc, epi;
  int64_t a_stride, w_stride, out_stride;
  float p0, p1, p2;
  lg_linear_groups_t groups;
  const int* offsets;      // as for SmallArgs (NULL: one range of rows)
  const int* row_idx;
};

__global__ void __launch_bounds__(256)
linear_f32_kernel(F32Args p) {
  lg::pdl_prologue();
  __shared__ float as[16][68], ws[16][68];
  int first = 0;
  if (p.offsets) {
    first = p.offsets[blockIdx.z];
    p.m = p.offsets[blockIdx.z + 1] - first;
    if ((int)blockIdx.y * 64 >= p.m) return;
  }
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int n0 = blockIdx.x * 64, m0 = blockIdx.y * 64;
  const float* A = p.a + (size_t)blockIdx.z * p.a_stride + (p.epi == kEpiGroups ? (size_t)group_of(p.groups, n0) * p.m * p.lda : 0);
  const __nv_bfloat16* W = p.w + (size_t)blockIdx.z * p.w_stride;
  float acc[4][4] = {};
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  int a_row = m0 + lr;
  if (p.offsets && a_row < p.m) a_row = p.row_idx ? p.row_idx[first + a_row] : first + a_row;
  for (int k0 = 0; k0 < p.k; k0 += 16) {
    float4 av = make_float4(0.f, 0.f, 0.f, 0.f);
    if (m0 + lr < p.m) av = *reinterpret_cast<const float4*>(A + (size_t)a_row * p.lda + k0 + lk);
    float wv[4] = {0.f, 0.f, 0.f, 0.f};
    if (n0 + lr < p.n) {
      const uint2 u = __ldg(reinterpret_cast<const uint2*>(W + (size_t)(n0 + lr) * p.k + k0 + lk));
      const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
      wv[0] = a.x; wv[1] = a.y; wv[2] = b.x; wv[3] = b.y;
    }
    as[lk][lr] = av.x; as[lk + 1][lr] = av.y; as[lk + 2][lr] = av.z; as[lk + 3][lr] = av.w;
#pragma unroll
    for (int i = 0; i < 4; ++i) ws[lk + i][lr] = wv[i];
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 16; ++kk) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i] = as[kk][4 * ty + i];
      y[0] = ws[kk][2 * tx]; y[1] = ws[kk][2 * tx + 1]; y[2] = ws[kk][32 + 2 * tx]; y[3] = ws[kk][33 + 2 * tx];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
  float* out = p.out + (size_t)blockIdx.z * p.out_stride + (size_t)first * p.ldc;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = m0 + 4 * ty + i;
    if (r >= p.m) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + (j >> 1) * 32 + 2 * tx + (j & 1);
      if (c < p.n && p.bias && (p.epi != kEpiGroups || c < p.groups.n_main)) acc[i][j] += p.bias[c];
    }
    if (p.epi == LG_EPI_GLU_CLAMP) {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        if (n0 + 2 * tx + j >= p.n) continue;
        const float g = fminf(acc[i][j], p.p1), u = fminf(fmaxf(acc[i][j + 2], -p.p1), p.p1);
        out[(size_t)r * p.ldc + (n0 >> 1) + 2 * tx + j] = g / (1.0f + expf(-p.p0 * g)) * (u + p.p2);
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = n0 + (j >> 1) * 32 + 2 * tx + (j & 1);
      if (c >= p.n) continue;
      if (p.epi == kEpiGroups) {
        const float v = acc[i][j];
        if (c < p.groups.n_main) out[(size_t)r * p.ldc + c] = c >= p.groups.silu_begin && c < p.groups.silu_end ? v / (1.0f + expf(-v)) : v;
        else reinterpret_cast<float*>(p.groups.tail)[(size_t)r * p.groups.ld_tail + c - p.groups.n_main] = p.groups.tail_cap > 0.0f ? p.groups.tail_cap * tanhf(v / p.groups.tail_cap) : v;
        continue;
      }
      if (p.epi == LG_EPI_RELU2) {
        const float v = fmaxf(acc[i][j], 0.0f);
        out[(size_t)r * p.ldc + c] = v * v;
        continue;
      }
      float* o = out + (size_t)r * p.ldc + c;
      if (p.epi == LG_EPI_RESID_F32) *o += acc[i][j];
      else *o = p.p0 > 0.0f ? p.p0 * tanhf(acc[i][j] / p.p0) : acc[i][j];
    }
  }
}

// the instantiation for a number of rows
uint32_t small_by_rows(const SmallArgs& p, int batch, cudaStream_t s) {
  const int m = p.m, n = p.n, k = p.k;
  const bool glu = p.epi == LG_EPI_SWIGLU || p.epi == LG_EPI_GLU_CLAMP;
  // two m16 tiles per CTA once that still leaves two CTAs per SM (the activations are then read half as often)
  const int64_t ctas2 = (int64_t)((n + 31) / 32) * batch;
  const bool two = glu || ctas2 >= 296;
  const int steps = k / 32;
  int warps = steps < 8 ? steps : 8;
  if (steps >= 128 && !two) warps = 16;
  const int nt = m <= 8 ? 1 : m <= 16 ? 2 : m <= 32 ? 4 : 8;
  if (two) {
    if (nt == 1) return launch_small<2, 1>(p, batch, warps, s);
    if (nt == 2) return launch_small<2, 2>(p, batch, warps, s);
    if (nt == 4) return launch_small<2, 4>(p, batch, warps, s);
    return launch_small<2, 8>(p, batch, warps, s);
  }
  if (nt == 1) return launch_small<1, 1>(p, batch, warps, s);
  if (nt == 2) return launch_small<1, 2>(p, batch, warps, s);
  if (nt == 4) return launch_small<1, 4>(p, batch, warps, s);
  return launch_small<1, 8>(p, batch, warps, s);
}

// ---- sums over slices of k -> the outputs of a grouped projection -----------------------------------
__global__ void __launch_bounds__(256)
groups_finish_kernel(float* __restrict__ acc, __nv_bfloat16* __restrict__ out, int m, int n, int ld_acc, int ldc, lg_linear_groups_t g) {
  lg::pdl_prologue();
  const int c = 4 * (blockIdx.x * 256 + threadIdx.x), r = blockIdx.y;
  if (c >= n) return;
  float4* src = reinterpret_cast<float4*>(acc + (size_t)r * ld_acc + c);
  float4 v = *src;
  *src = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < g.n_main) {
    if (g.bias) {
      const float4 b = __ldg(reinterpret_cast<const float4*>(reinterpret_cast<const float*>(g.bias) + c));
      v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
    }
    if (c >= g.silu_begin && c < g.silu_end) v = make_float4(silu_fast(v.x), silu_fast(v.y), silu_fast(v.z), silu_fast(v.w));
    *reinterpret_cast<uint2*>(out + (size_t)r * ldc + c) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
    return;
  }
  const int t = c - g.n_main, width = n - g.n_main;
  const float cap = g.tail_cap;
  if (cap > 0.0f) { v.x = cap * tanhf(v.x / cap); v.y = cap * tanhf(v.y / cap); v.z = cap * tanhf(v.z / cap); v.w = cap * tanhf(v.w / cap); }
  *reinterpret_cast<float4*>(reinterpret_cast<float*>(g.tail) + (size_t)r * g.ld_tail + t) = v;
  if (!g.tail_parts) return;
  __nv_bfloat16* parts = reinterpret_cast<__nv_bfloat16*>(g.tail_parts) + (size_t)r * 2 * width + t;
  const uint2 hi = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  const float2 a = unpack_bf16x2(hi.x), b = unpack_bf16x2(hi.y);
  *reinterpret_cast<uint2*>(parts) = hi;
  *reinterpret_cast<uint2*>(parts + width) = make_uint2(pack_bf16x2(v.x - a.x, v.y - a.y), pack_bf16x2(v.z - b.x, v.w - b.y));
}

}  // namespace

extern "C" {

uint32_t logismos_launch_linear_groups_finish(void* acc, void* out, int32_t m, int32_t n, int32_t ld_acc, int32_t ldc, const lg_linear_groups_t* groups, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!acc || !out || m <= 0 || m > 65535 || n <= 0 || n % 4 || ld_acc < n || ld_acc % 4 || ldc % 4 || !lg::groups_ok(groups, n, ldc) || groups->n_groups != 1 ||
      groups->n_main % 4 || (groups->n_main < n && groups->ld_tail % 4) || (((uintptr_t)acc | (uintptr_t)groups->bias | (uintptr_t)groups->tail) & 15) ||
      (((uintptr_t)out | (uintptr_t)groups->tail_parts) & 7))
    return lg::kInvalidValue;
  lg::launch(groups_finish_kernel, dim3((unsigned)((n / 4 + 255) / 256), (unsigned)m), dim3(256), 0, (cudaStream_t)stream, (float*)acc, (__nv_bfloat16*)out, m, n, ld_acc, ldc, *groups);
  return lg::launch_status();
}

static uint32_t small_any(const void* a, const void* w, const void* bias, void* out, int32_t m, int32_t n, int32_t k, int32_t lda, int32_t ldc,
                          int32_t batch, int64_t a_stride, int64_t w_stride, int64_t out_stride, int32_t epilogue, float p0, float p1, float p2,
                          const lg_linear_groups_t& groups, void* stream) {
  const bool glu = epilogue == LG_EPI_SWIGLU || epilogue == LG_EPI_GLU_CLAMP;
  if (m <= 0 || n <= 0 || k <= 0 || (k % 32) || batch <= 0 || batch > 65535 || (lda % 8) || lda < k || (a_stride % 8) || (w_stride % 8) ||
      (glu && (n % 64)) || ldc < (glu ? n / 2 : epilogue == kEpiGroups ? groups.n_main : n) || (((uintptr_t)a | (uintptr_t)w) & 15) || !out ||
      (m + 7) / 8 > 65535)
    return lg::kInvalidValue;
  const SmallArgs p{(const __nv_bfloat16*)a, (const __nv_bfloat16*)w, (const float*)bias, out, m, n, k, lda, ldc, epilogue,
                    a_stride, w_stride, out_stride, p0, p1, p2, groups};
  return small_by_rows(p, batch, (cudaStream_t)stream);
}

uint32_t logismos_launch_linear_small_tanh_norm(const void* a, const void* w, void* x, const lg_tanh_norm_t* post, void* h, const lg_tanh_norm_t* next, int32_t m,
                                                int32_t n, int32_t k, int32_t lda, int32_t ld, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!a || !w || !x || !post || !post->w || !post->b || (next && (!h || !next->w || !next->b)) || m <= 0 || (m + 7) / 8 > 65535 || n <= 0 || n > ld || k <= 0 || k % 32 || lda < k ||
      lda % 8 || (((uintptr_t)a | (uintptr_t)w) & 15))
    return lg::kInvalidValue;
  SmallArgs p{(const __nv_bfloat16*)a, (const __nv_bfloat16*)w, nullptr, x, m, n, k, lda, ld, kEpiTanhNorm, 0, 0, 0, 0, 0, 0, {}};
  p.post_alpha = post->alpha; p.post_w = (const float*)post->w; p.post_b = (const float*)post->b;
  if (next) { p.next_alpha = next->alpha; p.next_w = (const float*)next->w; p.next_b = (const float*)next->b; p.h = h; }
  return small_by_rows(p, 1, (cudaStream_t)stream);
}

uint32_t logismos_launch_linear_small_bf16(const void* a, const void* w, const void* bias, void* out, int32_t m, int32_t n, int32_t k,
                                           int32_t lda, int32_t ldc, int32_t batch, int64_t a_stride, int64_t w_stride,
                                           int64_t out_stride, int32_t epilogue, float p0, float p1, float p2, void* stream) {
  lg::LaunchScope launch_scope_;
  epilogue &= ~LG_EPI_STATIC_W;
  if (epilogue < 0 || epilogue > LG_EPI_RELU2) return lg::kInvalidValue;
  return small_any(a, w, bias, out, m, n, k, lda, ldc, batch, a_stride, w_stride, out_stride, epilogue, p0, p1, p2, {}, stream);
}

uint32_t logismos_launch_linear_groups_small_bf16(const void* a, const void* w, void* out, int32_t m, int32_t n, int32_t k, int32_t lda,
                                                  int32_t ldc, const lg_linear_groups_t* groups, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!lg::groups_ok(groups, n, ldc)) return lg::kInvalidValue;
  return small_any(a, w, groups->bias, out, m, n, k, lda, ldc, 1, 0, 0, 0, kEpiGroups, 0, 0, 0, *groups, stream);
}

uint32_t logismos_launch_linear_f32(const void* a, const void* w, const void* bias, void* out, int32_t m, int32_t n, int32_t k,
                                    int32_t lda, int32_t ldc, int32_t batch, int64_t a_stride, int64_t w_stride, int64_t out_stride,
                                    int32_t epilogue, float p0, float p1, float p2, void* stream) {
  lg::LaunchScope launch_scope_;
  epilogue &= ~LG_EPI_STATIC_W;
  const bool glu = epilogue == LG_EPI_GLU_CLAMP;
  if (m <= 0 || n <= 0 || k <= 0 || (k % 16) || batch <= 0 || batch > 65535 || (lda % 4) || lda < k || (a_stride % 4) || (w_stride % 4) ||
      (glu && (n % 64)) || ldc < (glu ? n / 2 : n) || ((uintptr_t)a & 15) || ((uintptr_t)w & 7) || !out || (m + 63) / 64 > 65535)
    return lg::kInvalidValue;
  if (epilogue != LG_EPI_RESID_F32 && epilogue != LG_EPI_F32 && epilogue != LG_EPI_RELU2 && !glu) return lg::kInvalidValue;
  const F32Args p{(const float*)a, (const __nv_bfloat16*)w, (const float*)bias, (float*)out, m, n, k, lda, ldc, epilogue,
                  a_stride, w_stride, out_stride, p0, p1, p2, {}};
  lg::launch(linear_f32_kernel, dim3((unsigned)((n + 63) / 64), (unsigned)((m + 63) / 64), (unsigned)batch), dim3(256), 0, (cudaStream_t)stream, p);
  return lg::launch_status();
}

uint32_t logismos_launch_linear_groups_f32(const void* a, const void* w, void* out, int32_t m, int32_t n, int32_t k, int32_t lda, int32_t ldc,
                                           const lg_linear_groups_t* groups, void* stream) {
  lg::LaunchScope launch_scope_;
  if (m <= 0 || n <= 0 || k <= 0 || (k % 16) || (lda % 4) || lda < k || ((uintptr_t)a & 15) || ((uintptr_t)w & 7) || !out || (m + 63) / 64 > 65535 ||
      !lg::groups_ok(groups, n, ldc))
    return lg::kInvalidValue;
  const F32Args p{(const float*)a, (const __nv_bfloat16*)w, (const float*)groups->bias, (float*)out, m, n, k, lda, ldc, kEpiGroups, 0, 0, 0, 0, 0, 0, *groups};
  lg::launch(linear_f32_kernel, dim3((unsigned)((n + 63) / 64), (unsigned)((m + 63) / 64)), dim3(256), 0, (cudaStream_t)stream, p);
  return lg::launch_status();
}

uint32_t logismos_launch_linear_experts_small_bf16(const void* a, const void* w, void* out, const void* offsets, const void* row_idx, int32_t n_groups,
                                                   int32_t max_group_rows, int32_t expected_group_rows, int32_t n, int32_t k, int32_t lda, int32_t ldc,
                                                   int32_t epilogue, float p0, float p1, float p2, void* stream) {
  lg::LaunchScope launch_scope_;
  epilogue &= ~LG_EPI_STATIC_W;
  const bool glu = epilogue == LG_EPI_SWIGLU || epilogue == LG_EPI_GLU_CLAMP;
  if (!a || !w || !out || !offsets || n_groups <= 0 || n_groups > 65535 || max_group_rows <= 0 || max_group_rows > (1 << 19) || n <= 0 || n % (glu ? 64 : 16) || k <= 0 ||
      k % 32 || lda < k || lda % 8 || ldc < (glu ? n / 2 : n) || (((uintptr_t)a | (uintptr_t)w) & 15) || (!glu && epilogue != LG_EPI_BF16))
    return lg::kInvalidValue;
  SmallArgs p{(const __nv_bfloat16*)a, (const __nv_bfloat16*)w, nullptr, out, 0, n, k, lda, ldc, epilogue, 0, (int64_t)n * k, 0, p0, p1, p2, {}, (const int*)offsets,
              (const int*)row_idx};
  const int steps = k / 32, warps = steps < 8 ? steps : 8, rows = expected_group_rows < max_group_rows ? expected_group_rows : max_group_rows;
  cudaStream_t s = (cudaStream_t)stream;
  if (rows <= 8) return launch_small_experts<1>(p, n_groups, max_group_rows, warps, s);
  if (rows <= 16) return launch_small_experts<2>(p, n_groups, max_group_rows, warps, s);
  return launch_small_experts<4>(p, n_groups, max_group_rows, warps, s);
}

uint32_t logismos_launch_linear_experts_f32(const void* a, const void* w, void* out, const void* offsets, const void* row_idx, int32_t n_groups,
                                            int32_t max_group_rows, int32_t n, int32_t k, int32_t lda, int32_t ldc, int32_t epilogue, float p0, float p1,
                                            float p2, void* stream) {
  lg::LaunchScope launch_scope_;
  epilogue &= ~LG_EPI_STATIC_W;
  const bool glu = epilogue == LG_EPI_GLU_CLAMP;
  if (!a || !w || !out || !offsets || n_groups <= 0 || n_groups > 65535 || max_group_rows <= 0 || (max_group_rows + 63) / 64 > 65535 || n <= 0 || (glu && n % 64) || k <= 0 ||
      k % 16 || lda < k || lda % 4 || ldc < (glu ? n / 2 : n) || ((uintptr_t)a & 15) || ((uintptr_t)w & 7) || (!glu && epilogue != LG_EPI_F32))
    return lg::kInvalidValue;
  const F32Args p{(const float*)a, (const __nv_bfloat16*)w, nullptr, (float*)out, 0, n, k, lda, ldc, epilogue, 0, (int64_t)n * k, 0, p0, p1, p2, {}, (const int*)offsets,
                  (const int*)row_idx};
  lg::launch(linear_f32_kernel, dim3((unsigned)((n + 63) / 64), (unsigned)((max_group_rows + 63) / 64), (unsigned)n_groups), dim3(256), 0, (cudaStream_t)stream, p);
  return lg::launch_status();
}

}  // extern "C"
