// Router of a mixture of experts (lg_moe_route_t): the choice of experts per token and the grouping of rows by expert.
//   few tokens    one CTA: choice, counts, offsets and row lists; the expert products read their rows through the list. Or a
//                 CTA per token that computes the token's logits too, the last one to finish then groups the rows
//   many tokens   choice with per-CTA histograms (a row's rank in its group is unique, its order is not fixed; rows of a
//                 group are independent), then a second launch that places the rows, copies them and lists the row tiles
// Logits, scores (softmax or sigmoid), choice and weights are fp32. A warp handles a token, a lane the experts lane, lane +
// 32, ... Choice by groups: the experts of all but the best groups are struck out first.
#include "common.cuh"
#include "logismos_kernels.h"

namespace {

using namespace lg;

constexpr int kMaxOut = 512, kMaxTop = 32, kMaxAlways = 64, kMaxGroups = kMaxOut + kMaxAlways;
constexpr int kFewThreads = 1024, kRouteThreads = 256, kRouteTokens = 32;

struct RouteArgs {
  float* logits;
  int ld, zero;
  const float* correction;
  int experts, identity, top, always;
  float* weights;
  int* pair_row;
  float* id_weight;
  int* offsets;
  int* row_token;
  int* counts;
  int* pair_expert;
  int4* tiles;
  int* n_tiles;
  int tokens;
  const __nv_bfloat16* h;     // with the product: [tokens, width]
  const __nv_bfloat16* w;     // [experts + identity, width]
  int width;
  int* arrived;
  int sigmoid, groups, keep_groups;
};

// float -> integer of the same order
LG_DEVINL uint32_t ordered(float x) {
  const uint32_t u = __float_as_uint(x);
  return u & 0x80000000u ? ~u : u | 0x80000000u;
}

// The largest c of a warp and the first output that has it (kMaxOut: all are -inf), struck out of c
template <int R>
LG_DEVINL int take_best(float (&c)[R], int lane, float* value) {
  float best = -INFINITY;
  int at = 0;
#pragma unroll
  for (int i = 0; i < R; ++i)
    if (c[i] > best) { best = c[i]; at = i; }
  const uint32_t key = ordered(best), top_key = __reduce_max_sync(0xffffffffu, key);
  const int id = __reduce_min_sync(0xffffffffu, key == top_key ? lane + 32 * at : kMaxOut);  // equal scores: the first
  float v = 0.0f;
#pragma unroll
  for (int i = 0; i < R; ++i)
    if (id == lane + 32 * i) { v = c[i]; c[i] = -INFINITY; }
  *value = __shfl_sync(0xffffffffu, v, id & 31);
  return id;
}

// c of the outputs outside the best groups is struck out; a group scores the sum of its two largest
template <int R>
LG_DEVINL void keep_best_groups(const RouteArgs& p, float (&c)[R], int lane) {
  const int n = p.experts + p.identity, size = n / p.groups;
  float score[R];   // of the groups lane, lane + 32, ...
#pragma unroll
  for (int i = 0; i < R; ++i) score[i] = -INFINITY;
  for (int g = 0; g < p.groups; ++g) {
    float own[R], sum, second = 0.0f;
#pragma unroll
    for (int i = 0; i < R; ++i) own[i] = (lane + 32 * i) / size == g && lane + 32 * i < n ? c[i] : -INFINITY;
    take_best<R>(own, lane, &sum);
    if (size > 1) take_best<R>(own, lane, &second);
#pragma unroll
    for (int i = 0; i < R; ++i)
      if (g == lane + 32 * i) score[i] = sum + second;
  }
  uint32_t kept = 0;   // of this lane's outputs
  for (int k = 0; k < p.keep_groups; ++k) {
    float unused;
    const int g = take_best<R>(score, lane, &unused);
#pragma unroll
    for (int i = 0; i < R; ++i)
      if ((lane + 32 * i) / size == g) kept |= 1u << i;
  }
#pragma unroll
  for (int i = 0; i < R; ++i)
    if (!(kept >> i & 1)) c[i] = -INFINITY;
}

// The experts by a token's logits z: lane i < top receives the i-th choice and its weight. R: logits per lane.
template <int R>
LG_DEVINL void choose(const RouteArgs& p, float* z, int lane, int& expert, float& weight) {
  const int n = p.experts + p.identity;
  float s[R], c[R], mx = -INFINITY, sum = 0.0f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    s[i] = lane + 32 * i < n ? z[lane + 32 * i] : -INFINITY;
    mx = fmaxf(mx, s[i]);
  }
  if (p.sigmoid) {
#pragma unroll
    for (int i = 0; i < R; ++i) s[i] = 1.0f / (1.0f + expf(-s[i]));
  } else {
    mx = warp_max(mx);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      s[i] = expf(s[i] - mx);
      sum += s[i];
    }
    sum = warp_sum(sum);
#pragma unroll
    for (int i = 0; i < R; ++i) s[i] /= sum;
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    c[i] = lane + 32 * i < n ? s[i] + (p.correction ? __ldg(p.correction + lane + 32 * i) : 0.0f) : -INFINITY;
    if (p.zero && lane + 32 * i < n) z[lane + 32 * i] = 0.0f;
  }
  if (p.groups > 0) keep_best_groups<R>(p, c, lane);
  expert = -1;
  float picked = 0.0f, total = 0.0f;
  for (int k = 0; k < p.top; ++k) {
    float unused, score = 0.0f;
    const int id = take_best<R>(c, lane, &unused);
#pragma unroll
    for (int i = 0; i < R; ++i)
      if (id == lane + 32 * i) score = s[i];
    score = __shfl_sync(0xffffffffu, score, id & 31);
    total += score;
    if (lane == k) { expert = id; picked = score; }
  }
  weight = picked / (total + 1e-20f);
}

// weights, the identity experts' share, and the group of each pair (-1: none)
LG_DEVINL int store_choice(const RouteArgs& p, int token, int lane, int expert, float weight) {
  const bool in = lane < p.top, none = in && expert >= p.experts;
  const float id = warp_sum(none ? weight : 0.0f);
  if (in) p.weights[(size_t)token * p.top + lane] = weight;
  if (lane == 0) p.id_weight[token] = id;
  return in && !none ? expert : -1;
}

// exclusive prefix of count[0 .. n) into start[0 .. n]; all threads of the CTA, n <= kMaxGroups
LG_DEVINL void prefix(const int* count, int* start, int n) {
  if (threadIdx.x < 32) {
    int base = 0;
    for (int g0 = 0; g0 < n; g0 += 32) {
      const int g = g0 + (int)threadIdx.x, own = g < n ? count[g] : 0;
      int x = own;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, o);
        if ((int)threadIdx.x >= o) x += y;
      }
      if (g < n) start[g] = base + x - own;
      base += __shfl_sync(0xffffffffu, x, 31);
    }
    if (threadIdx.x == 0) start[n] = base;
  }
  __syncthreads();
}

// the groups of all pairs, rank | group << 20 in pair_row (-1: none), counted in `count` -> offsets, rows and their tokens
LG_DEVINL void group_rows(const RouteArgs& p, const int* count, int* start) {
  const int groups = p.experts + p.always, pairs = p.top + p.always;
  prefix(count, start, groups);
  for (int g = threadIdx.x; g <= groups; g += blockDim.x) p.offsets[g] = start[g];
  for (int i = threadIdx.x; i < p.tokens * pairs; i += blockDim.x) {
    const int t = i / pairs, k = i - t * pairs;
    int row;
    if (k >= p.top) row = start[p.experts + k - p.top] + t;
    else {
      const int v = p.pair_row[i];
      if (v < 0) continue;
      row = start[v >> 20] + (v & 0xfffff);
    }
    p.pair_row[i] = row;
    p.row_token[row] = t;
  }
}

template <int R>
__global__ void __launch_bounds__(kFewThreads)
moe_route_few_kernel(RouteArgs p) {
  lg::pdl_prologue();
  __shared__ int count[kMaxGroups], start[kMaxGroups + 1];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, groups = p.experts + p.always, pairs = p.top + p.always;
  for (int g = tid; g < groups; g += kFewThreads) count[g] = g < p.experts ? 0 : p.tokens;
  __syncthreads();
  for (int t = warp; t < p.tokens; t += kFewThreads / 32) {
    int expert;
    float weight;
    choose<R>(p, p.logits + (size_t)t * p.ld, lane, expert, weight);
    const int g = store_choice(p, t, lane, expert, weight);
    if (lane < p.top) p.pair_row[(size_t)t * pairs + lane] = g < 0 ? -1 : atomicAdd(&count[g], 1) | (g << 20);
  }
  __syncthreads();
  group_rows(p, count, start);
}

// CTA = token: its logits (a warp per router row, fp32 sums in a fixed order), its choice; the last CTA groups the rows
template <int R>
__global__ void __launch_bounds__(kRouteThreads)
moe_router_kernel(RouteArgs p) {
  lg::pdl_prologue();
  __shared__ float z[kMaxOut];
  __shared__ int count[kMaxGroups], start[kMaxGroups + 1], last;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, t = blockIdx.x, n = p.experts + p.identity, pairs = p.top + p.always;
  const uint4* h = reinterpret_cast<const uint4*>(p.h + (size_t)t * p.width);
  for (int e = warp; e < n; e += kRouteThreads / 32) {
    const uint4* w = reinterpret_cast<const uint4*>(p.w + (size_t)e * p.width);
    float s = 0.0f;
#pragma unroll 4
    for (int c = lane; c < p.width / 8; c += 32) {
      const uint4 a = h[c], b = __ldg(w + c);
      const uint32_t aw[4] = {a.x, a.y, a.z, a.w}, bw[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 x = unpack_bf16x2(aw[i]), y = unpack_bf16x2(bw[i]);
        s = fmaf(x.x, y.x, fmaf(x.y, y.y, s));
      }
    }
    s = warp_sum(s);
    if (lane == 0) z[e] = s;
  }
  __syncthreads();
  if (warp == 0) {
    int expert;
    float weight;
    choose<R>(p, z, lane, expert, weight);
    const int g = store_choice(p, t, lane, expert, weight);
    if (lane < p.top) p.pair_row[(size_t)t * pairs + lane] = g;
    __threadfence();
    if (lane == 0) last = atomicAdd(p.arrived, 1) == (int)gridDim.x - 1;
  }
  __syncthreads();
  if (!last) return;
  __threadfence();
  if (tid == 0) *p.arrived = 0;
  for (int g = tid; g < p.experts + p.always; g += kRouteThreads) count[g] = g < p.experts ? 0 : p.tokens;
  __syncthreads();
  volatile int* groups = p.pair_row;
  for (int i = tid; i < p.tokens * p.top; i += kRouteThreads) {
    const int at = i / p.top * pairs + i % p.top, g = groups[at];
    if (g >= 0) groups[at] = atomicAdd(&count[g], 1) | (g << 20);
  }
  __syncthreads();
  group_rows(p, count, start);
}

template <int R>
__global__ void __launch_bounds__(kRouteThreads)
moe_route_kernel(RouteArgs p) {
  lg::pdl_prologue();
  __shared__ int count[kMaxOut], base[kMaxOut], group_s[kRouteTokens * kMaxTop], rank_s[kRouteTokens * kMaxTop];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int t0 = blockIdx.x * kRouteTokens, n = min(kRouteTokens, p.tokens - t0);
  for (int g = tid; g < p.experts; g += kRouteThreads) count[g] = 0;
  __syncthreads();
  for (int t = warp; t < n; t += kRouteThreads / 32) {
    int expert;
    float weight;
    choose<R>(p, p.logits + (size_t)(t0 + t) * p.ld, lane, expert, weight);
    const int g = store_choice(p, t0 + t, lane, expert, weight);
    if (lane < p.top) {
      group_s[t * p.top + lane] = g;
      rank_s[t * p.top + lane] = g < 0 ? 0 : atomicAdd(&count[g], 1);
    }
  }
  __syncthreads();
  for (int g = tid; g < p.experts; g += kRouteThreads) base[g] = count[g] ? atomicAdd(p.counts + g, count[g]) : 0;
  __syncthreads();
  for (int i = tid; i < n * p.top; i += kRouteThreads) {
    const int t = i / p.top, k = i - t * p.top, g = group_s[i];
    p.pair_expert[(size_t)(t0 + t) * p.top + k] = g < 0 ? -1 : (base[g] + rank_s[i]) | (g << 20);
  }
}

// A warp per (token, pair): final rows, and the copy of the token's row for the chosen experts. CTA 0 also lists the tiles.
__global__ void __launch_bounds__(kRouteThreads)
moe_place_kernel(RouteArgs p, const uint4* h, uint4* gathered, int vecs) {
  lg::pdl_prologue();
  __shared__ int count[kMaxGroups], start[kMaxGroups + 1], first[kMaxGroups + 1];
  const int tid = threadIdx.x, lane = tid & 31, groups = p.experts + p.always, pairs = p.top + p.always;
  for (int g = tid; g < groups; g += kRouteThreads) count[g] = g < p.experts ? p.counts[g] : p.tokens;
  __syncthreads();
  prefix(count, start, groups);
  const int64_t total = (int64_t)p.tokens * pairs;
  for (int64_t i = (int64_t)blockIdx.x * (kRouteThreads / 32) + (tid >> 5); i < total; i += (int64_t)gridDim.x * (kRouteThreads / 32)) {
    const int t = (int)(i / pairs), k = (int)(i - (int64_t)t * pairs);
    if (k >= p.top) {
      if (lane == 0) p.pair_row[i] = start[p.experts + k - p.top] + t;
      continue;
    }
    const int v = p.pair_expert[(size_t)t * p.top + k], row = v < 0 ? -1 : start[v >> 20] + (v & 0xfffff);
    if (lane == 0) p.pair_row[i] = row;
    if (row < 0) continue;
    for (int c = lane; c < vecs; c += 32) gathered[(size_t)row * vecs + c] = h[(size_t)t * vecs + c];
  }
  if (blockIdx.x) return;
  for (int g = tid; g < groups; g += kRouteThreads) count[g] = (count[g] + 127) >> 7;
  __syncthreads();
  prefix(count, first, groups);
  for (int g = tid; g < groups; g += kRouteThreads)
    for (int i = 0; i < count[g]; ++i) {
      const int row = start[g] + 128 * i;
      p.tiles[first[g] + i] = make_int4(g, row, start[g + 1], g < p.experts ? row : -1 - 128 * i);
    }
  if (tid == 0) *p.n_tiles = first[groups];
}

bool route_ok(const lg_moe_route_t* a, int tokens) {
  return a && tokens > 0 && tokens < (1 << 20) && (a->logits || a->h) && a->weights && a->pair_row && a->identity && a->n_experts > 0 &&
         a->n_identity >= 0 && a->n_experts + a->n_identity <= kMaxOut && (a->h || a->ld >= a->n_experts + a->n_identity) && a->top > 0 && a->top <= kMaxTop &&
         a->top <= a->n_experts + a->n_identity && a->n_always >= 0 && a->n_always <= kMaxAlways &&
         (a->scoring == LG_ROUTE_SOFTMAX || a->scoring == LG_ROUTE_SIGMOID) && a->groups >= 0 &&
         (a->groups == 0 || ((a->n_experts + a->n_identity) % a->groups == 0 && a->keep_groups > 0 && a->keep_groups <= a->groups &&
                             a->top <= (a->n_experts + a->n_identity) / a->groups * a->keep_groups));
}
RouteArgs route_args(const lg_moe_route_t* a, int tokens) {
  return RouteArgs{(float*)a->logits, a->ld, a->zero_logits, (const float*)a->correction, a->n_experts, a->n_identity, a->top, a->n_always, (float*)a->weights,
                   (int*)a->pair_row, (float*)a->identity, (int*)a->offsets, (int*)a->row_token, (int*)a->counts, (int*)a->pair_expert, (int4*)a->tiles,
                   (int*)a->n_tiles, tokens, (const __nv_bfloat16*)a->h, (const __nv_bfloat16*)a->w, a->width, (int*)a->arrived, a->scoring == LG_ROUTE_SIGMOID, a->groups, a->keep_groups};
}

}  // namespace

extern "C" {

// Measured (us, choice included, streamed / tiles; experts, top, width x ff): 16, 2, 1024 x 512 at 64 / 96 tokens 30 / 31, 35 /
// 31; 16, 2, 2048 x 1024 at 16 / 32 / 64 59 / 62, 63 / 61, 76 / 63; 16, 2, 4096 x 2048 at 4 / 8 / 16 102 / 112, 113 / 105, 159 /
// 139; 64, 8, 2048 x 512 at 8 / 16 79 / 80, 105 / 89: the tiles win once the experts in use hold some 200 MB.
int32_t logismos_moe_streams(int32_t tokens, int32_t top, int32_t n_experts, int32_t n_identity, int32_t n_always, int32_t width, int32_t ff) {
  if (tokens > 64) return 0;
  double idle = 1.0;
  for (int32_t i = 0; i < tokens; ++i) idle *= 1.0 - (double)top / (n_experts + n_identity);
  return (n_experts * (1.0 - idle) + n_always) * 6.0 * width * ff < 2e8 ? 1 : 0;
}

int32_t logismos_moe_max_tiles(int32_t tokens, int32_t top, int32_t n_experts, int32_t n_always) {
  return (int32_t)((int64_t)tokens * top / 128) + n_experts + (tokens + 127) / 128 * n_always;
}

// one launch when offsets are given, else the first of two
uint32_t logismos_launch_moe_route(const lg_moe_route_t* a, int32_t tokens, void* stream) {
  lg::LaunchScope launch_scope_;
  const bool few = a && a->offsets;
  if (!route_ok(a, tokens) || (few ? !a->row_token : !a->counts || !a->pair_expert)) return lg::kInvalidValue;
  if (a->h && (!few || !a->w || !a->arrived || a->width <= 0 || a->width % 8 || (((uintptr_t)a->h | (uintptr_t)a->w) & 15))) return lg::kInvalidValue;
  RouteArgs p = route_args(a, tokens);
  if (p.h) p.zero = 0;
  const dim3 grid(p.h ? (unsigned)tokens : few ? 1u : (unsigned)((tokens + kRouteTokens - 1) / kRouteTokens)), block(few && !p.h ? kFewThreads : kRouteThreads);
  auto go = [&](auto kern) -> uint32_t {
    lg::launch(kern, grid, block, 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
  const int n = p.experts + p.identity;
#define LG_ROUTE(R) (p.h ? go(moe_router_kernel<R>) : few ? go(moe_route_few_kernel<R>) : go(moe_route_kernel<R>))
  return n <= 32 ? LG_ROUTE(1) : n <= 64 ? LG_ROUTE(2) : n <= 128 ? LG_ROUTE(4) : n <= 256 ? LG_ROUTE(8) : LG_ROUTE(16);
#undef LG_ROUTE
}

uint32_t logismos_launch_moe_place(const lg_moe_route_t* a, const void* h, void* gathered, int32_t ld, int32_t tokens, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!route_ok(a, tokens) || !a->counts || !a->pair_expert || !a->tiles || !a->n_tiles || !h || !gathered || ld <= 0 || ld % 8 ||
      (((uintptr_t)h | (uintptr_t)gathered | (uintptr_t)a->tiles) & 15))
    return lg::kInvalidValue;
  const RouteArgs p = route_args(a, tokens);
  const int64_t warps = (int64_t)tokens * (p.top + p.always), ctas = (warps + kRouteThreads / 32 - 1) / (kRouteThreads / 32);
  lg::launch(moe_place_kernel, dim3((unsigned)(ctas < 148 * 8 ? ctas : 148 * 8)), dim3(kRouteThreads), 0, (cudaStream_t)stream, p, (const uint4*)h, (uint4*)gathered, ld / 8);
  return lg::launch_status();
}

}  // extern "C"
