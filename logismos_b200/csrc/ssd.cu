// State-space mixer with a scalar decay per head (Mamba-2, state-space duality). A projected row is [z | x | B | C]
// in the activation format, H heads of VP values and G groups of NP state channels, and dt per head in fp32. x, B
// and C pass a causal depthwise convolution and silu; then per head (B, C of its group)
//   dt <- softplus(dt + bias);  S <- exp(-exp(log_a) dt) S + dt B x^T;  y = S^T C + D x
// and over the heads y silu(z), each of several equal parts divided by its root mean square, times a gain.
// A fixed decay per head makes it linear attention over rows x | B | C = values | keys | queries, with every step of size one
// and no skip. State, step sizes, decays, convolution sums and norms are fp32. NP and VP are powers of two with zero padding.
// The last taps - 1 inputs of the convolution are its state: a slot holds two copies, a step reads the one its
// phase names and writes the other.
//
// ssd_conv_kernel: convolution and silu of all rows.
// ssd_step_kernel: CTA = (head, sequence), tokens one after the other. Decode steps, fp32, sizes beyond the next form.
// ssd_chunk_kernel: prompts. The chunked form resolves 64 tokens together: with c_i the sum of the
// log-decays up to token i of the chunk and S the state before it,
//   P_ij = (C_i . B_j) exp(c_i - c_j) dt_j (j <= i);   y_i = sum_j P_ij x_j + exp(c_i) S^T C_i + D x_i
//   S <- exp(c_last) S + sum_j B_j (dt_j exp(c_last - c_j) x_j)^T
// The products run on mma.sync with bf16 operands: B, C and x are bf16 already; the state, P and the weighted x go
// in as a rounded part and a remainder (two products), so that what is fp32 keeps about 16 bits; sums are fp32.
// Long prompts of few heads are cut in segments that run at once: every segment's own state from zero and its decay, a scan
// over the segments of a sequence, then the segments' outputs from the states that they start with.
#include "common.cuh"
#include "logismos_kernels.h"
#include "recurrent.cuh"

namespace {

using namespace lg;
using namespace lg::rec;

constexpr int kMaxTaps = 8;

struct SsdArgs {
  const void* proj;        // z at 0, x at heads * vp, B, C behind it
  int ld;
  const float* dt;         // [rows, ld_dt]
  int ld_dt;
  const float* conv_w;     // [taps][channels], the last tap is the current token's
  const float* conv_b;     // [channels]
  float* conv_state;       // [n_slots][2][taps - 1][channels]
  int taps;
  const float* dt_bias;
  const float* log_a;
  const float* skip;       // D
  float* state;            // [n_slots][heads][np][vp]
  const int* state_slots;
  const uint8_t* fresh;
  const uint8_t* phase;
  const int* cu;
  void* y;                 // activation format, [rows, ld_y], head h at h * vp
  int ld_y;
  int heads, groups, np, vp;
  void* xbc;               // convolved channels [rows, ld_xbc], activation format
  int ld_xbc;
  const float* decay;
  __host__ __device__ __forceinline__ int channels() const { return heads * vp + 2 * groups * np; }
};

template <typename T, bool FIXED>
__global__ void __launch_bounds__(kThreads, 5)
ssd_step_kernel(SsdArgs p, int in_smem) {
  lg::pdl_trigger();
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ __align__(16) float xs[256], bs[256], cs[256], red[1024];
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int vp = p.vp, np = p.np, group = head / (p.heads / p.groups), inner = p.heads * vp;
  const Tile t(np, vp);
  const bool fresh = p.fresh[seq] != 0;
  // the state of an earlier step and the weights do not depend on the kernels before this one
  State S(smem, in_smem, p.state + ((size_t)p.state_slots[seq] * p.heads + head) * np * vp);
  S.request(t, fresh);
  const int t0 = p.cu[seq], t1 = p.cu[seq + 1];
  const float bias = FIXED ? 0.0f : __ldg(p.dt_bias + head), a = FIXED ? 0.0f : expf(__ldg(p.log_a + head)), skip = FIXED ? 0.0f : __ldg(p.skip + head);
  const float fixed = FIXED ? __ldg(p.decay + 3 * head + 1) : 0.0f, dropped = FIXED ? __ldg(p.decay + 3 * head + 2) : 0.0f;
  lg::pdl_wait();
  for (int tok = t0; tok < t1; ++tok) {
    const T* row = reinterpret_cast<const T*>(p.xbc) + (size_t)tok * p.ld_xbc;
    const float dt = FIXED ? 1.0f : softplus_f(p.dt[(size_t)tok * p.ld_dt + head] + bias), decay = FIXED ? fixed : expf(-a * dt);
    if (tid < vp) xs[tid] = Io<T>::load(row + head * vp + tid);
    if (tid < np) {
      bs[tid] = dt * Io<T>::load(row + inner + group * np + tid);
      cs[tid] = Io<T>::load(row + inner + (p.groups + group) * np + tid);
    }
    __syncthreads();
    if (tok == t0) S.arrived();
    const float4 x4 = *reinterpret_cast<const float4*>(xs + t.c4);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    S.visit(t, fresh && tok == t0, tok + 1 == t1, [&](int r, float4& s) {
      const float b = bs[r], c = cs[r];
      float4 add = make_float4(b * x4.x, b * x4.y, b * x4.z, b * x4.w);
      // what the decay's rounding dropped joins the smaller term, where it is not rounded away: no drift over a thousand steps
      if (FIXED) add = make_float4(fmaf(dropped, s.x, add.x), fmaf(dropped, s.y, add.y), fmaf(dropped, s.z, add.z), fmaf(dropped, s.w, add.w));
      s = make_float4(fmaf(decay, s.x, add.x), fmaf(decay, s.y, add.y), fmaf(decay, s.z, add.z), fmaf(decay, s.w, add.w));
      o.x = fmaf(c, s.x, o.x); o.y = fmaf(c, s.y, o.y); o.z = fmaf(c, s.z, o.z); o.w = fmaf(c, s.w, o.w);
    });
    reduce_store(t, o, red);
    __syncthreads();
    if (tid < vp) Io<T>::store(reinterpret_cast<T*>(p.y) + (size_t)tok * p.ld_y + head * vp + tid, reduce_load(vp, red, tid) + skip * xs[tid]);
    if (tok + 1 < t1) __syncthreads();
  }
}

// Convolution and silu of ragged rows [row0, rows): a thread owns four channels and a run of RUN consecutive rows.
template <typename T> struct Raw4;
template <> struct Raw4<float> { typedef float4 type; };
template <> struct Raw4<__nv_bfloat16> { typedef uint2 type; };
LG_DEVINL float4 widen(float4 v) { return v; }
LG_DEVINL float4 widen(uint2 u) {
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
// z sigmoid(z) where bf16 is the result: sigmoid(z) = (1 + tanh(z / 2)) / 2 with the approximate tanh (relative error 2^-11)
LG_DEVINL float silu_bf16(float z) {
  float t;
  asm("tanh.approx.f32 %0, %1;\n" : "=f"(t) : "f"(0.5f * z));
  const float h = 0.5f * z;
  return fmaf(h, t, h);
}

template <typename T, int TAPS, int RUN>
__global__ void __launch_bounds__(128)
ssd_conv_kernel(SsdArgs p, const int* __restrict__ seq_ids, int row0, int rows) {
  lg::pdl_prologue();
  typedef typename Raw4<T>::type Raw;
  constexpr int HN = TAPS - 1;
  const int all = p.channels(), c0 = 4 * (blockIdx.y * blockDim.x + threadIdx.x);
  if (c0 >= all) return;
  const T* src = reinterpret_cast<const T*>(p.proj) + p.heads * p.vp + c0;
  T* dst = reinterpret_cast<T*>(p.xbc) + c0;
  auto load = [&](int t) { return *reinterpret_cast<const Raw*>(src + (size_t)t * p.ld); };
  const int first = row0 + blockIdx.x * RUN, last = min(rows, first + RUN);
  Raw in[RUN];
#pragma unroll
  for (int i = 0; i < RUN; ++i) in[i] = load(first + i < last ? first + i : first);
  float4 w[TAPS], prev[HN > 0 ? HN : 1];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = __ldg(reinterpret_cast<const float4*>(p.conv_w + (size_t)j * all + c0));
  const float4 bias = __ldg(reinterpret_cast<const float4*>(p.conv_b + c0));
  auto fma = [](float4 a, float4 x, float4 c) { return make_float4(fmaf(a.x, x.x, c.x), fmaf(a.y, x.y, c.y), fmaf(a.z, x.z, c.z), fmaf(a.w, x.w, c.w)); };
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  int cur = -1, t0 = 0, len = 0;
  float* next = nullptr;
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int t = first + i;
    if (t >= last) break;
    const int s = seq_ids[t];
    if (s != cur) {
      cur = s;
      t0 = p.cu[s];
      len = p.cu[s + 1] - t0;
      const bool fresh = p.fresh[s] != 0;
      const int ph = p.phase[s] & 1;
      const float* old = p.conv_state + ((size_t)p.state_slots[s] * 2 + ph) * HN * all + c0;
      next = p.conv_state + ((size_t)p.state_slots[s] * 2 + 1 - ph) * HN * all + c0;
#pragma unroll
      for (int j = 0; j < HN; ++j) {
        const int idx = t - t0 - HN + j;  // place inside the step's tokens of this sequence; negative: the state
        if (idx >= 0) prev[j] = widen(load(t0 + idx));
        else prev[j] = fresh ? zero : *reinterpret_cast<const float4*>(old + (size_t)(HN + idx) * all);
      }
      if (t == t0) {  // rows of the old state that stay in the new one
#pragma unroll
        for (int j = 0; j < HN; ++j)
          if (j + len < HN) *reinterpret_cast<float4*>(next + (size_t)j * all) = fresh ? zero : *reinterpret_cast<const float4*>(old + (size_t)(j + len) * all);
      }
    }
    const float4 x = widen(in[i]);
    float4 y = fma(w[TAPS - 1], x, bias);
#pragma unroll
    for (int j = 0; j < HN; ++j) y = fma(w[j], prev[j], y);
    if constexpr (sizeof(T) == 2)
      *reinterpret_cast<uint2*>(dst + (size_t)t * p.ld_xbc) = make_uint2(pack_bf16x2(silu_bf16(y.x), silu_bf16(y.y)), pack_bf16x2(silu_bf16(y.z), silu_bf16(y.w)));
    else
      *reinterpret_cast<float4*>(dst + (size_t)t * p.ld_xbc) = make_float4(silu_f(y.x), silu_f(y.y), silu_f(y.z), silu_f(y.w));
    const int keep = HN - (len - (t - t0));  // row of the new state this token becomes, if any
    if (keep >= 0) *reinterpret_cast<float4*>(next + (size_t)keep * all) = x;
#pragma unroll
    for (int j = 0; j + 1 < HN; ++j) prev[j] = prev[j + 1];
    if (HN > 0) prev[HN > 0 ? HN - 1 : 0] = x;
  }
}

template <typename T, int RUN>
uint32_t launch_conv(const SsdArgs& p, const int* seq_ids, int row0, int rows, cudaStream_t s) {
  const dim3 grid((unsigned)((rows - row0 + RUN - 1) / RUN), (unsigned)(((p.heads * p.vp + 2 * p.groups * p.np) / 4 + 127) / 128));
  auto go = [&](auto kern) {
    lg::launch(kern, grid, dim3(128), 0, s, p, seq_ids, row0, rows);
    return lg::launch_status();
  };
  switch (p.taps) {
    case 1: return go(ssd_conv_kernel<T, 1, RUN>);
    case 2: return go(ssd_conv_kernel<T, 2, RUN>);
    case 3: return go(ssd_conv_kernel<T, 3, RUN>);
    case 4: return go(ssd_conv_kernel<T, 4, RUN>);
    case 5: return go(ssd_conv_kernel<T, 5, RUN>);
    case 6: return go(ssd_conv_kernel<T, 6, RUN>);
    case 7: return go(ssd_conv_kernel<T, 7, RUN>);
    default: return go(ssd_conv_kernel<T, 8, RUN>);
  }
}

// CTA = (head, sequence), VP / 8 warps; shared memory as laid out by ssd_chunk_smem
constexpr int kPitchP = kChunk * 2 + 16;
inline size_t ssd_chunk_smem(int np, int vp) {
  return (size_t)kChunk * (2 * (2 * (2 * np + 16) + 2 * vp + 16) + 2 * kPitchP) + 4 * kChunk * 4;
}
// PART: whole sequences, or segments' states (all but a sequence's last), or segments' outputs. The segments of a sequence have
// consecutive entries of the scratch (state they start with, decay of the segment before them).
enum { kWhole = 0, kStates = 1, kOutputs = 2 };
constexpr int kSegment = 256;
struct Segments {
  float* state;   // [entries][heads][np][vp]
  float* decay;   // [entries][heads], log2
};
LG_DEVINL int first_entry(const int* cu, int seq) { return (cu[seq] - cu[0]) / kSegment + seq; }

template <int NP, bool FIXED, int PART>
__global__ void __launch_bounds__(512)
ssd_chunk_kernel(SsdArgs p, Segments segs) {
  lg::pdl_prologue();
  constexpr int NT = NP / 16, kPitchN = NP * 2 + 16;
  extern __shared__ __align__(16) uint8_t smem[];
  const int vp = p.vp, pitch_v = vp * 2 + 16;
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n_warps = blockDim.x >> 5;
  const int g = lane >> 2, t = lane & 3, v0 = 8 * warp;
  const int t0 = p.cu[seq] + (PART == kWhole ? 0 : (int)blockIdx.z * kSegment), end = p.cu[seq + 1], t1 = PART == kWhole ? end : min(end, t0 + kSegment);
  if (t1 <= t0 || (PART == kStates && t1 == end)) return;
  const int entry = PART == kWhole ? 0 : first_entry(p.cu, seq) + (int)blockIdx.z;
  const int group = head / (p.heads / p.groups), inner = p.heads * vp;
  uint8_t *Bt = smem, *Ct = Bt + 2 * kChunk * kPitchN, *Xt = Ct + 2 * kChunk * kPitchN, *Ph = Xt + 2 * kChunk * pitch_v, *Pl = Ph + kChunk * kPitchP;
  float *cums = reinterpret_cast<float*>(Pl + kChunk * kPitchP), *dtss = cums + 2 * kChunk;
  const __nv_bfloat16* xbc = reinterpret_cast<const __nv_bfloat16*>(p.xbc);
  const __nv_bfloat16 *xs = xbc + head * vp, *bs = xbc + inner + group * NP, *cs = bs + p.groups * NP;
  __nv_bfloat16* ys = reinterpret_cast<__nv_bfloat16*>(p.y) + head * vp;
  const float bias = FIXED ? 0.0f : p.dt_bias[head], a2 = FIXED ? -p.decay[3 * head] : expf(p.log_a[head]) * 1.4426950408889634f, skip = FIXED ? 0.0f : p.skip[head];
  float* st = p.state + ((size_t)p.state_slots[seq] * p.heads + head) * NP * vp;
  float S[NT][4];   // state channels 16 m + g, + 8; values v0 + 2 t, + 1
#pragma unroll
  for (int m = 0; m < NT; ++m) {
    float2 a = make_float2(0.f, 0.f), b = a;
    const float* from = PART == kOutputs ? segs.state + ((size_t)entry * p.heads + head) * NP * vp : st;
    if (PART == kOutputs || (PART == kWhole && !p.fresh[seq])) {
      a = *reinterpret_cast<const float2*>(from + (size_t)(16 * m + g) * vp + v0 + 2 * t);
      b = *reinterpret_cast<const float2*>(from + (size_t)(16 * m + g + 8) * vp + v0 + 2 * t);
    }
    S[m][0] = a.x; S[m][1] = a.y; S[m][2] = b.x; S[m][3] = b.y;
  }
  auto stage = [&](int tb, int buf) {
    const int n = min(kChunk, t1 - tb);
    stage_tile(Bt + buf * kChunk * kPitchN, kPitchN, bs + (int64_t)tb * p.ld_xbc, p.ld_xbc, n, NP);
    if (PART != kStates) stage_tile(Ct + buf * kChunk * kPitchN, kPitchN, cs + (int64_t)tb * p.ld_xbc, p.ld_xbc, n, NP);
    stage_tile(Xt + buf * kChunk * pitch_v, pitch_v, xs + (int64_t)tb * p.ld_xbc, p.ld_xbc, n, vp);
    cp_async_commit();
  };
  float dt_raw[2] = {0.f, 0.f};
  auto fetch_dt = [&](int tb) {
#pragma unroll
    for (int i = 0; i < 2 && !FIXED; ++i) dt_raw[i] = tb + lane + 32 * i < t1 ? p.dt[(size_t)(tb + lane + 32 * i) * p.ld_dt + head] : 0.0f;
  };
  // step sizes and log2-decays of a chunk summed up by one warp; tokens past the end take no step
  auto sum_decays = [&](int tb, int to) {
    const int n = min(kChunk, t1 - tb);
    const float d0 = lane < n ? (FIXED ? 1.0f : softplus_f(dt_raw[0] + bias)) : 0.0f, d1 = lane + 32 < n ? (FIXED ? 1.0f : softplus_f(dt_raw[1] + bias)) : 0.0f;
    float c0 = -a2 * d0, c1 = -a2 * d1;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float u0 = __shfl_up_sync(0xffffffffu, c0, d), u1 = __shfl_up_sync(0xffffffffu, c1, d);
      if (lane >= d) { c0 += u0; c1 += u1; }
    }
    c1 += __shfl_sync(0xffffffffu, c0, 31);
    cums[to * kChunk + lane] = c0; cums[to * kChunk + lane + 32] = c1;
    dtss[to * kChunk + lane] = d0; dtss[to * kChunk + lane + 32] = d1;
  };
  stage(t0, 0);
  if (warp == 0) { fetch_dt(t0); sum_decays(t0, 0); }
  float total = 0.0f;     // log2 of the decay so far
  int buf = 0, turn = 0;  // the warp whose turn it is prepares the next chunk's decays
  for (int tb = t0; tb < t1; tb += kChunk, buf ^= 1, turn = turn + 1 < n_warps ? turn + 1 : 0) {
    const int n = min(kChunk, t1 - tb);
    const float *cum = cums + buf * kChunk, *dts = dtss + buf * kChunk;
    cp_async_wait<0>();
    __syncthreads();
    if (tb + kChunk < t1) {
      stage(tb + kChunk, buf ^ 1);
      if (warp == turn) fetch_dt(tb + kChunk);
    }
    const uint32_t B_a = smem_u32(Bt + buf * kChunk * kPitchN), C_a = smem_u32(Ct + buf * kChunk * kPitchN), X_a = smem_u32(Xt + buf * kChunk * pitch_v);
    // ---- P: sixteen by sixteen blocks on and below the diagonal, dealt to the warps
    for (int b = warp; b < 10 && PART != kStates; b += n_warps) {
      const int I = b < 4 ? 3 : b < 7 ? 2 : b < 9 ? 1 : 0, J = b - (b < 4 ? 0 : b < 7 ? 4 : b < 9 ? 7 : 9);
      float acc[2][4] = {};
#pragma unroll
      for (int ks = 0; ks < NT; ++ks) {
        uint32_t a[4], bb[4];
        frag_a(a, C_a, kPitchN, 16 * I, 16 * ks, lane);
        frag_b(bb, B_a, kPitchN, 16 * J, 16 * ks, lane);
        mma(acc[0], a, bb[0], bb[1]);
        mma(acc[1], a, bb[2], bb[3]);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int i = 16 * I + g + 8 * h, j = 16 * J + 8 * nt + 2 * t;
          const float w0 = j <= i ? acc[nt][2 * h] * fast_exp2(cum[i] - cum[j]) * dts[j] : 0.0f;
          const float w1 = j + 1 <= i ? acc[nt][2 * h + 1] * fast_exp2(cum[i] - cum[j + 1]) * dts[j + 1] : 0.0f;
          uint32_t hi, lo;
          split2(w0, w1, hi, lo);
          *reinterpret_cast<uint32_t*>(Ph + i * kPitchP + j * 2) = hi;
          *reinterpret_cast<uint32_t*>(Pl + i * kPitchP + j * 2) = lo;
        }
    }
    __syncthreads();
    // ---- outputs of this warp's eight values
    float acc[4][4] = {};
#pragma unroll
    for (int ks = 0; ks < NT && PART != kStates; ++ks) {
      uint32_t hi[2], lo[2];
      state_operand(S[ks], hi, lo);
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) {
        uint32_t a[4];
        frag_a(a, C_a, kPitchN, 16 * mt, 16 * ks, lane);
        mma(acc[mt], a, hi[0], hi[1]);
        mma(acc[mt], a, lo[0], lo[1]);
      }
    }
    uint32_t xb[2][4];
    frag_bt(xb[0], X_a, pitch_v, 0, v0, lane);
    frag_bt(xb[1], X_a, pitch_v, 32, v0, lane);
    const uint32_t Ph_a = smem_u32(Ph), Pl_a = smem_u32(Pl);
#pragma unroll
    for (int mt = 0; mt < 4 && PART != kStates; ++mt) {
      const float e0 = fast_exp2(cum[16 * mt + g]), e1 = fast_exp2(cum[16 * mt + g + 8]);
      acc[mt][0] *= e0; acc[mt][1] *= e0; acc[mt][2] *= e1; acc[mt][3] *= e1;
#pragma unroll
      for (int kt = 0; kt <= mt; ++kt) {
        uint32_t a[4];
        frag_a(a, Ph_a, kPitchP, 16 * mt, 16 * kt, lane);
        mma(acc[mt], a, xb[kt >> 1][2 * (kt & 1)], xb[kt >> 1][2 * (kt & 1) + 1]);
        frag_a(a, Pl_a, kPitchP, 16 * mt, 16 * kt, lane);
        mma(acc[mt], a, xb[kt >> 1][2 * (kt & 1)], xb[kt >> 1][2 * (kt & 1) + 1]);
      }
#pragma unroll
      for (int h = 0; h < 2; ++h) {  // D x; the result takes the place of x (columns that only this warp reads)
        uint32_t* at = reinterpret_cast<uint32_t*>(Xt + buf * kChunk * pitch_v + (16 * mt + g + 8 * h) * pitch_v + (v0 + 2 * t) * 2);
        const float2 x = unpack_bf16x2(*at);
        *at = pack_bf16x2(fmaf(skip, x.x, acc[mt][2 * h]), fmaf(skip, x.y, acc[mt][2 * h + 1]));
      }
    }
    // ---- state
    const float c_last = cum[kChunk - 1], e_last = fast_exp2(c_last);
    total += c_last;
#pragma unroll
    for (int m = 0; m < NT; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[m][e] *= e_last;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      uint32_t hi[2], lo[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int j = 16 * kt + 8 * h + 2 * t;
        const float2 x = unpack_bf16x2(xb[kt >> 1][2 * (kt & 1) + h]);
        split2(x.x * dts[j] * fast_exp2(c_last - cum[j]), x.y * dts[j + 1] * fast_exp2(c_last - cum[j + 1]), hi[h], lo[h]);
      }
#pragma unroll
      for (int m = 0; m < NT; ++m) {
        uint32_t a[4];
        frag_at(a, B_a, kPitchN, 16 * m, 16 * kt, lane);
        mma(S[m], a, hi[0], hi[1]);
        mma(S[m], a, lo[0], lo[1]);
      }
    }
    if (warp == turn && tb + kChunk < t1) sum_decays(tb + kChunk, buf ^ 1);
    __syncthreads();
    const int pieces_v = vp >> 3, lg_v = 31 - __clz(pieces_v);
    for (int e = tid; e < n * pieces_v && PART != kStates; e += blockDim.x) {
      const int row = e >> lg_v, piece = e & (pieces_v - 1);
      *reinterpret_cast<uint4*>(ys + (int64_t)(tb + row) * p.ld_y + piece * 8) =
          *reinterpret_cast<const uint4*>(Xt + buf * kChunk * pitch_v + row * pitch_v + piece * 16);
    }
  }
  if (PART == kOutputs && t1 < end) return;
  float* to = PART == kStates ? segs.state + ((size_t)(entry + 1) * p.heads + head) * NP * vp : st;
  if (PART == kStates && tid == 0) segs.decay[(size_t)(entry + 1) * p.heads + head] = total;
#pragma unroll
  for (int m = 0; m < NT; ++m) {
    *reinterpret_cast<float2*>(to + (size_t)(16 * m + g) * vp + v0 + 2 * t) = make_float2(S[m][0], S[m][1]);
    *reinterpret_cast<float2*>(to + (size_t)(16 * m + g + 8) * vp + v0 + 2 * t) = make_float2(S[m][2], S[m][3]);
  }
}

// The states that the segments of a sequence start with: a thread owns four values of one head
__global__ void __launch_bounds__(256)
ssd_scan_kernel(SsdArgs p, Segments segs) {
  lg::pdl_prologue();
  const int seq = blockIdx.y, len = p.cu[seq + 1] - p.cu[seq], n = (len + kSegment - 1) / kSegment, per_head = p.np * p.vp / 4;
  const int64_t width = (int64_t)p.heads * per_head, at = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (at >= width || n == 0) return;
  const int head = (int)(at / per_head);
  float4* entry = reinterpret_cast<float4*>(segs.state) + first_entry(p.cu, seq) * width + at;
  const float* decay = segs.decay + (size_t)first_entry(p.cu, seq) * p.heads + head;
  float4 S = p.fresh[seq] ? make_float4(0.f, 0.f, 0.f, 0.f) : reinterpret_cast<const float4*>(p.state)[p.state_slots[seq] * width + at];
  entry[0] = S;
  constexpr int kBatch = 4;   // segments in flight
  for (int g0 = 1; g0 < n; g0 += kBatch) {
    float4 own[kBatch];
    float e[kBatch];
#pragma unroll
    for (int i = 0; i < kBatch; ++i) {
      const bool in = g0 + i < n;
      own[i] = in ? entry[(g0 + i) * width] : make_float4(0.f, 0.f, 0.f, 0.f);
      e[i] = in ? exp2f(decay[(size_t)(g0 + i) * p.heads]) : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < kBatch; ++i) {
      S = make_float4(fmaf(e[i], S.x, own[i].x), fmaf(e[i], S.y, own[i].y), fmaf(e[i], S.z, own[i].z), fmaf(e[i], S.w, own[i].w));
      if (g0 + i < n) entry[(g0 + i) * width] = S;
    }
  }
}

// y silu(z), normalised in equal parts of `width` contiguous bf16 channels: a warp per (row, part), NV times eight
// channels per lane. AFTER: y is normalised and then multiplied by sigmoid(z).
template <int NV, bool AFTER>
__global__ void __launch_bounds__(256)
gated_norm_warp_kernel(const __nv_bfloat16* __restrict__ y, int ld_y, const __nv_bfloat16* __restrict__ z, int ld_z, const float* __restrict__ gain,
                       __nv_bfloat16* __restrict__ out, int ld_out, int rows, int parts, int width, float eps) {
  lg::pdl_prologue();
  const int64_t item = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= (int64_t)rows * parts) return;
  const int r = (int)(item / parts), c0 = (int)(item % parts) * width, lane = threadIdx.x & 31;
  uint4 a[NV], b[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = 8 * (lane + 32 * i);
    a[i] = b[i] = make_uint4(0u, 0u, 0u, 0u);
    if (c < width) {
      a[i] = *reinterpret_cast<const uint4*>(y + (size_t)r * ld_y + c0 + c);
      b[i] = *reinterpret_cast<const uint4*>(z + (size_t)r * ld_z + c0 + c);
    }
  }
  float x[NV][8], ss = 0.0f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const uint32_t wa[4] = {a[i].x, a[i].y, a[i].z, a[i].w}, wb[4] = {b[i].x, b[i].y, b[i].z, b[i].w};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 fa = unpack_bf16x2(wa[k]), fb = unpack_bf16x2(wb[k]);
      x[i][2 * k] = AFTER ? fa.x : fa.x * silu_bf16(fb.x);
      x[i][2 * k + 1] = AFTER ? fa.y : fa.y * silu_bf16(fb.y);
      ss = fmaf(x[i][2 * k], x[i][2 * k], fmaf(x[i][2 * k + 1], x[i][2 * k + 1], ss));
    }
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)width + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = 8 * (lane + 32 * i);
    if (c >= width) continue;
    const float4 g0 = __ldg(reinterpret_cast<const float4*>(gain + c0 + c)), g1 = __ldg(reinterpret_cast<const float4*>(gain + c0 + c + 4));
    if (AFTER) {
      const uint32_t wb[4] = {b[i].x, b[i].y, b[i].z, b[i].w};
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 fb = unpack_bf16x2(wb[k]);
        x[i][2 * k] *= __fdividef(1.0f, 1.0f + __expf(-fb.x));
        x[i][2 * k + 1] *= __fdividef(1.0f, 1.0f + __expf(-fb.y));
      }
    }
    *reinterpret_cast<uint4*>(out + (size_t)r * ld_out + c0 + c) =
        make_uint4(pack_bf16x2(x[i][0] * inv * g0.x, x[i][1] * inv * g0.y), pack_bf16x2(x[i][2] * inv * g0.z, x[i][3] * inv * g0.w),
                   pack_bf16x2(x[i][4] * inv * g1.x, x[i][5] * inv * g1.y), pack_bf16x2(x[i][6] * inv * g1.z, x[i][7] * inv * g1.w));
  }
}

// The same for any width and format, a CTA per (row, part). VEC: channels are contiguous (no
// padding between heads) and eight of them are moved at once.
// KM: pieces of eight channels per thread
template <typename T, bool VEC, bool AFTER, int KM = 1>
__global__ void __launch_bounds__(512)
gated_group_norm_kernel(const T* __restrict__ y, int ld_y, const T* __restrict__ z, int ld_z, const float* __restrict__ gain, T* __restrict__ out,
                        int ld_out, int width, int v, int vp, float eps) {
  lg::pdl_prologue();
  __shared__ float red[32];
  const int r = blockIdx.x, c0 = blockIdx.y * width;
  const T *yr = y + (size_t)r * ld_y, *zr = z + (size_t)r * ld_z;
  T* o = out + (size_t)r * ld_out;
  if constexpr (VEC) {
    float x[KM][8], after[AFTER ? KM : 1][8];  // width <= KM * 8 * 512
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < KM; ++i) {
      const int c = 8 * (threadIdx.x + i * blockDim.x);
      if (c >= width) break;
      float a[8], g[8];
      if constexpr (sizeof(T) == 2) {
        const uint4 ua = *reinterpret_cast<const uint4*>(yr + c0 + c), ug = *reinterpret_cast<const uint4*>(zr + c0 + c);
        const uint32_t wa[4] = {ua.x, ua.y, ua.z, ua.w}, wg[4] = {ug.x, ug.y, ug.z, ug.w};
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float2 fa = unpack_bf16x2(wa[k]), fg = unpack_bf16x2(wg[k]);
          a[2 * k] = fa.x; a[2 * k + 1] = fa.y; g[2 * k] = fg.x; g[2 * k + 1] = fg.y;
        }
      } else {
#pragma unroll
        for (int k = 0; k < 8; ++k) { a[k] = yr[c0 + c + k]; g[k] = zr[c0 + c + k]; }
      }
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        x[i][k] = AFTER ? a[k] : a[k] * (sizeof(T) == 2 ? __fdividef(g[k], 1.0f + __expf(-g[k])) : silu_f(g[k]));
        if (AFTER) after[AFTER ? i : 0][k] = sizeof(T) == 2 ? __fdividef(1.0f, 1.0f + __expf(-g[k])) : sigmoid_f(g[k]);
        ss += x[i][k] * x[i][k];
      }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
#pragma unroll
    for (int i = 0; i < KM; ++i) {
      const int c = 8 * (threadIdx.x + i * blockDim.x);
      if (c >= width) break;
      const float4 g0 = __ldg(reinterpret_cast<const float4*>(gain + c0 + c)), g1 = __ldg(reinterpret_cast<const float4*>(gain + c0 + c + 4));
      float w[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
#pragma unroll
      for (int k = 0; k < 8 && AFTER; ++k) w[k] *= after[AFTER ? i : 0][k];
      if constexpr (sizeof(T) == 2) {
        uint32_t u[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) u[k] = pack_bf16x2(x[i][2 * k] * inv * w[2 * k], x[i][2 * k + 1] * inv * w[2 * k + 1]);
        *reinterpret_cast<uint4*>(o + c0 + c) = make_uint4(u[0], u[1], u[2], u[3]);
      } else {
#pragma unroll
        for (int k = 0; k < 8; ++k) o[c0 + c + k] = x[i][k] * inv * w[k];
      }
    }
  } else {
    auto col = [&](int c) { const int ch = c0 + c; return (ch / v) * vp + ch % v; };
    float ss = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      const float x = Io<T>::load(yr + col(c)) * (AFTER ? 1.0f : silu_f(Io<T>::load(zr + col(c))));
      ss += x * x;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      const int k = col(c);
      const float g = Io<T>::load(zr + k);
      Io<T>::store(o + k, Io<T>::load(yr + k) * (AFTER ? sigmoid_f(g) : silu_f(g)) * inv * gain[k]);
    }
  }
}

bool pow2(int v, int lo, int hi) { return v >= lo && v <= hi && (v & (v - 1)) == 0; }

bool args_ok(const lg_ssd_t* a, int n_seqs) {
  if (a && a->decay)
    return n_seqs > 0 && n_seqs <= 65535 && a->xbc && a->state && a->state_slots && a->fresh && a->cu && a->y && a->heads > 0 && a->groups == a->heads && pow2(a->np, 16, 256) &&
           pow2(a->vp, 16, 256) && a->ld_y >= a->heads * a->vp;
  return a && n_seqs > 0 && n_seqs <= 65535 && a->proj && a->dt && a->conv_w && a->conv_b && a->dt_bias && a->log_a && a->skip && a->state && a->state_slots &&
         a->fresh && a->phase && a->cu && a->y && a->taps >= 1 && a->taps <= kMaxTaps && (a->taps == 1 || a->conv_state) && a->heads > 0 && a->groups > 0 &&
         a->heads % a->groups == 0 && pow2(a->np, 16, 256) && pow2(a->vp, 16, 256) && a->ld >= 2 * a->heads * a->vp + 2 * a->groups * a->np &&
         a->ld_y >= a->heads * a->vp && a->ld_dt >= a->heads;
}

SsdArgs make_args(const lg_ssd_t* a) {
  return SsdArgs{a->proj, a->ld, (const float*)a->dt, a->ld_dt, (const float*)a->conv_w, (const float*)a->conv_b, (float*)a->conv_state, a->taps,
                 (const float*)a->dt_bias, (const float*)a->log_a, (const float*)a->skip, (float*)a->state, (const int*)a->state_slots,
                 (const uint8_t*)a->fresh, (const uint8_t*)a->phase, (const int*)a->cu, a->y, a->ld_y, a->heads, a->groups, a->np, a->vp, a->xbc, a->ld_xbc, (const float*)a->decay};
}

template <bool AFTER>
uint32_t launch_gated_norm(const void* y, int32_t ld_y, const void* z, int32_t ld_z, const void* gain_f32, void* out, int32_t ld_out, int32_t is_f32,
                           int32_t rows, int32_t heads, int32_t v, int32_t vp, int32_t parts, float eps, void* stream) {
  if (!y || !z || !gain_f32 || !out || rows <= 0 || heads <= 0 || v <= 0 || vp < v || parts <= 0 || parts > 65535 || (heads * v) % parts || ld_y < heads * vp ||
      ld_z < heads * vp || ld_out < heads * vp)
    return lg::kInvalidValue;
  const int width = heads * v / parts;
  const bool vec = v == vp && width % 8 == 0 && width <= 4 * 8 * 512 && ld_y % 8 == 0 && ld_z % 8 == 0 && ld_out % 8 == 0;
  int threads = ((vec ? width / 8 : width) + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  if (!is_f32 && vec && width <= 2048) {
    auto warp = [&](auto kern) {
      lg::launch(kern, dim3((unsigned)(((int64_t)rows * parts + 7) / 8)), dim3(256), 0, (cudaStream_t)stream, (const __nv_bfloat16*)y, ld_y, (const __nv_bfloat16*)z, ld_z,
                 (const float*)gain_f32, (__nv_bfloat16*)out, ld_out, rows, parts, width, eps);
      return lg::launch_status();
    };
    return width <= 256 ? warp(gated_norm_warp_kernel<1, AFTER>) : width <= 512 ? warp(gated_norm_warp_kernel<2, AFTER>) : width <= 1024 ? warp(gated_norm_warp_kernel<4, AFTER>)
                                                                                                           : warp(gated_norm_warp_kernel<8, AFTER>);
  }
  const dim3 grid((unsigned)rows, (unsigned)parts);
  auto go = [&](auto kern, auto* t) {
    using T = std::remove_pointer_t<decltype(t)>;
    lg::launch(kern, grid, dim3((unsigned)threads), 0, (cudaStream_t)stream, (const T*)y, ld_y, (const T*)z, ld_z, (const float*)gain_f32, (T*)out, ld_out, width, v, vp, eps);
    return lg::launch_status();
  };
  auto pick = [&](auto* t) {
    using T = std::remove_pointer_t<decltype(t)>;
    if (!vec) return go(gated_group_norm_kernel<T, false, AFTER>, t);
    return width <= 4096 ? go(gated_group_norm_kernel<T, true, AFTER, 1>, t) : go(gated_group_norm_kernel<T, true, AFTER, 4>, t);
  };
  return is_f32 ? pick((float*)nullptr) : pick((__nv_bfloat16*)nullptr);
}

}  // namespace

extern "C" {

uint32_t logismos_launch_ssd_step(const lg_ssd_t* a, int32_t n_seqs, int32_t is_f32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!args_ok(a, n_seqs)) return lg::kInvalidValue;
  if (!a->xbc || a->ld_xbc < make_args(a).channels()) return lg::kInvalidValue;
  const SsdArgs p = make_args(a);
  const size_t smem = state_smem(p.np, p.vp);
  auto go = [&](auto kern) -> uint32_t {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
    lg::launch(kern, dim3((unsigned)p.heads, (unsigned)n_seqs), dim3(kThreads), smem, (cudaStream_t)stream, p, smem > 0 ? 1 : 0);
    return lg::launch_status();
  };
  if (p.decay) return is_f32 ? go(ssd_step_kernel<float, true>) : go(ssd_step_kernel<__nv_bfloat16, true>);
  return is_f32 ? go(ssd_step_kernel<float, false>) : go(ssd_step_kernel<__nv_bfloat16, false>);
}

int32_t logismos_ssd_has_chunked(int32_t np, int32_t vp) { return pow2(np, 32, 128) && pow2(vp, 16, 128) ? 1 : 0; }

uint32_t logismos_launch_ssd_conv(const lg_ssd_t* a, const void* seq_ids_i32, int32_t row0, int32_t rows, int32_t single, int32_t is_f32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!args_ok(a, 1) || a->decay || !seq_ids_i32 || row0 < 0 || rows <= row0 || !a->xbc || a->ld % 4 || a->ld_xbc % 4 || a->ld_xbc < make_args(a).channels()) return lg::kInvalidValue;
  const SsdArgs p = make_args(a);
  const int* ids = (const int*)seq_ids_i32;
  cudaStream_t s = (cudaStream_t)stream;
  if (is_f32) return launch_conv<float, 1>(p, ids, row0, rows, s);
  return single ? launch_conv<__nv_bfloat16, 1>(p, ids, row0, rows, s) : launch_conv<__nv_bfloat16, 16>(p, ids, row0, rows, s);
}

int32_t logismos_ssd_segments(int32_t rows, int32_t n_seqs, int32_t longest, int32_t heads) {
  // Measured (us, whole / segments; 64 x 128 states): 4 prompts of 1024, 8 / 16 / 32 heads 71 / 40, 71 / 60, 73 / 107; one of 16384, 8 /
  // 32 heads 1075 / 126, 1077 / 415. Whole sequences take 4.4 us per 64 tokens of the longest, segments 0.052 us per 64 tokens and head.
  return longest > 2 * kSegment && (int64_t)rows * heads < (int64_t)72 * longest ? rows / kSegment + n_seqs + 1 : 0;
}

size_t logismos_ssd_scratch_bytes(int32_t entries, int32_t heads, int32_t np, int32_t vp) {
  return entries <= 0 ? 0 : (size_t)entries * heads * ((size_t)np * vp + 4) * 4;
}

uint32_t logismos_launch_ssd_chunked_bf16(const lg_ssd_t* a, int32_t n_seqs, void* stream) { return logismos_launch_ssd_segmented_bf16(a, n_seqs, 0, nullptr, 0, stream); }

uint32_t logismos_launch_ssd_segmented_bf16(const lg_ssd_t* a, int32_t n_seqs, int32_t longest, void* scratch, int32_t entries, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!args_ok(a, n_seqs) || !logismos_ssd_has_chunked(a->np, a->vp) || !a->xbc || a->ld_xbc % 8 || a->ld_y % 8 || (((uintptr_t)a->xbc | (uintptr_t)a->y) & 15) ||
      (entries > 0 && (!scratch || ((uintptr_t)scratch & 15) || longest <= 0 || longest > 65535 * kSegment)))
    return lg::kInvalidValue;
  const SsdArgs p = make_args(a);
  const size_t smem = ssd_chunk_smem(a->np, a->vp);
  const bool cut = entries > 0;
  Segments segs{(float*)scratch, (float*)scratch + (size_t)(cut ? entries : 0) * p.heads * p.np * p.vp};
  const int per_seq = cut ? (longest + kSegment - 1) / kSegment : 1;
  auto go = [&](auto kern, int n) -> uint32_t {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
    lg::launch(kern, dim3((unsigned)p.heads, (unsigned)n_seqs, (unsigned)n), dim3((unsigned)(4 * p.vp)), smem, (cudaStream_t)stream, p, segs);
    return lg::launch_status();
  };
#define LG_PART(FIXED, PART, N) (a->np == 32 ? go(ssd_chunk_kernel<32, FIXED, PART>, N) : a->np == 64 ? go(ssd_chunk_kernel<64, FIXED, PART>, N) : go(ssd_chunk_kernel<128, FIXED, PART>, N))
  if (!cut) return p.decay ? LG_PART(true, kWhole, 1) : LG_PART(false, kWhole, 1);
  if (per_seq > 1)
    if (uint32_t rc = p.decay ? LG_PART(true, kStates, per_seq - 1) : LG_PART(false, kStates, per_seq - 1)) return rc;
  const int64_t width = (int64_t)p.heads * p.np * p.vp / 4;
  lg::launch(ssd_scan_kernel, dim3((unsigned)((width + 255) / 256), (unsigned)n_seqs), dim3(256), 0, (cudaStream_t)stream, p, segs);
  if (uint32_t rc = lg::launch_status()) return rc;
  return p.decay ? LG_PART(true, kOutputs, per_seq) : LG_PART(false, kOutputs, per_seq);
#undef LG_PART
}

uint32_t logismos_launch_gated_group_norm(const void* y, int32_t ld_y, const void* z, int32_t ld_z, const void* gain_f32, void* out, int32_t ld_out,
                                          int32_t is_f32, int32_t rows, int32_t heads, int32_t v, int32_t vp, int32_t parts, float eps,
                                          void* stream) {
  lg::LaunchScope launch_scope_;
  return launch_gated_norm<false>(y, ld_y, z, ld_z, gain_f32, out, ld_out, is_f32, rows, heads, v, vp, parts, eps, stream);
}

uint32_t logismos_launch_norm_gate(const void* y, int32_t ld_y, const void* z, int32_t ld_z, const void* gain_f32, void* out, int32_t ld_out, int32_t is_f32,
                                   int32_t rows, int32_t heads, int32_t v, int32_t vp, float eps, void* stream) {
  lg::LaunchScope launch_scope_;
  return launch_gated_norm<true>(y, ld_y, z, ld_z, gain_f32, out, ld_out, is_f32, rows, heads, v, vp, 1, eps, stream);
}

}  // extern "C"
