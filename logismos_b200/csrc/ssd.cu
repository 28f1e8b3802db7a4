// State-space mixer with a scalar decay per head (Mamba-2, state-space duality). A projected row is [z | x | B | C]
// in the activation format, H heads of VP values and G groups of NP state channels, and dt per head in fp32. x, B
// and C pass a causal depthwise convolution and silu; then per head (B, C of its group)
//   dt <- softplus(dt + bias);  S <- exp(-exp(log_a) dt) S + dt B x^T;  y = S^T C + D x
// and over the heads y silu(z), each of several equal parts divided by its root mean square, times a gain.
// State, step sizes, decays, convolution sums and norms are fp32. NP and VP are powers of two with zero padding.
// The last taps - 1 inputs of the convolution are its state: a slot holds two copies, a step reads the one its
// phase names and writes the other.
//
// ssd_step_kernel: CTA = (head, sequence), tokens one after the other, convolution included. Decode steps, fp32.
#include "common.cuh"
#include "logismos_kernels.h"
#include "recurrent.cuh"

namespace {

using namespace lg;
using namespace lg::rec;

constexpr int kMaxTaps = 8, kMaxChannels = 768;  // VP + 2 NP of a head

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
  const void* xbc;         // convolved channels (the chunked form)
  int ld_xbc;
  LG_DEVINL int channels() const { return heads * vp + 2 * groups * np; }
};

template <typename T, int PT>
__global__ void __launch_bounds__(kThreads)
ssd_step_kernel(SsdArgs p) {
  lg::pdl_trigger();
  constexpr int NP = PT ? PT : 1;
  extern __shared__ float hist[];   // [taps - 1][local channels] raw inputs
  __shared__ float act[kMaxChannels], red[8 * 128];
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int vp = p.vp, np = p.np, group = head / (p.heads / p.groups), inner = p.heads * vp, nch = vp + 2 * np, all = p.channels();
  const bool owns_group = head % (p.heads / p.groups) == 0;
  const Tile t(np, vp);
  const size_t slot = (size_t)p.state_slots[seq];
  float* st = p.state + (slot * p.heads + head) * np * vp;
  const bool fresh = p.fresh[seq] != 0;
  const int ph = p.phase[seq] & 1, keep = p.taps - 1;
  const float* old = p.conv_state + (slot * 2 + ph) * keep * all;
  float* next = p.conv_state + (slot * 2 + 1 - ph) * keep * all;
  const int t0 = p.cu[seq], t1 = p.cu[seq + 1];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  // channel of the convolution behind local channel c
  auto chan = [&](int c) { return c < vp ? head * vp + c : c < vp + np ? inner + group * np + c - vp : inner + (p.groups + group) * np + c - vp - np; };
  // states of an earlier step and weights do not depend on the kernels before this one
  float4 S[NP];
  if (PT) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int row = t.r0 + i * t.step;
      S[i] = !fresh && row < np ? *reinterpret_cast<const float4*>(st + (size_t)row * vp + t.c4) : zero;
    }
  }
  for (int e = tid; e < keep * nch; e += kThreads) hist[e] = fresh ? 0.0f : old[(size_t)(e / nch) * all + chan(e % nch)];
  const float bias = __ldg(p.dt_bias + head), a = expf(__ldg(p.log_a + head)), skip = __ldg(p.skip + head);
  lg::pdl_wait();
  __syncthreads();
  int at = 0;  // oldest row of hist
  for (int tok = t0; tok < t1; ++tok) {
    const T* row = reinterpret_cast<const T*>(p.proj) + (size_t)tok * p.ld + inner;
    const float dt = softplus_f(p.dt[(size_t)tok * p.ld_dt + head] + bias), decay = expf(-a * dt);
    for (int c = tid; c < nch; c += kThreads) {  // a thread meets the same channels for every token
      const int g = chan(c);
      const float cur = Io<T>::load(row + g);
      float s = fmaf(__ldg(p.conv_w + (size_t)keep * all + g), cur, __ldg(p.conv_b + g));
      for (int j = 0; j < keep; ++j) {
        const int r = at + j < keep ? at + j : at + j - keep;
        s = fmaf(__ldg(p.conv_w + (size_t)j * all + g), hist[r * nch + c], s);
      }
      if (keep > 0) hist[at * nch + c] = cur;
      act[c] = silu_f(s);
    }
    if (keep > 0 && ++at == keep) at = 0;
    __syncthreads();
    const float4 x4 = *reinterpret_cast<const float4*>(act + t.c4);
    const float4 dx = make_float4(dt * x4.x, dt * x4.y, dt * x4.z, dt * x4.w);
    float4 o = zero;
    auto visit = [&](int r, float4& s) {
      const float b = act[vp + r], c = act[vp + np + r];
      s = make_float4(fmaf(decay, s.x, b * dx.x), fmaf(decay, s.y, b * dx.y), fmaf(decay, s.z, b * dx.z), fmaf(decay, s.w, b * dx.w));
      o.x = fmaf(c, s.x, o.x); o.y = fmaf(c, s.y, o.y); o.z = fmaf(c, s.z, o.z); o.w = fmaf(c, s.w, o.w);
    };
    if (PT) {
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int r = t.r0 + i * t.step;
        if (r < np) visit(r, S[i]);
      }
    } else {
      for (int r = t.r0; r < np; r += t.step) {
        float4* q = reinterpret_cast<float4*>(st + (size_t)r * vp + t.c4);
        float4 s = fresh && tok == t0 ? zero : *q;
        visit(r, s);
        *q = s;
      }
    }
    reduce_store(t, o, red);
    __syncthreads();
    if (tid < vp) Io<T>::store(reinterpret_cast<T*>(p.y) + (size_t)tok * p.ld_y + head * vp + tid, reduce_load(vp, red, tid) + skip * act[tid]);
    if (tok + 1 < t1) __syncthreads();
  }
  if (PT) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int row = t.r0 + i * t.step;
      if (row < np) *reinterpret_cast<float4*>(st + (size_t)row * vp + t.c4) = S[i];
    }
  }
  __syncthreads();
  for (int e = tid; e < keep * nch; e += kThreads) {
    const int j = e / nch, c = e % nch;
    if (c < vp || owns_group) next[(size_t)j * all + chan(c)] = hist[((at + j) % keep) * nch + c];
  }
}

// y silu(z), normalised in equal parts of `width` channels. CTA = (row, part). VEC: channels are contiguous (no
// padding between heads) and eight of them are moved at once.
template <typename T, bool VEC>
__global__ void __launch_bounds__(512)
gated_group_norm_kernel(const T* __restrict__ y, int ld_y, const T* __restrict__ z, int ld_z, const float* __restrict__ gain, T* __restrict__ out,
                        int ld_out, int width, int v, int vp, float eps) {
  lg::pdl_prologue();
  __shared__ float red[32];
  const int r = blockIdx.x, c0 = blockIdx.y * width;
  const T *yr = y + (size_t)r * ld_y, *zr = z + (size_t)r * ld_z;
  T* o = out + (size_t)r * ld_out;
  if constexpr (VEC) {
    constexpr int kMax = 4;  // width <= 4 * 8 * 512
    float x[kMax][8];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < kMax; ++i) {
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
      for (int k = 0; k < 8; ++k) { x[i][k] = a[k] * (sizeof(T) == 2 ? __fdividef(g[k], 1.0f + __expf(-g[k])) : silu_f(g[k])); ss += x[i][k] * x[i][k]; }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
#pragma unroll
    for (int i = 0; i < kMax; ++i) {
      const int c = 8 * (threadIdx.x + i * blockDim.x);
      if (c >= width) break;
      const float4 g0 = __ldg(reinterpret_cast<const float4*>(gain + c0 + c)), g1 = __ldg(reinterpret_cast<const float4*>(gain + c0 + c + 4));
      const float w[8] = {g0.x, g0.y, g0.z, g0.w, g1.x, g1.y, g1.z, g1.w};
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
      const float x = Io<T>::load(yr + col(c)) * silu_f(Io<T>::load(zr + col(c)));
      ss += x * x;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
      const int k = col(c);
      Io<T>::store(o + k, Io<T>::load(yr + k) * silu_f(Io<T>::load(zr + k)) * inv * gain[k]);
    }
  }
}

bool pow2(int v, int lo, int hi) { return v >= lo && v <= hi && (v & (v - 1)) == 0; }

bool args_ok(const lg_ssd_t* a, int n_seqs) {
  return a && n_seqs > 0 && n_seqs <= 65535 && a->proj && a->dt && a->conv_w && a->conv_b && a->dt_bias && a->log_a && a->skip && a->state && a->state_slots &&
         a->fresh && a->phase && a->cu && a->y && a->taps >= 1 && a->taps <= kMaxTaps && (a->taps == 1 || a->conv_state) && a->heads > 0 && a->groups > 0 &&
         a->heads % a->groups == 0 && pow2(a->np, 16, 256) && pow2(a->vp, 16, 256) && a->ld >= 2 * a->heads * a->vp + 2 * a->groups * a->np &&
         a->ld_y >= a->heads * a->vp && a->ld_dt >= a->heads;
}

SsdArgs make_args(const lg_ssd_t* a) {
  return SsdArgs{a->proj, a->ld, (const float*)a->dt, a->ld_dt, (const float*)a->conv_w, (const float*)a->conv_b, (float*)a->conv_state, a->taps,
                 (const float*)a->dt_bias, (const float*)a->log_a, (const float*)a->skip, (float*)a->state, (const int*)a->state_slots,
                 (const uint8_t*)a->fresh, (const uint8_t*)a->phase, (const int*)a->cu, a->y, a->ld_y, a->heads, a->groups, a->np, a->vp, a->xbc, a->ld_xbc};
}

}  // namespace

extern "C" {

uint32_t logismos_launch_ssd_step(const lg_ssd_t* a, int32_t n_seqs, int32_t is_f32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!args_ok(a, n_seqs)) return lg::kInvalidValue;
  const SsdArgs p = make_args(a);
  const size_t smem = (size_t)(p.taps - 1) * (p.vp + 2 * p.np) * 4;
  auto go = [&](auto kern) {
    lg::launch(kern, dim3((unsigned)p.heads, (unsigned)n_seqs), dim3(kThreads), smem, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
  const int pt = pieces(p.np, p.vp);
#define LG_STEP(T) pt == 1 ? go(ssd_step_kernel<T, 1>) : pt == 2 ? go(ssd_step_kernel<T, 2>) : pt == 4 ? go(ssd_step_kernel<T, 4>) : pt == 8 ? go(ssd_step_kernel<T, 8>) \
                   : pt == 16 ? go(ssd_step_kernel<T, 16>) : go(ssd_step_kernel<T, 0>)
  return is_f32 ? (LG_STEP(float)) : (LG_STEP(__nv_bfloat16));
#undef LG_STEP
}

uint32_t logismos_launch_gated_group_norm(const void* y, int32_t ld_y, const void* z, int32_t ld_z, const void* gain_f32, void* out, int32_t ld_out,
                                          int32_t is_f32, int32_t rows, int32_t heads, int32_t v, int32_t vp, int32_t parts, float eps,
                                          void* stream) {
  lg::LaunchScope launch_scope_;
  if (!y || !z || !gain_f32 || !out || rows <= 0 || heads <= 0 || v <= 0 || vp < v || parts <= 0 || parts > 65535 || (heads * v) % parts || ld_y < heads * vp ||
      ld_z < heads * vp || ld_out < heads * vp)
    return lg::kInvalidValue;
  const int width = heads * v / parts;
  const bool vec = v == vp && width % 8 == 0 && width <= 4 * 8 * 512 && ld_y % 8 == 0 && ld_z % 8 == 0 && ld_out % 8 == 0;
  int threads = ((vec ? width / 8 : width) + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const dim3 grid((unsigned)rows, (unsigned)parts);
  auto go = [&](auto kern, auto* t) {
    using T = std::remove_pointer_t<decltype(t)>;
    lg::launch(kern, grid, dim3((unsigned)threads), 0, (cudaStream_t)stream, (const T*)y, ld_y, (const T*)z, ld_z, (const float*)gain_f32, (T*)out, ld_out, width, v, vp, eps);
    return lg::launch_status();
  };
  if (is_f32) return vec ? go(gated_group_norm_kernel<float, true>, (float*)nullptr) : go(gated_group_norm_kernel<float, false>, (float*)nullptr);
  return vec ? go(gated_group_norm_kernel<__nv_bfloat16, true>, (__nv_bfloat16*)nullptr) : go(gated_group_norm_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)nullptr);
}

}  // extern "C"
