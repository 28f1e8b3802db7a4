// Time mixing with a decay per key channel that depends on the data (RWKV): per head, with r, k, the decay w and
// the bonus u over D key channels and v over D value channels,
//   o_t = (S + diag(u) k_t v_t^T)^T r_t;   S <- diag(w_t) S + k_t v_t^T;   w_t = exp(-exp(z_t))
// and the head's epilogue: o / rms(o) * gain * silu(g) * scale. State, decays, sums and norm are fp32.
// Heads are padded to DP = 32, 64, 128 or 256 channels with zeros.
//
// time_mix_step_kernel: CTA = (head, sequence), tokens one after the other. Decode steps, fp32, head sizes
// above 128. z comes from a buffer, or is computed from the low-rank activations: z = W2 low + w0.
#include "common.cuh"
#include "logismos_kernels.h"
#include "recurrent.cuh"

namespace {

using namespace lg;
using namespace lg::rec;

struct MixArgs {
  const void* proj;        // activation format; r, k, v, g of head h at column off_* + h * DP
  int ld, off_r, off_k, off_v, off_g;
  const float* z;          // [rows, ld_z], head h at h * DP (NULL: from low)
  int ld_z;
  const float* low;        // [rows, ld_low]
  int ld_low;
  const __nv_bfloat16* w2; // [heads * DP, ld_w2], rank columns used (a multiple of 32)
  int ld_w2, rank;
  const float* w0;         // [heads * DP]
  const float* u;
  const float* gain;
  float* state;            // [n_slots][heads][DP][DP]
  const int* state_slots;
  const uint8_t* fresh;
  const int* cu;
  void* out;               // activation format, head h at h * DP
  int ld_out;
  int heads, d, dp;
  float scale, eps;
};

template <typename T, int PT>
__global__ void __launch_bounds__(kThreads)
time_mix_step_kernel(MixArgs p) {
  lg::pdl_trigger();
  constexpr int NP = PT ? PT : 1;
  __shared__ float sr[256], sk[256], sv[256], sw[256], red[8 * 128], bred[32];
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int dp = p.dp, h0 = head * dp;
  const Tile t(dp, dp);
  float* st = p.state + ((size_t)p.state_slots[seq] * p.heads + head) * dp * dp;
  const bool fresh = p.fresh[seq] != 0;
  const int t0 = p.cu[seq], t1 = p.cu[seq + 1];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  // the state, left by an earlier step, and the weights do not depend on the kernels before this one
  float4 S[NP];
  if (PT) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int row = t.r0 + i * t.step;
      S[i] = !fresh && row < dp ? *reinterpret_cast<const float4*>(st + (size_t)row * dp + t.c4) : zero;
    }
  }
  float uu = 0.0f, w0 = 0.0f, gain = 0.0f;
  __shared__ float su[256];
  if (tid < dp) { uu = __ldg(p.u + h0 + tid); w0 = __ldg(p.w0 + h0 + tid); gain = __ldg(p.gain + h0 + tid); su[tid] = uu; }
  constexpr int kAhead = 4;  // 16-byte pieces of W2 per thread requested ahead: four threads per channel, 64 channels
  uint4 wv[kAhead];
  const int ch0 = tid >> 2, part = tid & 3;
#pragma unroll
  for (int j = 0; j < kAhead; ++j) {
    wv[j] = make_uint4(0u, 0u, 0u, 0u);
    if (!p.z && ch0 < dp && 32 * j < p.rank) wv[j] = __ldg(reinterpret_cast<const uint4*>(p.w2 + (size_t)(h0 + ch0) * p.ld_w2 + 32 * j + 8 * part));
  }
  lg::pdl_wait();
  for (int tok = t0; tok < t1; ++tok) {
    const T* row = reinterpret_cast<const T*>(p.proj) + (size_t)tok * p.ld + h0;
    float g = 0.0f, z = 0.0f;
    if (tid < dp) {
      sr[tid] = Io<T>::load(row + p.off_r + tid);
      sk[tid] = Io<T>::load(row + p.off_k + tid);
      sv[tid] = Io<T>::load(row + p.off_v + tid);
      g = Io<T>::load(row + p.off_g + tid);
      if (p.z) z = p.z[(size_t)tok * p.ld_z + h0 + tid];
    }
    if (!p.z) {
      const float* low = p.low + (size_t)tok * p.ld_low;
      for (int ch = ch0; ch < dp; ch += 64) {
        float s = 0.0f;
        for (int j0 = 0; j0 < p.rank; j0 += 32 * kAhead) {
#pragma unroll
          for (int j = 0; j < kAhead; ++j) {
            const int c = j0 + 32 * j + 8 * part;
            if (c - 8 * part >= p.rank) break;
            const uint4 w = ch == ch0 && j0 == 0 ? wv[j] : __ldg(reinterpret_cast<const uint4*>(p.w2 + (size_t)(h0 + ch) * p.ld_w2 + c));
            const float4 a = *reinterpret_cast<const float4*>(low + c), b = *reinterpret_cast<const float4*>(low + c + 4);
            const float2 w01 = unpack_bf16x2(w.x), w23 = unpack_bf16x2(w.y), w45 = unpack_bf16x2(w.z), w67 = unpack_bf16x2(w.w);
            s = fmaf(a.x, w01.x, fmaf(a.y, w01.y, fmaf(a.z, w23.x, fmaf(a.w, w23.y, s))));
            s = fmaf(b.x, w45.x, fmaf(b.y, w45.y, fmaf(b.z, w67.x, fmaf(b.w, w67.y, s))));
          }
        }
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        if (part == 0) sw[ch] = s;
      }
      __syncthreads();
      if (tid < dp) z = sw[tid] + w0;
    }
    if (tid < dp) sw[tid] = expf(-expf(z));
    __syncthreads();
    const float4 v4 = *reinterpret_cast<const float4*>(sv + t.c4);
    float4 o = zero;
    auto visit = [&](int r, float4& s) {
      const float kr = sk[r], rr = sr[r], wr = sw[r], ur = su[r];
      const float4 kv = make_float4(kr * v4.x, kr * v4.y, kr * v4.z, kr * v4.w);
      o.x = fmaf(rr, fmaf(ur, kv.x, s.x), o.x);
      o.y = fmaf(rr, fmaf(ur, kv.y, s.y), o.y);
      o.z = fmaf(rr, fmaf(ur, kv.z, s.z), o.z);
      o.w = fmaf(rr, fmaf(ur, kv.w, s.w), o.w);
      s = make_float4(fmaf(wr, s.x, kv.x), fmaf(wr, s.y, kv.y), fmaf(wr, s.z, kv.z), fmaf(wr, s.w, kv.w));
    };
    if (PT) {
#pragma unroll
      for (int i = 0; i < NP; ++i) {
        const int r = t.r0 + i * t.step;
        if (r < dp) visit(r, S[i]);
      }
    } else {
      for (int r = t.r0; r < dp; r += t.step) {
        float4* at = reinterpret_cast<float4*>(st + (size_t)r * dp + t.c4);
        float4 s = fresh && tok == t0 ? zero : *at;
        visit(r, s);
        *at = s;
      }
    }
    reduce_store(t, o, red);
    __syncthreads();
    const float oc = tid < dp ? reduce_load(dp, red, tid) : 0.0f;
    const float inv = 1.0f / sqrtf(block_sum(oc * oc, bred) / (float)p.d + p.eps);  // its barriers also free the vectors above
    if (tid < dp) Io<T>::store(reinterpret_cast<T*>(p.out) + (size_t)tok * p.ld_out + h0 + tid, oc * inv * gain * silu_f(g) * p.scale);
  }
  if (PT) {
#pragma unroll
    for (int i = 0; i < NP; ++i) {
      const int row = t.r0 + i * t.step;
      if (row < dp) *reinterpret_cast<float4*>(st + (size_t)row * dp + t.c4) = S[i];
    }
  }
}

bool args_ok(const lg_time_mix_t* a, int n_seqs) {
  return a && n_seqs > 0 && n_seqs <= 65535 && a->proj && a->state && a->state_slots && a->fresh && a->cu && a->out && a->u && a->gain && a->heads > 0 &&
         (a->dp == 32 || a->dp == 64 || a->dp == 128 || a->dp == 256) && a->d > 0 && a->d <= a->dp && a->ld_out >= a->heads * a->dp &&
         (a->z ? a->ld_z >= a->heads * a->dp : a->low && a->w2 && a->w0 && a->rank > 0 && a->rank % 32 == 0 && a->ld_low >= a->rank && a->ld_low % 4 == 0 &&
                                                   a->ld_w2 >= a->rank && a->ld_w2 % 8 == 0 && (((uintptr_t)a->low | (uintptr_t)a->w2) & 15) == 0);
}

MixArgs make_args(const lg_time_mix_t* a) {
  return MixArgs{a->proj, a->ld, a->off_r, a->off_k, a->off_v, a->off_g, (const float*)a->z, a->ld_z, (const float*)a->low, a->ld_low,
                 (const __nv_bfloat16*)a->w2, a->ld_w2, a->rank, (const float*)a->w0, (const float*)a->u, (const float*)a->gain, (float*)a->state,
                 (const int*)a->state_slots, (const uint8_t*)a->fresh, (const int*)a->cu, a->out, a->ld_out, a->heads, a->d, a->dp, a->scale, a->eps};
}

}  // namespace

extern "C" {

uint32_t logismos_launch_time_mix_step(const lg_time_mix_t* a, int32_t n_seqs, int32_t is_f32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!args_ok(a, n_seqs)) return lg::kInvalidValue;
  const MixArgs p = make_args(a);
  auto go = [&](auto kern) {
    lg::launch(kern, dim3((unsigned)p.heads, (unsigned)n_seqs), dim3(kThreads), 0, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
#define LG_STEP(T) p.dp == 32 ? go(time_mix_step_kernel<T, 1>) : p.dp == 64 ? go(time_mix_step_kernel<T, 4>) : p.dp == 128 ? go(time_mix_step_kernel<T, 16>) : go(time_mix_step_kernel<T, 0>)
  return is_f32 ? (LG_STEP(float)) : (LG_STEP(__nv_bfloat16));
#undef LG_STEP
}

}  // extern "C"
