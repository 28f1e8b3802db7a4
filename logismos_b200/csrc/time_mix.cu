// Linear attention with a decay per key channel that depends on the data: per head, with r, k and the decay w over the
// key channels and v over the value channels, in two forms (LG_DECAY_*)
//   time mixing (RWKV)  o_t = (S + diag(u) k_t v_t^T)^T r_t;   S <- diag(w_t) S + k_t v_t^T;   w_t = exp(-exp(z_t))
//   gated               S <- diag(w_t) S + k_t v_t^T;   o_t = q_scale S^T r_t;   w_t = sigmoid(z_t)^(1 / tau)
// and the head's epilogue: o / rms(o) * gain * silu(g) * scale. State, decays, sums and norm are fp32.
// Key and value heads are padded to 32, 64, 128 or 256 channels with zeros.
//
// time_mix_step_kernel: CTA = (head, sequence), tokens one after the other. Decode steps, fp32, head sizes
// above 128. z comes from a buffer, or is computed from the low-rank activations: z = W2 low + w0.
//
// time_mix_chunk_kernel: prompts, CTA = (head, sequence), 64 tokens at a time in four blocks of 16. With c_i the sum
// of log w inside a block up to its token i, T the block's total and S the state before the block,
//   R_i = r_i exp(c_(i-1));  K_j = k_j exp(T - c_j)
//   o_i = S^T R_i + sum_(j < i) (R_i exp(-T) . K_j) v_j + (r_i . u k_i) v_i;   S <- diag(exp(T)) S + sum_j K_j v_j^T
// (the gated form: R_i = q_scale r_i exp(c_i), the last product with 1 for u).
// R and K need one exponential per element and stay below r and k in size; the product with exp(-T) is taken where
// exp(T) does not underflow, else the block's coefficients are summed directly. The products run on mma.sync; what
// is fp32 (R, K, the state, the coefficients) goes in as a rounded bf16 part and a remainder.
#include "common.cuh"
#include "logismos_kernels.h"
#include "recurrent.cuh"

namespace {

using namespace lg;
using namespace lg::rec;

struct MixArgs {
  const void* proj;        // activation format; r, k of head h at column off_* + h * dp, v, g at off_* + h * vp
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
  float* state;            // [n_slots][heads][dp][vp]
  const int* state_slots;
  const uint8_t* fresh;
  const int* cu;
  void* out;               // activation format, head h at h * vp
  int ld_out;
  int heads, d, dp, vp;
  float scale, eps, tau, q_scale;
};

// log2 of the gated form's decay, sigmoid(z)^(1 / tau)
LG_DEVINL float gated_log2(float z, float inv_tau) { return -1.4426950408889634f * inv_tau * (fmaxf(-z, 0.0f) + log1pf(expf(-fabsf(z)))); }

template <typename T, bool GATED>
__global__ void __launch_bounds__(kThreads, 4)
time_mix_step_kernel(MixArgs p, int in_smem) {
  lg::pdl_trigger();
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ __align__(16) float sr[256], sk[256], sv[256], sw[256], su[256], red[1024], ssq[8];
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int dp = p.dp, vp = GATED ? p.vp : dp, h0 = head * dp, v0 = head * vp;
  const Tile t(dp, vp);
  const bool fresh = p.fresh[seq] != 0;
  // the state, left by an earlier step, and the weights do not depend on the kernels before this one
  State S(smem, in_smem, p.state + ((size_t)p.state_slots[seq] * p.heads + head) * dp * vp);
  S.request(t, fresh);
  const int t0 = p.cu[seq], t1 = p.cu[seq + 1];
  float w0 = 0.0f, gain = 0.0f;
  if (tid < dp) {
    w0 = __ldg(p.w0 + h0 + tid);
    if (!GATED) su[tid] = __ldg(p.u + h0 + tid);
  }
  if (tid < vp) gain = __ldg(p.gain + v0 + tid);
  lg::pdl_wait();
  for (int tok = t0; tok < t1; ++tok) {
    const T* row = reinterpret_cast<const T*>(p.proj) + (size_t)tok * p.ld;
    float z = 0.0f, g = 0.0f;
    if (tid < vp) {
      sv[tid] = Io<T>::load(row + p.off_v + v0 + tid);
      g = Io<T>::load(row + p.off_g + v0 + tid);
    }
    if (tid < dp) {
      sr[tid] = Io<T>::load(row + p.off_r + h0 + tid) * (GATED ? p.q_scale : 1.0f);
      sk[tid] = Io<T>::load(row + p.off_k + h0 + tid);
      if (p.z) z = p.z[(size_t)tok * p.ld_z + h0 + tid];
    }
    if (!p.z) {  // four threads per channel, eight of its columns at a time
      const float* low = p.low + (size_t)tok * p.ld_low;
      for (int ch = tid >> 2; ch < dp; ch += 64) {
        const __nv_bfloat16* wr = p.w2 + (size_t)(h0 + ch) * p.ld_w2;
        float s = 0.0f;
#pragma unroll 2
        for (int c = 8 * (tid & 3); c < p.rank; c += 32) {
          const uint4 w = __ldg(reinterpret_cast<const uint4*>(wr + c));
          const float4 a = *reinterpret_cast<const float4*>(low + c), b = *reinterpret_cast<const float4*>(low + c + 4);
          const float2 w01 = unpack_bf16x2(w.x), w23 = unpack_bf16x2(w.y), w45 = unpack_bf16x2(w.z), w67 = unpack_bf16x2(w.w);
          s = fmaf(a.x, w01.x, fmaf(a.y, w01.y, fmaf(a.z, w23.x, fmaf(a.w, w23.y, s))));
          s = fmaf(b.x, w45.x, fmaf(b.y, w45.y, fmaf(b.z, w67.x, fmaf(b.w, w67.y, s))));
        }
        s += __shfl_xor_sync(0xffffffffu, s, 1);
        s += __shfl_xor_sync(0xffffffffu, s, 2);
        if ((tid & 3) == 0) sw[ch] = s;
      }
      __syncthreads();
      if (tid < dp) z = sw[tid] + w0;
    }
    if (tid < dp) sw[tid] = GATED ? exp2f(gated_log2(z, 1.0f / p.tau)) : expf(-expf(z));
    __syncthreads();
    if (tok == t0) S.arrived();
    const float4 v4 = *reinterpret_cast<const float4*>(sv + t.c4);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    S.visit(t, fresh && tok == t0, tok + 1 == t1, [&](int r, float4& s) {
      const float kr = sk[r], rr = sr[r], wr = sw[r];
      const float4 kv = make_float4(kr * v4.x, kr * v4.y, kr * v4.z, kr * v4.w);
      if (!GATED) {
        const float ur = su[r];
        o.x = fmaf(rr, fmaf(ur, kv.x, s.x), o.x);
        o.y = fmaf(rr, fmaf(ur, kv.y, s.y), o.y);
        o.z = fmaf(rr, fmaf(ur, kv.z, s.z), o.z);
        o.w = fmaf(rr, fmaf(ur, kv.w, s.w), o.w);
      }
      s = make_float4(fmaf(wr, s.x, kv.x), fmaf(wr, s.y, kv.y), fmaf(wr, s.z, kv.z), fmaf(wr, s.w, kv.w));
      if (GATED) {
        o.x = fmaf(rr, s.x, o.x);
        o.y = fmaf(rr, s.y, o.y);
        o.z = fmaf(rr, s.z, o.z);
        o.w = fmaf(rr, s.w, o.w);
      }
    });
    reduce_store(t, o, red);
    __syncthreads();
    const float oc = tid < vp ? reduce_load(vp, red, tid) : 0.0f;
    const float part = warp_sum(oc * oc);
    if ((tid & 31) == 0) ssq[tid >> 5] = part;
    __syncthreads();
    if (tid < vp) {
      float ss = 0.0f;
      for (int i = 0; i < vp / 32; ++i) ss += ssq[i];
      Io<T>::store(reinterpret_cast<T*>(p.out) + (size_t)tok * p.ld_out + v0 + tid, oc * (p.scale / sqrtf(ss / (float)p.d + p.eps)) * gain * silu_f(g));
    }
    if (tok + 1 < t1) __syncthreads();
  }
}

template <int DP, int VP> struct ChunkCfg {
  static constexpr int kMax = DP > VP ? DP : VP, kThreadsC = 4 * kMax, kPitch = DP * 2 + 16, kTile = kChunk * kPitch, kPitchV = VP * 2 + 16, kTileV = kChunk * kPitchV,
                       kPitchC = kMax + 8, kPitchA = 16 * 2 + 16;
  // r, k, v twice; remainders of R and K; block sums (later the outputs) fp32; coefficients, two parts; totals, bonus, u, gain
  static constexpr size_t kSmem = 6 * (size_t)kTile + 2 * kTileV + kChunk * kPitchC * 4 + 2 * kChunk * kPitchA + 4 * DP * 4 + kChunk * 4 + (DP + VP) * 4;
};
constexpr float kMaxSpan = 100.0f;  // log2 of the decay over a block up to which exp(-T) is taken

template <int DP, int VP, bool GATED>
__global__ void __launch_bounds__(4 * (DP > VP ? DP : VP))
time_mix_chunk_kernel(MixArgs p) {
  lg::pdl_prologue();
  using C = ChunkCfg<DP, VP>;
  constexpr int NT = DP / 16, kOct = DP / 8, kOctV = VP / 8, kPitch = C::kPitch, kPitchV = C::kPitchV, kPitchC = C::kPitchC, kPitchA = C::kPitchA;
  extern __shared__ __align__(16) uint8_t smem[];
  uint8_t *Rt = smem, *Kt = Rt + 2 * C::kTile, *Vt = Kt + 2 * C::kTile, *Rl = Vt + 2 * C::kTileV, *Kl = Rl + C::kTile;
  float* cs = reinterpret_cast<float*>(Kl + C::kTile);
  uint8_t *Ah = reinterpret_cast<uint8_t*>(cs + kChunk * kPitchC), *Al = Ah + kChunk * kPitchA;
  float *tot = reinterpret_cast<float*>(Al + kChunk * kPitchA), *bonus = tot + 4 * DP, *us = bonus + kChunk, *gains = us + DP;
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t = lane & 3, v0 = 8 * warp, h0 = head * DP, hv = head * VP;
  const bool owner = DP <= VP || warp < kOctV;  // of eight value columns
  const int t0 = p.cu[seq], t1 = p.cu[seq + 1];
  if (t1 <= t0) return;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(p.proj);
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + hv;
  float* st = p.state + ((size_t)p.state_slots[seq] * p.heads + head) * DP * VP;
  const float inv_tau = GATED ? 1.0f / p.tau : 0.0f, q_scale = GATED ? p.q_scale : 1.0f;
  float S[NT][4];   // key channels 16 m + g, + 8; values v0 + 2 t, + 1
#pragma unroll
  for (int m = 0; m < NT; ++m) {
    float2 a = make_float2(0.f, 0.f), b = a;
    if (owner && !p.fresh[seq]) {
      a = *reinterpret_cast<const float2*>(st + (size_t)(16 * m + g) * VP + v0 + 2 * t);
      b = *reinterpret_cast<const float2*>(st + (size_t)(16 * m + g + 8) * VP + v0 + 2 * t);
    }
    S[m][0] = a.x; S[m][1] = a.y; S[m][2] = b.x; S[m][3] = b.y;
  }
  auto stage = [&](int tb, int buf) {
    const int n = min(kChunk, t1 - tb);
    const __nv_bfloat16* row = proj + (int64_t)tb * p.ld;
    stage_tile(Rt + buf * C::kTile, kPitch, row + p.off_r + h0, p.ld, n, DP);
    stage_tile(Kt + buf * C::kTile, kPitch, row + p.off_k + h0, p.ld, n, DP);
    stage_tile(Vt + buf * C::kTileV, kPitchV, row + p.off_v + hv, p.ld, n, VP);
    cp_async_commit();
  };
  const int zc = tid % DP, zb = tid / DP;  // channel and block of 16 tokens whose log-decays this thread sums
  const bool sums = DP >= VP || zb < 4;
  float z[16];
  auto fetch_z = [&](int tb) {
#pragma unroll
    for (int i = 0; i < 16; ++i) z[i] = sums && tb + 16 * zb + i < t1 ? p.z[(size_t)(tb + 16 * zb + i) * p.ld_z + h0 + zc] : GATED ? INFINITY : -INFINITY;
  };
  stage(t0, 0);
  fetch_z(t0);
  if (!GATED && tid < DP) us[tid] = p.u[h0 + tid];
  if (tid < VP) gains[tid] = p.gain[hv + tid];
  int buf = 0;
  for (int tb = t0; tb < t1; tb += kChunk, buf ^= 1) {
    const int n = min(kChunk, t1 - tb);
    if (sums) {
      float c = 0.0f;
#pragma unroll
      for (int i = 0; i < 16; ++i) {  // past the end: no decay
        c = GATED ? c + gated_log2(z[i], inv_tau) : fmaf(fast_exp2(z[i] * 1.4426950408889634f), -1.4426950408889634f, c);
        cs[(16 * zb + i) * kPitchC + zc] = c;
      }
      tot[zb * DP + zc] = c;
    }
    cp_async_wait<0>();
    __syncthreads();
    if (tb + kChunk < t1) {
      stage(tb + kChunk, buf ^ 1);
      fetch_z(tb + kChunk);
    }
    uint8_t *R = Rt + buf * C::kTile, *K = Kt + buf * C::kTile;
    // ---- R and K in two parts (the rounded ones in place), and r . u k
    for (int e = tid; e < kChunk * kOct; e += C::kThreadsC) {
      const int row = e / kOct, d0 = 8 * (e % kOct);
      const uint4 ru = *reinterpret_cast<const uint4*>(R + row * kPitch + d0 * 2), ku = *reinterpret_cast<const uint4*>(K + row * kPitch + d0 * 2);
      const uint32_t rw[4] = {ru.x, ru.y, ru.z, ru.w}, kw[4] = {ku.x, ku.y, ku.z, ku.w};
      uint32_t rh[4], rl[4], kh[4], kl[4];
      float dot = 0.0f;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int d = d0 + 2 * q;
        const float2 r = unpack_bf16x2(rw[q]), k = unpack_bf16x2(kw[q]);
        const float2 c = *reinterpret_cast<const float2*>(cs + row * kPitchC + d), tt = *reinterpret_cast<const float2*>(tot + (row >> 4) * DP + d);
        const float2 cp = GATED ? c : (row & 15) ? *reinterpret_cast<const float2*>(cs + (row - 1) * kPitchC + d) : make_float2(0.f, 0.f);
        const float2 u = GATED ? make_float2(q_scale, q_scale) : *reinterpret_cast<const float2*>(us + d);
        dot = fmaf(r.x * u.x, k.x, fmaf(r.y * u.y, k.y, dot));
        split2(r.x * q_scale * fast_exp2(cp.x), r.y * q_scale * fast_exp2(cp.y), rh[q], rl[q]);
        split2(k.x * fast_exp2(tt.x - c.x), k.y * fast_exp2(tt.y - c.y), kh[q], kl[q]);
      }
#pragma unroll
      for (int o = 1; o < kOct; o <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
      if (d0 == 0) bonus[row] = dot;
      *reinterpret_cast<uint4*>(R + row * kPitch + d0 * 2) = make_uint4(rh[0], rh[1], rh[2], rh[3]);
      *reinterpret_cast<uint4*>(Rl + row * kPitch + d0 * 2) = make_uint4(rl[0], rl[1], rl[2], rl[3]);
      *reinterpret_cast<uint4*>(K + row * kPitch + d0 * 2) = make_uint4(kh[0], kh[1], kh[2], kh[3]);
      *reinterpret_cast<uint4*>(Kl + row * kPitch + d0 * 2) = make_uint4(kl[0], kl[1], kl[2], kl[3]);
    }
    __syncthreads();
    const uint32_t R_a = smem_u32(R), K_a = smem_u32(K), V_a = smem_u32(Vt + buf * C::kTileV), Rl_a = smem_u32(Rl), Kl_a = smem_u32(Kl);
    // the gates of the epilogue, requested now
    uint4 gate[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int e = tid + i * C::kThreadsC, row = e / kOctV;
      gate[i] = row < n ? *reinterpret_cast<const uint4*>(proj + (int64_t)(tb + row) * p.ld + p.off_g + hv + 8 * (e % kOctV)) : make_uint4(0u, 0u, 0u, 0u);
    }
    // ---- coefficients inside the blocks, eight columns j at a time
    for (int task = warp; task < 8; task += C::kThreadsC / 32) {
      const int I = task >> 1, nt = task & 1;
      float worst = 0.0f;
      for (int d = lane; d < DP; d += 32) worst = fmaxf(worst, -tot[I * DP + d]);
      float acc[4] = {}, low1[4] = {}, low2[4] = {};
      if (__all_sync(0xffffffffu, worst <= kMaxSpan)) {
#pragma unroll
        for (int ks = 0; ks < NT; ++ks) {
          uint32_t ah[4], al[4], bh[4], bl[4];
          frag_a(ah, R_a, kPitch, 16 * I, 16 * ks, lane);
          frag_a(al, Rl_a, kPitch, 16 * I, 16 * ks, lane);
          frag_b(bh, K_a, kPitch, 16 * I, 16 * ks, lane);
          frag_b(bl, Kl_a, kPitch, 16 * I, 16 * ks, lane);
          const uint32_t h0 = nt ? bh[2] : bh[0], h1 = nt ? bh[3] : bh[1], l0 = nt ? bl[2] : bl[0], l1 = nt ? bl[3] : bl[1];
#pragma unroll
          for (int q = 0; q < 4; ++q) {  // columns 2 t (+ 8 for q >= 2)
            const float2 f = *reinterpret_cast<const float2*>(tot + I * DP + 16 * ks + 8 * (q >> 1) + 2 * t);
            const float2 x = unpack_bf16x2(ah[q]), y = unpack_bf16x2(al[q]);
            split2((x.x + y.x) * fast_exp2(-f.x), (x.y + y.y) * fast_exp2(-f.y), ah[q], al[q]);
          }
          mma(acc, ah, h0, h1);
          mma(low1, al, h0, h1);
          mma(low2, ah, l0, l1);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[e] += low1[e] + low2[e];
      } else {  // some channel decays too far: term by term, with exponents c_(i-1) - c_j <= 0
        const __nv_bfloat16 *rs = proj + p.off_r + h0, *ks_ = proj + p.off_k + h0;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = 16 * I + g + 8 * (e >> 1), j = 16 * I + 8 * nt + 2 * t + (e & 1);
          if (j >= i || i >= n) continue;
          float s = 0.0f;
          for (int d = 0; d < DP; ++d)
            s = fmaf(__bfloat162float(rs[(int64_t)(tb + i) * p.ld + d]) * __bfloat162float(ks_[(int64_t)(tb + j) * p.ld + d]),
                     fast_exp2(cs[(GATED ? i : i - 1) * kPitchC + d] - cs[j * kPitchC + d]), s);
          acc[e] = s * q_scale;
        }
      }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int i = g + 8 * h, j = 8 * nt + 2 * t;
        const float b = bonus[16 * I + i];
        uint32_t hi, lo;
        split2(j < i ? acc[2 * h] : j == i ? b : 0.0f, j + 1 < i ? acc[2 * h + 1] : j + 1 == i ? b : 0.0f, hi, lo);
        *reinterpret_cast<uint32_t*>(Ah + (16 * I + i) * kPitchA + j * 2) = hi;
        *reinterpret_cast<uint32_t*>(Al + (16 * I + i) * kPitchA + j * 2) = lo;
      }
    }
    __syncthreads();
    // ---- outputs of this warp's eight values and the state, block by block
    if (owner) {
    uint32_t vb[2][4];
    frag_bt(vb[0], V_a, kPitchV, 0, v0, lane);
    frag_bt(vb[1], V_a, kPitchV, 32, v0, lane);
    const uint32_t Ah_a = smem_u32(Ah), Al_a = smem_u32(Al);
#pragma unroll
    for (int I = 0; I < 4; ++I) {
      const uint32_t b0 = vb[I >> 1][2 * (I & 1)], b1 = vb[I >> 1][2 * (I & 1) + 1];
      float acc[4] = {}, low1[4] = {}, low2[4] = {};  // separate sums: the products do not wait for one another
      uint32_t a[4];
      frag_a(a, Ah_a, kPitchA, 16 * I, 0, lane);
      mma(low1, a, b0, b1);
      frag_a(a, Al_a, kPitchA, 16 * I, 0, lane);
      mma(low2, a, b0, b1);
#pragma unroll
      for (int ks = 0; ks < NT; ++ks) {
        uint32_t hi[2], lo[2];
        state_operand(S[ks], hi, lo);
        frag_a(a, R_a, kPitch, 16 * I, 16 * ks, lane);
        mma(acc, a, hi[0], hi[1]);
        mma(low1, a, lo[0], lo[1]);
        frag_a(a, Rl_a, kPitch, 16 * I, 16 * ks, lane);
        mma(low2, a, hi[0], hi[1]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[e] += low1[e] + low2[e];
      *reinterpret_cast<float2*>(cs + (16 * I + g) * kPitchC + v0 + 2 * t) = make_float2(acc[0], acc[1]);  // the block sums are no longer needed
      *reinterpret_cast<float2*>(cs + (16 * I + g + 8) * kPitchC + v0 + 2 * t) = make_float2(acc[2], acc[3]);
#pragma unroll
      for (int m = 0; m < NT; ++m) {
        const float e0 = fast_exp2(tot[I * DP + 16 * m + g]), e1 = fast_exp2(tot[I * DP + 16 * m + g + 8]);
        S[m][0] *= e0; S[m][1] *= e0; S[m][2] *= e1; S[m][3] *= e1;
        frag_at(a, K_a, kPitch, 16 * m, 16 * I, lane);
        mma(S[m], a, b0, b1);
        frag_at(a, Kl_a, kPitch, 16 * m, 16 * I, lane);
        mma(S[m], a, b0, b1);
      }
    }
    }
    __syncthreads();
    // ---- norm over the head, gain, gate
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int e = tid + i * C::kThreadsC, row = e / kOctV, d0 = 8 * (e % kOctV);
      if (DP > VP && row >= kChunk) continue;  // whole warps
      const float4 a = *reinterpret_cast<const float4*>(cs + row * kPitchC + d0), b = *reinterpret_cast<const float4*>(cs + row * kPitchC + d0 + 4);
      float o[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w}, ss = 0.0f;
#pragma unroll
      for (int q = 0; q < 8; ++q) ss = fmaf(o[q], o[q], ss);
#pragma unroll
      for (int s = 1; s < kOctV; s <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
      if (row >= n) continue;
      const float inv = p.scale / sqrtf(ss / (float)p.d + p.eps);
      const uint4 gu = gate[i];
      const uint32_t gw[4] = {gu.x, gu.y, gu.z, gu.w};
      uint32_t w[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 gg = unpack_bf16x2(gw[q]), gn = *reinterpret_cast<const float2*>(gains + d0 + 2 * q);
        w[q] = pack_bf16x2(o[2 * q] * inv * gn.x * __fdividef(gg.x, 1.0f + __expf(-gg.x)), o[2 * q + 1] * inv * gn.y * __fdividef(gg.y, 1.0f + __expf(-gg.y)));
      }
      *reinterpret_cast<uint4*>(out + (int64_t)(tb + row) * p.ld_out + d0) = make_uint4(w[0], w[1], w[2], w[3]);
    }
    __syncthreads();
  }
  if (!owner) return;
#pragma unroll
  for (int m = 0; m < NT; ++m) {
    *reinterpret_cast<float2*>(st + (size_t)(16 * m + g) * VP + v0 + 2 * t) = make_float2(S[m][0], S[m][1]);
    *reinterpret_cast<float2*>(st + (size_t)(16 * m + g + 8) * VP + v0 + 2 * t) = make_float2(S[m][2], S[m][3]);
  }
}

int value_dim(const lg_time_mix_t* a) { return a->vp ? a->vp : a->dp; }
bool padded_ok(int d) { return d == 32 || d == 64 || d == 128 || d == 256; }

bool args_ok(const lg_time_mix_t* a, int n_seqs) {
  return a && n_seqs > 0 && n_seqs <= 65535 && a->proj && a->state && a->state_slots && a->fresh && a->cu && a->out && a->gain && a->heads > 0 &&
         padded_ok(a->dp) && padded_ok(value_dim(a)) && a->d > 0 && a->d <= value_dim(a) && a->ld_out >= a->heads * value_dim(a) &&
         (a->mode == LG_DECAY_GATED ? a->tau > 0.0f : a->mode == LG_DECAY_TIME_MIX && a->u && value_dim(a) == a->dp) &&
         (a->z ? a->ld_z >= a->heads * a->dp : a->low && a->w2 && a->rank > 0 && a->rank % 32 == 0 && a->ld_low >= a->rank && a->ld_low % 4 == 0 &&
                                                   a->ld_w2 >= a->rank && a->ld_w2 % 8 == 0 && (((uintptr_t)a->low | (uintptr_t)a->w2) & 15) == 0) && a->w0;
}

MixArgs make_args(const lg_time_mix_t* a) {
  return MixArgs{a->proj, a->ld, a->off_r, a->off_k, a->off_v, a->off_g, (const float*)a->z, a->ld_z, (const float*)a->low, a->ld_low,
                 (const __nv_bfloat16*)a->w2, a->ld_w2, a->rank, (const float*)a->w0, (const float*)a->u, (const float*)a->gain, (float*)a->state,
                 (const int*)a->state_slots, (const uint8_t*)a->fresh, (const int*)a->cu, a->out, a->ld_out, a->heads, a->d, a->dp, value_dim(a), a->scale, a->eps,
                 a->tau, a->q_scale};
}

}  // namespace

extern "C" {

uint32_t logismos_launch_time_mix_step(const lg_time_mix_t* a, int32_t n_seqs, int32_t is_f32, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!args_ok(a, n_seqs)) return lg::kInvalidValue;
  const MixArgs p = make_args(a);
  const size_t smem = state_smem(p.dp, p.vp);
  auto go = [&](auto kern) -> uint32_t {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
    lg::launch(kern, dim3((unsigned)p.heads, (unsigned)n_seqs), dim3(kThreads), smem, (cudaStream_t)stream, p, smem > 0 ? 1 : 0);
    return lg::launch_status();
  };
  if (a->mode == LG_DECAY_GATED) return is_f32 ? go(time_mix_step_kernel<float, true>) : go(time_mix_step_kernel<__nv_bfloat16, true>);
  return is_f32 ? go(time_mix_step_kernel<float, false>) : go(time_mix_step_kernel<__nv_bfloat16, false>);
}

int32_t logismos_time_mix_has_chunked(int32_t dp, int32_t vp) { return padded_ok(dp) && padded_ok(vp) && dp <= 128 && vp <= 128 ? 1 : 0; }

uint32_t logismos_launch_time_mix_chunked_bf16(const lg_time_mix_t* a, int32_t n_seqs, void* stream) {
  lg::LaunchScope launch_scope_;
  if (!args_ok(a, n_seqs) || !a->z || !logismos_time_mix_has_chunked(a->dp, value_dim(a)) || ((a->ld | a->ld_out | a->off_r | a->off_k | a->off_v | a->off_g) % 8) ||
      (((uintptr_t)a->proj | (uintptr_t)a->out) & 15))
    return lg::kInvalidValue;
  const MixArgs p = make_args(a);
  auto go = [&](auto kern, size_t smem, int threads) -> uint32_t {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (uint32_t)e;
    lg::launch(kern, dim3((unsigned)p.heads, (unsigned)n_seqs), dim3((unsigned)threads), smem, (cudaStream_t)stream, p);
    return lg::launch_status();
  };
#define LG_CHUNK(DP, VP, GATED) go(time_mix_chunk_kernel<DP, VP, GATED>, ChunkCfg<DP, VP>::kSmem, ChunkCfg<DP, VP>::kThreadsC)
  if (a->mode == LG_DECAY_TIME_MIX) return p.dp == 32 ? LG_CHUNK(32, 32, false) : p.dp == 64 ? LG_CHUNK(64, 64, false) : LG_CHUNK(128, 128, false);
  if (p.dp == 32) return p.vp == 32 ? LG_CHUNK(32, 32, true) : p.vp == 64 ? LG_CHUNK(32, 64, true) : LG_CHUNK(32, 128, true);
  if (p.dp == 64) return p.vp == 32 ? LG_CHUNK(64, 32, true) : p.vp == 64 ? LG_CHUNK(64, 64, true) : LG_CHUNK(64, 128, true);
  return p.vp == 32 ? LG_CHUNK(128, 32, true) : p.vp == 64 ? LG_CHUNK(128, 64, true) : LG_CHUNK(128, 128, true);
#undef LG_CHUNK
}

}  // extern "C"
