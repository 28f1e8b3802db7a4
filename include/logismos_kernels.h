/*
 * logismos_kernels.h - C ABI of the sm_100a kernel launchers.
 *
 * Convention of the reference's launchers (crates/kernels/src/<op>/mod.rs `unsafe extern "C"`
 * blocks; e.g. matmul/mod.rs:36-56 and matmul/hip/matmul_launchers.cpp:14-52), kept for every
 * entry point here:
 *   - the caller owns every buffer; all pointers are DEVICE pointers unless a parameter is
 *     named host_*; a launcher never allocates and never synchronises;
 *   - dims are int32; `stream` is a cudaStream_t passed as void* (NULL = the null stream);
 *   - the return value is the raw runtime status read right after the launch (0 = success); a
 *     shape the kernel cannot address is rejected before launching with cudaErrorInvalidValue
 *     (1), the counterpart of the Rust-side guards check_matmul_shape / check_rope_shape
 *     (matmul/mod.rs:89-117, rope/mod.rs:79-132).
 * The library is built as liblogismos_kernels.so (and .a, the archive name the reference's
 * build script links, crates/kernels/build.rs:117-122).
 */
#ifndef LOGISMOS_KERNELS_H
#define LOGISMOS_KERNELS_H
#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* Process-wide switch for bit-reproducible results. By default two GEMM paths split the reduction over
 * k across CTAs when few output tiles would leave SMs idle (the accumulating epilogue of
 * logismos_launch_linear_t_bf16 and the spans of logismos_launch_qlinear_int4_g32_acc_f32); the
 * slices meet in fp32 reductions whose order is not fixed, so the last bits of a result can differ
 * between runs and between a row computed alone and inside a batch (within the 2e-2 parity bar, but
 * not bit-identical). With the switch on, those splits are not used: every output element is summed in
 * one fixed order, at some cost in speed for small steps. The environment variable
 * LOGISMOS_DETERMINISTIC=1 sets the initial value. No reference counterpart (its CPU path is
 * deterministic by construction). */
void logismos_set_deterministic(int32_t on);
int32_t logismos_get_deterministic(void);

/* Process-wide switch, on by default (LOGISMOS_DEPENDENT_LAUNCH=0 sets the initial value to off): the
 * kernels of the model steps are launched with programmatic stream serialisation, i.e. the next kernel
 * of the same stream is scheduled while the current one drains and waits on the device for its
 * completion before touching memory. Results do not change; the gaps between dependent launches
 * shrink. Off, every launch is an ordinary stream-ordered launch. No reference counterpart. */
void logismos_set_dependent_launch(int32_t on);
int32_t logismos_get_dependent_launch(void);

/* ====================================================================================
 * The reference's four fp16 launchers, same symbols and argument lists.
 * ==================================================================================== */

/* crates/kernels/src/matmul/mod.rs:37-45 -> matmul_naive.hip. D[M,N] = A[M,K] B[K,N], row-major
 * fp16, fp32 accumulate. */
uint32_t logismos_launch_matmul_naive_fp16(const void* a_fp16, const void* b_fp16, void* d_fp16,
                                           int32_t m, int32_t n, int32_t k, void* stream);
/* crates/kernels/src/matmul/mod.rs:47-55 -> matmul_wmma.hip. Same contract on tensor cores; M, N,
 * K must be multiples of 16 (the only case crates/praxis/src/matmul.rs:113-117 selects it). */
uint32_t logismos_launch_matmul_wmma_fp16(const void* a_fp16, const void* b_fp16, void* d_fp16,
                                          int32_t m, int32_t n, int32_t k, void* stream);
/* crates/kernels/src/rms_norm/mod.rs:33-43 -> rms_norm.hip */
uint32_t logismos_launch_rms_norm_fp16(const void* x_fp16, const void* w_fp16, void* y_fp16,
                                       int32_t m, int32_t n, float eps, void* stream);
/* crates/kernels/src/softmax/mod.rs:28-36 -> softmax.hip. An all -inf row yields 1/n. */
uint32_t logismos_launch_softmax_fp16(const void* x_fp16, void* y_fp16, int32_t m, int32_t n,
                                      void* stream);
/* crates/kernels/src/rope/mod.rs:44-54 -> rope.hip. In-place interleaved-pair rotation of
 * (batch, seq, heads, head_dim) fp16 with an fp32 (seq, head_dim) table of (cos, sin) pairs. */
uint32_t logismos_launch_rope_fp16(void* qk_fp16, const void* cos_sin_f32, int32_t batch,
                                   int32_t seq, int32_t heads, int32_t head_dim, void* stream);

/* ====================================================================================
 * Encoder / prefill path (bf16 storage, fp32 accumulation). Each entry replaces the CPU
 * function of crates/kernels/src/cpu_f32/mod.rs named beside it.
 * ==================================================================================== */

/* cpu_f32::embed_lookup (mod.rs:106-127): out[i,:] = table[ids[i],:]; an id >= vocab yields a
 * zero row. table bf16 [vocab, hidden]; out f32 [n_ids, hidden] (the fp32 residual stream). */
uint32_t logismos_launch_embed_lookup_bf16(const void* table_bf16, const void* ids_u32,
                                           void* out_f32, int32_t n_ids, int32_t hidden,
                                           int32_t vocab, void* stream);

/* cpu_f32::rms_norm (mod.rs:137-159) over the fp32 residual stream: y = x * rsqrt(mean(x^2)+eps)
 * * w. x f32 [rows, n], w f32 [n]; y bf16 [rows, n] (out_f32 == 0) or f32 (out_f32 != 0). */
uint32_t logismos_launch_rms_norm_f32(const void* x_f32, const void* w_f32, void* y, int32_t rows,
                                      int32_t n, float eps, int32_t out_f32, void* stream);

/* cpu_f32::linear_t (mod.rs:271-345) on the tcgen05 tensor cores:  C = A W^T (+ bias).
 * A bf16 [m, k] row-major (row stride lda elements), W bf16 [n, k] row-major (the HF [out, in]
 * layout, untransposed). k % 64 == 0, n % 16 == 0, lda % 8 == 0, pointers 16-byte aligned.
 * epilogue selects what is stored:
 *   LG_EPI_BF16      out bf16 [m, n]      = acc + bias
 *   LG_EPI_RESID_F32 out f32  [m, n]     += acc + bias       (residual add, in place)
 *   LG_EPI_SWIGLU    out bf16 [m, n / 2]  = silu(gate) * up, W holding gate and up rows
 *                    interleaved in blocks of 32 rows (32 gate rows, then the 32 matching up
 *                    rows); n % 64 == 0; fuses cpu_f32::silu + hadamard (mod.rs:349-374)
 * bias_f32 may be NULL. ldc is the row stride of out in elements. status_i32 (may be NULL)
 * receives a value whose low byte is 2 if a bounded wait inside the kernel expired (the output is
 * then invalid); the next byte names the kernel family (1 dense GEMM, 2 fused-dequant linear, 3
 * tensor-core attention).
 * With few output tiles and a long reduction the accumulating epilogue splits k over CTAs; the
 * slices meet in the fp32 reduce-add, so the last bits of the sum can differ between runs.
 *
 * LG_EPI_STATIC_W, or-ed into `epilogue`, is the caller's promise that no work still in flight on the
 * stream writes `w_bf16` (model weights uploaded once). With dependent launch on, the kernel then
 * requests its first weight stages before the preceding kernel has finished. Without the flag the
 * weights are read only after everything before the launch has completed. */
enum { LG_EPI_BF16 = 0, LG_EPI_RESID_F32 = 1, LG_EPI_SWIGLU = 2, LG_EPI_STATIC_W = 0x100 };
uint32_t logismos_launch_linear_t_bf16(const void* a_bf16, const void* w_bf16,
                                       const void* bias_f32, void* out, int32_t m, int32_t n,
                                       int32_t k, int32_t lda, int32_t ldc, int32_t epilogue,
                                       void* status_i32, void* stream);
/* The same launch with the epilogues that take constants (the three epilogues above ignore them):
 *   LG_EPI_F32        out f32 [m, n]       = acc + bias, then p0 tanh(. / p0) when p0 > 0 (soft cap);
 *                     any n, ldc >= n
 *   LG_EPI_GLU_CLAMP  out bf16 [m, n / 2]  = g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u =
 *                     clamp(up, -limit, limit), alpha = p0, limit = p1, shift = p2; rows (and bias)
 *                     interleaved as for LG_EPI_SWIGLU, n % 64 == 0 */
enum { LG_EPI_F32 = 3, LG_EPI_GLU_CLAMP = 4 };
/*   LG_EPI_RELU2      out bf16 [m, n]      = max(acc + bias, 0)^2 */
enum { LG_EPI_RELU2 = 5 };
uint32_t logismos_launch_linear_t_act_bf16(const void* a_bf16, const void* w_bf16, const void* bias_f32,
                                           void* out, int32_t m, int32_t n, int32_t k, int32_t lda,
                                           int32_t ldc, int32_t epilogue, float p0, float p1, float p2,
                                           void* status_i32, void* stream);
/* The same contract for few rows (decode steps): the weights are streamed once and shared by up to 64
 * rows, the reduction order is fixed. W must be static (it is requested before the preceding kernel has
 * finished: LG_EPI_STATIC_W is implied). batch independent products are done in one launch, entry b at
 * a + b * a_stride, w + b * w_stride, out + b * out_stride (elements). All six epilogues; k % 32 == 0,
 * lda % 8 == 0, strides of a and w multiples of 8; a and w 16-byte aligned. */
uint32_t logismos_launch_linear_small_bf16(const void* a_bf16, const void* w_bf16, const void* bias_f32,
                                           void* out, int32_t m, int32_t n, int32_t k, int32_t lda,
                                           int32_t ldc, int32_t batch, int64_t a_stride, int64_t w_stride,
                                           int64_t out_stride, int32_t epilogue, float p0, float p1,
                                           float p2, void* stream);
/* The same for an output projection whose norms need no statistics: x f32 [m, ld] += post(a W^T), then h bf16 [m, ld] =
 * next(x) (next NULL: none); n <= ld columns (lg_tanh_norm_t below). */
struct lg_tanh_norm;
uint32_t logismos_launch_linear_small_tanh_norm(const void* a_bf16, const void* w_bf16, void* x_f32,
                                                const struct lg_tanh_norm* post, void* h_bf16,
                                                const struct lg_tanh_norm* next, int32_t m, int32_t n, int32_t k,
                                                int32_t lda, int32_t ld, void* stream);
/* Several projections of the same rows in one launch, each block of columns with its own input: columns
 * [end[g - 1], end[g]) of the output are rows of W applied to activation copy g, copy g standing at a + g * m *
 * lda. Columns below n_main go to out (bf16 [m, n_main], row stride ldc), the others to tail (fp32, row stride
 * ld_tail), with a soft cap tail_cap tanh(. / tail_cap) when tail_cap > 0, and (bf16 routes) when tail_parts is given
 * also there as bf16 [m, 2 (n - n_main)]: the rounded values, then what rounding dropped, so that a GEMM over [W | W]
 * sees them to about 16 bits. The ends and n_main are multiples of
 * 128 (the last end is n), n a multiple of 16. The three launchers take the routes of the three above: tcgen05
 * tiles, weights streamed once for few rows, and fp32 (out and tail fp32). */
#define LG_MAX_LINEAR_GROUPS 8
typedef struct lg_linear_groups {
  int32_t n_groups;
  int32_t end[LG_MAX_LINEAR_GROUPS];
  int32_t n_main;
  void* tail;
  int32_t ld_tail;
  float tail_cap;
  void* tail_parts;
  const void* bias;             /* f32 [n_main], added to the main columns (NULL: none) */
  int32_t silu_begin, silu_end; /* main columns that leave as z sigmoid(z); multiples of 32 (equal: none) */
} lg_linear_groups_t;
uint32_t logismos_launch_linear_groups_tc_bf16(const void* a_bf16, const void* w_bf16, void* out, int32_t m, int32_t n,
                                               int32_t k, int32_t lda, int32_t ldc, const lg_linear_groups_t* groups,
                                               void* status_i32, void* stream);
uint32_t logismos_launch_linear_groups_small_bf16(const void* a_bf16, const void* w_bf16, void* out, int32_t m, int32_t n,
                                                  int32_t k, int32_t lda, int32_t ldc, const lg_linear_groups_t* groups,
                                                  void* stream);
/* The same of one group from its sums acc f32 [m, ldc] over all n columns (which are cleared): bias, rounding and the tail.
 * For a number of rows at which accumulating over slices of k is faster than whole tiles. */
uint32_t logismos_launch_linear_groups_finish(void* acc_f32, void* out_bf16, int32_t m, int32_t n, int32_t ld_acc, int32_t ldc,
                                              const lg_linear_groups_t* groups, void* stream);
uint32_t logismos_launch_linear_groups_f32(const void* a_f32, const void* w_bf16, void* out_f32, int32_t m, int32_t n,
                                           int32_t k, int32_t lda, int32_t ldc, const lg_linear_groups_t* groups,
                                           void* stream);
/* A stack of matrices, one per group of rows: rows offsets[g] .. offsets[g + 1] of the output are rows of the input
 * times w[g] (w bf16 [n_groups][n][k]). offsets i32 [n_groups + 1] on the device. row_idx (NULL: none) gives the input row
 * of every output row. max_group_rows bounds the rows of one group (host value). Epilogues LG_EPI_BF16, LG_EPI_SWIGLU and
 * LG_EPI_GLU_CLAMP (small), LG_EPI_F32 and LG_EPI_GLU_CLAMP (fp32), with the constants p0, p1, p2 of the last. The first
 * streams the weights of the groups that have rows. */
uint32_t logismos_launch_linear_experts_small_bf16(const void* a_bf16, const void* w_bf16, void* out, const void* offsets_i32,
                                                   const void* row_idx_i32, int32_t n_groups, int32_t max_group_rows,
                                                   int32_t expected_group_rows, int32_t n, int32_t k, int32_t lda, int32_t ldc,
                                                   int32_t epilogue, float p0, float p1, float p2, void* stream);
uint32_t logismos_launch_linear_experts_f32(const void* a_f32, const void* w_bf16, void* out_f32, const void* offsets_i32,
                                            const void* row_idx_i32, int32_t n_groups, int32_t max_group_rows, int32_t n,
                                            int32_t k, int32_t lda, int32_t ldc, int32_t epilogue, float p0, float p1, float p2,
                                            void* stream);
/* The same on the tcgen05 tiles, with the row tiles of 128 listed by logismos_launch_moe_place: tiles i32 [.][4] = group,
 * first output row, last output row + 1, and -1 - input row for tiles that read a_direct; the others read the rows of a
 * that they write (with a_direct NULL: all do). n_tiles i32 [1]; both on the device. max_tiles bounds their number.
 * a [a_rows, lda], a_direct [direct_rows, lda]. */
uint32_t logismos_launch_linear_experts_tc_bf16(const void* a_bf16, int32_t a_rows, const void* a_direct_bf16,
                                                int32_t direct_rows, const void* w_bf16, void* out_bf16, const void* tiles_i32,
                                                const void* n_tiles_i32, int32_t max_tiles, int32_t n_groups, int32_t n,
                                                int32_t k, int32_t lda, int32_t ldc, int32_t epilogue, float p0, float p1,
                                                float p2, void* status_i32, void* stream);
/* The batched contract with fp32 activations and outputs, true fp32 products and sums over the bf16
 * weights (which fp32 represents exactly). Epilogues LG_EPI_F32, LG_EPI_RESID_F32, LG_EPI_GLU_CLAMP, LG_EPI_RELU2 (fp32
 * out); k % 16 == 0, lda % 4 == 0, strides of a and w multiples of 4. */
uint32_t logismos_launch_linear_f32(const void* a_f32, const void* w_bf16, const void* bias_f32, void* out_f32,
                                    int32_t m, int32_t n, int32_t k, int32_t lda, int32_t ldc, int32_t batch,
                                    int64_t a_stride, int64_t w_stride, int64_t out_stride, int32_t epilogue,
                                    float p0, float p1, float p2, void* stream);
/* The same contract one thread per output, as the on-device correctness anchor (the role
 * matmul_naive.hip plays in the reference). LG_EPI_SWIGLU is not supported here. */
uint32_t logismos_launch_linear_t_naive_bf16(const void* a_bf16, const void* w_bf16,
                                             const void* bias_f32, void* out, int32_t m, int32_t n,
                                             int32_t k, int32_t lda, int32_t ldc, int32_t epilogue,
                                             void* stream);

/* cpu_f32::rope_halves_in_place (mod.rs:502-547) with RopeTable::gather (crates/transformers/
 * src/rope.rs:50-92) folded in: rotates, in place, the first n_rot_heads heads of every token row
 * of a packed bf16 [n_tokens, row_stride] buffer (q heads followed by k heads), head h at
 * column h * head_dim, using cos/sin f32 [max_pos, head_dim/2] rows selected by positions[token].
 * A position >= max_pos leaves the row untouched and sets *status (may be NULL) to 1. */
uint32_t logismos_launch_rope_halves_bf16(void* qk_bf16, const void* cos_f32, const void* sin_f32,
                                          const void* positions_i32, int32_t n_tokens,
                                          int32_t n_rot_heads, int32_t head_dim,
                                          int32_t row_stride, int32_t max_pos, void* status_i32,
                                          void* stream);

/* cpu_f32::silu + hadamard (mod.rs:349-374): out[t, j] = silu(gu[t, j]) * gu[t, inter + j].
 * gu bf16 [rows, 2*inter] (gate columns then up columns), out bf16 [rows, inter]. */
uint32_t logismos_launch_swiglu_bf16(const void* gu_bf16, void* out_bf16, int32_t rows,
                                     int32_t inter, void* stream);

/* QwenAttention::forward's score/softmax/PV stage (crates/transformers/src/attention.rs
 * :226-296) for a ragged batch, without materialising scores. qkv bf16 [n_tokens, row_stride]
 * with q heads at column 0, k heads at k_off, v heads at v_off (RoPE already applied); sequence
 * i owns token rows cu_seqlens[i] .. cu_seqlens[i+1]; q head j reads kv head j / (n_heads /
 * n_kv_heads) (attention.rs:366-382). causal = 0 is the reference's bidirectional encoder
 * attention, causal = 1 masks keys after the query. head_dim must be 128. out bf16
 * [n_tokens, n_heads * head_dim]. max_seqlen bounds the grid. */
uint32_t logismos_launch_varlen_attention_bf16(const void* qkv_bf16, const void* cu_seqlens_i32,
                                               void* out_bf16, int32_t n_seqs, int32_t max_seqlen,
                                               int32_t n_heads, int32_t n_kv_heads,
                                               int32_t head_dim, int32_t row_stride, int32_t k_off,
                                               int32_t v_off, int32_t causal, void* stream);

/* The same stage (attention.rs:226-296, head_dim 128 or 256) on the tcgen05 tensor cores: S = Q K^T and
 * O += P V as tcgen05.mma with the accumulators and P in tensor memory, operands moved by TMA. Same
 * layout contract as logismos_launch_varlen_attention_bf16; n_tokens = cu_seqlens[n_seqs]. scratch:
 * logismos_varlen_attention_tc_scratch_bytes(n_tokens, n_seqs, n_kv_heads, head_dim) bytes, 256-byte aligned
 * (receives V transposed per kv head with every sequence padded to a multiple of 8 keys). qkv and out
 * 16-byte aligned. Two launches. status (int32, may be NULL) is set to 2 (low byte; see logismos_launch_linear_t_bf16) if a bounded wait inside
 * the kernel expired. */
size_t logismos_varlen_attention_tc_scratch_bytes(int32_t n_tokens, int32_t n_seqs, int32_t n_kv_heads,
                                                  int32_t head_dim);
uint32_t logismos_launch_varlen_attention_tc_bf16(const void* qkv_bf16, const void* cu_seqlens_i32,
                                                  void* out_bf16, void* scratch, int32_t n_tokens,
                                                  int32_t n_seqs, int32_t max_seqlen, int32_t n_heads,
                                                  int32_t n_kv_heads, int32_t head_dim, int32_t row_stride,
                                                  int32_t k_off, int32_t v_off, int32_t causal,
                                                  void* status, void* stream);

/* The same with the halves-RoPE of the q and k heads (logismos_launch_rope_halves_bf16's contract:
 * the first n_rot_heads heads of every row are rotated in place by cos/sin f32 [max_pos, head_dim/2]
 * at positions[token]; a position outside [0, max_pos) sets status to 1) done by extra blocks of the
 * V-transposing launch, so the pair is still two launches. qkv is modified in place. */
uint32_t logismos_launch_rope_varlen_attention_tc_bf16(void* qkv_bf16, const void* cos_f32,
                                                       const void* sin_f32, const void* positions_i32,
                                                       int32_t n_rot_heads, int32_t max_pos,
                                                       const void* cu_seqlens_i32, void* out_bf16,
                                                       void* scratch, int32_t n_tokens, int32_t n_seqs,
                                                       int32_t max_seqlen, int32_t n_heads,
                                                       int32_t n_kv_heads, int32_t head_dim,
                                                       int32_t row_stride, int32_t k_off, int32_t v_off,
                                                       int32_t causal, void* status, void* stream);

/* A prefill chunk that continues a cached sequence (the reference has no scheduler, crates/sched/src/
 * lib.rs:1-30, and no paged cache; the anchors are QwenAttention::forward's score stage, crates/
 * transformers/src/attention.rs:226-296, made causal, and KvCache::get, crates/cache/src/flat.rs:254-304):
 * sequence s brings the query rows cu_seqlens_q[s] .. cu_seqlens_q[s+1] of q bf16 [n_q_tokens,
 * q_row_stride] (q heads at column 0, RoPE applied) and attends to its kv_lens[s] tokens in the paged
 * cache (k_pool / v_pool bf16 [n_pool_blocks, 16, n_kv_heads * head_dim], block_tables i32 [n_seqs,
 * max_blocks]); the K/V rows of the chunk's own tokens must already be stored there, so kv_lens[s] =
 * cached + new >= new, and query i sees keys 0 .. kv_lens[s] - new + i. out bf16 [n_q_tokens,
 * n_heads * head_dim]. total_kv_tokens >= sum(kv_lens), max_q_len / max_kv_len bound the grids (host
 * values). scratch: logismos_paged_prefix_attention_scratch_bytes(total_kv_tokens, n_seqs, n_kv_heads,
 * head_dim) bytes, 256-byte aligned: the first launch gathers each sequence's K rows and transposed V
 * through its block table into it, the second is the tcgen05 kernel of
 * logismos_launch_varlen_attention_tc_bf16. status (int32, may be NULL): 1 if a block id fell outside
 * the pool (zero rows are used) or kv_lens[s] is below the number of queries, 2 if a bounded wait
 * expired. head_dim 128 or 256. */
size_t logismos_paged_prefix_attention_scratch_bytes(int32_t total_kv_tokens, int32_t n_seqs,
                                                     int32_t n_kv_heads, int32_t head_dim);
uint32_t logismos_launch_paged_prefix_attention_tc_bf16(
    const void* q_bf16, int32_t q_row_stride, const void* cu_seqlens_q_i32, const void* kv_lens_i32,
    const void* k_pool_bf16, const void* v_pool_bf16, const void* block_tables_i32, int32_t max_blocks,
    int32_t n_pool_blocks, void* out_bf16, void* scratch, int32_t n_q_tokens, int32_t total_kv_tokens,
    int32_t n_seqs, int32_t max_q_len, int32_t max_kv_len, int32_t n_heads, int32_t n_kv_heads,
    int32_t head_dim, void* status, void* stream);

/* The same attention over a cache of TurboQuant 3-bit rows (logismos_launch_paged_kv_store_turbo3
 * below; pools u8 [n_pool_blocks, 16, n_kv_heads * head_dim / 128 * 56]): the gathering launch decodes
 * each head chunk (decode_turbo3_0_head, crates/quant/src/lib.rs:378-413) to bf16 on its way into the
 * scratch; everything else as above, a decode token included (one query per sequence). */
uint32_t logismos_launch_paged_prefix_attention_turbo3_bf16(
    const void* q_bf16, int32_t q_row_stride, const void* cu_seqlens_q_i32, const void* kv_lens_i32,
    const void* k_pool_t3, const void* v_pool_t3, const void* block_tables_i32, int32_t max_blocks,
    int32_t n_pool_blocks, void* out_bf16, void* scratch, int32_t n_q_tokens, int32_t total_kv_tokens,
    int32_t n_seqs, int32_t max_q_len, int32_t max_kv_len, int32_t n_heads, int32_t n_kv_heads,
    int32_t head_dim, void* status, void* stream);

/* Causal attention of query rows over keys and values given contiguously: q bf16 [n_q_tokens, q_row_stride]
 * (head h at column h * head_dim), k bf16 [n_kv_rows, n_kv_heads * head_dim], v_t bf16 [n_kv_heads *
 * head_dim, n_kv_rows] (transposed). Sequence s has the queries cu_seqlens_q[s] .. cu_seqlens_q[s+1] and the
 * kv_lens[s] keys at rows / columns kv_start[s] .. (kv_start a multiple of 8; what lies between sequences
 * must be finite); query i sees its first kv_lens[s] - new + i + 1 keys. Scores are scaled by `scale` (> 0).
 * out bf16, rows out_row_stride apart. head_dim 64, 128 or 256; n_kv_rows % 8 == 0. One launch of the
 * tcgen05 kernel above. status as there. gate (f32 [n_q_tokens, ld_gate], NULL: none): head h of a row is multiplied by
 * the sigmoid of its column h. */
uint32_t logismos_launch_varlen_attention_kv_tc_bf16(
    const void* q_bf16, int32_t q_row_stride, const void* cu_seqlens_q_i32, const void* kv_lens_i32,
    const void* kv_start_i32, const void* k_bf16, const void* v_t_bf16, int32_t n_kv_rows, void* out_bf16,
    int32_t out_row_stride, int32_t n_q_tokens, int32_t n_seqs, int32_t max_q_len, int32_t n_heads,
    int32_t n_kv_heads, int32_t head_dim, float scale, const void* gate_f32, int32_t ld_gate, void* status_i32,
    void* stream);

/* mean_pool_masked -> l2_normalize -> linear_t(head) -> l2_normalize (cpu_f32 mod.rs:553-591 as
 * composed by StellaModel::encode_raw, crates/embed/src/stella.rs:231-246), mask all ones.
 * hidden f32 [n_tokens, hidden]; head_w bf16 [dim, hidden]; head_b f32 [dim]; out f32
 * [n_seqs, dim]; scratch_f32 [n_seqs, hidden] receives the pooled means. A sequence of length 0
 * pools to zeros. Three launches. */
uint32_t logismos_launch_pool_head_f32(const void* hidden_f32, const void* cu_seqlens_i32,
                                       const void* head_w_bf16, const void* head_b_f32,
                                       void* out_f32, void* scratch_f32, int32_t n_seqs,
                                       int32_t hidden, int32_t dim, void* stream);

/* ====================================================================================
 * Decode path. No reference GPU or CPU implementation exists for these; the anchors are the
 * contracts named beside each.
 * ==================================================================================== */

/* int4 group-32 dequant GEMV / skinny GEMM: y[b,n] = sum_g s[n,g] sum_{k in g} q[n,k] x[b,k].
 * codes u8 [n, k/2]: value k of a row in byte k/2, even k in the low nibble (the nibble order of
 * Turbo4Block, crates/quant/src/lib.rs:272-301), two's-complement 4-bit; scales fp16 [n, k/32];
 * x bf16 [batch, k]; y bf16 [batch, n]. 1 <= batch <= 64, k % 128 == 0. */
uint32_t logismos_launch_gemv_int4_g32_bf16(const void* codes_u8, const void* scales_f16,
                                            const void* x_bf16, void* y_bf16, int32_t batch,
                                            int32_t n, int32_t k, void* stream);
/* The same product with the fp32 accumulators stored unrounded, y f32 [batch, n]: the lm_head of a
 * decode step, whose logits go to decode::greedy (crates/decode/src/lib.rs:73-83), which takes the
 * first strict maximum of fp32 logits (a bf16 rounding would turn near-ties into ties). */
uint32_t logismos_launch_gemv_int4_g32_f32(const void* codes_u8, const void* scales_f16,
                                           const void* x_bf16, void* y_f32, int32_t batch, int32_t n,
                                           int32_t k, void* stream);

/* The same product, y bf16 [batch, n], with the kernel chosen by shape and batch
 * (logismos_skinny_int4_route: 0 = the streaming GEMV, 1 = the fused-dequant tensor-core linear below,
 * taken above 16 rows, for k >= 3 n, and from 8 rows up to n = 16384; needs k % 256 == 0, n % 4 == 0).
 * Route 1 accumulates in workspace_f32 [batch, n] (16-byte aligned, ALL ZERO on entry, left all zero
 * on return) and rounds once to bf16: two launches. workspace_f32 == NULL keeps the GEMV at every
 * batch. status_i32 as for logismos_launch_qlinear_int4_g32_acc_f32. */
int32_t logismos_skinny_int4_route(int32_t batch, int32_t n, int32_t k);
uint32_t logismos_launch_skinny_int4_g32_bf16(const void* codes_u8, const void* scales_f16,
                                              const void* x_bf16, void* y_bf16, int32_t batch, int32_t n,
                                              int32_t k, void* workspace_f32, void* status_i32, void* stream);

/* Expands int4 group-32 weights (same storage as above) to bf16 [n, k]: w = bf16(scale * code).
 * The prefill side of a mixed step runs its contractions on the tcgen05 GEMM over this expansion.
 * k % 32 == 0. */
uint32_t logismos_launch_dequant_int4_g32_bf16(const void* codes_u8, const void* scales_f16,
                                               void* out_bf16, int32_t n, int32_t k, void* stream);

/* Quantises fp32 weights [n, k] to the int4 group-32 storage above, on the device: per group of 32
 * values along k, scale = fp16(max|w| / 7), code = clamp(round-half-even(w / scale), -8, 7) (0 for an
 * all-zero group), packed in the Turbo4Block nibble order (crates/quant/src/lib.rs:272-301). The
 * reference has no quantiser (turbo4 encode returns Unsupported, crates/quant/src/lib.rs:361-367);
 * the output is integer and is checked bit for bit against the CPU definition. k % 32 == 0. */
uint32_t logismos_launch_quantize_int4_g32(const void* w_f32, void* codes_u8, void* scales_f16,
                                           int32_t n, int32_t k, void* stream);

/* acc[m, n] += A[m, k] * dequant(W)[n, k]^T for 1 <= m <= 256 tokens, int4 group-32 weights (storage
 * as above), dequantisation fused into the tensor-core operand pipeline. The linear of decode and
 * small mixed steps: linear_t (cpu_f32/mod.rs:271-345) on the dequantised matrix. a bf16 [m, k]
 * rows lda apart; acc fp32 [m, n] rows ldc apart (the fp32 residual stream itself for the output
 * projections, or a zeroed workspace finished by the call below). Weights enter the MMA as
 * bf16(code) * bf16(scale). k % 256 == 0. Slices of k meet in fp32 reductions: with several slices
 * the last bits of acc may differ between runs. status_i32 as for logismos_launch_linear_t_bf16. */
uint32_t logismos_launch_qlinear_int4_g32_acc_f32(const void* a_bf16, const void* codes_u8,
                                                  const void* scales_f16, void* acc_f32, int32_t m,
                                                  int32_t n, int32_t k, int32_t lda, int32_t ldc,
                                                  void* status_i32, void* stream);
/* The same launch with the caller's promise that no work still in flight on the stream writes the
 * codes or scales (model weights uploaded once): with dependent launch on, the kernel fills its weight
 * ring before the preceding kernel has finished. */
uint32_t logismos_launch_qlinear_int4_g32_acc_f32_static(const void* a_bf16, const void* codes_u8,
                                                         const void* scales_f16, void* acc_f32,
                                                         int32_t m, int32_t n, int32_t k, int32_t lda,
                                                         int32_t ldc, void* status_i32, void* stream);
/* Finishes an accumulation workspace: out bf16 [m, n] = acc (+ bias), or with swiglu != 0,
 * out bf16 [m, n/2] = silu(gate) * up over columns interleaved in blocks of 32 (the LG_EPI_SWIGLU
 * row order); acc is left zeroed for the next accumulation. n % 4 == 0 (n % 64 == 0 for swiglu). */
uint32_t logismos_launch_qlinear_finish_bf16(void* acc_f32, const void* bias_f32, void* out_bf16,
                                             int32_t m, int32_t n, int32_t ld_acc, int32_t ldc,
                                             int32_t swiglu, void* stream);

/* Paged-attention decode with fused KV append. The paged cache keeps the row layout of
 * FlatKvCache (crates/cache/src/flat.rs:36-69: one row = all kv heads of one token, contiguous):
 * k_pool / v_pool bf16 [n_pool_blocks, block_size = 16, n_kv_heads * head_dim]; logical token t
 * of sequence s lives in block block_tables[s * max_blocks + t / 16], slot t % 16.
 * For each sequence: the new token's k/v row (new_k / new_v bf16 [n_seqs, n_kv_heads*head_dim])
 * is written at position context_lens[s] - 1 (context_lens counts the new token), then
 * q bf16 [n_seqs, n_heads * head_dim] attends causally to positions 0 .. context_lens[s] - 1.
 * new_k == NULL skips the append. head_dim 128 or 256, n_heads / n_kv_heads <= 16. Every
 * context_lens[s] must be >= 1 (a sequence without a key would get no chunk and its output row
 * would stay unwritten; logismos_build_decode_chunks rejects such a batch).
 * Work is split along the context in chunks of `chunk_tokens` (a multiple of 64):
 * chunk_offsets i32 [n_seqs + 1] is the exclusive prefix sum of ceil(context_lens / chunk_tokens)
 * and total_chunks its last entry (host copy). scratch must hold
 * logismos_paged_decode_scratch_bytes(total_chunks, n_heads, head_dim) bytes. status_i32 (may be
 * NULL) receives 1 if a block id fell outside the pool (that block is then skipped). */
size_t logismos_paged_decode_scratch_bytes(int32_t total_chunks, int32_t n_heads, int32_t head_dim);
uint32_t logismos_launch_paged_attention_decode_bf16(
    const void* q_bf16, void* k_pool_bf16, void* v_pool_bf16, const void* new_k_bf16,
    const void* new_v_bf16, const void* block_tables_i32, const void* context_lens_i32,
    const void* chunk_offsets_i32, void* out_bf16, void* scratch, void* status_i32, int32_t n_seqs,
    int32_t total_chunks, int32_t chunk_tokens, int32_t max_blocks, int32_t n_pool_blocks,
    int32_t n_heads, int32_t n_kv_heads, int32_t head_dim, void* stream);

/* Paged-attention decode for callers that cannot allocate device memory where they decode (an
 * engine that has given all free HBM to its KV pool, a thread where an allocation's device-wide
 * synchronisation is unacceptable). It has no counterpart in the reference. Same arguments and
 * results as logismos_launch_paged_attention_decode_bf16 minus `scratch`: the per-chunk partials
 * go to a buffer of LOGISMOS_PAGED_DECODE_STATIC_SCRATCH_BYTES built into the library image (each
 * GPU that loads the library holds it until exit). The call allocates nothing.
 *   - Limit: logismos_paged_decode_scratch_bytes(total_chunks, n_heads, head_dim) must not exceed
 *     the constant (8 MiB: e.g. 1008 chunks at 16 heads x 128); beyond it the call returns
 *     cudaErrorMemoryAllocation (2) without launching and says why on stderr.
 *   - The first call on each device looks up the buffer's device address (that device must be
 *     current, as for any launch) and caches it; make that first call before starting any stream
 *     capture on the device. "Allocates nothing" holds from then on: the buffer belongs to the
 *     library's device code, which the CUDA runtime may load lazily at the first call into the
 *     library on a device, and loading takes device memory (the 8 MiB included). A host that then
 *     grabs all free HBM for its KV pool must therefore make one small valid call of this entry
 *     point on each device BEFORE that grab.
 *   - All calls share the one buffer and it keeps the previous call's contents; nothing in it needs
 *     clearing, since a launch only reads partials it wrote itself. For the same reason two calls
 *     whose kernels can overlap on the GPU (different streams, or threads) race on it: serialise
 *     them, or use the entry point with caller scratch. */
#define LOGISMOS_PAGED_DECODE_STATIC_SCRATCH_BYTES (8u * 1024u * 1024u)
uint32_t logismos_launch_paged_attention_decode_noalloc_bf16(
    const void* q_bf16, void* k_pool_bf16, void* v_pool_bf16, const void* new_k_bf16,
    const void* new_v_bf16, const void* block_tables_i32, const void* context_lens_i32,
    const void* chunk_offsets_i32, void* out_bf16, void* status_i32, int32_t n_seqs,
    int32_t total_chunks, int32_t chunk_tokens, int32_t max_blocks, int32_t n_pool_blocks,
    int32_t n_heads, int32_t n_kv_heads, int32_t head_dim, void* stream);

/* KvCache::put for a ragged batch (crates/cache/src/lib.rs:57-82): row i of k/v bf16
 * [n_tokens, row_elems] is stored at physical slot slot_mapping[i] (i64: block * 16 + offset).
 * A slot outside the pool is skipped and sets *status to 1. */
uint32_t logismos_launch_paged_kv_store_bf16(const void* k_bf16, const void* v_bf16,
                                             int32_t src_row_stride, void* k_pool_bf16,
                                             void* v_pool_bf16, const void* slot_mapping_i64,
                                             int32_t n_tokens, int32_t row_elems,
                                             int64_t n_pool_slots, void* status_i32, void* stream);
/* KvCache::get: the first len rows of one sequence gathered through its block table into
 * contiguous bf16 [len, row_elems] buffers (bit-exact copy). */
uint32_t logismos_launch_paged_kv_gather_bf16(const void* k_pool_bf16, const void* v_pool_bf16,
                                              const void* block_table_i32, int32_t table_len,
                                              int32_t len, int32_t row_elems,
                                              int32_t n_pool_blocks, void* k_out_bf16,
                                              void* v_out_bf16, void* status_i32, void* stream);

/* The same cache with TurboQuant 3-bit rows: KvCache::put / get (crates/cache/src/lib.rs:57-82) through
 * encode_turbo3_0_head / decode_turbo3_0_head (crates/quant/src/lib.rs:316-413: L2 norm, 128-point
 * Walsh-Hadamard transform, 8-centroid codebook, four 14-byte blocks per 128-value head chunk). A pool
 * row holds row_elems / 128 chunks of 56 bytes (logismos_turbo3_row_bytes) instead of row_elems bf16:
 * pools are u8 [n_pool_blocks, 16, row_bytes]. The store encodes rows of k / v bf16 [n_tokens,
 * row_elems] (widened to fp32 first) into slot_mapping's slots; the gather decodes the first len rows of
 * one sequence to bf16 [len, row_elems] (fp32 decode rounded once). Bytes and values are identical to
 * the CPU definition (the arithmetic follows it operation by operation). row_elems % 128 == 0. */
size_t logismos_turbo3_row_bytes(int32_t row_elems);
uint32_t logismos_launch_paged_kv_store_turbo3(const void* k_bf16, const void* v_bf16, int32_t src_row_stride,
                                               void* k_pool_t3, void* v_pool_t3, const void* slot_mapping_i64,
                                               int32_t n_tokens, int32_t row_elems, int64_t n_pool_slots,
                                               void* status_i32, void* stream);
uint32_t logismos_launch_paged_kv_gather_turbo3(const void* k_pool_t3, const void* v_pool_t3,
                                                const void* block_table_i32, int32_t table_len, int32_t len,
                                                int32_t row_elems, int32_t n_pool_blocks, void* k_out_bf16,
                                                void* v_out_bf16, void* status_i32, void* stream);

/* dst[r, :] = src[idx[r], :] for fp32 rows (bit-exact copy): picks the last token row of every
 * sequence of a packed step before the final norm and the lm_head. An index outside
 * [0, n_src_rows) yields a zero row and sets *status to 1. width % 4 == 0. */
uint32_t logismos_launch_gather_rows_f32(const void* src_f32, const void* idx_i32, void* dst_f32,
                                         int32_t n_rows, int32_t width, int32_t n_src_rows,
                                         void* status_i32, void* stream);

/* gated_delta_rule_recurrent_fwd (crates/kernels/src/gated_delta_rule/cpu.rs:92-182), one decode
 * step for a batch of sequences and heads: state f32 [n_seqs, heads, K=128, V=128] updated in
 * place; q,k f32/bf16 ... see gdn.cu. q, k bf16 [n_seqs, heads, 128]; v bf16 [n_seqs, heads, 128];
 * g, beta f32 [n_seqs, heads]; o bf16 [n_seqs, heads, 128]. */
uint32_t logismos_launch_gdn_decode_step(void* state_f32, const void* q_bf16, const void* k_bf16,
                                         const void* v_bf16, const void* g_f32,
                                         const void* beta_f32, void* o_bf16, int32_t n_seqs,
                                         int32_t heads, float scale, void* stream);

/* One decode token per sequence straight from the fp32 accumulation workspace of the fused input
 * projection (logismos_launch_qlinear_int4_g32_acc_f32 over the row blocks q | k | v | z | a | b):
 * logismos_launch_gdn_finish and the one-token case of logismos_launch_gdn_prefill (with the output gate)
 * in a single launch, same arithmetic in the same order. acc f32 [n_seqs, ld_acc] is left zeroed. Row i
 * is sequence i; o bf16 [n_seqs, heads, 128]; state pool, state_slots and fresh as below. pair_count i32
 * [n_seqs * heads], all zero on entry and on return. The states, state_slots and fresh must not be
 * written by work still in flight on the stream (they are read ahead of the dependency wait). */
uint32_t logismos_launch_gdn_decode_from_acc(void* state_f32, void* acc_f32, int32_t ld_acc,
                                             const void* A_log_f32, const void* dt_bias_f32, void* o_bf16,
                                             const void* state_slots_i32, const void* fresh_u8,
                                             void* pair_count_i32, int32_t n_seqs, int32_t heads,
                                             float scale, void* stream);

/* gated_delta_rule_chunk_fwd / recurrent_fwd over a ragged batch (cpu.rs:92-249): sequence i owns
 * token rows cu_seqlens[i] .. cu_seqlens[i+1] of q, k, v bf16 [n_tokens, heads, 128], g, beta f32
 * [n_tokens, heads]; state f32 [n_seqs, heads, 128, 128] is the initial state on entry and the
 * final state on return; o bf16 [n_tokens, heads, 128]. Tokens are processed in order.
 * q, k, v may be column blocks of a wider projection output: token t, head h starts at
 * t * qkv_stride + h * 128 (elements; qkv_stride % 8 == 0, 16-byte aligned bases). state_slots i32 [n_seqs] (may be NULL = identity) selects
 * each sequence's slot in a state pool [n_slots, heads, 128, 128]; fresh u8 [n_seqs] (may be NULL)
 * marks sequences that start here and therefore begin from the zero state. gate_z bf16 (may be
 * NULL), addressed like q, k, v, applies the layer's output gate in the same pass:
 * o *= silu(z) in fp32 before the bf16 rounding. mode selects the kernel shape: 1 = throughput (64
 * value columns per CTA; decode and many sequences), 2 = latency (32 columns per CTA: more
 * CTAs per head for a few long sequences), 0 = by the number of (sequence, head) pairs.
 * LG_GDN_STATIC_STATE, or-ed into mode, is the caller's promise that no work still in flight on the
 * stream writes the state pool, cu_seqlens, state_slots or fresh (they were left by an earlier model
 * step that has completed): with dependent launch on, the kernel then reads its states while the
 * kernels that produce q, k, v and the gates are still running. */
enum { LG_GDN_STATIC_STATE = 0x100 };
uint32_t logismos_launch_gdn_prefill(void* state_f32, const void* q_bf16, const void* k_bf16,
                                     const void* v_bf16, const void* g_f32, const void* beta_f32,
                                     void* o_bf16, const void* gate_z_bf16, const void* cu_seqlens_i32,
                                     const void* state_slots_i32, const void* fresh_u8, int32_t n_seqs,
                                     int32_t heads, int32_t qkv_stride, float scale, int32_t mode,
                                     void* stream);
/* The same function in chunk-parallel form (gated_delta_rule_chunk_fwd, cpu.rs:201-249): the 64 tokens
 * of a chunk are resolved together by matrix products (a triangular solve for the in-chunk
 * dependencies, tensor-core products against the carried state), so a long prompt is not bound by a
 * token-serial chain. Arguments as logismos_launch_gdn_prefill. The state stays fp32 and enters the
 * products rounded to bf16: outputs within 2e-2 of the recurrence, final state within 1e-2.
 * scratch (128-byte aligned, logismos_gdn_chunked_scratch_bytes(n_tokens, n_seqs, heads) bytes, n_tokens
 * = cu_seqlens[n_seqs] - cu_seqlens[0] or more) selects the two-launch form: everything of a chunk that
 * does not involve the carried state is computed for all chunks of the batch at once (a CTA per chunk
 * and head) and parked in scratch, then each sequence's chunks are chained with the three products that
 * touch the state. scratch == NULL keeps the one-launch form (a CTA per sequence, head and value-column
 * half does all of it chunk after chunk). Same results within the stated tolerance. */
size_t logismos_gdn_chunked_scratch_bytes(int32_t n_tokens, int32_t n_seqs, int32_t heads);
uint32_t logismos_launch_gdn_chunked(void* state_f32, const void* q_bf16, const void* k_bf16,
                                     const void* v_bf16, const void* g_f32, const void* beta_f32,
                                     void* o_bf16, const void* gate_z_bf16, const void* cu_seqlens_i32,
                                     const void* state_slots_i32, const void* fresh_u8, int32_t n_seqs,
                                     int32_t heads, int32_t qkv_stride, float scale, void* scratch,
                                     int32_t n_tokens, void* stream);
/* Inputs of the recurrence from the layer's projections (no reference code; the formulas are
 * those of research/14-gdn-aiter-preflight.md:190-198, :209-219): q, k bf16 [n_tokens, heads, 128]
 * are L2-normalised per head row in place (l2_norm_in_place, cpu.rs:19-34);
 * g = -exp(A_log[h]) * softplus(a + dt_bias[h]) (softplus(x) = x for x > 20), beta = sigmoid(b),
 * g, beta f32 [n_tokens, heads], A_log, dt_bias f32 [heads]. q, k rows start at
 * t * qk_stride + h * 128; a, b are read at t * ab_stride + h (f32). */
uint32_t logismos_launch_gdn_prepare(void* q_bf16, void* k_bf16, const void* a_f32, const void* b_f32,
                                     const void* A_log_f32, const void* dt_bias_f32, void* g_f32,
                                     void* beta_f32, int32_t n_tokens, int32_t heads,
                                     int32_t qk_stride, int32_t ab_stride, void* stream);
/* logismos_launch_gdn_prepare fused with the finishing of the input projection's fp32 accumulation
 * workspace (logismos_launch_qlinear_int4_g32_acc_f32 into acc f32 [n_tokens, ld_acc], columns
 * q | k | v | z [heads * 128 each] | a | b [heads each]): q and k are L2-normalised in fp32, q, k, v, z
 * are rounded to bf16 once into proj [n_tokens, ld_proj] (columns q | k | v | z), g and beta f32
 * [n_tokens, heads] are computed from a and b, and the workspace is left zeroed. */
uint32_t logismos_launch_gdn_finish(void* acc_f32, int32_t ld_acc, const void* A_log_f32, const void* dt_bias_f32,
                                    void* proj_bf16, int32_t ld_proj, void* g_f32, void* beta_f32,
                                    int32_t n_tokens, int32_t heads, void* stream);
/* x[t, j] *= sigmoid(gate[t, j]) (mode 0) or silu(gate[t, j]) (mode 1), bf16 in place, fp32 math;
 * rows of x and gate have their own strides (elements). The output gates of the hybrid decoder's
 * attention and linear-attention layers. n % 8 == 0. */
uint32_t logismos_launch_gated_mul_bf16(void* x_bf16, int32_t x_stride, const void* gate_bf16,
                                        int32_t gate_stride, int32_t rows, int32_t n, int32_t mode,
                                        void* stream);

/* x[i] += d[i], fp32, n % 4 == 0: joins a partial sum that was reduced across tensor-parallel ranks
 * into the residual stream (no reference counterpart: the reference has no tensor parallelism). */
uint32_t logismos_launch_add_f32(void* x_f32, const void* d_f32, int64_t n, void* stream);

/* decode::greedy (crates/decode/src/lib.rs:73-83): argmax per row, first maximum wins, NaN
 * never selected. logits bf16 or f32 [rows, n]; out u32 [rows]. */
uint32_t logismos_launch_greedy_argmax(const void* logits, int32_t logits_f32, void* out_u32,
                                       int32_t rows, int32_t n, void* stream);

/* ====================================================================================
 * Mechanisms of parallel-block decoders with latent attention (no reference counterpart: the reference has
 * no decoder model). Rows of fp32 data are `ld` columns wide, a multiple of 4; columns n .. ld are
 * padding and must hold zeros in weights, gains and filters.
 * ==================================================================================== */

/* Depth average and RMS norm: x = sum_{j < n_hist} coef[j] X_j, X_j f32 rows at hist + j * hist_stride
 * (elements), h = x / sqrt(mean over n of x^2 + eps) * gain. Row r reads source row row_idx[r] (NULL: r;
 * an index outside [0, n_src_rows) raises status to 1). Any of x (f32 [rows, ld]), inv_rms (f32 [rows]) and
 * norm_out ([rows, ld], bf16 or with out_f32 f32; needs gain) may be NULL. ld <= 16384. */
uint32_t logismos_launch_depth_mix_f32(const void* hist_f32, int64_t hist_stride, int32_t n_hist,
                                       const void* coef_f32, const void* row_idx_i32, int32_t n_src_rows,
                                       void* x_f32, void* inv_rms_f32, const void* gain_f32, void* norm_out,
                                       int32_t out_f32, int32_t rows, int32_t n, int32_t ld, float eps,
                                       void* status_i32, void* stream);
/* Input convolution over a ragged batch: h = x * inv_rms * gain per row, o1 = h + sum_j w1[j] *
 * h_(t - taps + 1 + j) and the same for o2 with w2 (o2 may be NULL; w1 / w2 NULL: no filter), causal inside
 * each sequence. w f32 [taps, ld], taps 1..8. Row t belongs to sequence seq_ids[t], whose rows are
 * cu_seqlens[s] .. cu_seqlens[s+1]. state f32 [n_slots, 2, taps - 1, ld]: the last taps - 1 rows h of a
 * sequence in slot state_slots[s]; read from copy phase[s] (zeros when fresh[s]), the new state goes to copy
 * 1 - phase[s]. o1, o2 bf16 or with out_f32 f32, [rows, ld]. */
uint32_t logismos_launch_norm_conv(const void* x_f32, const void* inv_rms_f32, const void* gain_f32,
                                   const void* w1_f32, const void* w2_f32, void* o1, void* o2, int32_t out_f32,
                                   void* state_f32, const void* state_slots_i32, const void* fresh_u8,
                                   const void* phase_u8, const void* seq_ids_i32, const void* cu_seqlens_i32,
                                   int32_t rows, int32_t ld, int32_t taps, void* stream);
/* Both of the above in one launch for a step whose sequences bring one token each (row = sequence). gain, w1,
 * w2, the state and the three index arrays must not be written by work still in flight on the stream (they
 * may be read ahead of the dependency wait). */
uint32_t logismos_launch_depth_mix_conv_decode(const void* hist_f32, int64_t hist_stride, int32_t n_hist,
                                               const void* coef_f32, void* x_f32, const void* gain_f32,
                                               const void* w1_f32, const void* w2_f32, void* o1, void* o2,
                                               int32_t out_f32, void* state_f32, const void* state_slots_i32,
                                               const void* fresh_u8, const void* phase_u8, int32_t rows,
                                               int32_t n, int32_t ld, float eps, int32_t taps, void* stream);

/* Latent attention. A token's cache row is its normed key/value latent, c_width values: pool bf16 or f32
 * [n_pool_blocks, 16, c_width].
 * norm_store: raw f32 [rows, ld] holds the query latent in columns 0 .. q_width and the key/value latent in
 * q_width .. q_width + c_width; both are RMS-normed (means over the first q_n and c_n columns) with their
 * gains; the first goes to q_latent [rows, q_width], the second to the pool at slot_mapping[row] (a slot
 * outside the pool is skipped and raises status to 1). is_f32 selects the type of both. zero_raw != 0 leaves
 * raw zeroed, ready to be accumulated into again.
 * rotary (NULL: none): the key/value latent takes the first `at` of the c_width columns (a multiple of 4, c_n of them not
 * padding), the next dims columns are one rotated key part; raw columns q_width + c_width .. + n_gate go to gate f32
 * [rows, ld_gate] as they are. */
typedef struct lg_latent_rotary {
  const void* table;            /* f32 [positions][dims / 2][2] */
  const void* positions;        /* i32 [rows] */
  int32_t at, dims;
  void* gate;
  int32_t n_gate, ld_gate;
} lg_latent_rotary_t;
uint32_t logismos_launch_latent_norm_store(void* raw_f32, int32_t ld, const void* gain_q_f32,
                                           const void* gain_c_f32, void* q_latent, void* pool,
                                           const void* slot_mapping_i64, int32_t rows, int32_t q_width,
                                           int32_t q_n, int32_t c_width, int32_t c_n, float eps,
                                           int64_t n_pool_slots, int32_t is_f32, int32_t zero_raw,
                                           const lg_latent_rotary_t* rotary, void* status_i32, void* stream);
/* The cached rows of whole sequences made contiguous: out bf16 [logismos_latent_gather_rows(total, n_seqs),
 * width], sequence s at kv_start[s] (written, a multiple of 8), gaps zeroed. */
int32_t logismos_latent_gather_rows(int32_t total_kv_tokens, int32_t n_seqs);
uint32_t logismos_launch_latent_gather_bf16(const void* pool, const void* block_tables_i32, int32_t max_blocks,
                                            int32_t n_pool_blocks, const void* kv_lens_i32, void* out,
                                            void* kv_start_i32, int32_t total_kv_tokens, int32_t n_seqs,
                                            int32_t max_kv_len, int32_t width, void* status_i32, void* stream);
/* Decode in the latent space, one query row per sequence: out[r, h] = sum_j softmax_j(scale q[r, h] . c_j)
 * c_j over the first context_lens[r] cached rows. q, out bf16 [rows, heads, rank]; rank % 64 == 0, rank <=
 * 1024. chunk_offsets as for the paged decode kernel, with chunk_tokens % 64 == 0
 * (logismos_pick_latent_chunk, whose choice leaves at most logismos_latent_max_chunks(rows) chunks). scratch:
 * logismos_latent_decode_scratch_bytes(total_chunks, heads, rank). A second launch merges split contexts. The
 * index arrays, and every cached row but the last of each context, must not be written by work still in
 * flight on the stream (they may be read ahead of the dependency wait). gate (f32 [rows, ld_gate], NULL: none): head h of
 * a row is multiplied by the sigmoid of its column h. rot_table (NULL: none; f32 [positions][rot_dims / 2][2]): channels
 * rot_at .. rot_at + rot_dims (rot_at % 8 == 0) of q are turned by the angles of position context_lens - 1 as they are read. */
int32_t logismos_pick_latent_chunk(const int32_t* host_context_lens, int32_t n_seqs, int32_t heads);
int32_t logismos_latent_max_chunks(int32_t max_rows);
size_t logismos_latent_decode_scratch_bytes(int32_t total_chunks, int32_t heads, int32_t rank);
uint32_t logismos_launch_latent_decode_bf16(const void* q_bf16, const void* pool_bf16, const void* block_tables_i32,
                                            const void* context_lens_i32, const void* chunk_offsets_i32,
                                            void* out_bf16, void* scratch, int32_t rows, int32_t total_chunks,
                                            int32_t chunk_tokens, int32_t max_blocks, int32_t n_pool_blocks,
                                            int32_t heads, int32_t rank, float scale, const void* gate_f32,
                                            int32_t ld_gate, const void* rot_table_f32, int32_t rot_at, int32_t rot_dims,
                                            void* status_i32, void* stream);
/* The fp32 form for any rows of a step: row t of sequence seq_ids[t] sees keys 0 .. positions[t]. */
uint32_t logismos_launch_latent_attention_f32(const void* q_f32, const void* pool_f32, const void* block_tables_i32,
                                              const void* seq_ids_i32, const void* positions_i32, void* out_f32,
                                              int32_t rows, int32_t max_blocks, int32_t n_pool_blocks,
                                              int32_t heads, int32_t rank, float scale, const void* gate_f32,
                                              int32_t ld_gate, void* status_i32, void* stream);

/* ====================================================================================
 * Sampling chain on the device: the logit processors and the multinomial sampler of
 * crates/decode (chain.rs:33-76 runs processors in insertion order, then the sampler), each as one
 * launch over fp32 logits [rows, n] IN PLACE, so a caller keeps the reference's free ordering. Rows are
 * independent. Rows must hold at least one finite logit.
 * ==================================================================================== */

/* TemperatureScale (processors.rs:18-28): t = max(temperature, 1e-6); |t - 1| < 1e-9 is the identity;
 * otherwise every logit is divided by t. */
uint32_t logismos_launch_temperature_f32(void* logits_f32, int32_t rows, int32_t n, float temperature,
                                         void* stream);
/* TopK (processors.rs:50-82): k == 0 or k >= n is the identity; otherwise every NaN and every logit
 * below the k-th largest becomes -inf (ties with the k-th largest survive). Exact. */
uint32_t logismos_launch_top_k_f32(void* logits_f32, int32_t rows, int32_t n, int32_t k, void* stream);
/* TopP (processors.rs:89-122): p clamped to [0, 1]; p >= 1 is the identity; otherwise the smallest
 * prefix of the tokens in order of descending probability (equal probabilities in index order) whose
 * softmax mass reaches p is kept, the rest becomes -inf. The reference normalises by a sequential
 * fp32 sum over the vocabulary (about 1e-5 to 1e-4 of relative rounding error at 151936 terms); the
 * device sums pairwise, so the two nuclei can differ by the tokens whose cumulative mass lies within
 * that error of p. */
uint32_t logismos_launch_top_p_f32(void* logits_f32, int32_t rows, int32_t n, float p, void* stream);
/* MinP (processors.rs:130-146): p clamped; p <= 0 is the identity; tokens whose probability is below
 * p times the largest probability become -inf. */
uint32_t logismos_launch_min_p_f32(void* logits_f32, int32_t rows, int32_t n, float p, void* stream);
/* RepetitionPenalty (processors.rs:160-181): row r lists counts[r] <= max_tokens token ids in
 * tokens_u32 [rows, max_tokens]; for each in order (a token listed twice is penalised twice; ids >= n
 * are skipped) a positive logit is divided by penalty, any other multiplied. |penalty - 1| < 1e-9 is
 * the identity. */
uint32_t logismos_launch_repetition_penalty_f32(void* logits_f32, int32_t rows, int32_t n,
                                                const void* tokens_u32, const void* counts_i32,
                                                int32_t max_tokens, float penalty, void* stream);
/* MultinomialSampler::sample (sampler.rs:31-58) with the uniform draw of every row supplied by the
 * caller (uniforms_f32 [rows], each in [0, 1); the reference draws it from its RNG at that point):
 * probabilities are exp(l - max) of the finite logits over their sum; the token is the first index
 * whose cumulative probability exceeds the draw; a row without mass falls back to greedy; out u32
 * [rows]. */
uint32_t logismos_launch_multinomial_f32(const void* logits_f32, int32_t rows, int32_t n,
                                         const void* uniforms_f32, void* out_u32, void* stream);

/* ====================================================================================
 * Host-side index builders (no device work). crates/sched is an empty scaffold in the reference
 * (src/lib.rs:1-30); these define the packing of a mixed prefill/decode step.
 * ==================================================================================== */

/* For sequence i with cached_lens[i] tokens already in the cache and new_lens[i] new tokens:
 * cu_seqlens [n+1], positions [total] (continuing from the cached length), slot_mapping [total]
 * (block * block_size + offset through block_tables [n, max_blocks]), seq_ids [total].
 * Returns the total token count, or -1 if a needed table entry is negative or >= n_pool_blocks. */
int64_t logismos_build_packing(const int32_t* host_cached_lens, const int32_t* host_new_lens,
                               int32_t n_seqs, const int32_t* host_block_tables,
                               int32_t max_blocks, int32_t block_size, int32_t n_pool_blocks,
                               int32_t* host_cu_seqlens, int32_t* host_positions,
                               int64_t* host_slot_mapping, int32_t* host_seq_ids);
/* chunk_offsets [n+1] for the paged decode kernel; returns total_chunks, or -1 if a context length
 * is below 1 or the chunk count overflows. */
int32_t logismos_build_decode_chunks(const int32_t* host_context_lens, int32_t n_seqs,
                                     int32_t chunk_tokens, int32_t* host_chunk_offsets);
/* chunk_tokens for one step's contexts: the largest of 512, 1024, 2048 that leaves the decode launch at
 * least 32768 / head_dim CTAs (chunks x kv heads); 512 otherwise. Host-side, no device work. */
int32_t logismos_pick_decode_chunk(const int32_t* host_context_lens, int32_t n_seqs,
                                   int32_t n_kv_heads, int32_t head_dim);

/* ---- decoder stacks of state-space and parallel attention / time-mixing layers ------------------------------ */

/* Output norm of a sublayer: x f32 [rows, ld] += layer_norm(src) * w + b over n columns; h (may be NULL) receives
 * the new row in the activation format (bf16, or fp32 with out_f32). x NULL: h = layer_norm(src row) alone.
 * w NULL: no norm, h = x. row_idx_i32 (may be NULL) selects the rows of src. zero_src: src is cleared once read (an
 * accumulation buffer). */
uint32_t logismos_launch_post_norm(void* src_f32, int32_t zero_src, const void* row_idx_i32, int32_t n_src_rows,
                                   void* x_f32, const void* w_f32, const void* b_f32, void* h, int32_t out_f32,
                                   int32_t rows, int32_t n, int32_t ld, float eps, void* status_i32, void* stream);
/* The same for one token per sequence, with the mixes of the next sublayer: copy 0 of h [1 + n_mix][rows][ld] is x,
 * copy s is x + (x' - x) * mu[s - 1] with x' the previous token's row (state f32 [slots][2][ld]; the copy `phase`
 * names is read, the other written). */
uint32_t logismos_launch_post_norm_shift_decode(void* src_f32, int32_t zero_src, void* x_f32, const void* w_f32,
                                                const void* b_f32, void* h, int32_t out_f32, const void* mu_f32,
                                                int32_t n_mix, void* state_f32, const void* state_slots_i32,
                                                const void* fresh_u8, const void* phase_u8, int32_t rows, int32_t n,
                                                int32_t ld, float eps, void* stream);
/* The mixes of ragged sequences from x (seq_ids [rows], cu_seqlens). */
uint32_t logismos_launch_token_shift(const void* x_f32, void* h, int32_t out_f32, const void* mu_f32, int32_t n_mix,
                                     void* state_f32, const void* state_slots_i32, const void* fresh_u8,
                                     const void* phase_u8, const void* seq_ids_i32, const void* cu_seqlens_i32,
                                     int32_t rows, int32_t ld, void* stream);

/* Linear attention with a data-dependent decay per key channel; key heads padded to dp, value heads to vp, each 32, 64,
 * 128 or 256, with zeros:
 *   LG_DECAY_TIME_MIX  o_t = (S + diag(u) k_t v_t^T)^T r_t;  S <- diag(exp(-exp(z_t))) S + k_t v_t^T     (vp = dp)
 *   LG_DECAY_GATED     S <- diag(sigmoid(z_t)^(1 / tau)) S + k_t v_t^T;  o_t = q_scale S^T r_t
 *   out = o / rms(o) * gain * silu(g) * scale          (rms over the d true value channels)
 * proj holds r, k of head h at columns off_* + h * dp, v, g at off_* + h * vp. z f32 [rows, ld_z] or, when NULL, z = W2 low + w0 with
 * low f32 [rows, ld_low] and w2 bf16 [heads * dp, ld_w2] (rank columns, a multiple of 32). Sequence i owns rows
 * cu[i] .. cu[i + 1] and state slot state_slots[i] of state f32 [slots][heads][dp][vp]; fresh[i]: it starts here. */
enum { LG_DECAY_TIME_MIX = 0, LG_DECAY_GATED = 1 };
typedef struct lg_time_mix {
  const void* proj;
  int32_t ld, off_r, off_k, off_v, off_g;
  const void* z;
  int32_t ld_z;
  const void* low;
  int32_t ld_low;
  const void* w2;
  int32_t ld_w2, rank;
  const void *w0, *u, *gain;    /* f32 [heads * dp], u only for time mixing; gain [heads * vp] */
  void* state;
  const void *state_slots, *fresh, *cu;
  void* out;
  int32_t ld_out, heads, d, dp;
  float scale, eps;
  int32_t mode, vp;             /* vp 0: dp */
  float tau, q_scale;
} lg_time_mix_t;
/* Token by token: decode steps, fp32, any dp. */
uint32_t logismos_launch_time_mix_step(const lg_time_mix_t* args, int32_t n_seqs, int32_t is_f32, void* stream);
/* Prompts, 64 tokens at a time on the tensor cores: bf16 activations, dp and vp <= 128, z given. */
int32_t logismos_time_mix_has_chunked(int32_t dp, int32_t vp);
uint32_t logismos_launch_time_mix_chunked_bf16(const lg_time_mix_t* args, int32_t n_seqs, void* stream);

/* State-space mixer with a scalar decay per head; np and vp are powers of two in 16 .. 256 with zero padding:
 *   x, B, C <- silu(conv);  dt <- softplus(dt + dt_bias)
 *   S <- exp(-exp(log_a) dt) S + dt B x^T;  y = S^T C + skip x
 * proj holds z [heads * vp] | x [heads * vp] | B [groups * np] | C [groups * np]; dt f32 [rows, ld_dt]. conv_w f32
 * [taps][channels], channels = heads * vp + 2 groups * np; conv_state f32 [slots][2][taps - 1][channels] (phase as
 * above); state f32 [slots][heads][np][vp]. */
typedef struct lg_ssd {
  const void* proj;
  int32_t ld;
  const void* dt;
  int32_t ld_dt;
  const void *conv_w, *conv_b;
  void* conv_state;
  int32_t taps;
  const void *dt_bias, *log_a, *skip;
  void* state;
  const void *state_slots, *fresh, *phase, *cu;
  void* y;
  int32_t ld_y, heads, groups, np, vp;
  void* xbc;                    /* activation format [rows, ld_xbc]: the convolved channels x | B | C */
  int32_t ld_xbc;
  /* given: f32 [heads][3], a fixed decay per head as its log2 (at least -1e4), its value and what the value's rounding dropped.
   * Every step then has size one, S <- decay S + B x^T, y = S^T C (linear attention: x, B, C its values, keys and queries); only
   * xbc, state and its indices, y and the sizes are used. */
  const void* decay;
} lg_ssd_t;
/* Convolution and silu of rows [row0, rows) from proj into xbc (seq_ids [rows]; cu, slots, fresh and phase indexed by
 * them). single: rows are one token per sequence. */
uint32_t logismos_launch_ssd_conv(const lg_ssd_t* args, const void* seq_ids_i32, int32_t row0, int32_t rows, int32_t single,
                                  int32_t is_f32, void* stream);
/* The recurrence over xbc token by token: decode steps, fp32, any size. */
uint32_t logismos_launch_ssd_step(const lg_ssd_t* args, int32_t n_seqs, int32_t is_f32, void* stream);
/* Prompts: the recurrence 64 tokens at a time on the tensor cores (np 32 .. 128, vp <= 128). */
int32_t logismos_ssd_has_chunked(int32_t np, int32_t vp);
uint32_t logismos_launch_ssd_chunked_bf16(const lg_ssd_t* args, int32_t n_seqs, void* stream);
/* The same with sequences cut in segments that run side by side, for few heads and long prompts: entries = logismos_ssd_segments
 * of the step's prompt rows (0: not worth it, the launch above), scratch of logismos_ssd_scratch_bytes, longest >= every
 * sequence. */
int32_t logismos_ssd_segments(int32_t rows, int32_t n_seqs, int32_t longest, int32_t heads);
size_t logismos_ssd_scratch_bytes(int32_t entries, int32_t heads, int32_t np, int32_t vp);
uint32_t logismos_launch_ssd_segmented_bf16(const lg_ssd_t* args, int32_t n_seqs, int32_t longest, void* scratch, int32_t entries,
                                            void* stream);
/* out = y silu(z), divided in `parts` equal parts of the heads * v true channels by each part's root mean square,
 * times gain. Rows are laid out [heads][vp]. */
uint32_t logismos_launch_gated_group_norm(const void* y, int32_t ld_y, const void* z, int32_t ld_z, const void* gain_f32,
                                          void* out, int32_t ld_out, int32_t is_f32, int32_t rows, int32_t heads,
                                          int32_t v, int32_t vp, int32_t parts, float eps, void* stream);

/* out = y / rms(y) * gain * sigmoid(z) over the heads * v true channels, laid out [heads][vp]. */
uint32_t logismos_launch_norm_gate(const void* y, int32_t ld_y, const void* z, int32_t ld_z, const void* gain_f32,
                                   void* out, int32_t ld_out, int32_t is_f32, int32_t rows, int32_t heads, int32_t v,
                                   int32_t vp, float eps, void* stream);

/* Attention whose scores are capped and biased by distance: score = cap tanh(q . k scale / cap) + bias(i - j), with
 * queries and keys of unit root mean square and an output gate. bias f32 [n_heads][far + 1] in units of log2, the
 * entry `far` standing for every larger distance; cap 0: no cap. gate: activation format, head h of a row at h *
 * head_dim; the output is multiplied by sigmoid(gate) * gate_scale. */
typedef struct lg_score_bias {
  float scale, cap;
  const void* bias;
  int32_t far;
  float max_abs_bias;           /* largest |bias|, natural units */
  float max_abs_qk;             /* bound of |q . k|, 0: unknown */
  const void* gate;
  int32_t ld_gate;
  float gate_scale;
} lg_score_bias_t;
/* Queries (in place) and keys of packed rows q [n_heads * head_dim] | k [n_kv * head_dim] | v are divided by their
 * root mean square over dim channels, queries multiplied by 1 + coef ln(floor((pos + 1) / every) + 1) (coef 0:
 * none); keys and values go to their cache slots. head_dim 64, 128 or 256. */
uint32_t logismos_launch_unit_qk_store(void* qkv, int32_t ld, void* k_pool, void* v_pool, const void* slot_mapping_i64,
                                       const void* positions_i32, int32_t rows, int32_t n_heads, int32_t n_kv_heads,
                                       int32_t head_dim, int32_t dim, float eps, float coef, float every,
                                       int64_t n_pool_slots, int32_t is_f32, void* status_i32, void* stream);
/* Decode rows (one query per sequence; q row stride ld_q): the cache already holds the new token. Scratch as
 * logismos_paged_decode_scratch_bytes; any number of query heads per key head. */
uint32_t logismos_launch_bias_attention_decode_bf16(const void* q, int32_t ld_q, const void* k_pool, const void* v_pool,
                                                    const void* block_tables, const void* context_lens,
                                                    const void* chunk_offsets, void* out, int32_t ld_out, void* scratch,
                                                    int32_t n_seqs, int32_t total_chunks, int32_t chunk_tokens,
                                                    int32_t max_blocks, int32_t n_pool_blocks, int32_t n_heads,
                                                    int32_t n_kv_heads, int32_t head_dim, const lg_score_bias_t* score,
                                                    void* status_i32, void* stream);
/* Prompt rows over their sequences' cached keys (gathered through the block tables into scratch,
 * logismos_paged_prefix_attention_scratch_bytes), causal, on the tcgen05 tiles. */
uint32_t logismos_launch_bias_attention_prefix_bf16(const void* q, int32_t ld_q, const void* cu_seqlens_q, const void* kv_lens,
                                                    const void* k_pool, const void* v_pool, const void* block_tables,
                                                    int32_t max_blocks, int32_t n_pool_blocks, void* out, int32_t ld_out,
                                                    void* scratch, int32_t n_q_tokens, int32_t total_kv_tokens,
                                                    int32_t n_seqs, int32_t max_q_len, int32_t max_kv_len, int32_t n_heads,
                                                    int32_t n_kv_heads, int32_t head_dim, const lg_score_bias_t* score,
                                                    void* status_i32, void* stream);
/* Every row over its sequence's cached keys in fp32 (seq_ids, positions per row). */
uint32_t logismos_launch_bias_attention_f32(const void* q_f32, int32_t ld_q, const void* k_pool, const void* v_pool,
                                            const void* block_tables, const void* seq_ids_i32, const void* positions_i32,
                                            void* out_f32, int32_t ld_out, int32_t rows, int32_t max_blocks,
                                            int32_t n_pool_blocks, int32_t n_heads, int32_t n_kv_heads, int32_t head_dim,
                                            const lg_score_bias_t* score, void* status_i32, void* stream);

/* ---- norms without statistics, rotary positions, windows, mixtures of experts ---------------------------------- */

/* tanh(alpha x) w + b, w and b f32 [ld] with zeros in the padding. */
typedef struct lg_tanh_norm {
  float alpha;
  const void *w, *b;
} lg_tanh_norm_t;
/* What a mixture of experts returns, rows of the experts still to be summed: sum over the token's n_pairs pairs i of
 * weights[i] (1 from top on) * rows[pair_row[i]], plus identity[token] times the row of h before this call. pair_row i32
 * [tokens, n_pairs] (negative: an identity expert). counts i32 [n_counts] are cleared. */
typedef struct lg_mixture_out {
  const void* rows;             /* activation format [., ld] */
  const void *pair_row, *weights, *identity;   /* weights f32 [tokens, top], identity f32 [tokens] */
  int32_t n_pairs, top;
  void* counts;
  int32_t n_counts;
} lg_mixture_out_t;
/* x += post(y) (y f32 [rows, ld], with zero_y cleared once read, or the sum `mixture`; post NULL: x stays), then
 * h = next(x) in the activation format (next NULL: none). row_idx selects rows of x (then post is NULL). */
uint32_t logismos_launch_tanh_norm(void* y_f32, int32_t zero_y, const lg_mixture_out_t* mixture, const void* row_idx_i32,
                                   int32_t n_src_rows, void* x_f32, const lg_tanh_norm_t* post, void* h,
                                   const lg_tanh_norm_t* next, int32_t out_f32, int32_t rows, int32_t ld, void* status_i32,
                                   void* stream);

/* Rotary positions in the interleaved layout: channels 2 i, 2 i + 1 of the first dims channels of a vector turn by the
 * angle whose amplitude-scaled cosine and sine are table[position][i] (f32 [positions][dims / 2][2]). */

/* Packed rows q [n_heads * head_dim] | k [n_kv * head_dim] | v [n_kv * head_dim]: all of q (and all of k) is divided by
 * its root mean square over its n_* * dim channels, times gain f32 [n_* * head_dim], and its heads are rotated; q in
 * place, keys and values to their cache slots. head_dim % 8 == 0. */
uint32_t logismos_launch_qk_norm_rotary_store(void* qkv, int32_t ld, void* k_pool, void* v_pool, const void* slot_mapping_i64,
                                              const void* positions_i32, int32_t rows, int32_t n_heads, int32_t n_kv_heads,
                                              int32_t head_dim, int32_t dim, const void* gain_q_f32, const void* gain_k_f32,
                                              float eps, const void* table_f32, int32_t rot_dims, int64_t n_pool_slots,
                                              int32_t is_f32, void* status_i32, void* stream);
/* Channels at .. at + dims of every head (head_dim apart, at % 8 == 0), in place. */
uint32_t logismos_launch_rotary_heads(void* q, int32_t ld, const void* positions_i32, int32_t rows, int32_t n_heads,
                                      int32_t head_dim, int32_t at, const void* table_f32, int32_t dims, int32_t is_f32,
                                      void* stream);

/* Attention over a window: a query at position i sees the keys j <= i with i - j < size or j < keep_first (size 0: all);
 * chunked: those in its own chunk of `size` positions, counted from 0. sink: one is added to the softmax denominator. gate
 * f32 [rows, ld_gate]: head h of a row is multiplied by the sigmoid of its column h (NULL: none). Scores are scaled by scale
 * (> 0).
 * pool > 0: a query also sees the blocks of `pool` positions, as a key and a value each (block b: b pool .. b pool + pool - 1)
 * that lie wholly before it. They are rows of k_mean and v_mean [n_pool_blocks][ceil(16 / pool)], as wide as the cache's:
 * block b is kept with the cache block that holds its last token, the blocks ending there one after the other
 * (logismos_launch_pool_blocks). */
typedef struct lg_window {
  float scale;
  int32_t size, keep_first, sink;
  const void* gate;
  int32_t ld_gate;
  int32_t chunked, pool;        /* of these and keep_first at most one */
  const void *k_mean, *v_mean;
  int32_t out_f32;              /* the output is fp32 whatever the queries are */
} lg_window_t;
/* Decode launches split what a query sees, leading and window blocks, as one context of this length; keys that the prompt
 * launch gathers for a sequence of kv_len keys whose last new_len are its queries. */
int32_t logismos_window_view_context(const lg_window_t* window, int32_t context_len);
int32_t logismos_window_view_keys(const lg_window_t* window, int32_t kv_len, int32_t new_len);
/* The same of a sliding window with kept keys. */
int32_t logismos_window_context(int32_t context_len, int32_t size, int32_t keep_first);
int32_t logismos_window_keys(int32_t kv_len, int32_t new_len, int32_t size, int32_t keep_first);
/* As logismos_launch_bias_attention_decode_bf16 (chunk_offsets over logismos_window_view_context of the context lengths),
 * logismos_launch_bias_attention_prefix_bf16 (total_keys and max_keys over logismos_window_view_keys) and
 * logismos_launch_bias_attention_f32. */
uint32_t logismos_launch_window_attention_decode_bf16(const void* q, int32_t ld_q, const void* k_pool, const void* v_pool,
                                                      const void* block_tables, const void* context_lens,
                                                      const void* chunk_offsets, void* out, int32_t ld_out, void* scratch,
                                                      int32_t n_seqs, int32_t total_chunks, int32_t chunk_tokens,
                                                      int32_t max_blocks, int32_t n_pool_blocks, int32_t n_heads,
                                                      int32_t n_kv_heads, int32_t head_dim, const lg_window_t* window,
                                                      void* status_i32, void* stream);
uint32_t logismos_launch_window_attention_prefix_bf16(const void* q, int32_t ld_q, const void* cu_seqlens_q, const void* kv_lens,
                                                      const void* k_pool, const void* v_pool, const void* block_tables,
                                                      int32_t max_blocks, int32_t n_pool_blocks, void* out, int32_t ld_out,
                                                      void* scratch, int32_t n_q_tokens, int32_t total_keys, int32_t n_seqs,
                                                      int32_t max_q_len, int32_t max_keys, int32_t n_heads, int32_t n_kv_heads,
                                                      int32_t head_dim, const lg_window_t* window, void* status_i32,
                                                      void* stream);
uint32_t logismos_launch_window_attention_f32(const void* q_f32, int32_t ld_q, const void* k_pool, const void* v_pool,
                                              const void* block_tables, const void* seq_ids_i32, const void* positions_i32,
                                              void* out_f32, int32_t ld_out, int32_t rows, int32_t max_blocks,
                                              int32_t n_pool_blocks, int32_t n_heads, int32_t n_kv_heads, int32_t head_dim,
                                              const lg_window_t* window, void* status_i32, void* stream);

/* Router of a mixture of experts: scores s = softmax over the n_experts + n_identity logits of a token (f32 [tokens, ld]),
 * the `top` largest s + correction are chosen, with the weights s / (sum of the chosen s + 1e-20). n_always further
 * experts (a shared one) take every token with weight 1; together n_experts + n_always groups of rows. Identity experts
 * have no rows: their weights add up in identity [tokens].
 * pair i of a token (top + n_always of them) has its row of the groups in pair_row i32 [tokens, top + n_always] (-1: identity).
 * logits are cleared with zero_logits. One launch for few tokens: offsets i32 [groups + 1], row_token i32 [pairs] included.
 * Many tokens: route (counts i32 [n_experts], zero on entry) and then place, which also copies the tokens' rows of h (bf16
 * [tokens, ld]) of the chosen experts to gathered [., ld] and lists the row tiles (logismos_launch_linear_experts_tc_bf16;
 * the tiles of the n_always groups read h itself). At most 512 router outputs, top <= 32.
 * scoring LG_ROUTE_SIGMOID: s = sigmoid(logit). groups > 0: the outputs form that many equal groups of neighbours, a group
 * scores the sum of its two largest s + correction, and only the outputs of the best keep_groups groups are chosen from. */
enum { LG_ROUTE_SOFTMAX = 0, LG_ROUTE_SIGMOID = 1 };
typedef struct lg_moe_route {
  void* logits;
  int32_t ld, zero_logits;
  const void* correction;       /* f32 [n_experts + n_identity], NULL: none */
  int32_t n_experts, n_identity, top, n_always;
  void *weights, *pair_row, *identity;
  void *offsets, *row_token;    /* few tokens, fp32 */
  void *counts, *pair_expert;   /* many tokens; pair_expert i32 [tokens, top]: group << 20 | rank in the group, -1: identity */
  void *tiles, *n_tiles;
  const void *h, *w;            /* few tokens: the logits are w h (bf16 [outputs, width], [tokens, width], fp32 sums) instead */
  int32_t width;
  void* arrived;                /* i32, zero on entry and on return */
  int32_t scoring, groups, keep_groups;
} lg_moe_route_t;
/* 1: so few tokens are best served by the one-launch form and products that stream the experts' weights. */
int32_t logismos_moe_streams(int32_t tokens, int32_t top, int32_t n_experts, int32_t n_identity, int32_t n_always, int32_t width,
                             int32_t ff);
int32_t logismos_moe_max_tiles(int32_t tokens, int32_t top, int32_t n_experts, int32_t n_always);
uint32_t logismos_launch_moe_route(const lg_moe_route_t* args, int32_t tokens, void* stream);
uint32_t logismos_launch_moe_place(const lg_moe_route_t* args, const void* h_bf16, void* gathered_bf16, int32_t ld,
                                   int32_t tokens, void* stream);

/* ---- per-head norms, pooled blocks, differences of two attentions, gated residuals -------------------------------- */

/* Packed rows q [heads * maps * hd] | k [n_kv * maps * hd] | v [n_kv * maps * hd]: every one of the q and k pieces of hd
 * channels (a multiple of 8, at most 256) is divided by its root mean square over dim of them, times gain f32 [hd], and
 * rotated; keys and values go to their cache slots. maps 1: queries in place. maps 2: the pieces of q are ordered by key
 * head, map, query head of the key head; they go to q_out [rows][heads * 2][2 hd], each to the half of its map and zeros to
 * the other, so that one attention over keys [map 1 | map 2] gives both maps' scores.
 * pool > 0: for the rows below pool_rows (one per sequence, in the order of the tables) whose token ends a block of `pool`
 * positions, the means of the block's cached keys and values go to k_mean and v_mean (lg_window_t). */
typedef struct lg_head_norm {
  void* qkv;
  int32_t ld, rows, heads, n_kv, maps, hd, dim;
  const void *gain_q, *gain_k;
  float eps;
  const void* table;            /* rotation (NULL: none) */
  int32_t rot_dims;
  void* q_out;
  int32_t ld_q;
  void *k_pool, *v_pool;
  const void *slots_i64, *positions_i32;
  int64_t n_pool_slots;
  int32_t pool, pool_rows;
  void *k_mean, *v_mean;
  const void *tables_i32, *seq_ids_i32;
  int32_t max_blocks, n_pool_blocks;
} lg_head_norm_t;
uint32_t logismos_launch_head_norm_store(const lg_head_norm_t* args, int32_t is_f32, void* status_i32, void* stream);
/* The means for the rows from pool_rows on, once all rows of the step are stored. */
uint32_t logismos_launch_pool_blocks(const lg_head_norm_t* args, int32_t is_f32, void* status_i32, void* stream);

/* Difference of two attentions over the same values: a f32 [rows, ld_a] holds heads * 2 outputs of vp channels ordered by key
 * head, map, query head of the key head; out = (a1 - lambda a2) / rms over the v true channels * scale, [rows, ld_out] with
 * head h at h * vp. */
uint32_t logismos_launch_attention_difference(const void* a_f32, int32_t ld_a, void* out, int32_t ld_out, int32_t is_f32,
                                              int32_t rows, int32_t heads, int32_t n_kv, int32_t v, int32_t vp,
                                              float lambda, float scale, float eps, void* stream);

/* Decode rows of differential attention: queries as logismos_launch_head_norm_store leaves them (2 * heads of head_dim), the
 * window's attention for both maps, and the difference above where their chunks are merged; out bf16 [n_seqs, ld_out], head h
 * at h * head_dim. Otherwise as logismos_launch_window_attention_decode_bf16, scratch for 2 * heads. */
uint32_t logismos_launch_differential_decode_bf16(const void* q, int32_t ld_q, const void* k_pool, const void* v_pool,
                                                  const void* block_tables, const void* context_lens,
                                                  const void* chunk_offsets, void* out, int32_t ld_out, void* scratch,
                                                  int32_t n_seqs, int32_t total_chunks, int32_t chunk_tokens,
                                                  int32_t max_blocks, int32_t n_pool_blocks, int32_t heads,
                                                  int32_t n_kv_heads, int32_t head_dim, const lg_window_t* window, int32_t v,
                                                  float lambda, float scale, float eps, void* status_i32, void* stream);

/* The same of prompt rows, both maps in one pass over the keys (head_dim 64 or 128: logismos_differential_has_prompts); a window
 * or chunks. Otherwise as logismos_launch_window_attention_prefix_bf16. */
int32_t logismos_differential_has_prompts(int32_t head_dim);
uint32_t logismos_launch_differential_prefix_bf16(const void* q, int32_t ld_q, const void* cu_seqlens_q, const void* kv_lens,
                                                  const void* k_pool, const void* v_pool, const void* block_tables,
                                                  int32_t max_blocks, int32_t n_pool_blocks, void* out, int32_t ld_out,
                                                  void* scratch, int32_t n_q_tokens, int32_t total_keys, int32_t n_seqs,
                                                  int32_t max_q_len, int32_t max_keys, int32_t heads, int32_t n_kv_heads,
                                                  int32_t head_dim, const lg_window_t* window, int32_t v, float lambda,
                                                  float scale, float eps, void* status_i32, void* stream);

/* Residual stream with RMS norms of one gain and gated sublayers, one launch between two sublayers:
 *   y = branch[0] (one branch), half the sum of both, each divided by its root mean square, times its gain, or a mixture
 *   x += y sigmoid(gate);   kept = x;   x += embed[ids] + step;   h = x / rms(x) * gain
 * whatever is NULL is left out. branch f32 [rows, ld], cleared once read with zero_branches; gate in the activation format;
 * embed bf16. n true columns, ld a multiple of 4, padding zero throughout. row_idx selects rows of x (no sublayer then). */
typedef struct lg_gated_residual {
  void* x;
  void* branch[2];
  int32_t zero_branches;
  const void* branch_gain[2];   /* f32 [ld], of two branches */
  const lg_mixture_out_t* mixture;
  const void* gate;
  int32_t ld_gate;
  void* kept;
  const void *embed, *ids, *step;
  int32_t vocab;
  void* h;
  float gain, eps;
  const void* row_idx;
  int32_t n_src_rows, rows, n, ld, is_f32;
} lg_gated_residual_t;
uint32_t logismos_launch_gated_residual(const lg_gated_residual_t* args, void* status_i32, void* stream);

#ifdef __cplusplus
}
#endif
#endif
