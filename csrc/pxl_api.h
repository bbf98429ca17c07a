// C ABI of libpxl_kernels.so — the sm_100a kernel library of parallax_b200.
//
// Conventions
//   * every pointer is a device pointer unless its name ends in `_host`;
//   * bf16 tensors are passed as `void*`; shapes are row-major, innermost last;
//   * `stream` is a cudaStream_t passed as an opaque pointer;
//   * launchers return 0 (PXL_OK) or a PxlStatus error code; they never
//     synchronise and never allocate device memory unless stated otherwise;
//   * `status` is an optional device int. Kernels with bounded waits or index
//     checks write a non-zero PxlStatus code there instead of trapping.
#pragma once
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef struct CUstream_st* pxl_stream_t;

// GEMM epilogues
#define PXL_EPI_NONE 0      // C = A W^T (+bias)                      bf16 out
#define PXL_EPI_RESIDUAL 1  // C = A W^T (+bias) + residual           bf16 out
#define PXL_EPI_SILU_MUL 2  // C[:, j] = silu(gate_j) * up_j          bf16 out, N/2 columns
#define PXL_EPI_F32 3       // C = A W^T (+bias)                      fp32 out
#define PXL_EPI_RS 4        // partial sums scattered to the owning rank + reduce (pxl_gemm_bf16_rs)
#define PXL_EPI_SCATTER 5   // every output row stored through its own pointer, possibly on a peer GPU
#define PXL_EPI_SPLITK_T 6  // internal: small-M path (operands swapped, split along K, fp32 slabs + last-CTA finish)
#define PXL_EPI_SPLITK_C 7  // internal: small-M path, the K ranges of a tile form a cluster and reduce over DSMEM
#define PXL_EPI_SPLITK_CN 8 // internal: mid-M path (operands not swapped), K ranges of a tile reduce inside a cluster
#define PXL_EPI_GATE 9      // internal: C = (A W^T) * sigmoid(gate)      bf16 out (pxl_gemm_bf16_heads)
#define PXL_EPI_GLU 11      // act(gate) * up (* sigmoid(row gate)), arranged alike (pxl_gemm_bf16_act_glu)
#define PXL_EPI_ACT 12      // act(A W^T) (* table[ids[row], column])       bf16 out (pxl_gemm_bf16_act)
#define PXL_EPI_CLIP_GLU 10 // clipped GLU of gate / up groups arranged as for PXL_EPI_SILU_MUL (pxl_gemm_bf16_glu)

#define PXL_NORM_LAYER 0    // (x - mean) / sqrt(variance + eps)
#define PXL_NORM_RMS 1      // x / sqrt(mean(x^2) + eps)

// ---- gemm_tcgen05.cu -------------------------------------------------------
// C[M,N] = A[M,K] * W[N,K]^T. lda/ldw/ldc in elements. `bn` = tile width (64/128/256)
// or 0 to pick automatically. For PXL_EPI_SILU_MUL the rows of W must be arranged in
// groups of 128: 64 gate rows followed by the 64 up rows of the same outputs (bn >= 128).
int pxl_gemm_bf16(const void* A, const void* W, void* C, const void* residual, const void* bias,
                  int M, int N, int K, int lda, int ldw, int ldc, int epi, int bn, int* status,
                  pxl_stream_t stream);
int pxl_gemm_bf16_pick_bn(int M, int N, int epi);
// Small-M (decode) GEMM, M <= 128: the weight matrix takes the 128-row operand slot of the tensor
// core, the few activation rows the narrow one, and K is split over `splitk` CTAs per 128 output
// columns (0 = automatic) so that every SM streams weights. mode 2: the CTAs of one tile form a
// thread-block cluster (splitk <= 8), exchange their fp32 partial sums through distributed shared
// memory and each finishes a slice of the tokens (+ bias, + residual, bf16 out). mode 1: partial
// sums meet in an fp32 scratch owned by the library (one per stream) and the CTA that arrives last
// finishes the tile. mode 0 picks. Sums are formed in K order either way (bitwise repeatable).
// pxl_gemm_bf16 takes this path by itself when bn == 0 and the shape qualifies.
int pxl_gemm_bf16_small_m(const void* A, const void* W, void* C, const void* residual, const void* bias,
                          int M, int N, int K, int lda, int ldw, int ldc, int splitk, int mode, int* status,
                          pxl_stream_t stream);
// Clipped GLU in the epilogue: g = min(gate, limit), u = clamp(up, -limit, limit), C = g sigmoid(1.702 g) (u + 1).
// W rows in groups of 128 (64 gate rows, the 64 up rows of the same outputs); C has N / 2 columns.
int pxl_gemm_bf16_glu(const void* A, const void* W, void* C, int M, int N, int K, int lda, int ldw, int ldc, float limit,
                      int bn, int* status, pxl_stream_t stream);
// C = act(A W^T), times table[ids[row] * ld_table + column] if table is given (bf16). act 2 = gelu (tanh form), 3 = square
// of relu.
int pxl_gemm_bf16_act(const void* A, const void* W, void* C, int M, int N, int K, int lda, int ldw, int ldc, int act,
                      const void* table, int64_t ld_table, const int* ids, int64_t num_ids, int* status, pxl_stream_t stream);
// Gated activation in the epilogue: C = act(g) u, act 0 = silu, 2 = gelu (tanh form); with row_gate (fp32) row m times
// sigmoid(row_gate[m * ld_row_gate]). W and C as above.
int pxl_gemm_bf16_act_glu(const void* A, const void* W, void* C, int M, int N, int K, int lda, int ldw, int ldc, int act,
                          const float* row_gate, int64_t ld_row_gate, int bn, int* status, pxl_stream_t stream);
// One product per attention head in one launch: for every head h < heads
//   C[m, h * c_head + n] = sum_k A[m, h * a_head + k] * W[h * N + n, k]   (n < N, k < K)
// optionally times sigmoid(gate[m, h * N + n]). bf16; K, N, strides and head offsets multiples of 8, pointers 16-byte
// aligned.
int pxl_gemm_bf16_heads(const void* A, const void* W, void* C, const void* gate, int M, int heads, int N, int K, int lda,
                        int a_head, int ldw, int ldc, int c_head, int ldg, int* status, pxl_stream_t stream);
// 1 when pxl_gemm_bf16(bn = 0) would use the small-M path for this shape and epilogue.
int pxl_gemm_bf16_uses_small_m(int M, int N, int K, int epi);

// ---- elementwise.cu ----------------------------------------------------------
// out = x * rsqrt(mean(x^2) + eps) * (w + w_offset). If residual != NULL:
// residual += x first (in place) and the norm is taken of the sum.
int pxl_rmsnorm(const void* x, const void* weight, void* out, void* residual, int T, int H,
                float eps, float w_offset, pxl_stream_t stream);
// Same without residual for rows with their own strides (a column slice of a wider matrix; out may be x).
int pxl_rmsnorm_strided(const void* x, int64_t ldx, const void* weight, void* out, int64_t ldo, int T, int H,
                        float eps, float w_offset, pxl_stream_t stream);
// Per-head q/k RMSNorm (optional) + rotary embedding (neox pairing, first `rot_dim`
// dims) on a packed qkv activation [T, (Hq + 2*Hkv) * D], writing q in place and
// scattering k, v into the paged cache [blocks, Hkv, page, D] at slot_mapping[t]
// (slot < 0: skip). cos_sin: fp32 [max_pos, rot_dim] = cos | sin halves. A position outside [0, max_pos)
// sets PXL_DEV_BAD_POSITION and leaves its row unrotated (max_pos <= 0: not checked).
int pxl_qk_norm_rope_cache(void* qkv, const void* q_norm_w, const void* k_norm_w,
                           const float* cos_sin, const int* positions, const int64_t* slot_mapping,
                           void* k_cache, void* v_cache, int T, int Hq, int Hkv, int D, int rot_dim,
                           int page_size, int64_t num_slots, float eps, float norm_w_offset,
                           int max_pos, int* status, pxl_stream_t stream);
// Plain scatter of k, v [T, Hkv, D] (row strides in elements) into the paged cache.
int pxl_reshape_and_cache(const void* k, const void* v, int64_t k_stride, int64_t v_stride,
                          const int64_t* slot_mapping, void* k_cache, void* v_cache, int T,
                          int Hkv, int Dk, int Dv, int page_size, int64_t num_slots, int* status,
                          pxl_stream_t stream);
// e4m3 KV cache ("fp8 KV"): the caches hold one byte per element; K is stored as k / k_scale and V as
// v / v_scale (saturating, scales > 0) and the *_fp8 attention entry points undo the scaling. Same
// arguments as the bf16 functions plus the two scales.
int pxl_qk_norm_rope_cache_fp8(void* qkv, const void* q_norm_w, const void* k_norm_w,
                               const float* cos_sin, const int* positions,
                               const int64_t* slot_mapping, void* k_cache, void* v_cache, int T,
                               int Hq, int Hkv, int D, int rot_dim, int page_size, int64_t num_slots,
                               float eps, float norm_w_offset, float k_scale, float v_scale,
                               int max_pos, int* status, pxl_stream_t stream);
int pxl_reshape_and_cache_fp8(const void* k, const void* v, int64_t k_stride, int64_t v_stride,
                              const int64_t* slot_mapping, void* k_cache, void* v_cache, int T,
                              int Hkv, int Dk, int Dv, int page_size, int64_t num_slots,
                              float k_scale, float v_scale, int* status, pxl_stream_t stream);
int pxl_attn_decode_fp8(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache,
                        const int* block_tables, const int* ctx_lens, void* out, float* workspace,
                        const float* sinks, int B, int Hq, int Hkv, int D, int page_size,
                        int max_blocks, int64_t num_blocks, float scale, int window, int num_splits,
                        int max_ctx, float k_scale, float v_scale, int* status, pxl_stream_t stream);
int pxl_attn_prefill_fp8(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache,
                         const int* block_tables, const int* cu_q, const int* ctx_lens, void* out,
                         int64_t out_stride, const float* sinks, int B, int max_q_len, int Hq,
                         int Hkv, int D, int page_size, int max_blocks, int64_t num_blocks,
                         float scale, int window, float k_scale, float v_scale, int* status,
                         pxl_stream_t stream);
// out[T, I] = act(x[:, :I]) * x[:, I:]; mode 0 = silu, 1 = clipped swiglu-oai
// (alpha 1.702, limit), 2 = gelu-tanh.
int pxl_act_mul(const void* x, void* out, int T, int I, int mode, float limit, pxl_stream_t stream);
// out[t, :] = table[ids[t], :]  (ids int32 or int64 per `ids_are_i64`)
int pxl_gather_rows(const void* table, const void* ids, void* out, int T, int H, int64_t num_rows,
                    int ids_are_i64, int* status, pxl_stream_t stream);
// Bounded-wait self-test (see elementwise.cu): waits for *flag >= epoch like a fused kernel waits for a peer;
// *result = 1 when it arrived, 0 when the wait ran out (then *status = PXL_DEV_TIMEOUT_PEER).
int pxl_selftest_bounded_wait(const uint32_t* flag, uint32_t epoch, int* result, int* status, pxl_stream_t stream);
// dst[dst_idx[i]] = src[src_idx[i]] for i < n (int32 words; indices checked against dst_len / src_len)
int pxl_patch_i32(int* dst, const int* dst_idx, const int* src, const int* src_idx, int n, int dst_len, int src_len,
                  int* status, pxl_stream_t stream);
// y += x (bf16), n elements (multiple of 8)
int pxl_add_inplace(void* y, const void* x, int64_t n, pxl_stream_t stream);

// ---- attention_decode.cu -----------------------------------------------------
// Single-query GQA attention over the paged cache [blocks, Hkv, page, D] (D = 64 or 128).
// q [B, Hq, D] with row stride q_stride elements; out [B, Hq, D]; block_tables [B, max_blocks]; ctx_lens [B].
// window <= 0: full attention; with a window the sequence's first keep_first keys stay visible. sinks: optional fp32 [Hq] logits added to the
// softmax denominator. workspace: fp32, >= B*Hq*num_splits*(D+2) floats when
// num_splits > 1. num_splits = 0 picks automatically (see pxl_attn_decode_splits).
int pxl_attn_decode(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache,
                    const int* block_tables, const int* ctx_lens, void* out, float* workspace,
                    const float* sinks, int B, int Hq, int Hkv, int D, int page_size,
                    int max_blocks, int64_t num_blocks, float scale, int window, int keep_first, int num_splits,
                    int max_ctx, float softcap, const float* sig_bias, int* status, pxl_stream_t stream);
int pxl_attn_decode_splits(int B, int Hkv, int max_ctx);

// softcap > 0: scores become softcap * tanh(score / softcap). sig_bias [Hq]: the weight of a key is sigmoid(score + bias) and
// nothing normalises the weights (sinks do not count then). The same in the prefill entry points.

// ---- attention_prefill.cu ----------------------------------------------------
// Ragged causal attention of new query tokens against the paged cache, which must
// already hold K/V of the new tokens and of any cached prefix. q/out [T, Hq, D]
// with row stride q_stride/out_stride elements; cu_q [B+1] token offsets;
// ctx_lens[b] = prefix + new length of sequence b.
int pxl_attn_prefill(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache,
                     const int* block_tables, const int* cu_q, const int* ctx_lens, void* out,
                     int64_t out_stride, const float* sinks, int B, int max_q_len, int Hq, int Hkv,
                     int D, int page_size, int max_blocks, int64_t num_blocks, float scale,
                     int window, int keep_first, float softcap, const float* sig_bias, int* status, pxl_stream_t stream);

// ---- attention_prefill_tc.cu ------------------------------------------------------
// Same contract on the tcgen05 tensor cores (D = 128, page 16 / 32 / 64). total_q = rows of q / out.
int pxl_attn_prefill_tc(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache,
                        const int* block_tables, const int* cu_q, const int* ctx_lens, void* out,
                        int64_t out_stride, const float* sinks, int B, int max_q_len, int total_q, int Hq,
                        int Hkv, int D, int page_size, int max_blocks, int64_t num_blocks, float scale,
                        int window, int keep_first, float softcap, const float* sig_bias, int* status, pxl_stream_t stream);

// ---- sampler.cu ----------------------------------------------------------------
// Greedy arg-max over logits [B, V] (bf16 if logits_bf16 else fp32, row stride ld).
// A row without a finite maximum (all NaN) yields token 0 and sets PXL_DEV_NONFINITE_LOGITS in *status
// (status may be null).
int pxl_argmax(const void* logits, int logits_bf16, int64_t ld, int B, int V, int* out_ids,
               float* out_logprob, int* status, pxl_stream_t stream);
// Temperature / top-k / top-p / min-p sampling, one uniform random number per row.
// temperature <= 0 or top_k == 1 selects arg-max for that row.
int pxl_sample(const void* logits, int logits_bf16, int64_t ld, int B, int V,
               const float* temperature, const int* top_k, const float* top_p, const float* min_p,
               const float* uniform, int* out_ids, float* out_prob, int* status, pxl_stream_t stream);

// ---- moe.cu ------------------------------------------------------------------
// Router: scores [T, E] fp32/bf16 logits -> top-k expert ids and weights.
// Scores: softmax (mode 0) or sigmoid (mode 1). Selection by score + e_bias (optional), limited to the topk_group
// best of n_group groups (1/1 = none; a group counts as the sum of its group_top best, group_top 1 or 2). Weights =
// scores, optionally renormalised, times routed_scale. ld: elements between rows of logits.
int pxl_moe_route(const void* logits, int64_t ld, int logits_bf16, const float* e_bias, int T, int E, int k,
                  int mode, int renorm, int n_group, int topk_group, int group_top, float routed_scale,
                  int* out_ids, float* out_w, pxl_stream_t stream);

int pxl_moe_align(const int* ids, int T, int k, int E, int e_lo, int e_hi, int* counts,
                  int* offsets, int* cursor, int* mt_expert, int* mt_row0, int* mt_row_end,
                  int* num_mt, int max_mt, int* pos_of, int* src_tok, pxl_stream_t stream);
int pxl_moe_gather(const void* x, const int* src_tok, const int* n_rows, void* x_perm,
                   int max_rows, int H, pxl_stream_t stream);
// x_perm[pos_of[t, j]] = w[t, j] * x[t] (pos_of < 0: no row); any width, bf16 or fp32
int pxl_moe_scatter_rows(const void* x, int64_t ldx, const int* pos_of, const float* w, void* x_perm, int T, int k, int H,
                         int is_f32, pxl_stream_t stream);
int pxl_moe_combine(const void* y_perm, const int* pos_of, const float* w, const void* base,
                    void* out, int T, int k, int H, pxl_stream_t stream);
// Grouped GEMM over experts (see gemm_tcgen05.cu).
int pxl_gemm_bf16_grouped(const void* A, const void* W, void* C, const void* bias, int P, int E, int N, int K,
                          int lda, int ldw, int ldc, const int* mt_expert, const int* mt_row0,
                          const int* mt_row_end, const int* num_mt, int max_m_tiles, int epi, float limit,
                          int bn, int* status, pxl_stream_t stream);

// Fused tensor-parallel collectives (see gemm_tcgen05.cu for the buffer contracts).
int pxl_gemm_bf16_rs(const void* A, const void* W, void* out, const void* residual,
                     void* const* stage_ptrs, void* const* flag_ptrs, int rank, int tp,
                     int rows_per_rank, int N, int K, int lda, int ldw, int ldo, uint32_t epoch,
                     int bn, int* status, pxl_stream_t stream);
int pxl_gemm_bf16_ag(void* const* x_ptrs, void* const* ready_ptrs, void* tile_flags, const void* W,
                     void* C, const void* bias, int rank, int tp, int rows_per_rank, int N, int K,
                     int lda, int ldw, int ldc, int epi, uint32_t epoch, int ncopy, int bn,
                     int* status, pxl_stream_t stream);

// ---- mla.cu: multi-head latent attention on the compressed cache [blocks, page, 512 + 64] ----
// RMSNorm(latent) + interleaved RoPE(k_pe) of ckv [T, 576] (row stride ld) written to the cache.
int pxl_mla_kv_prep(const void* ckv, int64_t ld, const void* norm_w, const float* cos_sin,
                    const int* positions, const int64_t* slots, void* cache, int T, int latent,
                    int rope, int64_t num_slots, float eps, int* status, pxl_stream_t stream);
// q [T, H, nope + 64] -> q_nope_hm [H, Tpad, nope] (head-major, input of the absorb GEMM) and
// q_pe [T, H, 64] with interleaved RoPE applied.
int pxl_mla_q_prep(const void* q, int64_t ld, const float* cos_sin, const int* positions,
                   void* q_nope_hm, void* q_pe, int T, int Tpad, int H, int nope, int rope,
                   pxl_stream_t stream);
// Absorbed attention for tokens [tok_begin, tok_begin + n_tok): q_lat [H, Tpad, 512], q_pe
// [T, H, 64] -> out [H, Tpad, 512]. Query token t sits at positions[t] of sequence
// cu_q-lookup(t) (cu_q NULL: sequence t - tok_begin) and attends keys 0..positions[t], or, when
// topk != NULL and topk[t][0] >= 0, the listed positions only (topk rows indexed by t).
int pxl_mla_attn(const void* q_lat, const void* q_pe, const void* cache, const int* block_tables,
                 const int* cu_q, const int* positions, const int* topk, void* out, int tok_begin,
                 int n_tok, int Tpad, int H, int B, int max_blocks, int page, int latent, int rope,
                 int topk_k, int topk_stride, float scale, pxl_stream_t stream);

// ---- dsa.cu: lightning indexer -------------------------------------------------------------
// scores[t, j] = sum_h relu(q[t,h,:] . k_j) * w[t,h] for j <= positions[t], -inf beyond;
// ld_scores >= ceil(max_ctx / 64) * 64.
int pxl_dsa_index_scores(const void* q, const float* w, const void* index_cache,
                         const int* block_tables, const int* cu_q, const int* positions,
                         float* scores, int64_t ld_scores, int T, int B, int Hi, int Di,
                         int max_blocks, int page, int max_ctx, pxl_stream_t stream);
// Positions of the k largest scores among [0, positions[t]] per row (unordered); rows with at
// most k candidates are filled with -1 ("attend densely").
int pxl_topk_select(const float* scores, int64_t ld, const int* positions, int T, int k, int* out,
                    int64_t ld_out, pxl_stream_t stream);
// Indexer pre-processing of a step (Di == 128): q_idx [T, Hi*Di] gets the interleaved rotation on the first R
// dims of every head in place; the index key kv[t, k_off : k_off+Di] is layer-normed (w, optional b), rotated
// on its first R dims and stored at cache[slots[t]]; w_out[t, h] = kv[t, w_off+h] * w_scale (fp32).
int pxl_dsa_index_prep(void* q_idx, int64_t ldq, const void* kv, int64_t ldkv, int k_off, int w_off,
                       const void* ln_w, const void* ln_b, float ln_eps, const float* cos_sin,
                       const int* positions, int max_pos, const int64_t* slots, void* cache, int64_t num_slots,
                       float* w_out, float w_scale, int T, int Hi, int Di, int R, int* status,
                       pxl_stream_t stream);
// cache[slots[t], :] = src[t, :] (slot < 0: skip)
int pxl_store_rows(const void* src, int64_t ld, const int64_t* slots, void* cache, int T, int D,
                   int64_t num_slots, int* status, pxl_stream_t stream);

// ---- gemm_fp8.cu: block-scaled e4m3 GEMM (1x128 activation groups, weight scales per 64 rows x 128 cols)
// C[M,N] bf16 = sum over 128-wide K blocks of a_s[m,kb] * w_s[n/64,kb] * (A_kb W_kb^T). K % 128 == 0,
// N % 128 == 0. epi: PXL_EPI_NONE / PXL_EPI_RESIDUAL / PXL_EPI_SILU_MUL (W rows interleaved as for bf16).
int pxl_gemm_fp8_block(const void* A, const float* a_s, const void* W, const float* w_s, void* C,
                       const void* residual, int M, int N, int K, int lda, int ldw, int ldc, int epi,
                       int* status, pxl_stream_t stream);
int pxl_gemm_fp8_block_grouped(const void* A, const float* a_s, const void* W, const float* w_s, void* C,
                               int P, int E, int N, int K, int lda, int ldw, int ldc, const int* mt_expert,
                               const int* mt_row0, const int* mt_row_end, const int* num_mt, int max_m_tiles,
                               int epi, int* status, pxl_stream_t stream);
// x [T,K] bf16 (row stride ld) -> q [T,K] e4m3 + scales [T, K/128]: x ~= q * scale per group
int pxl_quant_fp8_rows(const void* x, int64_t ld, void* q, float* scales, int T, int K, pxl_stream_t stream);

// ---- moe_ep.cu + the scatter epilogue of gemm_tcgen05.cu: expert parallelism over peer memory ----
int pxl_ep_dispatch(const void* x, int64_t ldx, const int* ids, int n_rows, int k, int H,
                    int experts_per_rank, int cap, int rank, int ep, void* const* recv_x_ptrs,
                    void* const* recv_meta_ptrs, void* const* recv_cnt_ptrs, void* const* flag_ptrs,
                    int* cursor, uint32_t* done_counter, uint32_t epoch, int* status, pxl_stream_t stream);
int pxl_ep_recv_ids(const int* recv_meta, const int* recv_cnt, const void* disp_flag, int ep, int cap,
                    uint32_t epoch, int* ids_out, int* status, pxl_stream_t stream);
int pxl_ep_row_ptrs(const int* src_slot, const int* n_rows, const int* recv_meta, int cap, int H, int ep,
                    void* const* comb_ptrs, void** row_ptrs, int max_rows, pxl_stream_t stream);
int pxl_gemm_bf16_grouped_scatter(const void* A, const void* W, void* const* row_ptrs, int P, int E, int N,
                                  int K, int lda, int ldw, const int* mt_expert, const int* mt_row0,
                                  const int* mt_row_end, const int* num_mt, int max_m_tiles,
                                  void* const* flag_ptrs, uint32_t* done_counter, int rank, int ep_size,
                                  uint32_t epoch, int* status, pxl_stream_t stream);
int pxl_ep_combine(const void* comb, const float* w, const void* base, int64_t ld_base, void* out,
                   int64_t ld_out, const void* ret_flag, int ep, uint32_t epoch, int n_rows, int k, int H,
                   int* status, pxl_stream_t stream);

// ---- linear_attn.cu: gated delta-net layers (per-request state slots) ---------------------------
// y = silu(causal_conv(x)) per channel with the last K-1 inputs carried in conv_state [slots, C, K-1];
// sequence b covers tokens [seq_cu[b], seq_cu[b+1]) and uses slot seq_slots[b]; a sequence whose
// first token has position 0 starts from zeros.
int pxl_causal_conv1d_silu(const void* x, int64_t ldx, const void* w, const void* bias, void* conv_state,
                           const int* seq_cu, const int* seq_slots, const int* positions, void* out,
                           int64_t ldo, int B, int C, int K, pxl_stream_t stream);
// Gated delta rule over qkv [T, 2*Hk*Dk + Hv*Dv] (q | k | v), gates a, b [T, Hv] (shared row stride),
// output gate z [T, Hv*Dv]; rec_state [slots, Hv, Dv, Dk] fp32; out [T, Hv*Dv] after the gated RMSNorm.
int pxl_gated_delta_rule(const void* qkv, int64_t ld_qkv, const void* a, const void* b, int64_t ld_ab,
                         const float* A_log, const float* dt_bias, const void* z, int64_t ld_z,
                         const void* norm_w, float* rec_state, const int* seq_cu, const int* seq_slots,
                         const int* positions, void* out, int64_t ld_out, int B, int Hk, int Hv, int Dk,
                         int Dv, float eps, pxl_stream_t stream);
// out = x * sigmoid(gate), rows of N elements with their own strides
int pxl_sigmoid_gate_mul(const void* x, int64_t ldx, const void* gate, int64_t ldg, void* out, int64_t ldo,
                         int T, int N, pxl_stream_t stream);

// out = (res +) x * sigmoid(gate[:, col / group]); gate [T, N / group]; res may be null; group % 8 == 0
int pxl_gate_mul_grouped(const void* x, int64_t ldx, const void* gate, int64_t ldg, const void* res, int64_t ldr,
                         void* out, int64_t ldo, int T, int N, int group, pxl_stream_t stream);
// out[t] = x[t, :K] . w[:K] (bf16 out)
int pxl_row_dot(const void* x, int64_t ldx, const void* w, void* out, int T, int K, pxl_stream_t stream);

// ---- msa.cu: block-sparse attention indexer --------------------------------------------------
// scores[t, j] = max over index heads and visible tokens of 128-token block j of scale * iq . ik
int pxl_msa_block_scores(const void* iq, const void* index_cache, const int* block_tables, const int* cu_q,
                         const int* positions, float* scores, int64_t ld, int T, int B, int Hi, int Di,
                         int max_blocks, int page, int sparse_block, int max_ctx, float scale,
                         pxl_stream_t stream);
// top-k blocks per query (first init_blocks and the last local_blocks always kept) expanded into a
// virtual block table v_tables [T, topk * sparse_block / page] and visible-token count v_ctx [T]
int pxl_msa_select(const float* scores, int64_t ld, const int* positions, const int* block_tables,
                   const int* cu_q, int T, int B, int max_blocks, int page, int sparse_block, int topk,
                   int init_blocks, int local_blocks, int* v_tables, int64_t ld_vt, int* v_ctx,
                   pxl_stream_t stream);

// ---- gemm_simt.cu: fp32 operands, and bf16 shapes the TMA rules exclude -----------------------------
// C[m, h*c_head + n] = sum_k A[m, h*a_head + k] * W[h*N + n, k] (+ bias[h*N + n]) (+ residual at C's place)
// (* sigmoid(gate[m, h*N + n])); fp32 accumulation in K order. in_f32: operands, bias and gate are fp32.
int pxl_gemm_simt(const void* A, const void* W, void* C, const void* bias, const void* residual, const void* gate, int M,
                  int N, int K, int64_t lda, int64_t ldw, int64_t ldc, int64_t ldg, int heads, int64_t a_head,
                  int64_t c_head, int in_f32, int out_f32, pxl_stream_t stream);
// Grouped form over the device tile lists of pxl_moe_align: C[r, :N] = A[a_rows ? a_rows[r] : r] . W_expert^T
int pxl_gemm_simt_grouped(const void* A, const void* W, void* C, const int* a_rows, int N, int K, int64_t lda, int64_t ldw,
                          int64_t ldc, const int* mt_expert, const int* mt_row0, const int* mt_row_end, const int* num_mt,
                          int max_m_tiles, int is_f32, pxl_stream_t stream);

// ---- residual.cu: fp32 residual stream -----------------------------------------------------------------
// out[t] = table[ids[t]] * scale (+ hash[row]), row = (prev[t] * mul_prev + ids[t] * mul_cur) mod buckets, or
// `buckets` when prev[t] < 0. hash may be null.
int pxl_embed_rows(const void* table, const int* ids, float scale, const void* hash, const int* prev, int64_t mul_prev,
                   int64_t mul_cur, int64_t buckets, float* out, int T, int W, int64_t num_rows, int is_f32, int* status,
                   pxl_stream_t stream);
int pxl_f32_to_bf16(const float* x, void* out, int64_t n, pxl_stream_t stream);
// x += mult * norm(y) * w in place; low (bf16) receives the sum when y is bf16. kind: PXL_NORM_*.
int pxl_residual_norm(float* x, const void* y, const float* w, void* low, int T, int W, float eps, float mult, int kind,
                      int y_f32, pxl_stream_t stream);
// out[t] = norm(x[rows ? rows[t] : t]) * w; groups > 1 (RMS): statistics of each of that many equal parts of the row
int pxl_row_norm(const float* x, const float* w, const int* rows, int64_t num_rows, void* out, int T, int W, float eps,
                 int kind, int groups, int out_f32, int* status, pxl_stream_t stream);
// fp32 form of pxl_act_mul
int pxl_act_mul_f32(const float* x, float* out, int T, int I, int mode, float limit, pxl_stream_t stream);

// x += y (+ sum_j weights[t, j] * (pos_of[t, j] >= 0 ? rows[pos_of[t, j]] : h[t])) in place; with a norm weight w:
// low = x / sqrt(mean(x^2) + eps) * w, the mean taken over each of `groups` equal parts of the row. y may be null. With y2:
// x += mult * (y / rms(y) * yw + y2 / rms(y2) * y2w) instead of y. y, y2, rows, h and low are bf16, or fp32 when y_f32.
int pxl_residual_add(float* x, const void* y, int64_t ldy, const void* rows, int64_t ldr, int64_t num_rows,
                     const int* pos_of, const float* weights, int k, const void* h, const float* w, void* low, int T, int W,
                     float eps, const float* yw, const void* y2, const float* y2w, float mult, int groups, int y_f32,
                     int* status, pxl_stream_t stream);
// out[t, c] = act(gate) * up (* sigmoid(row_gate[t * ldg])) of x [T, 2 I] with gate / up columns in alternating groups
// of 64; mode 0 = silu, 1 = clipped GLU with `limit`, 2 = gelu (tanh form)
int pxl_glu_act(const void* x, const float* row_gate, int64_t ldg, void* out, int64_t ldo, int T, int I, int mode, float limit,
                int is_f32, pxl_stream_t stream);

// ---- attn_prep.cu: in front of and behind softmax attention with grouped heads ---------------------------
// proj [T, ld]: q (H x dk columns from q_off), k (G x dk), v (G x dv; G == 0: no keys and values). Convolution taps
// conv_w [taps, q | k | v channels] (null: none) over each sequence's tokens with the state slots conv_state
// [slots, taps - 1, channels]; RMS norm over the whole q and k rows; rotation of the first `rot` dimensions of a head
// (pairs i, i + rot / 2). q_out [T, H, cols] and the pages get heads padded with zeros to `cols`. Sequences: seq_cu
// [n + 1], the first prefill_seqs are slices (prefill_tokens tokens), each later one is one decoded token.
int pxl_conv_qkv_prep(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int G, int dk, int dv, int cols,
                      int rot, int taps, const void* conv_w, void* conv_state, int num_state_slots, const float* q_norm,
                      const float* k_norm, const float* cos_sin, const int* positions, int max_pos, const int* seq_cu,
                      const int* seq_slots, int prefill_seqs, int prefill_tokens, int T, const int64_t* slots,
                      int64_t num_slots, int page, void* k_cache, void* v_cache, void* q_out, float eps, int is_f32,
                      int* status, pxl_stream_t stream);
// Without convolution and norm weights (all null) q and k are only rotated.
// out[t, h * dv + d] = x[t, h, d] (, RMS-normed over all heads, or per head, * norm_w) * sigmoid(gate[t, h * dv + d]) * scale;
// columns up to out_cols are zeroed. x [T, heads, x_cols].
int pxl_gated_rows(const void* x, int heads, int x_cols, int dv, const void* gate, int64_t ldg, const float* norm_w, float eps,
                   int per_head, float scale, void* out, int64_t ldo, int out_cols, int T, int is_f32, pxl_stream_t stream);

// Heads normed one by one without weights: rotation of the first `rot` dimensions (0: none), q and k over their root mean
// square, queries times head_scale [H] and pos_scale [max_pos], values (1 - v_mix) v + v_mix v_first ([T, ldf]; null: v).
int pxl_head_qkv_prep(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int G, int dk, int dv, int cols, int rot,
                      float eps, const float* cos_sin, const float* pos_scale, const float* head_scale, const int* positions,
                      int max_pos, const void* v_first, int64_t ldf, float v_mix, const int64_t* slots, int64_t num_slots, int page,
                      void* k_cache, void* v_cache, void* q_out, int T, int is_f32, int* status, pxl_stream_t stream);
// out[t] = x[t] * silu(gate[t]) over the root mean square of each of `groups` equal parts, times w; zeros behind the row
int pxl_gated_norm_rows(const void* x, int n, const void* gate, int64_t ldg, const float* w, int groups, float eps, void* out,
                        int64_t ldo, int out_cols, int T, int is_f32, pxl_stream_t stream);

// ---- attention_any.cu: paged attention of any head size, bf16 or fp32, on the FMA pipes ------------------
// Arguments as pxl_attn_prefill; cu_q null: token i is the only query of sequence i.
int pxl_attn_any(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache, const int* block_tables,
                 const int* cu_q, const int* ctx_lens, void* out, int64_t out_stride, const float* sinks, int B, int max_q,
                 int Hq, int Hkv, int D, int page, int max_blocks, int64_t num_blocks, float scale, int window, int keep_first,
                 float softcap, const float* sig_bias, int is_f32, int* status, pxl_stream_t stream);

// ---- lightning_attn.cu: linear attention with a fixed decay per head ------------------------------------
// q, k [T, H x dk] and v [T, H x dv] are columns of proj, all passed through silu here. state [slots, H, dk, dv] fp32,
// decay_pow [H, pow_len = 65]: decay^0 .. decay^64. Sequences as for pxl_conv_qkv_prep.
int pxl_lightning_attn(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int dk, int dv,
                       const float* decay_pow, int pow_len, float* state, int num_slots, const int* seq_cu,
                       const int* seq_slots, const int* positions, void* out, int64_t ldo, int prefill_seqs, int decode_seqs,
                       int is_f32, int* status, pxl_stream_t stream);

// ---- latent_attn.cu / latent_attn_tc.cu: latent attention of any widths, window, sinks -------------------
// proj [T, ld]: `heads` query heads of q_width columns (rotated part of R dims at q_rot_off) and, at kv_off, the raw
// latent (L) | key part (R). Writes cache[slots[t]] = RMSnorm(latent) * norm_w | rotated key and the rotated query
// parts to q_cat[t, h, L:]. Interleaved pairs; the first `rot` of the R dims are rotated. cos_sin [max_pos, rot].
int pxl_latent_prep(const void* proj, int64_t ld, int kv_off, int heads, int q_width, int q_rot_off, const float* norm_w,
                    const float* cos_sin, const int* positions, int max_pos, const int64_t* slots, void* cache,
                    int64_t num_slots, void* q_cat, int T, int L, int R, int rot, float eps, int is_f32, int* status,
                    pxl_stream_t stream);
// The same for queries that go through a latent of their own: pxl_latent_rows writes the cache rows and
// c_q[t] = RMSnorm(proj[t, q_off : q_off + q_rank]) * q_norm, pxl_latent_queries the rotated parts of q [T, ldq].
int pxl_latent_rows(const void* proj, int64_t ld, int q_off, int q_rank, const float* q_norm, void* c_q, int kv_off,
                    const float* norm_w, const float* cos_sin, const int* positions, int max_pos, const int64_t* slots,
                    void* cache, int64_t num_slots, int T, int L, int R, int rot, float eps, int is_f32, int* status,
                    pxl_stream_t stream);
int pxl_latent_queries(const void* q, int64_t ldq, int heads, int q_width, int q_rot_off, const float* cos_sin,
                       const int* positions, int max_pos, void* q_cat, int T, int L, int R, int rot, int is_f32, int* status,
                       pxl_stream_t stream);
// out[t, h, :L] = attention of q[t, h, :L+R] over the cached rows of t's sequence (cu_q null: token t is the only
// query of sequence t). The queries are the last tokens of ctx_lens[b]. window <= 0: no window; sinks may be null.
int pxl_latent_attn(const void* q, const void* cache, const int* block_tables, const int* cu_q, const int* ctx_lens,
                    void* out, const float* sinks, int B, int max_q, int H, int L, int R, int page, int max_blocks,
                    int64_t num_blocks, float scale, int window, int is_f32, int* status, pxl_stream_t stream);
// bf16 tensor-core form of pxl_latent_attn (L and R multiples of 8, L + R <= 576, scale > 0; total_q = rows of q).
int pxl_latent_attn_tc_supported(int L, int R, int page, float scale);
int pxl_latent_attn_tc(const void* q, const void* cache, const int* block_tables, const int* cu_q, const int* ctx_lens,
                       void* out, const float* sinks, int B, int max_q, int total_q, int H, int L, int R, int page,
                       int max_blocks, int64_t num_blocks, float scale, int window, int* status, pxl_stream_t stream);

// ---- matrix_memory.cu: mLSTM ------------------------------------------------------------------------------
// q, k [T, H x dk] and v [T, H x dv] are columns of proj; gates [T, ldg] fp32: H input gates | H forget gates before
// bias [2 H] and the soft cap. state [slots, H, words] fp32, words >= dk * dv + ceil(dv / 32) * (dk + 1): S, then per 32
// columns of v a copy of the normaliser, then as many copies of the running maximum. out [T, ldo]: heads side by side.
// Sequences as for pxl_conv_qkv_prep.
int pxl_matrix_memory(const void* proj, int64_t ld, int q_off, int k_off, int v_off, int H, int dk, int dv, const float* gates,
                      int64_t ldg, const float* bias, float cap, float* state, int64_t words, int num_slots, const int* seq_cu,
                      const int* seq_slots, const int* positions, void* out, int64_t ldo, int prefill_seqs, int decode_seqs,
                      int is_f32, int* status, pxl_stream_t stream);

// Mamba-2 state space on the same kernels: x (H x dv), B and C (groups x n) are columns of x, dt [T, ldt] fp32 logits; S <-
// exp(-exp(A_log) d) S + d B x^T, out = S^T C + D x with d = softplus(dt + dt_bias); state [slots, H, n, dv] fp32.
int pxl_state_space(const void* x, int64_t ld, int x_off, int b_off, int c_off, int H, int groups, int n, int dv, const float* dt,
                    int64_t ldt, const float* dt_bias, const float* A_log, const float* D, float* state, int num_slots,
                    const int* seq_cu, const int* seq_slots, const int* positions, void* out, int64_t ldo, int prefill_seqs,
                    int decode_seqs, int is_f32, int* status, pxl_stream_t stream);

// ---- delta_rule.cu: gated delta rule with a decay per key channel ------------------------------------------
// q, k [T, Hk x dk] and v [T, H x dv] are columns of x; decay [T, ldd] (H x dk) and beta [T, ldb] (H) fp32 logits, state
// [slots, H, dk, dv] fp32. Prompt slices in bf16 need `work` (pxl_delta_rule_workspace bytes); without it they run token by token.
int64_t pxl_delta_rule_workspace(int H, int dk, int dv, int prefill_seqs, int prefill_tokens);
int pxl_delta_rule(const void* x, int64_t ld, int q_off, int k_off, int v_off, int H, int Hk, int dk, int dv, const float* decay,
                   int64_t ldd, const float* dt_bias, const float* A_log, const float* beta, int64_t ldb, float* state,
                   int num_slots, const int* seq_cu, const int* seq_slots, const int* positions, void* out, int64_t ldo,
                   int prefill_seqs, int prefill_tokens, int decode_seqs, void* work, int64_t work_bytes, int is_f32, int* status,
                   pxl_stream_t stream);

// ---- short_conv.cu: causal convolution per channel + SiLU ---------------------------------------------------
// x [T, ldx] (C channels), w [taps, C], bias [C] or null, state [slots, taps - 1, C] (the last inputs), out [T, C].
int pxl_short_conv(const void* x, int64_t ldx, int C, int taps, const void* w, const void* bias, void* state, int num_slots,
                   const int* positions, const int* seq_cu, const int* seq_slots, int prefill_seqs, int prefill_tokens, int T,
                   void* out, int is_f32, int* status, pxl_stream_t stream);

// ---- tanh_norm.cu: the fp32 residual between two products --------------------------------------------------
// In place: x += norm(y + sum_j weights[t, j] * rows[pos_of[t, j]]) (post 1: tanh(alpha z) w + b, 2: z / rms(z) * w),
// x += table[ids[t]], x += step; then low = x (pre 2) or tanh(pre_alpha x) pre_w + pre_b (pre 1). Null or 0: left out;
// null weights count as 1. y, rows, table and low are bf16, or fp32 when is_f32.
int pxl_residual_step(float* x, const void* y, int64_t ldy, const void* rows, int64_t ldr, int64_t num_rows, const int* pos_of,
                      const float* weights, int k, int post, const float* post_w, const float* post_b, float post_alpha, float eps,
                      const void* table, const int* ids, int64_t num_ids, const float* step, int pre, const float* pre_w,
                      const float* pre_b, float pre_alpha, void* low, int T, int W, int is_f32, int* status, pxl_stream_t stream);
// out[t] = tanh(alpha x[rows ? rows[t] : t]) w + b
int pxl_tanh_norm(const float* x, const float* w, const float* b, float alpha, const int* rows, int64_t num_rows, void* out,
                  int T, int W, int out_f32, int* status, pxl_stream_t stream);
// out[t, c] = act(x[t, c]) (* table[ids[t] * ldt + col + c]); act 2 = gelu (tanh form), 3 = square of relu
int pxl_act_rows(const void* x, int64_t ldx, int x_f32, int act, const void* table, int64_t ldt, int col, const int* ids,
                 int64_t num_ids, void* out, int64_t ldo, int out_f32, int T, int N, int* status, pxl_stream_t stream);

// ---- stage_exec.cu: all layers of a dense GQA stage for one step behind one call --------------
// The descriptor structs are defined in stage_exec.cu (mirrored by parallax_b200/engine/native_stage.py).
struct PxlStageDesc;
struct PxlStepDesc;
struct PxlStageWorkspace;
int pxl_stage_forward_dense(const struct PxlStageDesc* stage, const struct PxlStepDesc* step,
                            const struct PxlStageWorkspace* ws, const void* h_in, void** h_out, int* launches,
                            int* status, pxl_stream_t stream);

#ifdef __cplusplus
}
#endif
