// Host-callable launchers of every CUDA kernel in this library.  The .cu files are
// free of torch headers; bindings.cpp adapts torch tensors to these entry points.
// dtype codes: 0 = bf16, 1 = fp16, 2 = fp32.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "status.h"
#include "comm_params.h"
#include "epi.h"

namespace b200 {

// What follows the read-outs o of a linear-attention recurrence:
// out = out_scale * unit_rms(o) * norm_w * act(gate), act = sigmoid or silu.
struct GatedNormOut {
  const void* gate; int64_t gate_stride;      // [tokens, heads * vdim]
  const void* norm_w; int w_head_stride;      // [vdim] (stride 0) or [heads * vdim]
  void* out; int64_t out_stride;              // [tokens, heads * vdim]
  float eps, out_scale;
  int sigmoid_gate;
};

struct DecodeParams {
  void* out;                 // [T, Hq, D] (T dtype)
  float* part_out;           // [splits, T, Hq, D]
  float* part_lse;           // [splits, T, Hq]
  const void* q;             // [T, Hq, D] with token stride q_stride (elements)
  const void* k_cache;       // K of page 0; token rows of num_kv_heads * dqk elements
  const void* v_cache;       // V of page 0; token rows of num_kv_heads * dv elements
  int64_t page_stride;       // elements between two pages (of K and of V)
  const float* kv_scales;    // kinds 1, 2
  const int* block_table;    // [B, max_blocks]
  const int* seq_lens;       // [B]
  const int* query_start_loc;  // [B+1] or null (one token per sequence)
  const float* sinks;        // [Hq] or null
  const float* alibi_slopes; // [Hq] or null: score += slope * (kv position - query position)
  float* lse_out;            // [Hq, T] or null (natural-log LSE of the final result)
  int64_t q_stride;
  int num_q_heads, num_kv_heads, block_size, max_blocks, num_splits, total_tokens;
  int64_t num_blocks;
  int dqk, dv;               // head sizes (8-bit caches: both the tile size of the kernel)
  float scale, softcap, k_scale, v_scale;
  int window;                // <=0: none
  int causal;
  StatusWord* status;
  // what happens to scores and results beyond that (all optional)
  const float* bias = nullptr;   // [Hq, bias_len]: added to the scaled (and capped) score of a key by its distance
  int bias_len = 0;              //   ... from bias_len - 1 on: the last entry
  const float* bias_tiles = nullptr;   // prompt kernel: [Hq / gp, bias_len + 254, gp], the same times log2(e): entry y of a head
                                       //   is that of distance clamp(bias_len + 126 - y, 0, bias_len - 1)
  const void* gate = nullptr;    // [T, Hq * dv] (token stride gate_stride): the result is multiplied by its sigmoid
  int64_t gate_stride = 0;
  int gate_per_head = 0;         //   ... [T, Hq]: one number per head
  float out_scale = 1.f;
  int64_t out_stride = 0;        // elements between two tokens of out (0: packed)
  int chunk = 0;                 // > 0 (causal): a position sees its own chunk of this many positions, counted from 0
  const float* sigmoid_shift = nullptr;   // [Hq]: a key's weight is sigmoid(score + shift), no softmax over the keys
};

struct PrefillParams {
  void* out;                     // [T, Hq, DV]
  float* lse_out;                // [Hq, T] or null
  const int* block_table;        // [B, max_blocks] (paged) or null
  const int* seq_lens;           // [B] kv length (paged) ; contiguous: derived from kv_start_loc
  const int* query_start_loc;    // [B+1]
  const int* kv_start_loc;       // [B+1] (contiguous mode) or null
  const float* sinks;            // [Hq] or null
  const float* alibi_slopes;     // [Hq] or null
  int num_q_heads, num_kv_heads, gp;  // gp: heads packed per tile (divides 128)
  int block_size, max_blocks;
  int64_t num_blocks;
  int total_q;
  float scale, softcap;
  int window, causal, paged;
  int dqk, dv;                   // head sizes (the kernel's tiles are padded up to 64 / 128 / 192 by the TMA fill)
  int64_t k_head_stride, v_head_stride;   // contiguous mode, elements
  int64_t page_stride;           // paged mode: elements between two pages (of K and of V)
  StatusWord* status;
  // what happens to scores and results beyond that (all optional)
  const float* bias = nullptr;   // [Hq, bias_len]: added to the scaled (and capped) score of a key by its distance
  int bias_len = 0;              //   ... from bias_len - 1 on: the last entry
  const float* bias_tiles = nullptr;   // prompt kernel: [Hq / gp, bias_len + 254, gp], the same times log2(e): entry y of a head
                                       //   is that of distance clamp(bias_len + 126 - y, 0, bias_len - 1)
  const void* gate = nullptr;    // [T, Hq * dv] (token stride gate_stride): the result is multiplied by its sigmoid
  int64_t gate_stride = 0;
  int gate_per_head = 0;         //   ... [T, Hq]: one number per head
  float out_scale = 1.f;
  int64_t out_stride = 0;        // elements between two tokens of out (0: packed)
  int chunk = 0;                 // > 0 (causal): a position sees its own chunk of this many positions, counted from 0
  const float* sigmoid_shift = nullptr;   // [Hq]: a key's weight is sigmoid(score + shift), no softmax over the keys
};

struct MlaDecodeParams {
  void* out;                   // [T, H, 512]
  float* lse_out;              // [H, T] or null
  float* part_out;             // [splits, T, H, 512]
  float* part_lse;             // [splits, T, H]
  const void* q;               // [T, H, 576], token stride q_stride (elements)
  const void* cache;           // latent cache (bf16 576 rows or 656-byte fp8 records)
  const int* block_table;      // [B, max_blocks]
  const int* seq_lens;         // [B]
  const int* query_start_loc;  // [B+1] or null (one token per sequence)
  const int* topk_indices;     // [T, topk] per-request positions (-1 = none) or null (dense)
  int64_t q_stride;
  int window;                  // > 0: only the last `window` visible positions
  int kv_rank, row_elems, q_dim;   // latent columns; elements of a cache row; entries of a query head (512, 576, 576)
  int smem_row_bytes;          // set by the launcher
  int num_heads, block_size, max_blocks, num_splits, total_tokens, batch, topk;
  int64_t num_blocks;
  float scale;
  StatusWord* status;
};

// ---- gemm_tcgen05.cu
void gemm_tn(const void* A, const void* W, void* C, const void* bias, const void* residual, int M, int N, int K,
             int lda, int ldw, int ldc, int ldr, int dtype, cudaStream_t stream, void* status, int force_bn, Epi epi);
// `batches` independent products of one shape (16-bit operands; strides in elements; 1 = the plain product)
void gemm_tn_batched(const void* A, const void* W, void* C, int batches, int M, int N, int K, int lda, int ldw, int ldc,
                     int64_t a_batch, int64_t w_batch, int64_t c_batch, int dtype, cudaStream_t stream, void* status,
                     Epi epi);
// gemm_simt.cu: any shape, pitch and alignment, 16-bit or fp32 operands, fp32 accumulation on the CUDA cores; plain,
// batched, or grouped over expert-sorted 128-row blocks (block_expert / total_padded)
struct SimtGemmParams {
  const void* A; const void* W; void* C;
  const void* bias;              // [N] or null
  int batches, M, N, K;
  int64_t lda, ldw, ldc, a_batch, w_batch, c_batch;   // elements
  const int* block_expert;       // grouped: expert of every 128-row block (w_batch = elements per expert)
  const int* total_padded;
  int experts;
  Epi epi;
};
int gemm_simt(const SimtGemmParams& p, int dtype, cudaStream_t stream);
// gemm_streamk_tcgen05.cu: swap-AB CTA-pair stream-K for skinny problems (scratch supplied by the caller)
size_t gemm_streamk_workspace_bytes(int sms);
int gemm_streamk_max_tiles();
int gemm_tn_streamk(const void* A, const void* W, void* C, const void* bias, const void* residual, int M, int N, int K,
                    int lda, int ldw, int ldc, int ldr, int dtype, cudaStream_t stream, void* status, Epi epi,
                    float* ws, int* counters, int sms, const struct RowScatter* scatter = nullptr);
void gemm_tn_pair(const void* A, const void* W, void* C, const void* bias, const void* residual, int M, int N, int K,
                  int lda, int ldw, int ldc, int ldr, int dtype, cudaStream_t stream, void* status, Epi epi,
                  const struct RowScatter* scatter = nullptr);
// ---- comm_ar_norm.cu
int ar_norm_gather(const ArNormParams& p, int dtype, cudaStream_t stream);
int nvls_ar_norm(const NvlsArNormParams& p, int dtype, cudaStream_t stream);
// ---- gemm_splitk_tcgen05.cu
int gemm_splitk_choice(int M, int N, int K, int sms);
void gemm_tn_splitk(const void* A, const void* W, void* C, const void* bias, const void* residual, int M, int N, int K,
                    int lda, int ldw, int ldc, int ldr, int dtype, cudaStream_t stream, void* status, Epi epi,
                    int splits);
// ---- norm.cu
void rms_norm(void* out, void* x, void* residual, const void* weight, float eps, int tokens, int hidden,
              int64_t x_stride, int64_t out_stride, int dtype, int mode, cudaStream_t stream);
void head_rms_norm(void* x, const void* weight, float eps, int tokens, int heads, int head_dim, int64_t token_stride,
                   int dtype, cudaStream_t stream);
void rms_norm_quant(void* out_q, float* scale_out, const float* scale_in, const void* x, void* residual,
                    const void* weight, float eps, int tokens, int hidden, int dtype, int qmode, int group, int ue8m0,
                    float scale_ub, cudaStream_t stream);
// ---- rope_cache.cu
void rope_and_cache(const int64_t* positions, void* q, void* k, const void* v, const float* cos_sin, int rot,
                    int head_dim, int num_q, int num_kv, int64_t q_stride, int64_t k_stride, int64_t v_stride,
                    int is_neox, int rot_offset, int inverse, void* kv_cache, float* kv_scales,
                    const int64_t* slot_mapping, int block_size, int64_t num_slots, int cache_kind, float k_scale,
                    float v_scale, int tokens, int dtype, void* status, cudaStream_t stream);
void copy_blocks(void* cache, const int64_t* pairs, int num_pairs, int64_t block_bytes, cudaStream_t stream);
void concat_and_cache_mla(const void* kv_c, const void* k_pe, void* cache, const int64_t* slot_mapping, int tokens,
                          int rank, int rope, int64_t kvc_stride, int64_t kpe_stride, int64_t num_slots,
                          int fp8_record, int dtype, void* status, cudaStream_t stream);
void indexer_k_quant_and_cache(const void* k, void* cache, const int64_t* slot_mapping, int tokens, int head_dim,
                               int block_size, int64_t num_slots, int64_t k_stride, int ue8m0, int dtype, void* status,
                               cudaStream_t stream, int kind = 0);
// ---- activation.cu
void act_and_mul(void* out, const void* x, int tokens, int d, int64_t x_stride, int64_t out_stride, int act, float p0,
                 float p1, int dtype, cudaStream_t stream);
void activation(void* out, const void* x, int64_t n, int act, float p0, int dtype, cudaStream_t stream);
void act_and_mul_quant(void* out_q, float* scale_out, const float* scale_in, const void* x, int tokens, int d, int act,
                       float p0, float p1, int group, int ue8m0, int dtype, cudaStream_t stream);
// ---- attention
int paged_attention_decode(const DecodeParams& p, int kv_kind, int dtype, int batch, int max_q_len, cudaStream_t stream);
// paged_attn_simt.cu: the same on the CUDA cores for fp32 caches and head sizes beyond the tensor-core kernels
int paged_attn_simt(const DecodeParams& p, int dtype, int batch, cudaStream_t stream);
int attention_prefill(const PrefillParams& p, const void* q, int64_t q_stride, const void* k_src, const void* v_src,
                      int64_t k_tok_stride, int64_t v_tok_stride, int64_t total_kv, int dqk, int dv, int dtype,
                      int batch, int max_q_len, cudaStream_t stream);
// attn_prefill_pingpong.cu: two query tiles per CTA, P and O resident in TMEM
int attention_prefill_pp(const PrefillParams& p, const void* q, int64_t q_stride, const void* k_src, const void* v_src,
                      int64_t k_tok_stride, int64_t v_tok_stride, int64_t total_kv, int dqk, int dv, int dtype,
                      int batch, int max_q_len, cudaStream_t stream);
// ---- sampling.cu
void argmax(int64_t* out, const void* logits, int rows, int vocab, int64_t stride, int dtype, cudaStream_t stream);
void sample(int64_t* out, const void* logits, int rows, int vocab, int64_t stride, const float* temperature,
            const int* top_k, const float* top_p, const float* min_p, const float* uniform, int dtype,
            cudaStream_t stream);
void apply_penalties(void* logits, const int* prompt_mask, const int* output_counts, const float* rep,
                     const float* presence, const float* frequency, int rows, int vocab, int64_t stride, int dtype,
                     cudaStream_t stream);
void advance_step(int64_t* input_ids, int64_t* positions, int* seq_lens, int64_t* slot_mapping, const int64_t* sampled,
                  const int* block_table, int max_blocks, int block_size, int batch, int64_t* token_log, int log_col,
                  int log_stride, cudaStream_t stream);
void embedding(void* out, const void* table, const int64_t* ids, int tokens, int hidden, int64_t vocab,
               int64_t vocab_start, int dtype, cudaStream_t stream);

// ---- moe.cu / gemm_grouped_tcgen05.cu
// (rows of gating start `stride` elements apart)
void topk_gating(float* weights, int* ids, const void* gating, const float* bias, int tokens, int experts, int64_t stride,
                 int topk, int mode, int renorm, float scale, int dtype, cudaStream_t stream);
void grouped_topk(float* weights, int* ids, const void* gating, const float* bias, int tokens, int experts, int topk,
                  int n_group, int topk_group, int sigmoid, int renorm, float scale, int dtype, cudaStream_t stream);
void moe_align(int* sorted_ids, int* block_expert, int* total_padded, int* inv_pos, const int* topk_ids,
               const int* expert_map, int numel, int experts, int block, int max_padded, cudaStream_t stream);
// (weights given: a pair's row is multiplied by its weight)
void moe_gather(void* out, const void* x, const int* sorted_ids, const int* total_padded, const float* weights, int max_padded,
                int numel, int topk, int hidden, int dtype, cudaStream_t stream);
// (expert_ids / through given: a pair whose expert id is at least identity_from adds its weight times the row of `through`)
void moe_combine(void* out, const void* y, const float* weights, const int* inv_pos, const void* shared,
                 const int* expert_ids, const void* through, int identity_from, int tokens, int topk, int hidden, int dtype,
                 cudaStream_t stream);
void moe_sum(void* out, const void* in, int tokens, int topk, int hidden, int dtype, cudaStream_t stream);
void gemm_grouped(const void* A, int max_rows, int lda, const void* W, int E, int N, int K, void* C, int ldc,
                  const int* block_expert, const int* total_padded, Epi epi, int dtype, cudaStream_t stream,
                  void* status);
// ---- quant.cu / gemm_fp8_blockscale.cu
void per_token_group_quant(void* q, float* scales, const void* x, int64_t rows, int K, int group, int int8, int ue8m0,
                           int col_major, float eps, int dtype, cudaStream_t stream);
void scaled_fp8_quant(void* q, float* scale, const void* x, int64_t rows, int K, int mode, float scale_ub, int dtype,
                      cudaStream_t stream);
void scaled_int8_quant(void* q, float* scale, int* azp, const void* x, int64_t rows, int K, int mode, int dtype,
                       cudaStream_t stream);
void merge_attn_states(void* out, float* out_lse, const void* p_out, const float* p_lse, const void* s_out,
                       const float* s_lse, int tokens, int heads, int D, int dtype, cudaStream_t stream);
void gemm_fp8_blockscale(const void* A, int M, int lda, const void* W, int E, int N, int K, void* C, int ldc,
                         const float* a_scale, const float* w_scale, const int* block_expert,
                         const int* total_padded, int grouped, int out_dtype, cudaStream_t stream, void* status);
// ---- gemm_scaled_mm.cu
void gemm_scaled_mm(const void* A, int M, int lda, const void* W, int E, int N, int K, void* C, int ldc,
                    const float* a_scale, int a_per_row, const float* w_scale, int w_per_col, const int* azp,
                    const int* azp_adj, const void* bias, const int* block_expert, const int* total_padded,
                    int grouped, int kind, int out_dtype, cudaStream_t stream, void* status);
// ---- gemm_wna16_tcgen05.cu
int gemm_wna16_token_tile(int M);
int gemm_wna16_splits(int M, int N, int K, int bn);
void gemm_wna16(const void* A, int M, int lda, const void* Q, const void* scales, const void* zeros, int E, int N,
                int K, int group, int bits, void* C, int ldc, const void* bias, float* partial, int splits,
                const int* block_expert, const int* total_padded, int grouped, int token_tile, int epi, int dtype,
                cudaStream_t stream, void* status);
// ---- small_gemm.cu
int small_gemm(void* C, const void* A, const void* W, const void* bias, int M, int N, int K, int lda, int ldw, int ldc,
               int dtype, int out_kind, cudaStream_t stream);
// ---- fused_misc.cu
int qkv_norm_rope_insert(void* qkv, int64_t row_stride, const void* q_w, const void* k_w, const void* iq_w,
                         const void* ik_w, const float* cos_sin, const int64_t* positions, const int64_t* slot_mapping,
                         void* q_out, void* iq_out, void* kv_cache, void* idx_cache, int tokens, int insert_tokens, int hq,
                         int hk, int niq, int has_ik, int insert_v, int rot, int is_neox, int gemma, int idx_fp8,
                         int block_size, int64_t num_slots, float eps, int dtype, cudaStream_t stream);
int fused_qk_norm_rope(void* qkv, const void* q_weight, const void* k_weight, const float* cos_sin,
                       const int64_t* positions, int tokens, int hq, int hk, int hv, int head_dim, int rot, int is_neox,
                       float eps, int gemma, int dtype, cudaStream_t stream);
void mla_rope_and_cache(void* q_pe, void* k_pe, const void* kv_c, void* cache, const float* cos_sin,
                        const int64_t* positions, const int64_t* slots, int tokens, int heads, int64_t q_tok_stride,
                        int64_t kpe_stride, int64_t kvc_stride, int is_neox, int64_t num_slots, int dtype,
                        cudaStream_t stream);
void concat_mla_q(void* out, const void* nope, const void* pe, int64_t rows, int64_t nope_stride, int64_t pe_stride,
                  int dtype, cudaStream_t stream);
void permute_cols(void* out, const void* a, const int* perm, int64_t rows, int cols, int64_t lda, int dtype,
                  cudaStream_t stream);
void gather_mla_cache(void* dst, const void* cache, const int* block_table, const int* cu_seq_lens,
                      const int* seq_starts, int batch, int max_blocks, int block_size, int max_total, int records,
                      int row_elems, int dtype, cudaStream_t stream);
void gather_indexer_k(void* dst_k, float* dst_s, const void* cache, const int* block_table, const int* cu_seq_lens,
                      int batch, int max_blocks, int block_size, int max_total, cudaStream_t stream);
// ---- mamba_scan.cu
struct ScanParams {
  const void* u; const void* delta; const void* z; void* out;
  const float* A;                 // [dim, dstate]
  const void* B; const void* C;   // [(batch,) groups, dstate, tokens]
  const float* D;                 // [dim] or null
  const float* delta_bias;        // [dim] or null
  float* state;                   // [slots, dim, dstate] fp32
  const int* query_start_loc;     // [batch+1] or null (dense layout)
  const int* cache_indices;       // [batch] or null (slot = b)
  const uint8_t* has_initial_state;  // [batch] or null (no initial state)
  int batch, dim, dstate, groups, seqlen, total_tokens, softplus, pad_slot;
};
int selective_scan_fwd(const ScanParams& p, int dtype, cudaStream_t stream);
// ---- mhc.cu
struct MhcParams {
  const void* residual;   // [T, M, H] (input streams)
  void* residual_out;     // fused: new streams [T, M, H] (a different buffer than residual)
  const void* y;          // fused: sub-layer output [T, H]
  const float* post_in;   // fused: [T, M]
  const float* comb_in;   // fused: [T, M, M]
  const float* fn;        // [mix, M*H]
  const float* scale;     // [3] (head: [1])
  const float* base;      // [mix]
  float* post_out;        // [T, M]
  float* comb_out;        // [T, M, M]
  void* x_out;            // [T, H]
  int T, M, H, iters, head;
  float rms_eps, pre_eps, sinkhorn_eps, post_mult;
};
int mhc_pre(const MhcParams& p, int fused, int dtype, cudaStream_t stream);
void mhc_post(void* out, const void* y, const void* res, const float* post, const float* comb, int tokens, int M, int H,
              int dtype, cudaStream_t stream);
// ---- p2p_copy.cu
void p2p_copy(void* dst, const void* src, size_t nbytes, int ctas, int mode, void* status, cudaStream_t stream);
// ---- comm_ag_gemm.cu
int ag_gemm_copiers(int tp, int rows_per_rank);
int ag_gemm(const AgGemmParams& p, const void* W, int ldw, void* C, const void* bias, int dtype, cudaStream_t stream);
// ---- comm_moe_a2a.cu
void moe_a2a_dispatch(const MoeA2aParams& p, const void* x, const int* topk_ids, const float* topk_w, int dtype,
                      cudaStream_t stream);
void moe_a2a_combine(const MoeA2aParams& p, const void* y, void* out, const int* topk_ids, const void* shared_out,
                     int dtype, cudaStream_t stream);
void gather_rows(void* dst, const void* src, const int* idx, const int* count, int max_rows, int limit, int row_bytes,
                 int div, cudaStream_t stream);
// ---- v4_cache.cu
void v4_qnorm_rope_kv_insert(const void* q_in, int64_t q_stride_t, int64_t q_stride_h, const void* kv, int64_t kv_stride,
                             void* q_out, void* cache, int64_t block_stride, const int64_t* slot_mapping,
                             const int64_t* positions, const float* cos_sin, int tokens, int insert_tokens, int hq,
                             int hq_pad, int block_size, float eps, cudaStream_t stream);
void v4_gather_dequant(void* dst, const void* cache, int64_t block_stride, const int64_t* slots, int n, int block_size,
                       cudaStream_t stream);
void v4_inv_rope(void* out, const void* o, int64_t o_stride_t, int64_t o_stride_h, const int64_t* positions,
                 const float* cos_sin, int tokens, int heads, int hpg, int dtype, cudaStream_t stream);
void v4_indexer_q(void* q8, float* w_out, const void* q, int64_t q_stride_t, int64_t q_stride_h, const void* weights,
                  int64_t w_stride, const int64_t* positions, const float* cos_sin, int tokens, int heads, int rot,
                  float softmax_scale, float head_scale, int dtype, cudaStream_t stream);
// ---- gdn.cu
int gdn_recurrent(void* out, float* state, const void* q, const void* k, const void* v, const float* g, const float* beta,
                  const int* query_start_loc, const int* state_idx, int batch, int hq, int hv, int dk, int dv,
                  int64_t q_stride, int64_t k_stride, int64_t v_stride, float scale, int l2norm,
                  const int* has_initial, int dtype, cudaStream_t stream);
// ---- causal_conv1d.cu (depthwise causal convolution over ragged batches with a per-sequence carry)
int causal_conv1d(void* out, const void* x, int64_t x_stride, const void* w, const void* bias, void* state,
                  const int* query_start_loc, const int* state_idx, const int* has_init, int batch, int tokens,
                  int channels, int K, int silu, int dtype, cudaStream_t stream);
// ---- residual_conv.cu (post-norm residual add + short input convolution, fp32 residual stream)
struct ResidualConvParams {
  const void* y;           // [tokens, D] sublayer output (or the embedding rows when x is null)
  const float* x;          // [tokens, D] residual stream or null
  float* x_out;            // [tokens, D] new residual stream (another buffer than x)
  void* h;                 // [tokens, D] what the next sublayer reads
  const void* gain;        // 1 or D numbers, or null
  const void* w;           // [D, K]
  float* carry;            // [slots, K-1, D] or null
  const int* qsl;          // [batch + 1]
  const int* state_idx;    // [batch] or null
  const int* has_init;     // [batch] or null
  int gain_per_channel, batch, tokens, D, K, vec;
  float eps;
};
int residual_conv(const ResidualConvParams& p, int dtype, cudaStream_t stream);
// ---- residual_norm.cu (norm of a finished sublayer's output + residual add + norm in front of the next one)
struct ResidualNormParams {
  const void* y;           // [rows, D] sublayer output; its row for token t is t, ids[t], or a weighted sum (topk > 0)
  const int64_t* ids;      // [tokens] rows of y (an embedding table of `rows` rows), or null
  const float* weights;    // topk > 0: y holds expert-sorted rows, token t's is sum_k weights[t, k] * y[inv_pos[t, k]]
  const int* inv_pos;      //   ... pairs with inv_pos < 0 are skipped,
  const int* expert_ids;   //   ... unless expert_ids[t, k] >= identity_from: those add weights[t, k] * through[t]
  const void* through;     // [tokens, D] or null
  const void* shared;      // [tokens, D] added to the sum, or null
  const float* x;          // [tokens, D] residual stream, or null: x' = scale * y
  float* x_out;            // [tokens, D] new residual stream or null (may be x itself)
  void* h;                 // [tokens, D] x' normed
  const void* gain;        // norm of y: 1 or D numbers
  const void* gain2;       // norm of x': 1 or D numbers
  int gain_n, gain2_n, gain_f32;   // gain_f32: the gains are fp32 (else of y's type)
  int tokens, D, vec, topk, identity_from;
  int64_t rows;
  float eps, scale;
  StatusWord* status;
};
int residual_norm(const ResidualNormParams& p, int dtype, cudaStream_t stream);
// ---- prenorm.cu (residual add + layer norm in front of the next sublayer, or the operand of a loop's entry product)
struct PrenormParams {
  const void* y;           // [rows, D] as in ResidualNormParams; y_f32: fp32 rows
  const int64_t* ids;      // [tokens] rows of y, or null
  const float* weights;    // topk > 0: expert-sorted rows; null weights: ones
  const int* inv_pos;
  const void* shared;      // [tokens, D] or null
  const float* x;          // [tokens, D] or null
  const void* add;         // [D] or null
  float* x_out;            // [tokens, D] or null
  void* h;                 // [tokens, D]; with `table`: [tokens, 3 D] = x' in two 16-bit parts | table row (fp32: [tokens, 2 D])
  const void* gain;        // [D]
  const void* table;       // loop operand: rows of the embedding table ...
  const int64_t* table_ids;
  int tokens, D, vec, topk, y_f32;
  int64_t rows, table_rows;
  float eps;
  StatusWord* status;
};
int prenorm(const PrenormParams& p, int dtype, cudaStream_t stream);
// ---- stream_norm.cu (sublayer boundary of decoders whose residual is several streams)
constexpr int kMaxStreams = 8;
struct StreamNormParams {
  const void* y;           // [tokens, D] the finished sublayer's output, or null in front of the first one
  const float* x;          // [tokens, streams, D], or null: every stream is scale * table[ids]
  const void* table; const int64_t* ids; int64_t rows; float scale;
  const float* coef;       // [streams] read | [streams] write | [streams, streams] mix (from, to)
  const float* gain;       // [D]
  float* x_out;            // [tokens, streams, D] (may be x) or null
  void* h;                 // [tokens, D]
  int tokens, D, streams, vec;
  float eps;
  StatusWord* status;
};
int stream_norm(const StreamNormParams& p, int dtype, cudaStream_t stream);
// ---- head_norm_rope.cu (epilogue of a merged q | k | v product: head norms, partial rotation, paged cache write)
struct HeadNormRopeParams {
  const void* qkv; int64_t row_stride; int q_off, k_off, v_off;   // [tokens, ...], heads packed from these columns on
  void* q_out;                          // [tokens, heads, dim_pad] (heads = 0: keys and values only)
  void* k_cache; void* v_cache;         // K / V of page 0, or null: queries only
  int64_t page_stride, num_slots;       // elements between two pages
  const void* q_w; const void* k_w;     // [dim_pad] norm weights or null
  int normed;                           // 0: no norm (without weights a norm multiplies by one)
  const float* q_scale;                 // [heads]: factors of the queries, or null
  const float* angles;                  // [tokens, 2, rot / 2]: cosines, sines
  const int64_t* slots;
  int tokens, heads, kv_heads, dim, dim_pad, vdim_pad, rot, block_size, one_plus, vec;
  int whole_row, interleaved;           // one norm over all heads (weights [heads, dim_pad]); pairs (2i, 2i + 1)
  const int64_t* positions;             // with temp_coef: queries times 1 + temp_coef * ln((position + 1) / temp_every + 1)
  float temp_coef; int temp_every;
  float eps;
  StatusWord* status;
};
int head_norm_rope(const HeadNormRopeParams& p, int dtype, cudaStream_t stream);
// cos and sin of position * inv_freq, [tokens, 2, half]; whole turns are taken off in fp64
void rope_angles(float* out, const int64_t* positions, const double* inv_freq, int tokens, int half, cudaStream_t stream);
// ---- gla.cu (linear attention with a decay)
struct GlaParams {
  const void* qkvg;            // [tokens, row_stride]: q | k | v at the given element offsets
  int64_t row_stride;
  int q_off, k_off, v_off;
  const float* alpha;          // [tokens, heads * dim] decays per key channel, or null:
  const float* decay_tok;      // [tokens, heads], or null:
  const float* decay_head;     // [heads]
  const float* k_mul;          // matrix memory: [tokens, heads] factors of k,
  const float* floor;          //   [tokens, heads] least absolute value of the divisor,
  float* norm_state;           //   [slots, heads, ceil(vdim / 16), dim] (equal copies), or null
  GatedNormOut out;
  float* state;                // [slots, heads, dim, vdim]
  float* o_raw;                // set from the scratch: [tokens, heads * vdim] raw outputs of heads split over CTAs
  float* seg_state;            // set from the scratch: [segments, heads, dim, vdim] ...
  float* seg_decay;            // ... and [segments, heads, dim] ...
  float* seg_norm;             // ... twice, or null
  const int* qsl; const int* state_idx; const int* has_init;
  int batch, tokens, heads, dim, vdim, col_block, vec, chunk, silu_qkv, whole_row;
  float scale;
};
struct GlaScratch { int64_t raw, segments; };
GlaScratch gla_scratch(int batch, int tokens, int heads, int dim, int vdim, int max_query_len, int sms, bool whole_row);
int gla_recurrent(GlaParams p, float* scratch, int max_query_len, int sms, int dtype, cudaStream_t stream);
struct MemoryGatesParams {
  const float* logits; int64_t stride;   // [tokens, >= 2 heads]: input gates, forget gates
  const float* bias;                     // [2 heads]
  float* top;                            // [slots, heads]
  float* out;                            // [3, tokens, heads]: decay, k_mul, floor
  const int* qsl; const int* state_idx; const int* has_init;
  int batch, tokens, heads;
  float cap;
};
void memory_gates(const MemoryGatesParams& p, int max_query_len, cudaStream_t stream);
// ---- channel_delta.cu (gated delta rule with a decay per key channel)
struct ChannelDeltaParams {
  const void* qkv; int64_t row_stride; int q_off, k_off, v_off;
  const float* g; int64_t g_stride;            // [tokens, heads * dim] decays
  const float* beta; int64_t beta_stride;      // [tokens, heads] logits of the step sizes
  GatedNormOut out;
  float* state;                                // [slots, heads, dim, vdim]
  float4* lengths;                             // set from the scratch: [tokens, kv_heads] 1 / |q|, 1 / |k|, q . k, or null
  float* o_raw;                                // set from the scratch: [tokens, heads * vdim] where heads are split over CTAs
  const int* qsl; const int* state_idx; const int* has_init;
  int batch, tokens, heads, kv_heads, dim, vdim, col_block, lanes, vec, chunk;
};
int64_t channel_delta_scratch(int batch, int tokens, int heads, int kv_heads, int dim, int vdim, int max_query_len, int sms,
                              int shape);
int channel_delta(ChannelDeltaParams p, float* scratch, int max_query_len, int sms, int shape, int dtype, cudaStream_t stream);
// ---- rglru.cu (real-gated linear recurrent unit)
struct RgLruParams {
  const void* u; int64_t u_stride;       // [tokens, width] recurrence input
  const void* y; int64_t y_stride;       // [tokens, width] gate branch before its gelu
  float* gates;                          // [tokens, blocks, 2, width / blocks] logits without bias; overwritten
  const float* r_bias; const float* i_bias; const float* decay;   // [width]; decay = -8 softplus(lambda)
  float* state;                          // [slots, width]
  float* summary;                        // [chunks, 2, width] scratch, needed when a sequence spans several chunks
  void* out;                             // [tokens, width]
  const int* qsl; const int* state_idx; const int* has_init;
  int batch, tokens, width, block_width;
};
int rglru_chunk();                       // tokens per chunk
int rglru_scan(const RgLruParams& p, int max_query_len, int dtype, cudaStream_t stream);
// ---- latent_attn.cu (latent attention of any sizes: projection epilogues, fp32 attention)
struct LatentInsertParams {
  const void* a; int64_t a_stride; int q_off, kv_off;   // [tokens, ...]: query latent | key latent, rotated key part
  const void* q_w; const void* kv_w;                    // norm weights
  void* cq;                                             // [tokens, q_rank] (q_rank = 0: no query latent)
  void* cache; int64_t row_elems, num_slots;            // [slots, row_elems]
  const int64_t* slots;
  const float* angles;                                  // [tokens, 2, rot_dims / 2]: cosines, sines
  int tokens, q_rank, kv_rank, rot_dim, rot_dims;
  int interleaved;                                      // pairs (2i, 2i + 1) instead of (i, i + rot_dims / 2)
  float eps;
  StatusWord* status;
};
int latent_insert(const LatentInsertParams& p, int dtype, cudaStream_t stream);
// Rotates the first rot_dims of the rot_dim entries at src (per token and head) into dst and zeroes `pad` entries behind.
int latent_rope(const void* src, int64_t src_tok, int64_t src_head, void* dst, int64_t dst_tok, int64_t dst_head,
                const float* angles, int tokens, int heads, int rot_dim, int rot_dims, int pad, bool interleaved, int dtype,
                cudaStream_t stream);
int latent_attn_simt(const MlaDecodeParams& p, int dtype, cudaStream_t stream);
// ---- tq_cache.cu (TurboQuant KV cache, head_dim 128)
int tq_slot_bytes(int kbits, int vbits);
int tq_store(void* cache, const void* k, const void* v, int64_t k_stride, int64_t v_stride, const int64_t* slot_mapping,
             int tokens, int heads, int64_t num_slots, int kbits, int vbits, int nc, int dtype, cudaStream_t stream);
int tq_dequant(void* k_out, void* v_out, const void* cache, const int64_t* slots, int rows, int heads, int kbits, int vbits,
               int nc, int dtype, cudaStream_t stream);
int tq_decode(void* out, float* part_out, float* part_lse, const void* q, int64_t q_stride, const void* cache,
              const int* block_table, int max_blocks, const int* seq_lens, int batch, int hq, int hkv, int block_size,
              int64_t num_blocks, int splits, float scale, int kbits, int vbits, int nc, int dtype, cudaStream_t stream);
// ---- comm_allreduce.cu
int custom_allreduce(const CustomArParams& p, const void* in, void* out, int dtype, int mode, cudaStream_t stream);
int reduce_rms(const ReduceRmsParams& p, int dtype, cudaStream_t stream);
// ---- mla_decode.cu
// impl: 0 = choose (tcgen05 kernel for dense 16-bit caches from 64 heads per rank up), 1 = mma.sync kernel,
// 2 = tcgen05 kernel or fail.  Returns 0, or -1 when impl 2 was asked for and that kernel does not serve the call.
int mla_decode(const MlaDecodeParams& p, int fp8_records, int dtype, cudaStream_t stream, int impl = 1);
// ---- mla_decode_tcgen05.cu: 0 = launched, -1 = not served
int mla_decode_tc(const MlaDecodeParams& p, int dtype, cudaStream_t stream);
// ---- indexer.cu
void indexer_logits(float* logits, int64_t logits_stride, const void* q, const float* w, const void* cache,
                    const int* block_table, int max_blocks, const int* seq_lens, const int* query_start_loc,
                    int tokens, int batch, int heads, int block_size, int64_t num_blocks, int max_len, void* status,
                    cudaStream_t stream, int kind = 0);   // kind 1: int8 queries and keys
// ---- indexer_tcgen05.cu: returns -1 when the shapes are not served (caller falls back to indexer_logits)
int indexer_logits_tc(float* logits, int64_t logits_stride, const void* q, const float* w, const void* cache,
                      const int* block_table, int max_blocks, const int* seq_lens, const int* query_start_loc,
                      int tokens, int batch, int heads, int block_size, int64_t num_blocks, int max_len,
                      int max_query_len, void* status, cudaStream_t stream, int kind);
void topk_per_row(int* out, const float* x, int64_t stride, const int* row_len, int rows, int cols, int k,
                  cudaStream_t stream);
// ---- comm_gemm_ar_norm.cu (FusedArParams: comm_params.h)
struct FusedArParams;
int gemm_ar_norm(const FusedArParams& p, const void* A, int lda, const void* W, int ldw, int dtype,
                 cudaStream_t stream);

}  // namespace b200
