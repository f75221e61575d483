// C ABI of the sm_100a kernel library.  Kernel sources include only this header and CUDA headers
// (no libtorch), so they compile in seconds; bindings.cpp adapts torch tensors to these calls.
// Every launcher returns 0 on success, a cudaError_t value or a small positive code on bad arguments.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

// dtype codes: 0 = float32, 1 = bfloat16, 2 = float16

// ---- GEMM (tcgen05) -------------------------------------------------------------------------
typedef struct GemmArgs {
  void* out;          // [T, ldo] bf16/fp16
  const void* bias;   // [N] or null
  float* ws;          // stream-K partial tiles (tiles * max_contrib * bn * 128 floats)
  int* counters;      // per-tile arrival tickets, zero on entry, zero again on exit
  int* status;        // device status word: 0 = ok, otherwise the code of the wait that timed out
  int T, N, K;
  int n_tiles, t_tiles;
  int per_cta;        // stream-K: k-block units per CTA; 0 = whole tiles, strided over the grid
  int max_contrib;    // stream-K: workspace slots per tile
  int grid;
  int fmt;            // 1 = bf16, 0 = fp16
  int ldo;            // row stride of out (elements)
  int bn;             // token tile: 16 / 32 / 64 / 128 / 256
  int num_sms;
  int stages;         // 0 = choose from the shared-memory budget
  int ctas_per_sm;    // 0 = choose (2 for small token tiles)
  int act;            // 0 = plain; 1 silu, 2 gelu-tanh, 3 swigluoai on [64 gate | 64 up] interleaved weight tiles; 4 = square
                      // of relu on every output
  // collective fusion over peer memory (all zero / null = plain GEMM)
  void* rs_stage[8];  // reduce-scatter: staging area of every rank (peer mappings)
  void* rs_flags[8];  // reduce-scatter: per-(source, token tile) arrival counters on every rank
  const void* ag_flags;  // all-gather: local per-token-tile arrival counters
  int rs_on, rs_tloc, rs_rank, ag_on, ag_expect;
  unsigned spin_limit;
  // signed 8-bit operands (kind::i8): per-token activation scales [T], per-channel weight scales [N]; fmt = output type
  int i8;
  const float* a_scale;
  const float* w_scale;
} GemmArgs;
int b200_gemm_pick_bn(int T);
int b200_gemm_launch(const GemmArgs* a, const void* tmapW, const void* tmapX, cudaStream_t st);

// Decode-sized GEMM (one token tile of at most 32 rows): cluster split-K with the reduction in the leader CTA's
// shared memory; optional gated activation or tensor-parallel push epilogue (gemm/gemm_decode.cu).
typedef struct GemmDecodeArgs {
  void* out;            // [T, ldo]
  const void* bias;     // [N] or null
  int* status;
  int T, N, K;
  int n_tiles;          // ceil(N / 128)
  int S;                // CTAs per cluster = K splits per weight tile, 1..8 (at most 4 when bn = 32)
  int kb_per_cta;       // ceil(ceil(K / 64) / S); (S - 1) * kb_per_cta must be < ceil(K / 64)
  int fmt, ldo, bn;     // bn: 16 or 32
  int stages;           // 0 = choose
  int ctas_per_sm;      // 1 or 2: shared-memory budget per CTA
  int act;              // as in GemmArgs
  // row-parallel epilogue under tensor parallelism: store locally and push {data, epoch} units to every peer
  int ar_on, rank, nranks;
  void* ll_bufs[8];     // low-latency all-reduce buffers of all ranks (peer mappings)
  const void* epoch_word;  // device word holding the number of completed all-reduce calls
  int64_t ll_slot_bytes;
  // fp8 e4m3 operands with 128x128 weight block scales and 1x128 activation scales (fmt then names the output type;
  // a k-block is 128 elements, so kb_per_cta counts blocks of 128)
  int fp8;
  const float* a_scale;    // [ceil(K/128), a_stride] transposed activation scales
  const float* w_scale;    // [ceil(N/128), ceil(K/128)]
  int a_stride;
  int i8;  // signed 8-bit operands (kind::i8): a_scale [T] per token, w_scale [N] per channel; fmt = output type
  // 4-bit weights (AWQ / GPTQ after repacking): the weight tensor map covers the packed bytes [N, K / 2] (32-byte x
  // 128-row boxes, no swizzle); scale / zero [N, K / group] in the activation type; group a multiple of 64
  int w4, w4_group;
  const void* w4_scale;
  const void* w4_zero;
  // qkv epilogue (head_dim 128): split + optional q / k RMSNorm + rotary + K / V cache write; out = q [T, Hq * 128]
  int qk_on, qk_hq, qk_hkv, qk_neox, qk_gemma, qk_block_size;
  float qk_eps;
  const int64_t* qk_positions;
  const float* qk_cos_sin;
  const void* qk_q_w;
  const void* qk_k_w;
  void* qk_kv_cache;
  const int64_t* qk_slots;
  int64_t qk_num_blocks, qk_max_pos;
} GemmDecodeArgs;
int b200_gemm_decode_launch(const GemmDecodeArgs* a, const void* tmapW, const void* tmapX, cudaStream_t st);

// Grouped (rows sorted by expert) and/or fp8 block-scaled GEMM; lod == null -> one group of M rows.
typedef struct GroupedGemmArgs {
  void* out;             // [M, ldo] bf16/fp16
  const void* bias;      // [E, N] or null
  const int* lod;        // [E + 1] device, or null
  const float* a_scale;  // fp8: [ceil(K/128), a_stride] transposed activation scales
  const float* w_scale;  // fp8: [E, ceil(N/128), ceil(K/128)]
  int* status;
  int M, N, K, E, ldo, a_stride;
  int fp8;               // 1 = e4m3 inputs
  int fmt;               // 16-bit inputs: 1 = bf16, 0 = fp16
  int out_fmt;           // 1 = bf16, 0 = fp16, 2 = fp32 (16-bit inputs, no bias)
  int bn;                // token tile 16 / 32 / 64 / 128
  int grid;
  int act;               // 0, or 4 = square of relu (16-bit inputs)
} GroupedGemmArgs;
int b200_grouped_gemm_launch(const GroupedGemmArgs* a, const void* tmapW, const void* tmapX, cudaStream_t st);

// Encodes a 2-D row-major [rows, cols] tensor map with a [box_rows, box_cols] box and 128-byte
// swizzle into `out` (128 bytes).  elem_bytes = 1 or 2.
int b200_encode_tmap_2d(void* out, const void* base, uint64_t rows, uint64_t cols, uint64_t row_stride_bytes,
                        uint32_t box_rows, uint32_t box_cols, int elem_bytes);

// Same for a plain (unswizzled) byte tensor: [rows, row_bytes] with a [box_rows, box_bytes] box; box_bytes a multiple
// of 16.
int b200_encode_tmap_2d_raw(void* out, const void* base, uint64_t rows, uint64_t row_bytes, uint64_t row_stride_bytes,
                            uint32_t box_rows, uint32_t box_bytes);
// out [N, K] (bf16 / fp16) = (q - zero) * scale of 4-bit weights packed as [N, K / 2] (see quantization/int4.py)
int b200_dequant_w4(void* out, const void* packed, const void* scale, const void* zero, int64_t N, int K, int group,
                    int dtype, cudaStream_t st);

// ---- elementwise ----------------------------------------------------------------------------
int b200_rmsnorm(void* out, const void* x, void* residual, const void* w, int64_t rows, int H, float eps, int gemma,
                 int64_t x_stride, int64_t out_stride, int dtype, cudaStream_t st);
int b200_rownorm(void* out, const void* x, const void* z, const void* w, int64_t rows, int D, float eps, int mode,
                 int dtype, cudaStream_t st);
int b200_act_and_mul(void* out, const void* x, int64_t rows, int d, int act, float limit, int dtype, cudaStream_t st);
int b200_quick_gelu(void* out, const void* x, int64_t n, int dtype, cudaStream_t st);
int b200_embedding(void* out, const int64_t* ids, const void* w, int64_t T, int H, int64_t rows, int64_t vocab_start,
                   int dtype, cudaStream_t st);
// scratch_val / scratch_idx: rows * chunks entries each (partial maxima)
int b200_argmax(int64_t* out, const void* logits, int64_t rows, int V, int64_t stride, int dtype, float* scratch_val,
                int* scratch_idx, int chunks, cudaStream_t st);

// ---- rotary / cache -------------------------------------------------------------------------
int b200_qkv_split_norm_rope_cache(void* q_out, const void* qkv, const int64_t* positions, const float* cos_sin,
                                   const void* q_w, const void* k_w, float eps, int64_t T, int Hq, int Hkv, int D,
                                   int rot_dim, int neox, int gemma, void* kv_cache, const int64_t* slots,
                                   int block_size, int64_t num_blocks, int64_t max_pos, int64_t qkv_stride, int dtype,
                                   cudaStream_t st);
int b200_rope(void* q, void* k, const int64_t* positions, const float* cos_sin, int64_t T, int Hq, int Hk, int D,
              int rot_dim, int neox, int64_t max_pos, int64_t q_stride, int64_t k_stride, const int64_t* positions3,
              int sec0, int sec1, int interleaved, int dtype, cudaStream_t st);
int b200_reshape_and_cache(const void* k, const void* v, void* kv_cache, const int64_t* slots, int64_t T, int Hkv,
                           int D, int block_size, int64_t num_blocks, int64_t k_stride, int64_t v_stride, int dtype,
                           cudaStream_t st);
int b200_concat_and_cache_mla(const void* kv_c, const void* k_pe, void* cache, const int64_t* slots, int64_t T,
                              int rank, int rope, int64_t total_slots, int64_t kvc_stride, int64_t kpe_stride, int fp8,
                              int dtype, cudaStream_t st);
int b200_indexer_prep(const void* q, const void* k, const void* ln_w, const void* ln_b, const int64_t* positions,
                      const float* cos_sin, const void* head_w, float wscale, void* q_out, float* w_out, void* cache,
                      const int64_t* slots, int64_t T, int H, int64_t max_pos, int64_t total_slots, int64_t q_stride,
                      int64_t k_stride, int64_t hw_stride, float eps, int ue8m0, int64_t q_lo, int64_t q_hi, int block_size, int dtype,
                      cudaStream_t st);
int b200_indexer_k_quant_and_cache(const void* k, void* cache, const int64_t* slots, int64_t T, int64_t total_slots,
                                   int ue8m0, int64_t k_stride, int block_size, int dtype, cudaStream_t st);
int b200_convert_req_index(int32_t* out, const int32_t* req_id, const int32_t* block_table, const int32_t* idx,
                           int64_t T, int topk, int block_size, int max_blocks, int num_reqs, cudaStream_t st);
int b200_copy_blocks(void* cache, const int64_t* src, const int64_t* dst, int64_t n_pairs, int64_t bytes_per_block,
                     int64_t num_blocks, cudaStream_t st);
int b200_merge_attn_states(void* out, float* lse_out, const void* o1, const float* lse1, const void* o2,
                           const float* lse2, int64_t rows, int D, int dtype, cudaStream_t st);

// ---- attention ------------------------------------------------------------------------------
int b200_paged_attention(void* out, const void* q, const void* kv_cache, const int* block_tables, const int* seq_lens,
                         const int* qsl, const float* sinks, float* ws_o, float* ws_lse, int64_t T, int B, int Hq,
                         int Hkv, int D, int block_size, int max_blocks, int64_t num_blocks, int max_query_len,
                         int num_splits, int window, float scale, int decode_layout, int dtype, cudaStream_t st);

// Decode-shaped paged GQA attention on tcgen05 with TMA-fed KV tiles (attention/decode_umma.cu): head dim 128,
// at most 16 packed query rows per KV head, cache blocks of a multiple of 64 tokens.  `tmap`: the cache as a 2-D
// [blocks * 2 * Hkv * block_size, 128] tensor, 64 x 64 boxes, 128-byte swizzle.  Returns 3 for shapes it does not serve.
int b200_decode_attention_umma(void* out, const void* q, const void* tmap, const int* block_tables,
                               const int* seq_lens, const int* qsl, const float* sinks, float* ws_o, float* ws_lse,
                               int* status, int64_t T, int B, int Hq, int Hkv, int D, int block_size, int max_blocks,
                               int64_t num_blocks, int max_query_len, int num_splits, int window, float scale,
                               int early_meta, const float* bias, int bias_len, const void* gate, int64_t gate_stride,
                               int keep_first, int sigmoid, int dtype, cudaStream_t st);

// Dense paged MLA decode on tcgen05 (attention/mla_decode_umma.cu): cache blocks of 64 tokens, at most 32 query
// tokens per request.  `tmap`: the cache as a 2-D [blocks * 64, 576] 16-bit tensor, 64 x 64 boxes, 128-byte swizzle.
// early_meta as for b200_decode_attention_umma.  Returns 3 for shapes it does not serve.
int b200_mla_decode_umma(void* out, const void* q, const void* tmap, const int* block_tables, const int* seq_lens,
                         const int* qsl, const float* sinks, float* ws_o, float* ws_lse, int* status, int64_t T, int B, int N,
                         int block_size, int max_blocks, int64_t num_blocks, int max_query_len, int num_splits, int window,
                         float scale, int early_meta, int dtype, unsigned long long* trace, cudaStream_t st);

int b200_mla_decode_max_clusters(int R, int S, int dtype);
int b200_prefill_attention_umma(void* out, float* lse, const void* tmQ, const void* tmKV, const int* block_tables,
                                const int* seq_lens, const int* qsl, const float* sinks, int* status, int B, int Hq, int Hkv,
                                int D, int block_size, int max_blocks, int64_t num_blocks, int max_query_len, int window,
                                float scale, const float* bias, int bias_len, const void* gate, int64_t gate_stride,
                                int keep_first, int sigmoid, int dtype, unsigned long long* trace, cudaStream_t st);
int b200_mla_prefill_umma(void* out, float* lse, const void* tmQ, const void* tmKV, const void* tmKpe, const int* kv_starts,
                          const int* kv_lens, const int* qsl, const float* sinks, const void* gate, int64_t gate_stride,
                          int* status, int B, int Hq, int max_query_len, int causal, int window, float scale, int dtype,
                          unsigned long long* trace, cudaStream_t st);
int b200_gather_mla_rows(void* out, const void* cache, const int32_t* slots, int64_t M, int64_t total_slots, int fp8,
                         int dtype, cudaStream_t st);
int b200_quant_int8_token(void* q, float* scale, const void* x, const float* static_scale, int64_t rows, int K,
                          int64_t x_stride, int dtype, cudaStream_t st);
int b200_indexer_logits_umma(float* logits, const void* tmQ, const float* w, const void* cache, const void* tmK,
                             const int* block_tables, const int* seq_lens, const int* qsl, int* status, int B,
                             int max_query_len, int max_blocks, int64_t num_blocks, int64_t ld, int64_t t_lo, int64_t t_hi,
                             cudaStream_t st);

int b200_merge_splits(void* out, const float* ws_o, const float* ws_lse, int64_t rows, int Hq, int D, int splits,
                      int64_t T, int dtype, cudaStream_t st);
// Absorbed MLA attention over the latent cache: dense paged (indices == null) or sparse by index list.
int b200_mla_attention(void* out, const void* q, const void* kv, const int* block_tables, const int* seq_lens,
                       const int* qsl, const int* req_of_token, const int* indices, float* ws_o, float* ws_lse,
                       int64_t T, int B, int N, int block_size, int max_blocks, int64_t total_slots, int topk,
                       int num_splits, float scale, int dtype, cudaStream_t st);

// Lightning indexer: fp8 scores over the paged key cache (per block: key rows, then scales), then per-row top-k (unordered, -1 padded)
int b200_indexer_logits(float* logits, const void* q_fp8, const float* w, const void* k_cache, const int* block_tables,
                        const int* seq_lens, const int* qsl, const int* req_of_token, int64_t T, int B, int block_size,
                        int max_blocks, int64_t total_slots, int64_t ld_logits, int64_t t0, cudaStream_t st);
int b200_topk_rows(int* out, const float* logits, const int* row_len, int64_t rows, int64_t ld, int k, int64_t max_len,
                   cudaStream_t st);

// ---- MoE / fp8 activation quantisation --------------------------------------------------------
int b200_moe_route(float* out_w, int* out_ids, const void* logits, const float* bias, int64_t T, int E, int k, int mode,
                   int renorm, int n_group, int topk_group, int group_top, float scale, int64_t stride, int dtype,
                   cudaStream_t st);
int b200_moe_permute(void* x_sorted, int* pos_of_pair, int* lod, int* counts, int* cursor, const void* x, const int* ids,
                     const int* emap, const float* factors, int64_t T, int k, int H, int E_local, int E_global,
                     int64_t x_stride, int64_t max_rows, int dtype, cudaStream_t st);  // factors [T][k] (or null): times the rows
int b200_moe_unpermute(void* out, const void* y_sorted, const int* pos_of_pair, const float* w, int64_t T, int k, int H,
                       int dtype, cudaStream_t st);
int b200_router_gemm_small(float* out, const void* x, int64_t x_stride, const void* w, const void* bias,
                           int64_t T_, int N, int K, int dtype, cudaStream_t st);
int b200_router_route_small(float* out_w, int* out_ids, const void* x, int64_t x_stride, const void* w,
                            const void* wbias, const float* bias, int64_t T_, int E, int K, int k, int mode,
                            int renorm, int n_group, int topk_group, int group_top, float scale, int dtype, cudaStream_t st);
int b200_moe_small_pairs();
int b200_moe_prepare_small(void* x_sorted, float* scale_t, int64_t s_stride, int* pos_of_pair, int* lod,
                           const void* x, const int* ids, const int* emap, const float* factors, int64_t T_, int k,
                           int H, int E_local, int E_global, int64_t x_stride, int quant, int dtype, cudaStream_t st);
int b200_act_mul_quant_fp8(void* q, float* scale_t, const void* h, int64_t rows, int I, int64_t s_stride, int act,
                           const int* rows_valid_ptr, int dtype, cudaStream_t st);
int b200_quant_fp8_group(void* q, float* scale_t, const void* x, int64_t rows, int K, int64_t x_stride, int64_t s_stride,
                         int ue8m0, const int* rows_valid_ptr, int dtype, cudaStream_t st);

// ---- communication over NVLink peer memory ----------------------------------------------------
int b200_allreduce_max_ctas();
int64_t b200_allreduce_flag_bytes();
int b200_oneshot_allreduce(void* const* bufs, const void* in, void* out, void* residual, const void* weight,
                           uint32_t* epochs, int* status, int64_t parity_bytes, int64_t flags_offset, int rank,
                           int nranks, int rows, int H, float eps, int gemma, int grid, uint32_t spin_limit, int dtype,
                           cudaStream_t st);

int b200_ll_allreduce(void* const* bufs, const void* in, void* out, void* residual, const void* weight,
                      uint32_t* epochs, int* status, int64_t slot_bytes, int rank, int nranks, int rows, int H,
                      float eps, int gemma, int grid, uint32_t spin_limit, int skip_push, int dtype, cudaStream_t st);

// Reduce-scatter consumer: sum R partial rows + residual, RMSNorm, push the row to every rank (see rs_norm_ag.cu)
typedef struct RsNormArgs {
  const void* stage; const void* rs_flags;
  void* xfull[8]; void* ag_flags[8];
  void* reset_a; void* reset_b; int reset_a_n, reset_b_n;
  void* residual; const void* weight; int* status;
  int rank, R, Tloc, H, rs_bn, n_tiles, ag_bn, rows_per_cta, max_tt, gemma, dtype;
  float eps; unsigned spin_limit;
} RsNormArgs;
int b200_rs_norm_ag(const RsNormArgs* a, cudaStream_t st);
int b200_sp_wait(const void* flags, int n_tt, unsigned expect, unsigned spin_limit, int* status, cudaStream_t st);

// ---- sampling ---------------------------------------------------------------------------------
int b200_topk_topp_sample(int64_t* out, const void* logits, int64_t rows, int V, int64_t stride,
                          const float* temperature, const int* top_k, const float* top_p, const float* noise,
                          int64_t noise_stride, uint64_t seed, uint64_t step, int dtype, cudaStream_t st);
int b200_repetition_penalty(void* logits, int64_t rows, int V, int64_t stride, const int64_t* tokens,
                            int64_t tok_stride, int max_tokens, const int* n_tokens, const float* penalty,
                            uint32_t* seen, int dtype, cudaStream_t st);
int b200_rejection_sample(int64_t* out, int64_t B, int S, const int64_t* draft_ids, const int* cu_draft,
                          const float* target_probs, const float* draft_probs, int V, const int64_t* bonus,
                          const uint8_t* is_greedy, const float* uniform, const float* recover_q, uint64_t seed,
                          uint64_t step, cudaStream_t st);

// ---- layer norm / post-norm residual stream / unit-norm split (elementwise/layernorm.cu) ----------
int b200_embed_layernorm(float* x, void* h, const int64_t* ids, const int64_t* positions, const void* table,
                         const int64_t* freq, const float* w, int64_t T, int H, int ld, int64_t rows, float eps,
                         int dtype, cudaStream_t st);
int b200_layernorm_residual(float* x, void* h, const void* y1, int64_t y1_stride, float s1, const void* y2,
                            int64_t y2_stride, float s2, const float* w, int64_t T, int H, int ld, float eps, int add,
                            int dtype, cudaStream_t st);
int b200_gated_group_rmsnorm(void* out, int64_t out_stride, const float* o, int64_t o_stride, const void* gate,
                             int64_t gate_stride, const float* w, int64_t T, int groups, int D, float eps, int dtype,
                             cudaStream_t st);
int b200_qk_unit_norm_cache(void* q_out, const void* q, const void* k, const void* v, int64_t stride, void* kv_cache,
                            const int64_t* slots, int64_t T, int Hq, int Hkv, int D, int Dv, int Dc, int block_size,
                            int64_t num_blocks, float eps, int dtype, cudaStream_t st);

// ---- norms before and after every sublayer, polynomial activation, value-normed attention split (elementwise/sandwich.cu) ----
int b200_embed_rmsnorm(float* x, void* h, const int64_t* ids, const void* table, const float* w, int64_t T, int H, int ld,
                       int64_t rows, float eps, int dtype, cudaStream_t st);
// pos [T][k] (or null): rows of y that add up to a token's
int b200_sandwich_rmsnorm(float* x, void* h, const void* y, int64_t y_stride, const int* pos, int k, const float* w_post,
                          const float* w_pre, int64_t T, int H, int ld, float eps, int dtype, cudaStream_t st);
int b200_poly_norm(void* out, int64_t ldo, const void* z, int64_t ldz, const float* coeff, int64_t T, int F, int ld, float eps,
                   int dtype, cudaStream_t st);
typedef struct AttnPrepArgs {
  const void *q, *k, *v;     // [T][heads][head size] column slices of one projection, rows `stride` apart
  void *q_out, *cache;       // [T][Hq][Dc]; [block][2][Hkv][slot][Dc]
  const int64_t *slots, *positions;
  const float *q_norm, *k_norm;  // [D] weights of an RMS norm per head (null: none)
  const float* table;        // cos / sin pairs [T][pairs][2] of the first 2 pairs columns of q and k (null: no rotation)
  void* v_out;               // [T][Hkv * Dv] the values (before mixing) for later layers, or null
  const void* v_in;          // such values of an earlier layer, mixed in with `share`, or null
  int64_t stride, num_blocks, temp_every;  // temp_every 0: no temperature
  int Hq, Hkv, D, Dv, Dc, block_size, pairs, v_norm;  // v_norm: values are divided by their root mean square
  float share, temp_coef, eps;
} AttnPrepArgs;
int b200_attn_prep_cache(const AttnPrepArgs* args, int64_t T, int dtype, cudaStream_t st);

// ---- fp32 stream normalised on the sublayers' outputs, short convolution of their inputs (elementwise/postnorm.cu) ------
typedef struct PostNormArgs {
  float* x;                  // [T][ld] the stream, updated in place
  const void* table;         // start of a stream: x = table[ids[t]] * scale; null: x += LayerNorm(y) * weight
  const int64_t* ids;
  int64_t table_rows;
  // y = its row (or null: 0) + sum over k choices of weights[t][q] * (rows[places[t][q]], or pass[t] where the place is < 0)
  const void *y, *rows, *pass;
  const int* places;
  const float* weights;
  int64_t y_stride, rows_stride, pass_stride;
  const float* weight;       // [width]
  void* h;                   // [T][ld] x + conv(x) (taps > 0), or LayerNorm(x) * final_weight (if any), in the model's type
  const float *conv, *final_weight;  // [taps][ld]; [width]
  float* state;              // [slots][taps - 1][ld] the stream's last rows of every request
  const int *qsl, *slots, *has_init;
  int64_t T, num_slots;
  int k, taps, width, ld, num_reqs, max_query_len;
  float scale, eps;
} PostNormArgs;
int b200_postnorm(const PostNormArgs* args, int dtype, cudaStream_t st);    // taps > 0: requests of a few tokens
int b200_input_conv(const PostNormArgs* args, int dtype, cudaStream_t st);  // h = x + conv(x)

// ---- fp32 GEMM on the CUDA cores (gemm/gemm_f32.cu): out[T, N] = x[T, K] . w[N, K]^T (+ bias) -----------------
int b200_gemm_f32(float* out, int64_t ldo, const float* x, int64_t ldx, const float* w, int64_t ldw, const float* bias,
                  int64_t T, int N, int K, int relu2, cudaStream_t st);  // relu2: outputs pass the square of relu
int b200_gemm_f32_grouped(float* out, int64_t ldo, const float* x, int64_t ldx, const float* w, const int* lod, int64_t M,
                          int E, int N, int K, int relu2, cudaStream_t st);

// ---- latent attention of any size (attention/latent.cu) --------------------------------------------------
typedef struct LatentPrepArgs {
  const void *q_down, *kv_down;  // down-projections [T][q_rank], [T][kv_rank | rot_dim], rows `stride` apart
  const float *q_norm, *kv_norm, *table;  // RMS norm weights; cos / sin pairs [T][pairs][2]
  const int64_t* slots;
  void *q_out, *cache;           // [T][q_out_stride] (padded with zeros); latent cache, rows of `row` columns
  int64_t stride, total_slots;
  int q_out_stride, q_rank, kv_rank, rot_dim, rot_off, row, pairs, vec;
  float eps;
} LatentPrepArgs;
int b200_latent_prep(const LatentPrepArgs* args, int64_t T, int dtype, cudaStream_t st);
int b200_rotary_table(float* out, const int64_t* positions, const int64_t* turns, int64_t T, int pairs, cudaStream_t st);
int b200_rotate_heads(void* q, const float* table, int64_t T, int H, int D, int off, int pairs, int dtype, cudaStream_t st);
int b200_absorb_query(void* out, const void* q, const void* w, int64_t w_head, const float* table, int64_t T, int H, int D,
                      int R, int C, int rot_off, int row, int pairs, int dtype, cudaStream_t st);
int b200_expand_value(void* out, int64_t out_stride, const void* o, const void* w, int64_t w_head, const void* gate,
                      int64_t gate_stride, int64_t T, int H, int Dv, int C, int dtype, cudaStream_t st);
int b200_gather_window(void* out, const void* cache, const int* block_tables, const int* seq_lens, const int* starts,
                       const int* lens, int B, int max_len, int64_t max_blocks, int block_size, int64_t num_blocks,
                       int64_t row_bytes, int64_t total, cudaStream_t st);

// ---- fp32 stream with one norm per layer, gated summands and token shift (elementwise/gated_stream.cu) ------------
typedef struct StreamNormArgs {
  // source of a row: tables (table != null) or stream + gated summands (y1 may be null: the stream as it is)
  const void *table, *bigram_table;
  const int64_t *ids, *bigram_rows;
  int64_t table_rows, bigram_table_rows;
  const float* x_in;
  const void *y1, *g1, *y2, *g2;
  int64_t y1_stride, g1_stride, y2_stride, g2_stride;
  // results: stream (may be null), norm, norm mixed with the previous token's (may be null)
  float* x_out;
  void *h, *shifted;
  const float *weight, *mix;
  float* state;              // [slots][ld] norm of the last token of every request
  const int *req_of_token, *qsl, *slots, *has_init;
  int64_t T, num_slots;
  int width, ld, rows_per_cta;
  float scale, eps;
} StreamNormArgs;
int b200_stream_layernorm(const StreamNormArgs* args, int dtype, cudaStream_t st);
int b200_bigram_rows(int64_t* rows, const int64_t* ids, int64_t* state, const int* qsl, const int* slots, const int* has_init,
                     int B, int64_t num_slots, int64_t mul_prev, int64_t mul_cur, int64_t buckets, cudaStream_t st);

// ---- paged attention for any head size and for fp32 (attention/paged_generic.cu) -----------------
int b200_paged_attention_generic(void* out, const void* q, const void* kv_cache, const int* block_tables,
                                 const int* seq_lens, const int* qsl, const float* sinks, int64_t T, int B, int Hq,
                                 int Hkv, int D, int block_size, int max_blocks, int64_t num_blocks, int latent_dv,
                                 int window, float scale, const float* bias, int bias_len, const void* gate,
                                 int64_t gate_stride, int keep_first, int sigmoid, int dtype, cudaStream_t st);

// ---- gated delta net / conv / MTP glue --------------------------------------------------------
int b200_causal_conv1d_fwd(void* out, int64_t out_stride, const void* x, int64_t x_stride, const void* w,
                           const void* bias, const int* cu, int R, void* states, const int* slots,
                           const uint8_t* has_init, int C, int W, int act, int64_t T_, int dtype, cudaStream_t st);
int b200_causal_conv1d_update(void* out, int64_t out_stride, const void* x, int64_t x_stride, void* states,
                              const void* w, const void* bias, const int* slots, const int* has_init, int64_t B, int C,
                              int W, int act, int dtype, cudaStream_t st);
int b200_gdn_gating(float* g, float* beta, const void* a, int64_t a_stride, const void* b, int64_t b_stride,
                    const float* A_log, const float* dt_bias, int H, int64_t T_, int dtype, cudaStream_t st);
int b200_gdn_recurrent(void* out, int64_t o_stride, const void* q, const void* k, int64_t qk_stride, const void* v,
                       int64_t v_stride, const float* g, const float* beta, float* states, const int* cu,
                       const int* slots, const uint8_t* has_init, int R, int Hk, int Hv, int Dk, int Dv, float scale,
                       int l2norm, int dtype, cudaStream_t st);
// Linear recurrences with a matrix state (linear_attn/recurrence.cu); kind 0 = delta rule with a decay per key channel,
// 1 = fixed decay per head.  q, k: [T][Hk][Dk], v: [T][H][Dv] column slices of one row-strided tensor.
typedef struct RecurrenceArgs {
  float* out;                // [T][H][Dv], rows out_stride apart
  const void *q, *k, *v;     // raw (kind 1) or convolved (kind 0) projections, rows qkv_stride apart
  const void *a, *b;         // kind 0: raw decay [T][H][Dk] and step-size [T][H] projections; kind 2: a = raw forget gates
  const float *A_log, *dt_bias;  // kind 0: [H], [H][Dk]; kind 2: dt_bias = bias of the forget gates
  const float* decay;        // kind 1: [H]
  const float* lower;        // kind 2: [H][Dk] lower bound of the forget gates
  float* states;             // [slots][H][Dv][Dks]
  const int *cu, *slots, *has_init;
  int64_t out_stride, qkv_stride, a_stride, b_stride;
  int R, Hk, H, Dk, Dks, Dv, kind;
  int decode;                // the requests have one token each (any number is correct, one is fast)
  float scale, unit_eps;
} RecurrenceArgs;
int b200_linear_recurrence(const RecurrenceArgs* a, int dtype, cudaStream_t st);
int b200_chunk_decay(const RecurrenceArgs* a, int dtype, cudaStream_t st);  // kind 1, prompt portions (linear_attn/chunk_decay.cu)
int b200_chunk_gated_write(const RecurrenceArgs* a, int dtype, cudaStream_t st);  // kind 2, prompt portions (linear_attn/chunk_gated.cu)
// Element-wise gated recurrence with gates of the current token (linear_attn/blend.cu)
typedef struct BlendArgs {
  void* out;                 // [T][width] state * silu(g)
  const void *z, *x, *g;     // raw projections, rows `stride` apart
  const float *z_bias, *x_bias;
  float* state;              // [slots][width]
  const int *qsl, *slots, *has_init;
  int64_t stride, out_stride, num_slots;
  int R, width;
  int steps;                 // the requests have one token each (any number is correct, few are fast)
} BlendArgs;
int b200_gated_blend(const BlendArgs* args, int dtype, cudaStream_t st);
int b200_sigmoid_gate_mul(void* out, const void* o, const void* gate, int64_t gate_stride, int D, int64_t T_,
                          int dtype, cudaStream_t st);
int b200_mtp_concat_norm(void* out, const void* embed, const void* hidden, const void* we, const void* wh,
                         const int64_t* pos, int64_t T_, int H, float eps, int dtype, cudaStream_t st);

// ---- LoRA ---------------------------------------------------------------------------------------
int b200_lora_shrink(float* out, const void* x, int64_t x_stride, const void* A, const int* ids, int64_t T_, int r,
                     int K, float scale, int dtype, cudaStream_t st);
int b200_lora_expand(void* out, int64_t out_stride, int offset, const float* h, const void* B, const int* ids,
                     int64_t T_, int N, int r, int add, int dtype, cudaStream_t st);

// ---- expert-parallel dispatch / combine over peer memory (see comm/ep_a2a.cu) --------------------
typedef struct EpArgs {
  void* peer[8];             // every rank's symmetric buffer (index = rank)
  int64_t off_x, off_scale, off_ids, off_w, off_recv_flag, off_comb, off_comb_flag;
  const void* x;             // local payload rows [T][x_row_bytes] (bf16, or fp8 already quantised)
  const float* x_scale_t;    // fp8 payload: transposed scales [H/128][scale_stride], else null
  int64_t x_row_bytes, scale_stride;
  const int* topk_ids;       // [T][k] global expert ids
  const float* topk_w;       // [T][k]
  int* send_count;           // [R] zero between calls
  int* sent_slot;            // [T][R]
  int* recv_count;           // [R]
  int* prev_count;           // [R]
  int* ticket;               // [3] zero between calls
  uint32_t* epoch;           // [1]
  int* status;
  int64_t T;
  int rank, R, cap, H, k, E, row_bytes;
  unsigned spin_limit;
} EpArgs;
int b200_ep_dispatch(const EpArgs* a, cudaStream_t st);
int b200_ep_permute_scales(float* scale_t, int64_t s_stride, const float* recv_scale, const int* pos_of_pair,
                           int64_t pairs, int k, int ngroups, cudaStream_t st);
int b200_ep_combine(const EpArgs* a, const void* y_sorted, const int* pos_of_pair, void* out, const void* addend,
                    int dtype, cudaStream_t st);

#ifdef __cplusplus
}
#endif
