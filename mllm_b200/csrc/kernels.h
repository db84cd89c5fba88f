// Host-callable launchers of the sm_100a kernels (plain C++ signatures: raw
// device pointers + a stream, no framework types). The PyTorch binding in
// bindings.cpp validates tensors and forwards here; other hosts can link the
// same symbols.
#pragma once

#include <cuda_runtime.h>
#include <stdint.h>

namespace mb200 {

enum DType : int { kBF16 = 0, kF16 = 1, kF32 = 2 };

// Number of kernel launches issued through these launchers since load.
uint64_t launch_count();
void note_launch(int n = 1);

// ----- element-wise / normalisation --------------------------------------------------
void launch_rmsnorm(const void* x, const void* w, void* out, int rows, int hidden, int64_t x_stride,
                    int64_t out_stride, float eps, DType dt, cudaStream_t s);
void launch_fused_add_rmsnorm(void* x, void* residual, const void* w, int rows, int hidden, float eps, DType dt,
                              cudaStream_t s);
void launch_layernorm(const void* x, const void* w, const void* b, void* out, int rows, int hidden, float eps,
                      DType dt, cudaStream_t s);
// act: 0 = silu(gate)*up, 1 = gelu_tanh(gate)*up, 2 = clamped gate (see clamped_gate in common.cuh); x is [rows, 2*inter] = [gate | up]
void launch_act_and_mul(const void* x, void* out, int rows, int inter, int act, float limit, DType dt, cudaStream_t s);
// fp32 residual stream with a Dynamic Tanh norm: x += mult * y (y may be null), h = tanh(alpha x) * w + b
void launch_residual_dyt(float* x, const void* y, float mult, const float* alpha, const float* w, const float* b, void* h,
                         int rows, int width, DType dt, cudaStream_t s);
// embedding rows times `scale` in fp32; h (may be null): the same rounded to dt
void launch_embedding_f32(const int64_t* ids, const void* table, float scale, float* out, void* h, int tokens, int width, int vocab,
                          DType dt, int* status, cudaStream_t s);

// ----- row-wise kernels of decoders with an fp32 residual stream (row_ops.cu) -----------------
// x_out, h = rmsnorm(alpha * x + ls * (y + sum of the token's expert rows)) * w, x and x_out fp32 (x_out may be x, or null)
struct PostNormArgs {
  const float* x;           // [rows, width]
  float* x_out;             // [rows, width] or null
  const void* y;            // [rows, width] or null
  const float* ls;          // [width] or null (1)
  const float* w;           // [width]
  void* h;                  // [rows, width]
  // weighted sum of expert outputs (expert_rows null: none); choice j of token t is row sorted_pos[t * top + j] of
  // expert_rows, or, where that is negative and its id is >= identity_from > 0, the row t of token_in
  const void* expert_rows;
  const int* sorted_pos;
  const float* topk_w;
  const int* ids;
  const void* token_in;
  const float* y_logit;     // one per row, y_logit_ld apart, or null: y times its logistic function
  int64_t y_logit_ld;
  int rows, width, top, identity_from;
  int inner;                // 0: x <- norm(alpha * x + ls * y), 1: x <- alpha * x + ls * norm(y)
  float alpha, eps;
  DType dt;                 // of y, h, expert_rows, token_in
};
int launch_post_norm(const PostNormArgs& args, cudaStream_t s);
// out = rmsnorm over the whole row of x, times w and sigmoid(gate)
int launch_rmsnorm_sigmoid_gate(const void* x, const void* gate, int64_t gate_ld, const float* w, void* out, int64_t out_ld, int rows,
                                int width, float eps, DType dt, cudaStream_t s);
// rows [q | k | v] of tokens: RMS norm over all query heads and over all key heads, rotation of neighbouring features,
// q to q_out [tokens, heads, q_width] (zeros behind dim), k and v to the cache slots loc
struct RowNormRopeArgs {
  const void* row;          // row t at t * row_ld: heads * dim, kv_heads * dim and kv_heads * vdim features
  const float* q_w;         // [heads * dim]
  const float* k_w;         // [kv_heads * dim]
  const double* inv_freq;   // [rot_dims / 2]
  const int64_t* positions; // [tokens]
  const int64_t* loc;       // [tokens]
  void* q_out;
  void* k_cache;            // head h of slot s at s * tok + h * head (elements)
  void* v_cache;
  int* status;
  int64_t row_ld, k_tok_stride, k_head_stride, v_tok_stride, v_head_stride, num_slots;
  int tokens, heads, kv_heads, dim, vdim, q_width, rot_dims;
  float eps;
  DType dt;
};
int launch_rownorm_rope_kv(const RowNormRopeArgs& args, cudaStream_t s);
// rows [q | k | ..] of tokens: rotation of part of every query and key head, each head divided by its root mean square (norm),
// q to q_out [tokens, heads, q_width] (zeros behind dim), k and the unchanged values to the cache slots loc
struct HeadNormRopeArgs {
  const void* row;          // row t at t * row_ld: heads * dim and kv_heads * dim features, kv_heads * vdim values at v_at
  const double* inv_freq;   // [rot_dims / 2]
  const int64_t* positions; // [tokens]
  const int64_t* loc;       // [tokens]
  void* q_out;
  void* k_cache;            // head h of slot s at s * tok + h * head (elements)
  void* v_cache;
  int* status;
  int64_t row_ld, k_tok_stride, k_head_stride, v_tok_stride, v_head_stride, num_slots;
  int tokens, heads, kv_heads, dim, vdim, v_at, q_width, rot_dims;
  int halves;               // pairs are (i, i + rot_dims / 2); 0: neighbours (2i, 2i + 1)
  int norm;                 // 0: heads keep their length
  float eps, magnitude;     // magnitude: factor of the sines and cosines
  DType dt;
};
int launch_headnorm_rope_kv(const HeadNormRopeArgs& args, cudaStream_t s);
// out = rmsnorm of x * silu(gate), the mean over each of `groups` equal parts of the row, times w
int launch_gated_rmsnorm(const void* x, const void* gate, int64_t gate_ld, const float* w, void* out, int64_t out_ld, int rows, int width,
                         int groups, float eps, DType dt, cudaStream_t s);

// ----- the step between layers whose sublayers run side by side, with an average over depth (depth.cu) -----
// causal convolution of single tokens with their input added: row t is the next token of the request with state row slots[t]
struct ConvStepArgs {
  const void* w;            // [width, taps], column taps - 1 meets the token itself; null: no convolution
  void* state;              // [rows, width, taps - 1] the last inputs, oldest first; moved on
  const int* slots;
  int taps;
};
// normed rows of a stream: h = x / sqrt(mean(x^2) + eps) * g with a single number g; h1 may pass a convolution
struct DepthInputs {
  const float* g1;
  const float* g2;
  void* h1;                 // [rows, width]
  void* h2;                 // [rows, width] or null
  ConvStepArgs conv;
};
struct DepthStepArgs {
  const float* x;           // [rows, width] what the layer's sublayers read
  float* x_out;             // [rows, width] what goes on, or null; may be x
  float* results;           // results 0 .. n - 1, result_stride elements apart; result n is written where keep is set
  int64_t result_stride;
  int n, keep;
  const float* dwa;         // [n + 1] weights of the average, or null: the layer's result goes on
  const void* a;            // [rows, width] mixer output
  const void* b;            // [rows, width] a second one, or null; then mix = mix_scale * (norm(a) * a_w + norm(b) * b_w)
  const float* a_w;         // [width]
  const float* b_w;         // [width]
  float mix_scale;
  const void* f;            // [rows, width] feed-forward output or null
  const void* expert_rows;  // choice j of token t is row sorted_pos[t * top + j] (negative: none), or null
  const int* sorted_pos;
  const float* topk_w;      // [rows, top] or null (1)
  int top;
  DepthInputs in;
  int rows, width;
  float eps;
  DType dt;                 // of a, b, f, expert_rows, h1, h2, the convolution
};
int launch_depth_step(const DepthStepArgs& args, cudaStream_t s);
// x = embedding row / sqrt(mean of its squares + eps) * g, and the inputs of the first layer
struct EmbedNormArgs {
  const int64_t* ids;
  const void* table;        // [vocab, width]
  const float* g;
  float* x;                 // [rows, width]
  int* status;
  DepthInputs in;
  int rows, width, vocab;
  float eps;
  DType dt;
};
int launch_embed_norm(const EmbedNormArgs& args, cudaStream_t s);

void launch_soft_cap(const void* x, int64_t x_ld, float* out, int rows, int width, float cap, DType dt, cudaStream_t s);
void launch_relu_squared(void* x, int64_t n, DType dt, cudaStream_t s);
void launch_gelu_tanh(const void* x, void* out, int64_t n, DType dt, cudaStream_t s);
void launch_embedding(const int64_t* ids, const void* table, void* out, int tokens, int hidden, int vocab,
                      DType dt, int* status, cudaStream_t s);

// Per-head RMSNorm of q and k (weights may be null), NeoX rotary embedding and the
// write of K (normed, rotated) and V into the slot-indexed cache; q and k are updated
// in place inside the fused qkv activation. head_dim is 128.  kv_fmt 1 / 2: the caches hold unscaled e4m3 / e5m2
// bytes and K and V are rounded to that format on the way in.
// positions: [pos_rows, tokens] int64 with pos_rows 1 (plain RoPE) or 3 (M-RoPE: t,h,w);
// axis_map[head_dim/2] selects the position row per frequency (null -> row 0).
// The caches are addressed by strides (in elements): the row of head h of slot s starts at
// s * kv_tok_stride + h * kv_head_stride, which covers both the slot-major [slots, heads, D] and the head-major
// [heads, slots, D] layout.
void launch_qk_norm_rope_kv_write(void* qkv, const void* q_w, const void* k_w, const int64_t* positions,
                                  int pos_rows, const int8_t* axis_map, const float* inv_freq,
                                  const int64_t* cache_loc, void* k_cache, void* v_cache, int64_t kv_tok_stride,
                                  int64_t kv_head_stride, int tokens,
                                  int num_q_heads, int num_kv_heads, int head_dim, int64_t qkv_stride,
                                  int64_t num_slots, float eps, DType dt, int kv_fmt, int* status, cudaStream_t s);
void launch_kv_write(const void* k, const void* v, const int64_t* loc, void* k_cache, void* v_cache,
                     int64_t kv_tok_stride, int64_t kv_head_stride, int head_elems, int tokens,
                     int row_elems, int64_t k_stride, int64_t v_stride, int64_t num_slots, DType dt, int kv_fmt, int* status,
                     cudaStream_t s);

// Bookkeeping of one decode step of a static batch (see decode_prepare_kernel): one launch instead of a dozen
// small framework kernels.
void launch_decode_prepare(const int64_t* last_ids, const int32_t* req_rows, const int64_t* own, int64_t own_stride,
                           int used, int32_t* seq_lens, int32_t* req_to_token, int64_t rtt_stride,
                           int64_t* g_input_ids, int32_t* g_req_rows, int32_t* g_seq_lens, int64_t* g_out_loc,
                           int64_t* g_positions, int batch, cudaStream_t s);

// ----- quantisation -------------------------------------------------------------------
void launch_per_token_quant_int8(const void* x, int8_t* q, float* scale, int rows, int k, DType dt,
                                 cudaStream_t s);

// ----- sampling -------------------------------------------------------------------------
void launch_argmax(const void* logits, int64_t* out, int rows, int vocab, int64_t stride, DType dt,
                   cudaStream_t s);
// two-stage variant for few rows x wide vocabulary; part_val / part_idx hold rows * 32 entries
int launch_argmax_split(const void* logits, int64_t* out, float* part_val, int* part_idx, int rows, int vocab,
                        int64_t stride, DType dt, cudaStream_t s);

// one token per row: temperature (<= 1e-6: greedy), top-k (<= 0: off), top-p, min-p (may be null),
// inverse-CDF draw with uniform[row] in [0, 1)
void launch_sample(const void* logits, int64_t stride, int rows, int vocab, const float* temperature, const int* top_k,
                   const float* top_p, const float* min_p, const float* uniform, int64_t* out, DType dt, cudaStream_t s);
void launch_apply_penalties(float* logits, const int* counts, const uint8_t* prompt_mask, const float* freq,
                            const float* presence, const float* repetition, int rows, int vocab, cudaStream_t s);

// ----- GEMM (tcgen05 + TMEM + TMA) ---------------------------------------------------
struct GemmArgs {
  const void* a;         // [m, k] row-major activations
  const void* b;         // [n, k] row-major weights (out = a * b^T)
  void* out;             // [m, n_out] row-major
  const void* bias;      // [n] or null
  const void* residual;  // [m, n] or null (added before rounding)
  float act_limit;       // swiglu 4
  const float* a_scale;  // int8 only: per-row scale [m]
  const float* b_scale;  // int8 only: per-column scale [n]
  int m, n, k;
  int64_t lda, ldb, ldc, ld_res;
  int swiglu;            // 1: b rows alternate 128 gate / 128 up rows; out is [m, n/2] = silu(gate) * up; 2: gelu_tanh(gate) * up;
                         // 4: clamped_gate(gate + bias, up + bias, act_limit), the only gated form with a bias (rows as b's);
                         // 3: out is [m, n] = max(a b^T, 0)^2 (launch_gemm returns 1 for 9 to 256 rows: not fused there)
  DType dt;              // element type of a, b (kBF16 / kF16) ; out has the same type
  int is_int8;           // 1: a, b are int8, out type given by dt
  float* workspace;      // split-K partial sums (small-m path), may be null when not needed
  size_t workspace_bytes;
  int* counters;         // split-K tile tickets, zero-initialised, self-resetting
  int num_counters;
  int* status;           // device int, set non-zero when a bounded wait ran out
  int num_sms;
  int b_static;          // 1: b (the weights) is not written by kernels that precede this launch in its stream
  // ---- fused add + RMSNorm prologue, batches of up to 8 rows only (norm_weight null = off) ----
  // the product is taken of rmsnorm(a + norm_residual) * norm_weight; the 16-bit sum a + norm_residual (the new
  // residual stream) is written to norm_residual_out, which must not alias norm_residual (other CTAs still read it)
  const void* norm_weight;        // [k]
  const void* norm_residual;      // [m, k] or null
  void* norm_residual_out;        // [m, k] or null
  int64_t norm_residual_ld, norm_residual_out_ld;   // elements
  float norm_eps;
  // ---- tensor-parallel fusion, large-m tiling only (all zero = off) ----
  // all-gather -> GEMM: 128-row tile t of `a` is read only once gate_flags[t] >= gate_epoch
  const uint32_t* gate_flags;
  uint32_t gate_epoch;
  // GEMM -> reduce-scatter: m must be a multiple of 128 * rs_tp; 128-row tile t goes to rank
  // t / (m / 128 / rs_tp): stored at rs_out[owner] + local_row * rs_ld (this rank's slot of the owner's
  // inbox), and rs_flags[owner][local_tile * 8 + rs_rank] is set to rs_epoch when the row tile is complete.
  // rs_count: local int[m / 128], zero-initialised, self-resetting.  `out` is ignored.
  int rs_tp, rs_rank;
  uint32_t rs_epoch;
  int64_t rs_ld;
  uint64_t rs_out[8];
  uint64_t rs_flags[8];
  int* rs_count;
};
// Returns 0 on success, a negative code when the shape is unsupported (caller falls back / raises).
int launch_gemm(const GemmArgs& args, cudaStream_t s);
size_t gemm_workspace_bytes(int m, int n, int k, int num_sms);
// m <= 8, 16-bit operands: the weight matrix streamed through registers and warp-level MMAs (no tensor memory, no
// shared-memory ring, no split of k between CTAs).  Returns 0 when launched, 1 when the shape is not for it.
int launch_gemm_smallm(const GemmArgs& args, cudaStream_t s);

// ----- W4A16 GEMM (4-bit weights expanded in shared memory, tcgen05) ----------------------------
struct W4A16Args {
  const void* x;        // [m, k] activations (bf16 / fp16), row stride ldx
  const void* qweight;  // int32 [n, k/8]; nibble i of word j = element 8j + i, or (interleaved = 1) element
                        // 8j + 2p + h in nibble p + 4h
  const void* scales;   // [n, k/group] in the activation type
  const uint8_t* zeros; // [n, k/group] or null (zero point 8)
  const void* bias;     // [n] or null
  void* out;            // [m, n] row stride ldc
  float* workspace;     // split-K partials (may be null: no split)
  size_t workspace_bytes;
  int* status;
  int m, n, k, group;
  int64_t ldx, ldc;
  DType dt;
  int num_sms;
  int interleaved;
};
int launch_w4a16_gemm(const W4A16Args& args, cudaStream_t s);
// m <= 8, k <= 4096: packed weights streamed and expanded in registers (gemm_smallm_w4.cu).  0 launched, 1 not for it.
int launch_w4a16_smallm(const W4A16Args& args, cudaStream_t s);

// 128-byte-swizzled 2-D tensor map over a row-major [rows, k] matrix (box = 128 bytes of k x box_rows);
// map points at a CUtensorMap.  type: 0 bf16, 1 fp16, 2 uint8.
bool make_tma_operand_map(void* map, const void* base, int64_t rows, int64_t k, int64_t ld, int elem_bytes, int type,
                          int box_rows);

// ----- expert-parallel token exchange (ep_a2a.cu) -------------------------------------------
// Addresses of every rank's copy of the shared buffers (index = rank), this rank's id and the call's epoch.
struct EpA2AArgs {
  int ep, rank, experts, hidden, cap_rows;
  uint32_t epoch;
  uint64_t cnt_all[8];     // int32 [ep][experts]
  uint64_t cnt_flags[8];   // uint32 [ep]
  uint64_t recv_x[8];      // 16-bit [cap_rows][hidden]
  uint64_t recv_meta[8];   // int32 [cap_rows][2]
  uint64_t disp_flags[8];  // uint32 [ep]
  uint64_t ret_y[8];       // 16-bit [pairs capacity][hidden]
  uint64_t ret_flags[8];   // uint32 [ep]
};
int launch_ep_plan(const EpA2AArgs& a, const int* topk_ids, int pairs, int bn, int* pair_dst_rank, int* pair_dst_row,
                   int* expert_offsets, int* work, int* n_work, int max_work, int* recv_rows, int* status,
                   cudaStream_t s);
int launch_ep_dispatch(const EpA2AArgs& a, const void* x, int64_t x_stride, int pairs, int top_k, const int* pair_dst_rank,
                       const int* pair_dst_row, int* done_count, cudaStream_t s);
int launch_ep_return(const EpA2AArgs& a, const void* ys, const int* recv_rows, int* done_count, cudaStream_t s);

// ----- mixture of experts ----------------------------------------------------------------
// logits[t, e] = x[t] . w[e] in fp32 (products of 16-bit values are exact in it)
int launch_moe_router_logits(const void* x, int64_t x_ld, const void* w, float* logits, int tokens, int experts, int hidden,
                             int num_sms, DType dt, cudaStream_t s);
// router: fp32 scores of `experts` (<= 256) logits -> top_k (<= 32, sorted, lowest index wins ties).  The choice goes by
// the scores plus `correction`, the weights are the scores
struct RouteArgs {
  const void* logits;       // [tokens, >= experts], rows `stride` apart
  const float* correction;  // [experts] or null
  float* w;                 // [tokens, top_k]
  int* ids;                 // [tokens, top_k]
  int64_t stride;
  int tokens, experts, top_k;
  int sigmoid;              // scores: 0 softmax over the experts, 1 logistic function of each logit
  int renorm;               // weights divided by their sum + renorm_eps
  int groups, keep;         // keep < groups: only experts of the `keep` groups with the largest sums of two choice scores
  float renorm_eps, scale;  // scale: factor of the weights
  DType dt;                 // of the logits
};
int launch_moe_router_topk(const RouteArgs& args, cudaStream_t s);
// counting sort of the (token, choice) pairs by local expert.  sorted_pos[pair] = row in the sorted
// matrix or -1 (expert on another rank); src_token[row] = token; expert_offsets[experts + 1];
// work[i] = (expert, chunk of bn rows), *n_work items.  src_w (or null): src_w[row] = topk_w of the row's pair.
void launch_moe_align(const int* topk_ids, int pairs, int top_k, int expert_offset, int experts, int bn, int* sorted_pos,
                      int* src_token, int* expert_offsets, int* work, int* n_work, int max_work, const float* topk_w, float* src_w,
                      cudaStream_t s);
// rows of the pairs' tokens in expert order, each times src_w of its row
void launch_moe_gather_scaled(const void* x, int64_t x_stride, const int* src_token, const float* src_w, const int* expert_offsets, int experts,
                              void* xs, int pairs, int hidden, DType dt, cudaStream_t s);
void launch_moe_gather(const void* x, int64_t x_stride, const int* src_token, const int* expert_offsets, int experts,
                       void* xs, int pairs, int hidden, int elem_bytes, cudaStream_t s);
void launch_moe_combine(const void* y, const int* sorted_pos, const float* topk_w, void* out, int tokens, int hidden,
                        int top_k, DType dt, cudaStream_t s);
struct MoeGemmArgs {
  const void* x;    // [rows_cap, k] expert-sorted activations
  const void* w;    // [experts, n, k]
  void* out;        // [rows_cap, n_out]
  const int* expert_offsets;
  const int* work;
  const int* n_work;
  int* status;
  int64_t ldx, ldc;
  int rows_cap, experts, n, k, bn, max_work, swiglu, num_sms;
  int gelu;         // the exact GELU of the plain product
  DType dt;
};
int launch_moe_grouped_gemm(const MoeGemmArgs& args, cudaStream_t s);
// the plain product (no SwiGLU) for fp32 and for sizes that the tensor-core kernel does not take
int launch_moe_grouped_gemm_any(const MoeGemmArgs& args, cudaStream_t s);

// ----- attention over the slot-indexed KV pool (tcgen05, head_dim 128) -----------------
struct AttnArgs {
  const void* q;            // [T, Hq, 128], token stride q_stride elements
  const void* k_cache;      // row of head h of slot s at s * kv_tok_stride + h * kv_head_stride (elements)
  const void* v_cache;
  int64_t kv_tok_stride;    // slot-major [slots, Hkv, 128]: Hkv * 128 and 128; head-major [Hkv, slots, 128]:
  int64_t kv_head_stride;   // 128 and slots * 128 (consecutive slots of a head are then contiguous)
  void* out;                // [T, Hq, D], rows of a token out_stride apart (0: contiguous)
  float* part_o;            // decode with num_splits > 1: [B, Hq, splits, 128]
  float* part_lse;          // decode with num_splits > 1: [B, Hq, splits]
  const int* req_to_token;  // [reqs, rtt_stride]
  const int* req_pool_indices;  // [B]
  const int* seq_lens;          // [B]
  const int* prefix_lens;       // [B], prefill only
  const int* q_start;           // [B], prefill only: first query row of each request
  int* status;
  int64_t q_stride, out_stride, rtt_stride, num_slots;
  int batch, hq, hkv, head_dim;
  int max_q_len;            // prefill: longest run of new tokens in the batch
  int num_splits;           // decode
  int is_decode;
  int non_causal;           // prefill only: bidirectional attention inside each sequence
  float scale;
  int window;               // > 0: a query at position i sees keys i - window + 1 .. i only (causal attention)
  int chunk;                // > 0 (without a window): a query at position i sees keys i / chunk * chunk .. i only
  float logit_cap;          // > 0: scores pass through cap * tanh(score / cap) before the softmax
  DType dt;
  const float* sink;        // [Hq] or null: per head, exp(sink) joins the softmax denominator (no key, no value, unscaled)
  int kv_fmt;               // 0: the caches hold dt; 1 / 2: unscaled e4m3 / e5m2 bytes (strides then count bytes)
};
int launch_attention(const AttnArgs& args, cudaStream_t s);
int decode_num_splits(int batch, int hkv, int max_seq_len, int num_sms);

// ----- attention of single rows, any head sizes, fp32 arithmetic (attention_rows.cu) -----------
struct RowAttnArgs {
  const void* q;            // [rows, heads, dim], rows q_stride apart
  const void* k_cache;      // head g of slot s at s * tok + g * head (elements), dim features
  const void* v_cache;      // the same with vdim features
  void* out;                // [rows, heads, vdim], rows out_stride apart
  const int* req_to_token;
  const int* row_req;       // [rows] request-table row
  const int64_t* row_pos;   // [rows] position: keys 0 .. position (the last `window` of them when window > 0, those of its
                            // chunk of positions when chunk > 0)
  const float* sink;        // [heads] or null
  int* status;
  int64_t q_stride, out_stride, rtt_stride, num_slots, k_tok_stride, k_head_stride, v_tok_stride, v_head_stride;
  int rows, heads, kv_heads, dim, vdim, window, chunk;
  float scale, logit_cap;
  DType dt;
};
int launch_attention_rows(const RowAttnArgs& args, cudaStream_t s);

// ----- lightning attention (lightning.cu) --------------------------------------------------------
// Per request and head, S <- decay S + k v^T and o = S^T q with q, k, v = silu of the given rows (rounded to dt), S fp32.
// Ragged sequences as for the gated delta net below.
struct LightningArgs {
  const void* q;            // [T, heads, dk], token rows q_ld apart
  const void* k;
  const void* v;            // [T, heads, dv]
  void* out;                // [T, heads, dv] contiguous
  const float* decay;       // [heads]
  float* state;             // [rows, heads, dk, dv]
  const int* slots;
  const int* lens;
  const int* has_state;
  const int* q_start;
  // state-space duality (dt_raw null: lightning attention): rows activated already, q and k [T, k_heads, dk],
  // dt = softplus(dt_raw + dt_bias), decay exp(-exp(a_log) dt), S <- decay S + dt k v^T, o = S^T q + skip v
  const void* dt_raw;       // [T, heads], rows dt_ld apart
  const float* dt_bias;     // [heads]
  const float* a_log;       // [heads]
  const float* skip;        // [heads]
  int64_t dt_ld;
  int k_heads;
  int64_t q_ld, k_ld, v_ld;
  int batch, heads, dk, dv;
  // chunk kernel: > 1 cuts every request's tokens into this many segments of seg_tokens (a multiple of 64; segments *
  // seg_tokens >= the longest request) that run side by side; ws holds [batch][segments][heads][dk][dv] fp32
  int segments, seg_tokens;
  float* ws;
  float* ws_log;            // state-space duality with segments: [batch][segments][heads]
  DType dt;
};
int lightning_segments(int batch, int heads, int dv, int max_len, int num_sms);
// token by token; dk up to 512, any dv
int launch_lightning_recurrent(const LightningArgs& args, cudaStream_t s);
// 64 tokens at a time on the tensor cores; 16-bit types, dk up to 128
int launch_lightning_chunk(const LightningArgs& args, cudaStream_t s);
bool lightning_chunk_covers(const LightningArgs& args);

// ----- latent attention (one cached row of `rank` features per token, shared by all heads; `rot` rotated key features may
// follow them in the row) ------------
// Rows [q_rank | kv_rank | rot | ..] of the down projections: RMS norm of the first two, the first into cq, the second into
// the cache row loc[t], where the third follows it, its neighbouring features (halves: feature i with i + rot / 2) turned by
// positions[t] * inv_freq.  kv_rank 0: the layer reads another layer's rows and writes none; q_rank 0: queries have no latent.
struct LatentPrologueArgs {
  const void* y;            // [tokens, ..], rows ld apart
  const float* q_w;         // [q_rank]
  const float* kv_w;        // [kv_rank]
  const double* inv_freq;   // [rot / 2]
  const int64_t* positions; // [tokens]
  float2* turns;            // [tokens, rot / 2]: cosine and sine of every token, written
  void* cq;                 // [tokens, q_rank]
  const int64_t* loc;       // [tokens]
  void* cache;
  int* status;
  int64_t ld, cache_ld, num_slots;
  int tokens, q_rank, kv_rank, rot, halves;
  float eps;
  DType dt;
};
void launch_latent_prologue(const LatentPrologueArgs& args, cudaStream_t s);
// neighbouring features (halves: i and i + rot / 2) of x [tokens, heads, rot] (strided) turn by turns [tokens, rot / 2]; out may be x
void launch_turn_heads(const void* x, int64_t x_tok, int64_t x_head, const float2* turns, void* out, int64_t out_tok, int64_t out_head,
                       int tokens, int heads, int rot, int halves, DType dt, cudaStream_t s);
// out [tokens, heads, width] (strided, may be x) = x (strided) * sigmoid(gate[t, h]), rows of gate gate_ld apart; per_feature:
// gate is [tokens, heads * width], a number for every feature
void launch_gate_heads(const void* x, int64_t x_tok, int64_t x_head, const void* gate, int64_t gate_ld, void* out, int64_t out_tok,
                       int64_t out_head, int tokens, int heads, int width, int per_feature, DType dt, cudaStream_t s);
// out[start[b] + j] = latent of token first[b] + j of request b, j < lens[b] (first null: 0)
void launch_latent_gather(const void* cache, int64_t cache_ld, int rank, int elem_bytes, const int* rtt, int64_t rtt_stride,
                          const int* req, const int* lens, const int* start, const int* first, int batch, int max_len, void* out,
                          int64_t num_slots, int* status, cudaStream_t s);
// out[t, h, :N] = w[h] x[t, h, :K], times sigmoid(gate[t, h]) where gate is given; the `rot` features behind K are turned by
// turns [tokens, rot / 2] and put behind N.  K % 8 == 0, 16-bit types (else -1)
struct HeadLinearArgs {
  const void* x;
  const void* w;            // [heads, N, K]
  void* out;
  const void* gate;         // [tokens, heads] (gate_feat: [tokens, heads * N]) with rows gate_ld apart, or null
  const float2* turns;
  int64_t x_tok, x_head, out_tok, out_head, gate_ld;
  int tokens, heads, N, K, rot, halves, gate_feat;
  DType dt;
};
int launch_head_linear(const HeadLinearArgs& args, int num_sms, cudaStream_t s);
struct LatentAttnArgs {
  const void* q;            // [rows, heads, key] queries taken to the latent space, key >= rank
  const void* cache;        // row of slot s at s * cache_ld (elements): key features, values are the first rank of them
  void* out;                // [rows, heads, rank]
  float* part_o;            // splits > 1: [rows, heads, splits, rank]
  float* part_lse;          // splits > 1: [rows, heads, splits]
  const int* req_to_token;
  const int* row_req;       // [rows] request-table row of each query
  const int64_t* row_pos;   // [rows] its position: it sees keys 0 .. position, with window > 0 the last `window` of them
  const float* sink;        // [heads] or null
  int* status;
  int64_t rtt_stride, cache_ld, num_slots;
  int rows, heads, key, rank, splits, window;
  float scale;
  DType dt;
};
int launch_latent_attention(const LatentAttnArgs& args, cudaStream_t s);
int latent_num_splits(int rows, int heads, int max_seq_len, int num_sms);
bool latent_mma_covers(int key, int rank, int64_t cache_ld, DType dt);   // false: the fp32 kernel runs, splits must be 1

// ----- gated delta net (hybrid models): causal convolution (bias [C] or null; add_input: x + conv(x) instead of the SiLU), rule -----------------------------------------------------------
// Ragged sequences: request b owns rows q_start[b] .. q_start[b] + lens[b] of the token-major inputs and
// row slots[b] of the state tensors; has_state[b] != 0 resumes from the stored state.
int launch_gdn_conv1d_silu(const void* x, int64_t x_ld, const void* w, void* conv_state, const int* slots, const int* lens,
                           const int* has_state, const int* q_start, void* out, int batch, int max_tokens, int channels, int K,
                           const void* bias, int add_input, DType dt, cudaStream_t s);
// beta = sigmoid(b), g = -exp(a_log) * softplus(a + dt_bias); b and a [tokens, heads] with rows ld apart
void launch_gdn_gates(const void* b, const void* a, int64_t ld, const float* a_log, const float* dt_bias, float* g, float* beta,
                      int64_t tokens, int heads, DType dt, cudaStream_t s);
struct GdnRuleParams {
  const void* q;            // [T, k_heads, dk], token rows q_ld apart (elements)
  const void* k;            // [T, k_heads, dk]
  const void* v;            // [T, heads, dv]
  void* out;                // [T, heads, dv] contiguous
  const float* g;           // log decay [T, heads], or null: gates from the four fields below (recurrent kernel only)
  const float* beta;
  const void* b_raw;        // [T, heads] with rows gate_ld apart
  const void* a_raw;        // [T, heads]; with a decay per key channel (a_ld > 0) [T, heads * dk] with rows a_ld apart
  const float* a_log;       // [heads]
  const float* dt_bias;     // [heads], per channel [heads * dk]
  float* state;             // [rows, heads, dk, dv]
  const int* slots;
  const int* lens;
  const int* has_state;
  const int* q_start;
  int64_t q_ld, k_ld, v_ld, gate_ld, a_ld;
  int batch, heads, k_heads, dk, dv;
  int split_tf32;           // chunk kernel: two-term tf32 operands (fp32-like products)
  DType dt;
};
// token by token; dk up to 512, any dv
int launch_gdn_recurrent(const GdnRuleParams& p, cudaStream_t s);
// the same rule evaluated 64 tokens at a time with tensor-core products (prefill); dk up to 128, multiples of 8
int launch_gdn_chunk(const GdnRuleParams& p, int num_sms, cudaStream_t s);
bool gdn_chunk_covers(const GdnRuleParams& p);
// decays per key channel, 16 tokens at a time (prefill); dk up to 128, multiples of 8, gates formed inside.  The workspace
// holds `span` chunks of every request; longer runs loop over spans
struct GdnChannelPlan {
  int span;
  int64_t ws_floats;
};
GdnChannelPlan gdn_channel_plan(const GdnRuleParams& p, int max_len);
int launch_gdn_channel_chunk(const GdnRuleParams& p, float* ws, int span, int max_len, int num_sms, cudaStream_t s);
bool gdn_channel_chunk_covers(const GdnRuleParams& p);
// x, out [rows = tokens * heads, width] contiguous, gate [tokens, heads * width] with rows gate_ld apart
void launch_rmsnorm_gated(const void* x, const void* gate, int64_t gate_ld, const void* w, void* out, int64_t rows, int heads,
                          int width, float eps, int round_norm, int sigmoid, DType dt, cudaStream_t s);

// ----- vision tower helpers ------------------------------------------------------------------
// qkv [T, 3, H, D] (D <= 128, D % 8 == 0) -> q, k, v [T, H, 128] zero-padded; q and k get the 2-D rotary
// embedding: out[i] = x[i] c[i] - x[i + D/2] s[i], out[i + D/2] = x[i + D/2] c[i] + x[i] s[i], cos/sin fp32 [T, D/2].
void launch_vision_rope_split_pad(const void* qkv, const float* cos, const float* sin, void* q, void* k, void* v,
                                  int tokens, int heads, int head_dim, int out_dim, DType dt, cudaStream_t s);
// x[t, :] += sum_i w[i, t] * table[idx[i, t], :]  (i < 4: bilinear corners); idx int64 [4, T], w fp32 [4, T]
void launch_vision_pos_embed_add(void* x, const void* table, const int64_t* idx, const float* w, int tokens, int hidden,
                                 DType dt, cudaStream_t s);
void launch_gelu_erf(const void* x, void* out, int64_t n, DType dt, cudaStream_t s);

// ----- tensor-parallel reduction + residual add + RMSNorm over peer memory ----------------
// peer_data / peer_flags: host arrays of `tp` device addresses (every rank's partial-sum buffer
// and flag block, mapped into this process).  flags: uint32 [max_rows][8] per rank, zero-initialised;
// local_seq: uint32 [max_rows] on this device, zero-initialised.  weight may be null (plain sum).
int launch_tp_reduce_add_rmsnorm(const uint64_t* peer_data, const uint64_t* peer_flags, uint32_t* local_seq,
                                 void* residual, const void* weight, void* out, int rows, int hidden, int tp, int rank,
                                 int64_t row_stride, float eps, DType dt, int* status, cudaStream_t s);


// ----- tensor-parallel prefill: reduce-scatter + residual add + RMSNorm + all-gather -------
// This rank owns `rows` consecutive token rows (global rows rank * rows ...).  inbox: local
// [tp][inbox_rows_cap][hidden] partial sums written by every rank's GEMM epilogue; tile_flags: local
// uint32 [tiles][8], slot (tile, src) holds the epoch of src's last completed delivery of that 128-row
// tile.  For each own row: sum the tp partials in rank order, add the residual shard (in place; when
// residual is null the sum itself is the new residual... the caller passes the shard), normalise, and
// store the row into every rank's gathered buffer (peer_hidden[r] + global_row * hidden).  When a
// 128-row tile is complete, gather_flags[global tile] on every rank is set to `epoch`.
// ag_count: local int[tiles], zero-initialised, self-resetting.  rows must be a multiple of 128.
// n_src = partial sums per row in the inbox: tp for the reduce-scatter inbox; 1 with tile_flags == nullptr when
// the rows of this rank are already complete (output of the expert-parallel exchange).
int launch_tp_rs_add_rmsnorm_ag(const void* inbox, int64_t inbox_rows_cap, const uint32_t* tile_flags,
                                void* residual_shard, const void* weight, const uint64_t* peer_hidden,
                                const uint64_t* peer_gather_flags, int* ag_count, int rows, int hidden, int tp,
                                int n_src, int rank, uint32_t epoch, float eps, DType dt, int* status, cudaStream_t s);
// Bounded wait until flags[i] >= epoch for all i < n (makes peers' deliveries visible to later kernels).
int launch_tp_wait_flags(const uint32_t* flags, int n, uint32_t epoch, int* status, cudaStream_t s);

}  // namespace mb200
