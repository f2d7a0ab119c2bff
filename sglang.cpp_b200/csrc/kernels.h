// Internal launch interface shared by the C-ABI wrappers and the step runner.
// Every function enqueues work on `stream` and returns a B200_* status.
#pragma once

#include <cuda.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/b200_token_loop.h"

namespace b200 {

// Gated epilogues take two stacked halves of W (gate, up); the others one.
constexpr bool epilogue_is_gated(int epilogue) {
    return epilogue != B200_EPILOGUE_NONE && epilogue != B200_EPILOGUE_RELU2 && epilogue != B200_EPILOGUE_GELU_ERF &&
           epilogue != B200_EPILOGUE_F32;
}

int launch_rmsnorm(void* out, const void* x, const void* weight, int rows, int hidden, float eps,
                   cudaStream_t stream);
// round_sum_first: normalise the bf16-rounded sum (separate add then norm, as the Llama wiring
// does) instead of the fp32 sum (the fused FlashInfer form the Qwen3 wiring uses).
int launch_fused_add_rmsnorm(void* x, void* residual, const void* weight, int rows, int hidden,
                             float eps, bool round_sum_first, cudaStream_t stream);
int launch_qknorm_rope_store(void* qkv, const void* q_weight, const void* k_weight,
                             const float* cos_table, const float* sin_table,
                             const int32_t* positions, const int32_t* out_loc, void* k_cache,
                             void* v_cache, int tokens, int q_heads, int kv_heads, int head_dim,
                             int max_pos, int64_t num_slots, float eps, int write_k_back,
                             int* status, cudaStream_t stream);
int launch_act_and_mul(void* out, const void* in, int tokens, int d, bool gelu, cudaStream_t stream);
// ssq (optional, [ssq_slots, ssq_stride]): slot 0 receives each row's sum of squares in 2^-24 fixed
// point and the other slots are zeroed for the tokens of this call.
int launch_embedding(void* out, const void* table, const int32_t* ids, int tokens, int hidden,
                     int vocab, int* status, cudaStream_t stream, unsigned long long* ssq = nullptr,
                     int ssq_slots = 0, int ssq_stride = 0);
// out[n, k] = bf16(w[n, k] * scale[k]): a norm weight folded into the columns of the matrix that follows it.
int launch_scale_columns(void* out, const void* w, const void* scale, int64_t rows, int K, cudaStream_t stream);
// Optional write-back of the chosen tokens into the token pool by the kernel that chooses them
// (token_pool[table_idx[i], write_pos[i]] = token[i] for i < count, positions outside the table
// skipped): what a separate scatter launch would do behind it.
struct TokenWriteBack {
    int32_t* pool = nullptr;
    int64_t rows = 0, stride = 0, cols = 0;
    const int32_t* table_idx = nullptr;
    const int32_t* write_pos = nullptr;
    int count = 0;
};
// step_index_dev (optional): the step index is read from device memory instead of the argument, so a
// captured graph replays with a new value.
int launch_sample(int32_t* out, const void* logits, int rows, int vocab, int64_t ld,
                  const float* temperatures, const int32_t* top_k, const float* top_p,
                  const uint64_t* seeds, uint64_t step_index, uint8_t* mask, cudaStream_t stream,
                  const uint64_t* step_index_dev = nullptr, const TokenWriteBack* write_back = nullptr);
int launch_argmax_f32(int32_t* out, const float* logits, int rows, int vocab, int64_t ld, cudaStream_t stream,
                      const TokenWriteBack* write_back = nullptr);
int launch_argmax(int32_t* out, const void* logits, int rows, int vocab, int64_t ld,
                  cudaStream_t stream, const TokenWriteBack* write_back = nullptr);

// Tensor map of a 2-D bf16 tensor [outer, inner] copied in [box_outer, box_inner] boxes with the
// 128-byte swizzle, from a small per-thread cache (the same buffers come back every layer).
int cached_tmap(CUtensorMap* out, const void* base, uint64_t inner, uint64_t outer, uint64_t pitch,
                uint32_t box_inner, uint32_t box_outer);

// Large-M GEMM (prefill batches): persistent 128 x 256 output tiles on the tcgen05 tensor cores.
// act_limit (here and below): the limit of B200_EPILOGUE_CLAMPED_SWIGLU.
int launch_tile_gemm(void* y, const void* x, const void* w, const void* bias, int M, int N, int K,
                     int64_t ldx, int epilogue, int* status, cudaStream_t stream, float act_limit = 0.f);

int launch_grouped_tile_gemm(void* y, const void* x, const void* w, const int32_t* counts,
                             const int32_t* offsets, int num_groups, int64_t total_rows, int N, int K,
                             int epilogue, int* status, cudaStream_t stream, float act_limit = 0.f);

// Fusions of a split-K GEMM of at most 256 rows with the residual stream of a decode step.  Row
// statistics travel as sums of squares in 2^-24 fixed point (integer atomics: the same bits whatever
// order the CTAs finish in).
//  - ssq_in: the rows of x are un-normalised and w has the norm weight folded into its columns; the
//    accumulator of row m is multiplied by rsqrt(ssq_in[m] / 2^24 / norm_width + eps).
//  - residual: y is not written; residual[m, n] becomes bf16(bf16(acc) + residual[m, n]) and
//    ssq_out[m] grows by the squares of those sums (of the stored bf16 values if ssq_of_rounded).
//  - heads: the projection is a packed qkv projection with 128-wide heads; instead of y[:, all] the
//    epilogue writes the rotated (and, with norm weights, RMS-normalised) q heads into y and the k / v
//    heads into the pool at out_loc - what launch_qknorm_rope_store does after a plain projection.
struct HeadEpilogue {
    const void* q_norm_w = nullptr;   // [128] bf16 or NULL
    const void* k_norm_w = nullptr;
    const float* cos_t = nullptr;     // [max_pos, 64]
    const float* sin_t = nullptr;
    const int32_t* positions = nullptr;
    const int32_t* out_loc = nullptr;
    void* k_cache = nullptr;          // [num_slots, kv_heads, 128] bf16
    void* v_cache = nullptr;
    int q_heads = 0, kv_heads = 0, max_pos = 1;
    int64_t num_slots = 0;
    float eps = 0.f;
};
struct SkinnyFusion {
    const unsigned long long* ssq_in = nullptr;
    float eps = 0.f;
    int norm_width = 1;
    void* residual = nullptr;
    unsigned long long* ssq_out = nullptr;
    bool ssq_of_rounded = false;
    const HeadEpilogue* heads = nullptr;
};
// The K split launch_linear picks for a slab of this shape (the fusions need it above 1).
int skinny_gemm_split(int M, int N, int K, int epilogue);

// y[M, n_out] = x[M, K] w[N, K]^T (+bias / gated epilogue); any M (slabs of 256 rows).
int launch_linear(void* y, const void* x, const void* w, const void* bias, int M, int N, int K,
                  int64_t ldx, int epilogue, int* status, cudaStream_t stream,
                  const SkinnyFusion* fuse = nullptr, float act_limit = 0.f);

int launch_grouped_gemm(void* y, const void* x, const void* w, const int32_t* counts,
                        const int32_t* offsets, int num_groups, int max_rows_per_group,
                        int64_t total_rows, int N, int K, int epilogue, int* status,
                        cudaStream_t stream, float act_limit = 0.f);

int launch_linear_heads(void* y, const void* x, const void* w, int M, int heads, int N, int K, int* status,
                        cudaStream_t stream);
// fp32 GEMMs of every form the layer stack uses (linear_f32.cu); see b200_linear_f32.
int launch_linear_f32(float* y, const float* x, const float* w, int max_rows, int N, int K, int groups,
                      const int32_t* counts, const int32_t* offsets, int epilogue, cudaStream_t stream,
                      float act_limit = 0.f, const float* bias = nullptr);

// fp32 residual stream: add, norm, and the gather / scatter around them (residual.cu).
struct ResidualNorm {
    void* out = nullptr;
    const int32_t* out_rows = nullptr;
    int out_top = 1;
    float* residual = nullptr;
    const void* src = nullptr;
    const int32_t* src_rows = nullptr;
    int src_top = 1;
    int64_t src_count = 0;
    float src_scale = 1.f;
    bool init = false;
    const void* weight = nullptr;
    float weight_offset = 0.f, out_scale = 1.f;
    int tokens = 0, width = 0, padded = 0;
    float eps = 0.f;
};
int launch_residual_norm(const ResidualNorm& a, int dtype, int* status, cudaStream_t stream);

// The wiring with the norm on what is added: residual += add_weight * rms_normalise(sum_k src_weights[k] *
// src[src_rows[k]] + src2), out = residual (through the norm with out_weight if there is one).
struct ResidualPostNorm {
    void* out = nullptr;
    float* residual = nullptr;
    const void* src = nullptr;
    const int32_t* src_rows = nullptr;      // NULL: the token's own row
    const float* src_weights = nullptr;     // NULL: 1
    int src_top = 1;
    int64_t src_count = 0;
    const void* src2 = nullptr;             // optional second row per token
    // Both set: src and src2 are RMS-normalised with a weight each before they are added, and the sum is
    // multiplied by pair_scale.
    const void *pair_weight = nullptr, *pair_weight2 = nullptr;
    float pair_scale = 1.f;
    bool init = false;                      // the sum replaces the residual
    const void* add_weight = nullptr;       // NULL: what is added is not normalised
    const void* out_weight = nullptr;       // NULL: out is the residual itself
    // Layer norms instead of RMS norms (weight_offset and out_scale do not apply, nor do pairs).
    bool layer = false;
    const void *add_bias = nullptr, *out_bias = nullptr;
    const void* self = nullptr;             // what a source row of -1 stands for: the token's own row here
    float src_scale = 1.f;                  // with init: a factor on what is added
    float weight_offset = 0.f, out_scale = 1.f;   // as in ResidualNorm
    int tokens = 0, width = 0, padded = 0;
    float eps = 0.f;
    int32_t* clear = nullptr;               // integers set to zero on the way (counters of a later kernel)
    int clear_count = 0;
};
int launch_residual_post_norm(const ResidualPostNorm& a, int dtype, int* status, cudaStream_t stream);

// Expert placement of every table-routed layer of a step in one launch (moe.cu): one CTA per layer.
struct TableRouteLayer {
    const int32_t* table;     // [vocab, top]
    int32_t *rows, *counts, *offsets;
    int top, experts;
};
constexpr int kMaxTableExperts = 4096;
int launch_table_route(const TableRouteLayer* layers_dev, int num_layers, int max_experts, const int32_t* token_ids,
                       int tokens, int vocab, int* status, cudaStream_t stream);

// Routing by scores (moe.cu; b200_score_route): ids, weights and counts from fp32 logits, then a row for every choice
// and the token's activations copied there.  counts [experts] and the cursor [experts] are zero before.
struct ScoreRoute {
    const float* logits = nullptr;   // [tokens, ld]
    int64_t ld = 0;
    int tokens = 0, experts = 0, top = 1, groups = 1, keep = 1;
    float scale = 1.f;
    int score = B200_SCORE_SIGMOID;
    int identity = 0;                // logits behind those of the experts: experts that return their input
    const float* correction = nullptr;   // softmax scores: what a choice adds to a score, or NULL
    int32_t* ids = nullptr;          // [tokens, top]
    float* weights = nullptr;        // [tokens, top]
    int32_t* counts = nullptr;
};
int launch_score_route(const ScoreRoute& r, cudaStream_t stream);
int launch_score_place(void* xp, const void* x, int row_bytes, const ScoreRoute& r, int32_t* rows, int32_t* cursor,
                       int32_t* offsets, cudaStream_t stream);

// Latent attention (latent_attention.cu, latent_attention_tc.cu).
// The output of the joint down-projection [tokens, qp + rp] -> RMS-normalised query latent [tokens, qp]
// and RMS-normalised key/value latent straight into the pool (cache NULL: the joint rows are the query latent
// alone).  With a rotation, columns [rope_at, rope_at + rope_dim) of the key/value part are not normalised but
// rotated in neighbouring pairs; rope_at is a multiple of 8.
struct LatentNorm {
    void *q_latent = nullptr, *cache = nullptr;
    const void *joint = nullptr, *q_weight = nullptr, *kv_weight = nullptr;
    const int32_t *out_loc = nullptr, *positions = nullptr;
    int tokens = 0, q_rank = 0, qp = 0, kv_rank = 0, rp = 0;
    int rope_at = 0, rope_dim = 0, max_pos = 1;
    const float *cos_t = nullptr, *sin_t = nullptr;   // [max_pos, rope_dim / 2]
    int64_t num_slots = 0;
    float eps = 0.f;
    int* status = nullptr;
};
int launch_latent_norm_store(const LatentNorm& a, int dtype, cudaStream_t stream);
// The first `dims` elements of every head of x [tokens, heads, ld] rotated in place, in neighbouring pairs.
int launch_rotate_pairs(void* x, int tokens, int heads, int ld, int dims, const float* cos_t, const float* sin_t,
                        const int32_t* positions, int max_pos, int dtype, int* status, cudaStream_t stream);
struct LatentAttention {
    void* out = nullptr;              // [rows, heads, out_width]
    const void* q = nullptr;          // [rows, heads, width]
    const void* cache = nullptr;      // [num_slots, width]
    int64_t num_slots = 0;
    const int32_t* page_table = nullptr;
    int64_t pt_stride = 0;
    const int32_t* row_table = nullptr;   // page-table row of every query row
    const int32_t* row_len = nullptr;     // keys it sees
    int rows = 0, heads = 0, width = 0, page_size = 1;
    int out_width = 0;                    // only the first columns of a latent are averaged; 0: all of them
    float scale = 1.f;
    // Only key row_len[i] - 1 of row i was written by kernels that may still be running when this one
    // starts (a decode step), and the tables and lengths are complete: the rest is read ahead of them.
    bool only_last_key_new = false;
    void* workspace = nullptr;
    int64_t workspace_bytes = 0;
};
int64_t latent_attention_workspace_bytes(int rows, int heads, int width);
bool latent_attention_tc_supported(const LatentAttention& a);
int launch_latent_attention_tc(const LatentAttention& a, int* status, cudaStream_t stream);
int launch_latent_attention_plain(const LatentAttention& a, int dtype, int* status, cudaStream_t stream);
// Rows of a paged latent pool gathered into consecutive rows: request b's positions [0, seq_lens[b]) to
// rows base[b] + position (base[b] < 0: skipped).
int launch_gather_latents(void* out, const void* cache, int64_t num_slots, const int32_t* page_table,
                          int64_t pt_stride, const int32_t* table_idx, const int32_t* seq_lens,
                          const int32_t* base, int batch, int max_len, int rp, int* status, cudaStream_t stream);
// out[i] = in[rows[i]] (gather) or out[rows[i]] = in[i] (scatter) for rows of vec_per_row 16-byte vectors.
int launch_move_rows(void* out, const void* in, const int32_t* rows, int count, int vec_per_row, bool scatter,
                     cudaStream_t stream);

int64_t moe_workspace_bytes(int tokens, int E, int top_k, int H, int I);
int launch_moe_forward(void* out, const void* hidden, const void* router_logits, const void* gate_up,
                       const void* down, int tokens, int E, int top_k, int H, int I, int renorm,
                       int activation, int expert_begin, int num_local_experts, void* workspace,
                       int* status, cudaStream_t stream);

// Decode-step layer chain (decode_chain.cu): o_proj -> add + norm -> gate_up -> act -> down ->
// add + norm -> the next layer's qkv -> QK-norm -> RoPE -> KV store, as one persistent kernel.
struct DecodeChainArgs {
    int tokens, hidden, inter, q_heads, kv_heads, max_pos;
    float eps;
    bool round_first, gelu;
    const void* attn_out;        // [tokens, q_heads * 128] bf16, the attention output of this layer
    void* residual;              // [tokens, hidden] bf16, updated in place
    void* mlp_act;               // [tokens, inter] bf16 scratch (the activated gate_up output)
    void* x_out;                 // last layer only: [tokens, hidden] down_proj output (no residual add)
    void* qkv_out;               // [tokens, (q + 2 kv) * 128]: the q heads of the next layer are written
    const void *w_o, *w_gate_up, *w_down;
    const void* w_qkv_next;      // NULL for the last layer: the chain then ends after down_proj
    const void *post_norm_w, *next_input_norm_w, *q_norm_w, *k_norm_w;   // q / k norm weights may be NULL
    const float *cos_t, *sin_t;
    const int32_t *positions, *out_loc;
    void *k_cache_next, *v_cache_next;
    int64_t num_slots;
    void* scratch;               // decode_chain_scratch_bytes(hidden), zero-initialised once
    int* status;
};
int decode_chain_max_grid();
int64_t decode_chain_scratch_bytes(int hidden);
bool decode_chain_supported(int tokens, int hidden, int q_heads, int kv_heads, int head_dim, int inter,
                            bool has_bias);
int launch_decode_chain(const DecodeChainArgs& args, cudaStream_t stream);

// What the paged attention kernels take beside causal attention.
//  - A sliding window over the keys, the first ones kept: the query at position i sees key j <= i if
//    i - j < size or j < keep_first.  Or chunks of the sequence (chunk > 0, which replaces size): it sees j if
//    i / chunk = j / chunk.
//  - A sink: exp(sinks[h]) is added to the denominator of head h's softmax.
//  - A gate on the output: head h's element c is multiplied by sigmoid(gate[token, h * vdim + c]), or the whole
//    head by sigmoid(gate[token, h]).
//  - A constant factor on the output, whose rows may be part of wider ones.
struct AttentionWindow {
    int size = 0x7fffffff;
    int keep_first = 0;
    int chunk = 0;
    const float* sinks = nullptr;   // [heads]; NULL: none
    const void* gate = nullptr;     // of the attention's dtype; NULL: no gate
    int64_t gate_st = 0;            // its token stride in elements
    bool gate_per_head = false;
    float out_scale = 1.f;
    int64_t out_st = 0;             // token stride of the output; 0: its rows are dense
    // the oldest key in the window of the query at position `pos` (kept ones aside)
    __host__ __device__ int oldest(int pos) const {
        const int o = chunk > 0 ? pos / chunk * chunk : pos - size + 1;
        return o > 0 ? o : 0;
    }
};

// A pool [slots, kv heads, 128] in boxes of 64 elements of one head of kpc slots (attention_prefill_tc2.cu).
int make_kv_tile_tmap(CUtensorMap* out, const void* cache, int64_t num_slots, int kv_heads, int kpc);
int64_t decode_workspace_bytes(int max_batch, int q_heads, int kv_heads);
int make_kv_tmap(CUtensorMap* out, const void* cache, int64_t num_slots, int kv_heads, int page_size);
int launch_attention_decode(void* out, const void* q, int64_t q_st, int64_t q_sh,
                            const CUtensorMap& tmap_k, const CUtensorMap& tmap_v, int64_t num_slots,
                            const int32_t* page_table, int64_t pt_stride, const int32_t* table_idx,
                            const int32_t* seq_lens, int batch, int q_heads, int kv_heads,
                            int page_size, float sm_scale, void* workspace, int64_t workspace_bytes,
                            int* status, cudaStream_t stream, bool kv_evict_first = false,
                            const AttentionWindow* window = nullptr);
// Attention of layer stacks (window_attention.cu).  head_prepare: the rows of the joint projection's output
// [q heads | k heads | v heads | ...] to normalised, rotated queries (in place) and into the pools.
struct HeadPrepare {
    enum { kPlain = 0, kSave = 1, kMix = 2 };   // values: as they are, kept for later layers, mixed with the kept ones
    void* joint = nullptr;
    int64_t ld = 0;
    int tokens = 0, heads = 0, kv_heads = 0, dim = 0, dp = 0, vp = 0;
    const void *q_weight = nullptr, *k_weight = nullptr;   // [dp] or NULL
    float eps = 0.f;
    int rotary_dim = 0, max_pos = 1;
    const float *cos_t = nullptr, *sin_t = nullptr;        // [max_pos, rotary_dim / 2]
    const int32_t *positions = nullptr, *out_loc = nullptr;
    void *k_cache = nullptr, *v_cache = nullptr;           // [num_slots, kv_heads, dp | vp]
    int64_t num_slots = 0;
    int mix = kPlain;
    const float* lambda = nullptr;                         // v <- (1 - lambda) v + lambda first
    void* first_values = nullptr;                          // [tokens, kv_heads, vp]
    bool unit_norm = false;                                // RMS norms without weights
    int value_rotary = 0;                                  // values rotate over their first value_rotary elements
    const float *value_cos = nullptr, *value_sin = nullptr;
    int* status = nullptr;
};
int launch_head_prepare(const HeadPrepare& a, int dtype, cudaStream_t stream);
// Heads that mix their softmax weights, and values that are turned back (head_mix.cuh); see
// b200_window_attention_args.
struct HeadMix {
    const float* weights = nullptr;    // [heads, heads]; NULL: off
    int rotary = 0, max_pos = 1;
    const float *cos_t = nullptr, *sin_t = nullptr;
    const int32_t* positions = nullptr;
    float score_bound = 0.f;
    void* scratch = nullptr;           // [tokens, heads, kv_heads, vp] of the dtype
};
struct WindowAttention {
    void* out = nullptr;               // [tokens, heads, vp]
    const void* q = nullptr;           // token stride q_st, heads dp apart
    int64_t q_st = 0;
    const void *k_cache = nullptr, *v_cache = nullptr;
    int64_t num_slots = 0;
    const int32_t* page_table = nullptr;
    int64_t pt_stride = 0;
    const int32_t *table_idx = nullptr, *seq_lens = nullptr, *qo_indptr = nullptr;   // per request
    const int32_t *row_table = nullptr, *row_len = nullptr;                          // per token
    int tokens = 0, batch = 0, max_extend = 0;
    bool decode = false;               // one token per request, the tables complete ahead of the launch
    bool plain = false;                // never the tensor-core kernels
    int heads = 0, kv_heads = 0, dp = 0, vp = 0, page_size = 1;
    float scale = 1.f;
    AttentionWindow window;
    HeadMix mix;
    void* workspace = nullptr;
    int64_t workspace_bytes = 0;       // decode_workspace_bytes, or head_mix_workspace_bytes
    int* status = nullptr;
};
// The plain kernel over all key / value heads' values: what every head's weights make of each of them, in a.mix.scratch.
int launch_plain_all_values(const WindowAttention& a, int dtype, cudaStream_t stream);
bool window_attention_tc_supported(const WindowAttention& a, int dtype);
int launch_window_attention(const WindowAttention& a, int dtype, cudaStream_t stream);
// Mixing heads (talking_heads.cu; the decode kernel is attention_decode.cu's).
bool talking_heads_tc_supported(const WindowAttention& a, int dtype);
int launch_talking_heads(const WindowAttention& a, int dtype, cudaStream_t stream);
bool talking_decode_supported(int heads, int kv_heads);
int64_t head_mix_workspace_bytes(int max_batch, int heads, int kv_heads);
int launch_talking_decode(const WindowAttention& a, cudaStream_t stream);
// Recurrences with one decay per head (recurrence.cu); see b200_recurrence.
using Recurrence = b200_recurrence_args;
// Bytes of a step's scratch arrays.
struct RecurrenceScratch {
    int64_t mixed, steps, units, chunks;
};
RecurrenceScratch recurrence_scratch(int rule, int max_tokens, int max_batch, int heads, int kv_heads, int padded_dim,
                                     int padded_value_dim, int dtype);
bool recurrence_supported(int padded_value_dim, int padded_dim, int taps);
int64_t recurrence_memory_floats(int padded_dim, int padded_value_dim);   // per head
int launch_recurrence(const Recurrence& a, int dtype, cudaStream_t stream);
// Gated linear attention (linear_attention.cu): the recurrence, its norm and its gate; see
// b200_linear_attention.
using LinearAttention = b200_linear_attention_args;
bool linear_attention_supported(int padded_value_dim, int padded_dim);
int launch_linear_attention(const LinearAttention& a, int dtype, cudaStream_t stream);
bool attention_prefill_tc_supported(const void* q, int64_t q_st, int64_t q_sh, const void* out);
int launch_attention_prefill_tc(void* out, const void* q, int64_t q_st, int64_t q_sh, const void* k_cache,
                                const void* v_cache, int64_t num_slots, const int32_t* page_table,
                                int64_t pt_stride, const int32_t* table_idx, const int32_t* seq_lens,
                                const int32_t* qo_indptr, int batch, int max_extend_len, int q_heads,
                                int kv_heads, int page_size, float sm_scale, int* status,
                                cudaStream_t stream);
int launch_attention_prefill_tc2(void* out, const void* q, int64_t q_st, int64_t q_sh, const void* k_cache,
                                const void* v_cache, int64_t num_slots, const int32_t* page_table,
                                int64_t pt_stride, const int32_t* table_idx, const int32_t* seq_lens,
                                const int32_t* qo_indptr, int batch, int max_extend_len, int q_heads,
                                int kv_heads, int page_size, float sm_scale, int* status,
                                cudaStream_t stream, const AttentionWindow* window = nullptr);
int launch_attention_prefill(void* out, const void* q, int64_t q_st, int64_t q_sh, const void* k_cache,
                             const void* v_cache, int64_t num_slots, const int32_t* page_table,
                             int64_t pt_stride, const int32_t* table_idx, const int32_t* seq_lens,
                             const int32_t* qo_indptr, int batch, int max_extend_len, int q_heads,
                             int kv_heads, int page_size, float sm_scale, int* status,
                             cudaStream_t stream);

}  // namespace b200
