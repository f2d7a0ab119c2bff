/*
 * b200_token_loop.h — C ABI of the B200 (sm_100a) per-step token loop.
 *
 * This library replaces the device side of sglang.cpp's per-step forward pass
 * (Engine::forward_batch, src/engine/engine.cc:495-544 of the reference) with
 * hand-written sm_100a kernels.  Every entry point takes plain device pointers,
 * sizes, strides (in elements) and a CUDA stream; none allocates or touches
 * LibTorch types.  Each declaration cites the reference interface it stands in
 * for, by the file's path inside the reference project.
 *
 * Conventions
 *   - All entry points return B200_OK (0) or a B200_ERR_* code;
 *     b200_last_error() gives the text for the calling thread.
 *   - bf16 tensors are raw uint16 storage ("bf16*" below means const void* /
 *     void* pointing at __nv_bfloat16 data).  Index tensors are int32.
 *   - `stream` is a cudaStream_t passed as void*; NULL is the legacy default
 *     stream.  Calls are asynchronous unless stated otherwise.
 *   - Nothing here synchronises the device unless stated otherwise.
 */
#ifndef B200_TOKEN_LOOP_H_
#define B200_TOKEN_LOOP_H_

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define B200_API __attribute__((visibility("default")))

typedef void* b200_stream_t;

enum {
    B200_OK = 0,
    B200_ERR_INVALID_ARGUMENT = 1, /* the reference would TORCH_CHECK-fail here */
    B200_ERR_CUDA = 2,             /* a CUDA runtime / driver call failed */
    B200_ERR_TIMEOUT = 3,          /* a bounded in-kernel wait ran out */
    B200_ERR_UNSUPPORTED = 4,      /* shape / dtype outside what the kernels cover */
    B200_ERR_STATE = 5             /* object used in the wrong state */
};

/* ---- library ------------------------------------------------------------- */

/* Text of the last error returned to the calling thread ("" if none). */
B200_API const char* b200_last_error(void);

/* ABI version of this header (bumped on incompatible change). */
B200_API int b200_abi_version(void);

/* Reads (synchronously) and clears the device status words that kernels with
 * bounded waits or index checks write: out[0] = wait site that timed out (0 =
 * none), out[1] = offending index + 1 (0 = none).  Synchronises `stream`. */
B200_API int b200_read_device_status(int32_t out[2], b200_stream_t stream);

/* ---- normalisation (include/sglang/layers/normalization.h:6-22) ---------- */

/* RMSNorm::forward / forward_inplace (src/layers/normalization.cu:236-269):
 * out[r,:] = x[r,:] * rsqrt(mean(x[r,:]^2) + eps) * weight, fp32 math, bf16
 * storage.  out may alias x.  x, out: [rows, hidden] contiguous. */
B200_API int b200_rmsnorm(void* out, const void* x, const void* weight, int rows, int hidden,
                          float eps, b200_stream_t stream);

/* RMSNorm::fused_add_forward_inplace (src/layers/normalization.cu:386-416):
 * residual <- x + residual (fp32 add, stored bf16); x <- rmsnorm(fp32 sum) * weight. */
B200_API int b200_fused_add_rmsnorm(void* x, void* residual, const void* weight, int rows,
                                    int hidden, float eps, b200_stream_t stream);

/* fused_qk_rmsnorm_inplace_3d_strided and RMSNorm::forward_inplace_3d_strided
 * (src/layers/normalization.cu:271-384): per-(token, head) RMSNorm over head_dim,
 * in place, on strided views q [tokens, q_heads, head_dim] and k [tokens,
 * k_heads, head_dim].  Either of q / k may be NULL (with 0 heads) for the
 * single-tensor form.  Strides are in elements. */
B200_API int b200_qk_rmsnorm_strided(void* q, void* k, const void* q_weight, const void* k_weight,
                                     int tokens, int q_heads, int k_heads, int head_dim,
                                     int64_t q_stride_token, int64_t q_stride_head,
                                     int64_t k_stride_token, int64_t k_stride_head, float eps,
                                     b200_stream_t stream);

/* ---- rotary embedding (include/sglang/layers/rotary_embedding.h:11-22) ---- */

/* RotaryEmbedding::forward_inplace (src/layers/rotary_embedding.cu:96-190):
 * NeoX (rotate-half) RoPE applied in place to q [tokens, q_heads, head_dim] and
 * k [tokens, k_heads, head_dim] from fp32 tables cos/sin [max_pos, rotary_dim/2]
 * and int32 positions [tokens].  fp32 math, bf16 storage. */
B200_API int b200_rope_neox_inplace(void* q, void* k, const float* cos_table,
                                    const float* sin_table, const int32_t* positions, int tokens,
                                    int q_heads, int k_heads, int head_dim, int rotary_dim,
                                    int max_pos, int64_t q_stride_token, int64_t q_stride_head,
                                    int64_t k_stride_token, int64_t k_stride_head,
                                    b200_stream_t stream);

/* ---- KV pool (include/sglang/kvcache/base.h:78-90) ------------------------ */

/* MHAKVCache::store_kv (src/kvcache/mha_kvcache.cu:12-41,113-155):
 * k_cache[out_loc[t], :, :] = k[t, :, :] and the same for v.  k_cache / v_cache:
 * one layer's [slots, kv_heads, head_dim] contiguous; k / v: strided rows of
 * kv_heads*head_dim elements. */
B200_API int b200_store_kv(void* k_cache, void* v_cache, const void* k, const void* v,
                           const int32_t* out_loc, int tokens, int kv_heads, int head_dim,
                           int64_t k_stride_token, int64_t v_stride_token, int64_t num_slots,
                           b200_stream_t stream);

/* The three steps AttentionLayer::forward runs before attention
 * (src/layers/attention_layer.cc:17-47), as one pass over the packed qkv rows
 * [tokens, (q_heads + 2*kv_heads)*head_dim]: optional per-head QK RMSNorm
 * (q_weight/k_weight NULL = none), NeoX RoPE, then the KV-pool store of the
 * rotated k and of v at out_loc.  q is rewritten in place; with
 * write_k_back != 0 the k rows are too (as the reference leaves them).
 * Rounding points match the unfused sequence (bf16 after the norm, bf16 after
 * the rotation). */
B200_API int b200_qknorm_rope_store(void* qkv, const void* q_weight, const void* k_weight,
                                    const float* cos_table, const float* sin_table,
                                    const int32_t* positions, const int32_t* out_loc,
                                    void* k_cache, void* v_cache, int tokens, int q_heads,
                                    int kv_heads, int head_dim, int max_pos, int64_t num_slots,
                                    float eps, int write_k_back, b200_stream_t stream);

/* ---- activation (include/sglang/layers/activation.h:8-11) ----------------- */

/* silu_and_mul / gelu_and_mul (src/layers/activation.cu:15-75):
 * out[t, j] = act(in[t, j]) * in[t, d + j]; in [tokens, 2*d], out [tokens, d]. */
B200_API int b200_silu_and_mul(void* out, const void* in, int tokens, int d, b200_stream_t stream);
B200_API int b200_gelu_and_mul(void* out, const void* in, int tokens, int d, b200_stream_t stream);

/* ---- embedding and index tables ------------------------------------------- */

/* torch::nn::Embedding as used by the models (src/models/qwen3.cc:38-43,56):
 * out[t, :] = table[ids[t], :].  ids int32; an id outside [0, vocab) writes a
 * zero row and records the index in the device status word. */
B200_API int b200_embedding(void* out, const void* table, const int32_t* ids, int tokens,
                            int hidden, int vocab, b200_stream_t stream);

/* gather_int32_2d (src/kernels/token_pool.cu:31-49,93-133):
 * out[i] = table[req[i], pos[i]], 0 when either index is out of range. */
B200_API int b200_gather_int32_2d(int32_t* out, const int32_t* table, int64_t rows, int64_t stride,
                                  int64_t cols, const int32_t* req_indices,
                                  const int32_t* positions, int64_t count, b200_stream_t stream);

/* write_token_pool (src/kernels/token_pool.cu:10-29,53-91):
 * table[req[i], pos[i]] = tokens[i], skipped when either index is out of range. */
B200_API int b200_write_token_pool(int32_t* table, int64_t rows, int64_t stride, int64_t cols,
                                   const int32_t* req_indices, const int32_t* positions,
                                   const int32_t* tokens, int64_t count, b200_stream_t stream);

/* ---- linear (include/sglang/layers/linear.h:7-73) -------------------------- */

enum {
    B200_EPILOGUE_NONE = 0,
    /* y[m, j] = silu(bf16(acc[m, j])) * bf16(acc[m, N/2 + j]), j < N/2: the
     * gate_up projection followed by silu_and_mul (src/models/utils.cc:41-57). */
    B200_EPILOGUE_SWIGLU = 1,
    B200_EPILOGUE_GEGLU = 2,     /* tanh-approximated GELU, as gelu_and_mul (src/layers/activation.cu:11-13) */
    B200_EPILOGUE_GEGLU_ERF = 3, /* exact GELU, as torch::gelu in MoELayer::forward (src/moe/moe.cc:80) */
    /* y[m, n] = max(acc[m, n], 0)^2, not gated: N outputs (no counterpart in the reference). */
    B200_EPILOGUE_RELU2 = 4,
    /* y[m, n] = gelu(acc[m, n]), exact, not gated: N outputs (no counterpart in the reference). */
    B200_EPILOGUE_GELU_ERF = 5,
    /* g = min(gate, limit), u = clamp(up, -limit, limit): y = g sigmoid(1.702 g) (u + 1); gated, with a
     * limit beside it (no counterpart in the reference). */
    B200_EPILOGUE_CLAMPED_SWIGLU = 6,
    /* the fp32 accumulator itself: y is float [M, N] (no counterpart in the reference). */
    B200_EPILOGUE_F32 = 7
};

/* LinearBase::forward (src/layers/linear.cc:24-26): y = x W^T (+ bias), bf16 in,
 * fp32 accumulate on the tcgen05 tensor cores, bf16 out.  x [M, K] with row
 * stride ldx, w [N, K] contiguous, y [M, N_out] contiguous where N_out = N (or
 * N/2 with a gated epilogue).  K must be a multiple of 64, N of 16. */
B200_API int b200_linear(void* y, const void* x, const void* w, const void* bias, int M, int N,
                         int K, int64_t ldx, int epilogue, b200_stream_t stream);

/* ---- mixture of experts (include/sglang/moe/moe.h:9-35) -------------------- */

/* Bytes of scratch b200_moe_forward needs (routing tables and the permuted activations). */
B200_API int64_t b200_moe_workspace_bytes(int tokens, int num_experts, int top_k, int hidden_size,
                                          int intermediate_size);

/* The routing half of MoELayer::forward (src/moe/moe.cc:47-55): fp32 softmax of bf16 router
 * logits [tokens, num_experts], top_k largest per token (lower expert index on ties), optional
 * renormalisation w / (sum w + 1e-8), weights rounded to bf16 as the reference casts them.
 * topk_ids int32 [tokens, top_k], topk_weights float [tokens, top_k], expert_counts int32
 * [num_experts + 1] (histogram; cleared by the call). */
B200_API int b200_moe_route(int32_t* topk_ids, float* topk_weights, int32_t* expert_counts,
                            const void* router_logits, int tokens, int num_experts, int top_k,
                            int renormalize, b200_stream_t stream);

/* MoELayer::forward (src/moe/moe.cc:36-96) for tp_size 1 (the caller all-reduces under TP):
 * out[t] = sum over the token's top_k experts e, in k order with bf16 accumulation, of
 * w[t,k] * down_e(act(gate_e x_t) * up_e x_t).  hidden_states / out bf16 [tokens, hidden_size];
 * gate_up_proj bf16 [E, 2*I, hidden]; down_proj bf16 [E, hidden, I]; activation 0 = silu,
 * 1 = gelu (exact, as torch::gelu).  No host synchronisation: six launches. */
B200_API int b200_moe_forward(void* out, const void* hidden_states, const void* router_logits,
                              const void* gate_up_proj, const void* down_proj, int tokens,
                              int num_experts, int top_k, int hidden_size, int intermediate_size,
                              int renormalize, int activation, void* workspace,
                              int64_t workspace_bytes, b200_stream_t stream);

/* One rank's share of MoELayer::forward under expert parallelism.  No counterpart in the
 * reference, whose MoELayer gives every rank a slice of every expert's intermediate dimension
 * (src/moe/moe.cc:12-30); here the rank holds whole experts [expert_begin, expert_begin +
 * num_local_experts) of the router's num_experts: gate_up_proj bf16 [num_local_experts, 2*I,
 * hidden], down_proj bf16 [num_local_experts, hidden, I].  Routing runs over all experts; only
 * the local experts' terms are summed into out (rows with none are zero); the all-reduce the
 * caller runs next (tensor_model_parallel_all_reduce, src/moe/moe.cc:92-94) adds the ranks. */
B200_API int b200_moe_forward_local(void* out, const void* hidden_states, const void* router_logits,
                                    const void* gate_up_proj, const void* down_proj, int tokens,
                                    int num_experts, int top_k, int hidden_size,
                                    int intermediate_size, int renormalize, int activation,
                                    int expert_begin, int num_local_experts, void* workspace,
                                    int64_t workspace_bytes, b200_stream_t stream);

/* ---- attention (include/sglang/attention/backend.h:24-41) ------------------ */

/* Bytes of scratch b200_attention_decode needs for up to max_batch requests
 * with q_heads / kv_heads local heads. */
B200_API int64_t b200_attention_decode_workspace_bytes(int max_batch, int q_heads, int kv_heads,
                                                       int head_dim);

/* FlashInferBackend::forward for a decode batch
 * (src/attention/flashinfer_backend.cu:553-595): out[b, h, :] = softmax(q[b, h]
 * . K_b^T / sqrt(d)) V_b over the seq_lens[b] keys whose KV-pool slots are
 * page_table[table_idx[b], 0 .. seq_lens[b]).  page_table holds one slot per
 * token position; page_size states that positions [j*page_size, (j+1)*page_size)
 * of a row are consecutive slots starting at a multiple of page_size (1 = no
 * such guarantee, as the reference Engine runs).  q [batch, q_heads, head_dim]
 * with strides; out [batch, q_heads*head_dim] contiguous.  k_cache / v_cache:
 * one layer's [num_slots, kv_heads, head_dim].  workspace: zero-initialised
 * once by the caller, then owned by the calls (they leave it zeroed where it
 * must be).  Split-KV is decided on the device; no host plan. */
B200_API int b200_attention_decode(void* out, const void* q, int64_t q_stride_token,
                                   int64_t q_stride_head, const void* k_cache, const void* v_cache,
                                   int64_t num_slots, const int32_t* page_table,
                                   int64_t page_table_stride, const int32_t* table_idx,
                                   const int32_t* seq_lens, int batch, int q_heads, int kv_heads,
                                   int head_dim, int page_size, float sm_scale, void* workspace,
                                   int64_t workspace_bytes, b200_stream_t stream);

/* No counterpart in the reference.  The same computation as b200_attention_decode for callers
 * that cannot allocate device memory when they need it (a process whose device-memory budget is
 * already owned by one pool, or a step loop that must not run into cudaMalloc's device-wide
 * synchronisation): there is no workspace argument, the split-KV scratch is an 8 MiB array built
 * into the library image (every GPU that loads the library carries it until exit).  The call makes
 * no cudaMalloc / cudaFree and no other allocating call.  Shapes whose partial results need more
 * than that array (see b200_attention_decode_workspace_bytes; 64 requests x 16 query heads need
 * under 2 MiB) are refused with B200_ERR_UNSUPPORTED.  The first call on a device looks up the
 * array's device address (cudaGetSymbolAddress) with that device current; make that first call
 * before any stream capture begins.  All calls share the one array and it keeps the previous
 * call's contents (the call clears the words that must start at zero): two calls whose kernels
 * overlap on the GPU race.  What the kernel reports (a wait that ran out, a page-table slot out of
 * range) goes to two words inside the same array, NOT to the words b200_read_device_status reads:
 * read them with b200_attention_decode_noalloc_status. */
B200_API int b200_attention_decode_noalloc(void* out, const void* q, int64_t q_stride_token,
                                           int64_t q_stride_head, const void* k_cache,
                                           const void* v_cache, int64_t num_slots,
                                           const int32_t* page_table, int64_t page_table_stride,
                                           const int32_t* table_idx, const int32_t* seq_lens,
                                           int batch, int q_heads, int kv_heads, int head_dim,
                                           int page_size, float sm_scale, b200_stream_t stream);

/* No counterpart in the reference.  Reads what the kernels of b200_attention_decode_noalloc reported
 * on the current device since the last read, after synchronising `stream`: out[0] = site of a wait
 * that ran out (0 = none), out[1] = offending slot + 1 of a page-table entry outside the pool (0 =
 * none; the kernel read slot 0 instead, nothing faulted).  Non-zero words are cleared by the read, so
 * a report survives later calls until somebody looks.  Allocates nothing. */
B200_API int b200_attention_decode_noalloc_status(int32_t out[2], b200_stream_t stream);

/* FlashInferBackend::forward for a prefill (extend) batch
 * (src/attention/flashinfer_backend.cu:596-678): causal attention of ragged
 * query rows against paged keys.  Request b owns query rows
 * [qo_indptr[b], qo_indptr[b+1]), which are the LAST extend positions of its
 * seq_lens[b] keys (the first seq_lens[b] - extend_len are the cached prefix).
 * max_extend_len bounds the longest request's extend length (grid sizing). */
B200_API int b200_attention_prefill(void* out, const void* q, int64_t q_stride_token,
                                    int64_t q_stride_head, const void* k_cache,
                                    const void* v_cache, int64_t num_slots,
                                    const int32_t* page_table, int64_t page_table_stride,
                                    const int32_t* table_idx, const int32_t* seq_lens,
                                    const int32_t* qo_indptr, int batch, int max_extend_len,
                                    int q_heads, int kv_heads, int head_dim, int page_size,
                                    float sm_scale, b200_stream_t stream);

/* ---- sampler (include/sglang/engine/engine.h:36-55) ------------------------- */

/* Sampler::sample, all-greedy branch (src/engine/engine.cc:294-298): argmax over
 * bf16 logits [rows, vocab] (row stride ld), first index on ties, int32 out. */
B200_API int b200_argmax(int32_t* out, const void* logits, int rows, int vocab, int64_t ld,
                         b200_stream_t stream);

/* Sampler::sample, stochastic branch (src/engine/engine.cc:299-338) with the candidate set of
 * sample_row (engine.cc:126-158): logits / temperature, keep the top_k largest, then drop sorted
 * entries whose inclusive cumulative probability exceeds top_p (never the first), renormalise and
 * draw.  bf16 logits [rows, vocab]; temperatures / top_k / top_p per row as Sampler::prepare
 * clamps them (top_k, top_p may be NULL = off; a row with temperature <= 1e-6 is greedy).  The
 * draw uses Philox keyed by seeds[row] (NULL = row index) and step_index, so it is reproducible;
 * the reference draws from torch's global generator instead.  candidate_mask (NULL or uint8
 * [rows, vocab]) receives 1 for every token of the final candidate set.  Ties are ordered by
 * index. */
B200_API int b200_sample(int32_t* out, const void* logits, int rows, int vocab, int64_t ld,
                         const float* temperatures, const int32_t* top_k, const float* top_p,
                         const uint64_t* seeds, uint64_t step_index, uint8_t* candidate_mask,
                         b200_stream_t stream);

/* flashinfer_sample_from_probs / _top_k_ / _top_p_ / _top_k_top_p_sample_from_probs
 * (include/sglang/engine/sampling.h:12-34; src/engine/sampling.cu:65-192): one token per row of
 * fp32 probabilities [rows, vocab] (contiguous), drawn with the caller's uniform number
 * uniform[row] in [0, 1) by inverse CDF over the tokens FlashInfer's rejection samplers accept:
 * those among the top_k largest probabilities (ties included) whose strictly larger probabilities
 * sum to less than top_p.  top_k / top_p: per-row device arrays, or NULL to use the scalar
 * (top_k_value < 1 or >= vocab and top_p_value >= 1 switch the filter off).  Always succeeds (the
 * reference's `success` flags are all true).  Reproducible: masses are summed in fixed point. */
B200_API int b200_sample_from_probs(int32_t* out, const float* probs, int rows, int vocab,
                                    const int32_t* top_k, int top_k_value, const float* top_p,
                                    float top_p_value, const float* uniform, b200_stream_t stream);

/* ---- latent attention, table routing, fp32 residual (no counterparts in the reference) --------- */

/* Attention in the latent space: every query row attends over one shared latent per token that serves
 * as key and value of all heads (the per-head up-projections are absorbed into the query before and
 * applied to the result after).  Row i sees keys [0, row_len[i]) of page-table row row_table[i]:
 *   out[i, h, :] = softmax_j(scale * q[i, h] . c_j) c_j.
 * q, out [rows, heads, width] contiguous; cache [num_slots, width]; width a multiple of 128.
 * dtype B200_DTYPE_*.  bf16 with width <= 512 runs split-KV on the tcgen05 tensor cores; everything else
 * on a plain kernel (as it does with plain != 0).  workspace: b200_latent_attention_workspace_bytes. */
B200_API int64_t b200_latent_attention_workspace_bytes(int rows, int heads, int width);
B200_API int b200_latent_attention(void* out, const void* q, const void* cache, int64_t num_slots,
                                   const int32_t* page_table, int64_t page_table_stride,
                                   const int32_t* row_table, const int32_t* row_len, int rows, int heads,
                                   int width, int page_size, float scale, int dtype, int plain,
                                   void* workspace, int64_t workspace_bytes, b200_stream_t stream);
/* The same where only the first out_width columns of a latent are averaged (out [rows, heads, out_width], a multiple
 * of 128): the others, a rotated part of the keys for instance, take part in the scores alone.  The tensor-core
 * kernel takes widths of up to 640 with up to 512 of them averaged. */
B200_API int b200_latent_attention_part(void* out, const void* q, const void* cache, int64_t num_slots,
                                        const int32_t* page_table, int64_t page_table_stride,
                                        const int32_t* row_table, const int32_t* row_len, int rows, int heads,
                                        int width, int out_width, int page_size, float scale, int dtype, int plain,
                                        void* workspace, int64_t workspace_bytes, b200_stream_t stream);

/* residual[t, :] += sum_k src_scale * src[src_rows[t * src_top + k], :]   (src NULL: nothing added;
 * src_rows NULL: row t; init != 0: the sum replaces the residual instead, e.g. an embedding lookup), then
 *   out = out_scale * residual / sqrt(mean(residual^2) + eps) * (weight + weight_offset)
 * to row t, or to the rows out_rows[t * out_top + k].  residual fp32 [tokens, padded]; src, weight, out of
 * `dtype`; the mean is over `width`, columns [width, padded) are zero and stay so.  padded % 64 == 0.
 * A src row outside [0, src_count) adds nothing and is reported in the device status word. */
B200_API int b200_residual_norm(void* out, const int32_t* out_rows, int out_top, float* residual,
                                const void* src, const int32_t* src_rows, int src_top, int64_t src_count,
                                float src_scale, int init, const void* weight, float weight_offset,
                                float out_scale, int tokens, int width, int padded, float eps, int dtype,
                                b200_stream_t stream);

/* Expert placement for a table of token id -> experts ([vocab, top] int32): counts[e] rows of expert e,
 * offsets[e] their first row (offsets[experts] = the total) and rows[t * top + k], the row of token t's
 * k-th expert in the expert-sorted order. */
B200_API int b200_table_route(int32_t* rows, int32_t* counts, int32_t* offsets, const int32_t* table,
                              const int32_t* token_ids, int tokens, int vocab, int top, int experts,
                              b200_stream_t stream);

/* One projection per head in one launch: y[m, h*N + n] = sum_k x[m, h*K + k] w[h*N + n, k] for
 * h < heads.  x [M, heads*K], y [M, heads*N] contiguous, w [heads*N, K]. */
B200_API int b200_linear_heads(void* y, const void* x, const void* w, int M, int heads, int N, int K,
                               b200_stream_t stream);

/* The fp32 counterparts of b200_linear / the grouped expert GEMM / b200_linear_heads, in true fp32 (no
 * tensor cores): y[m, n] over `groups` problems.  counts/offsets (device, [groups]) non-NULL: group g
 * multiplies rows [offsets[g], offsets[g] + counts[g]) of x; NULL and groups > 1: per-head columns as in
 * b200_linear_heads.  max_rows bounds M or any count. */
B200_API int b200_linear_f32(float* y, const float* x, const float* w, int max_rows, int N, int K,
                             int groups, const int32_t* counts, const int32_t* offsets, int epilogue,
                             b200_stream_t stream);

/* b200_linear without a bias in either dtype, with the epilogues that take a limit (act_limit). */
B200_API int b200_linear_act(void* y, const void* x, const void* w, int M, int N, int K, int epilogue,
                             float act_limit, int dtype, b200_stream_t stream);

/* The wiring with the norm on what a block returned (layer_norm below: the same with layer norms):
 *   a = sum_k src_weights[t, k] src[src_rows[t, k], :] + src2[t, :]   (src_rows NULL: src[t, :]; weights NULL: 1),
 *   residual[t, :] += a / sqrt(mean(a^2) + eps) * add_weight          (add_weight NULL: += a; init: = instead of +=),
 *   out[t, :] = residual, or its RMS norm with out_weight when there is one.
 * Shapes as b200_residual_norm; every row of out is the token's own. */
B200_API int b200_residual_post_norm(void* out, float* residual, const void* src, const int32_t* src_rows,
                                     const float* src_weights, int src_top, int64_t src_count, const void* src2,
                                     int init, const void* add_weight, const void* out_weight, int tokens,
                                     int width, int padded, float eps, int dtype, b200_stream_t stream);

/* With y -> (y - mean) / sqrt(mean squared deviation + eps) * weight + bias as the norm:
 *   a = sum_k src_weights[t, k] src[src_rows[t, k], :]   (a row of -1: the token's own row of `self` instead),
 *   residual[t, :] += norm(a; add_weight, add_bias)      (NULL: += a; init: = a * src_scale instead of +=),
 *   out[t, :] = norm(residual; out_weight, out_bias), or the residual without a weight. */
B200_API int b200_residual_layer_norm(void* out, float* residual, const void* src, const int32_t* src_rows,
                                      const float* src_weights, int src_top, int64_t src_count, const void* self,
                                      float src_scale, int init, const void* add_weight, const void* add_bias,
                                      const void* out_weight, const void* out_bias, int tokens, int width, int padded,
                                      float eps, int dtype, b200_stream_t stream);

enum { B200_SCORE_SIGMOID = 0, B200_SCORE_SOFTMAX = 1 };
/* Routing by scores of fp32 logits [tokens, logits_ld], one per expert and then one per identity expert.
 * B200_SCORE_SIGMOID: only experts of the best keep_groups of
 * `groups` equal groups (a group counts for the sum of its two best scores), the best `top` of those, weights =
 * scores over their sum (+ 1e-20) times scale.  B200_SCORE_SOFTMAX: groups (which count for their best) and experts
 * are chosen by softmax score + correction (fp32 per output, or NULL), weights = softmax scores times scale.  ids, weights,
 * rows [tokens, top]: the chosen experts and the row each choice has in the expert-sorted order, -1 for an identity
 * expert; counts [2 * experts] (the second half is scratch), offsets
 * [experts + 1]; the token's row of x (row_bytes) is copied to its rows of xp. */
B200_API int b200_score_route(int32_t* ids, float* weights, int32_t* rows, int32_t* counts, int32_t* offsets,
                              void* xp, const void* x, int row_bytes, const float* logits, int64_t logits_ld,
                              int tokens, int experts, int top, int groups, int keep_groups, float scale,
                              int score, int identity_experts, const float* correction, b200_stream_t stream);

/* What lies between the joint projection of an attention layer and the attention: joint [tokens, joint_ld]
 * holds [heads * padded_dim | kv_heads * padded_dim | kv_heads * padded_value_dim | ...].  Queries (in place)
 * and keys (to k_cache [num_slots, kv_heads, padded_dim]) are RMS-normalised over `dim` with q_norm / k_norm
 * (NULL: not; unit_norm: without a weight), then element i of the first rotary_dim turns with element i + rotary_dim / 2.
 * Values go to v_cache; mix 1 keeps a copy in first_values, mix 2 stores (1 - lambda) v + lambda first_values.
 * value_rotary > 0: element i of the first value_rotary of a value turns with element i + value_rotary / 2. */
typedef struct b200_head_prepare_args {
    void* joint;
    int64_t joint_ld;
    int32_t tokens, heads, kv_heads, dim, padded_dim, padded_value_dim;
    const void *q_norm, *k_norm;
    float eps;
    int32_t rotary_dim, max_pos;
    const float *cos_table, *sin_table;   /* [max_pos, rotary_dim / 2] */
    const int32_t *positions, *out_loc;
    void *k_cache, *v_cache;
    int64_t num_slots;
    int32_t mix;
    const float* lambda;                  /* device */
    void* first_values;                   /* [tokens, kv_heads, padded_value_dim] */
    int32_t unit_norm, value_rotary;
    const float *value_cos, *value_sin;   /* [max_pos, value_rotary / 2] */
} b200_head_prepare_args;
B200_API int b200_head_prepare(const b200_head_prepare_args* args, int dtype, b200_stream_t stream);

/* Paged grouped-query attention through a window: the query at position i sees key j <= i if i - j < window or
 * j < keep_first.  out[t, h, :] = softmax(scale * q k) v, times sigmoid(gate[t, h, :]) when there is a gate.
 * q: heads padded_dim apart; out [tokens, heads, padded_value_dim].  Requests by table_idx / seq_lens /
 * qo_indptr (decode != 0: one token each), and per token its page-table row and the keys it could see without
 * a window (row_table, row_len).  bf16 with both paddings 128 runs on the tensor-core kernels where they take
 * the head counts, everything else (or plain != 0) on a plain kernel.
 * workspace: b200_attention_decode_workspace_bytes, or any 16 bytes where that refuses the head counts. */
typedef struct b200_window_attention_args {
    void* out;
    const void* q;
    int64_t q_stride;
    const void *k_cache, *v_cache;
    int64_t num_slots;
    const int32_t* page_table;
    int64_t page_table_stride;
    const int32_t *table_idx, *seq_lens, *qo_indptr, *row_table, *row_len;
    int32_t tokens, batch, max_extend, decode, plain;
    int32_t heads, kv_heads, padded_dim, padded_value_dim, page_size;
    float scale;
    int32_t window, keep_first;
    const void* gate;
    int64_t gate_stride;
    void* workspace;
    int64_t workspace_bytes;
    int32_t chunk;           /* > 0, instead of the window: key j is seen if i / chunk = j / chunk */
    const float* sinks;      /* [heads] or NULL: exp(sinks[h]) joins the softmax's denominator */
    int32_t gate_per_head;   /* the gate is [tokens, heads]: one number per head */
    float out_scale;         /* a factor on the output; 0 means 1 */
    int64_t out_stride;      /* token stride of out in elements; 0: dense */
    /* Heads that mix their weights: with p_g the softmax weights of head g, head h applies sum_g head_mix[h, g] p_g to
     * the values of its own key / value head.  value_rotary > 0: the result at position p is then turned back by p,
     * element i of the first value_rotary with element i + value_rotary / 2, before the gate.  No sinks. */
    const float* head_mix;   /* [heads, heads] or NULL */
    int32_t value_rotary, max_pos;
    const float *value_cos, *value_sin;   /* [max_pos, value_rotary / 2] */
    const int32_t* positions;             /* [tokens] */
    float score_bound;       /* no q . k is larger than this; 0: not known.  (A bound lets the tensor-core kernels of mixing
                                heads run without a running maximum; without one the plain kernel is used.) */
    void* mix_scratch;       /* b200_head_mix_scratch_bytes */
} b200_window_attention_args;
/* Per (token, head), what the head's weights make of the values of every key / value head. */
B200_API int64_t b200_head_mix_scratch_bytes(int tokens, int heads, int kv_heads, int padded_value_dim, int dtype);
/* The workspace of mixing heads instead of b200_attention_decode_workspace_bytes. */
B200_API int64_t b200_head_mix_workspace_bytes(int max_batch, int heads, int kv_heads);
B200_API int b200_window_attention(const b200_window_attention_args* args, int dtype, b200_stream_t stream);

/* Gated linear attention with one decay per key channel.  Per head, with state S [dim, value dim]:
 *   S <- diag(alpha) S + k v^T,   o = S^T (q * q_scale),   alpha = sigmoid(z)^(1 / tau),
 *   z = a up^T + bias for the low-rank row a that the joint projection returns,
 * and out = o / sqrt(mean(o^2) + eps) * norm * silu(gate) per head.  joint [tokens, joint_ld] holds
 * [q | k: heads * padded_dim each | v | gate: heads * padded_value_dim each | a: padded rank]; up
 * [heads * padded_dim, up_ld] of the dtype, bias fp32 [heads * padded_dim].  state fp32 [rows, heads, padded_dim,
 * padded_value_dim]: row table_idx[b] belongs to request b, whose tokens are [qo_indptr[b], qo_indptr[b + 1])
 * and whose first token has position cached[b]; a request that starts at position 0 starts from zeros.
 * decode != 0: every request brings one token.  plain != 0: never the chunked tensor-core kernel. */
typedef struct b200_linear_attention_args {
    void* out;
    const void* joint;
    int64_t joint_ld;
    int32_t tokens, batch, decode, plain;
    const int32_t *table_idx, *cached, *qo_indptr;
    float* state;
    int32_t heads, dim, padded_dim, value_dim, padded_value_dim, rank, up_ld;
    const void* up;
    const float* bias;
    const void* norm;
    float tau, eps, q_scale;
} b200_linear_attention_args;
B200_API int b200_linear_attention(const b200_linear_attention_args* args, int dtype, b200_stream_t stream);

/* Recurrences with one decay per head, the first two behind a short causal convolution.  joint [tokens, joint_ld] holds
 * [gate | v: heads * padded_value_dim each | k | q: kv_heads * padded_dim each | a of every head (none for lightning),
 * and for the delta rule and the matrix memory b of every head]; head h uses k / q head h / (heads / kv_heads).
 *   v, k, q <- silu(conv(.) + conv_bias): conv [taps, channels] per channel of [v | k | q], the last tap the
 *   current token's; conv_state [rows, taps, channels] of the dtype keeps the last inputs, that of position p at
 *   p mod taps
 * B200_RULE_STATE_SPACE:  dt = softplus(a + step_bias), g = exp(-exp(decay_log) dt)
 *   S <- g S + dt k v^T,  o = S^T q + skip * v,  out = rms(o * silu(gate)) * norm in norm_groups equal parts of the
 *   concatenated (true) heads; norm [heads * padded_value_dim]
 * B200_RULE_DELTA:  g = exp(-exp(decay_log) softplus(a + step_bias)), beta = sigmoid(b); k and q divided by
 *   sqrt(sum of squares + 1e-6), q also by sqrt(dim)
 *   S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q,  out = rms(o) * norm * silu(gate) per head; norm
 *   [padded_value_dim]
 * B200_RULE_LIGHTNING: v, k, q <- silu(.), g = exp(decay_log)
 *   S <- g S + k v^T,  o = S^T q,  out = rms(o) * norm * sigmoid(gate) in norm_groups parts as above
 * B200_RULE_MATRIX_MEMORY: v, k as they are, q / sqrt(dim); i = c tanh((a + step_bias[h]) / c),
 *   f = log sigmoid(c tanh((b + step_bias[heads + h]) / c)) with c = gate_cap; from S = 0, n = 0, m = 0
 *   m' = max(f + m, i),  S <- exp(f + m - m') S + exp(i - m') k v^T,  n likewise with k alone,  m <- m'
 *   o = S^T q / (max(|n . q|, exp(-m)) + 1e-6),  out = rms(o) * norm * sigmoid(gate) in norm_groups parts;
 *   memory fp32 [rows, heads, b200_recurrence_memory_bytes / 4] holds n and m
 * out [tokens, out_ld] is also multiplied by out_scale.  state fp32 [rows, heads, padded_dim, padded_value_dim];
 * rows, requests, decode and plain as for b200_linear_attention; a request brings at most max_extend tokens.  conv,
 * conv_bias (NULL: 0), decay_log, step_bias, skip are fp32.  Scratch: b200_recurrence_scratch. */
enum { B200_RULE_STATE_SPACE = 0, B200_RULE_DELTA = 1, B200_RULE_LIGHTNING = 2, B200_RULE_MATRIX_MEMORY = 3 };
typedef struct b200_recurrence_args {
    void* out;
    int64_t out_ld;
    const void* joint;
    int64_t joint_ld;
    int32_t rule, tokens, batch, max_extend, decode, plain;
    const int32_t *table_idx, *cached, *qo_indptr;
    float* state;
    void* conv_state;
    int32_t heads, kv_heads, dim, padded_dim, value_dim, padded_value_dim, taps, norm_groups;
    const float *conv, *conv_bias, *decay_log, *step_bias, *skip;
    const void* norm;
    float eps, out_scale;
    void* mixed;       /* [tokens, channels] of the dtype */
    float* steps;      /* [tokens, heads, 2]: log2 of the decay, weight of what is written (matrix memory: its log2) */
    float* units;      /* delta rule [tokens, 2 kv_heads]: factors that make k and q unit vectors; matrix memory
                          [tokens, heads]: what a chunk's tokens add to n . q */
    void* chunks;      /* per 64 tokens and head: matrices of the chunked kernel */
    float gate_cap;    /* matrix memory */
    float* memory;
} b200_recurrence_args;
B200_API int b200_recurrence(const b200_recurrence_args* args, int dtype, b200_stream_t stream);
/* Bytes per head of the matrix memory's n and m (one copy for every group of value columns that a CTA may work on). */
B200_API int64_t b200_recurrence_memory_bytes(int padded_dim, int padded_value_dim);
/* Bytes of mixed, steps, units and chunks for steps of at most max_tokens tokens of max_batch requests. */
B200_API int b200_recurrence_scratch(int rule, int max_tokens, int max_batch, int heads, int kv_heads, int padded_dim,
                                     int padded_value_dim, int dtype, int64_t* bytes);

/* residual_post_norm where what is added is the sum of two rows per token, each RMS-normalised with its own weight,
 * times pair_scale. */
B200_API int b200_residual_pair_norm(void* out, float* residual, const void* src, const void* src2,
                                     const void* weight, const void* weight2, float pair_scale, const void* add_weight,
                                     const void* out_weight, int tokens, int width, int padded, float eps, int dtype,
                                     b200_stream_t stream);

/* The first `dims` elements of every head of x [tokens, heads, ld] rotated in place, element 2i with its
 * neighbour, by the angles whose cosines and sines are in the tables [max_pos, dims / 2]. */
B200_API int b200_rotate_pairs(void* x, int tokens, int heads, int ld, int dims, const float* cos_table,
                               const float* sin_table, const int32_t* positions, int max_pos, int dtype,
                               b200_stream_t stream);

/* ---- tensor-parallel all-reduce (include/sglang/distributed/distributed.h:24) --- */

/* One process per GPU.  A communicator owns this rank's two exchange buffers (call parity 0 / 1)
 * of buffer_bytes each and a flag table, in device memory that the peers map through CUDA IPC.
 * Set-up (the part the reference does with an NCCL unique id, src/distributed/distributed.cc:
 * 142-173): every rank creates, exports its 64-byte handle, the host code gathers all handles
 * in rank order (torch.distributed / MPI / a file), every rank connects. */
typedef struct b200_comm b200_comm;
B200_API int b200_comm_create(int rank, int world, int64_t buffer_bytes, b200_comm** out);
B200_API int b200_comm_handle_bytes(void);
B200_API int b200_comm_export(b200_comm* comm, void* handle_out);
B200_API int b200_comm_connect(b200_comm* comm, const void* all_handles);
/* The same communicator over memory the host obtained elsewhere (a symmetric allocation): region =
 * this rank's block of b200_comm_region_bytes(buffer_bytes) zeroed bytes, 256-byte aligned;
 * peer_regions[world] = every rank's block as this process addresses it; multicast_region = the
 * NVLink multicast address of the blocks, or NULL.  With a multicast address the all-reduce is
 * summed inside the switch (multimem.ld_reduce) and delivered with one store (multimem.st); the
 * order of the additions is then the switch's, not rank order.  The memory stays the caller's. */
B200_API int64_t b200_comm_region_bytes(int64_t buffer_bytes);
B200_API int b200_comm_create_on(int rank, int world, int64_t buffer_bytes, void* region, b200_comm** out);
B200_API int b200_comm_connect_pointers(b200_comm* comm, const void* const* peer_regions,
                                        const void* multicast_region);
B200_API int b200_comm_uses_multicast(b200_comm* comm);
/* Device address of this rank's exchange buffer for the given parity: the producer of the
 * partial sum (the row-parallel GEMM) writes there. */
B200_API void* b200_comm_buffer(b200_comm* comm, int parity);
B200_API int b200_comm_destroy(b200_comm* comm);
/* The longest one kernel waits for its peers' announcement before it gives up, leaves its outputs
 * untouched and reports through the device status words (sites 401-403).  Default 2 s; the
 * reference's only time-out is the NCCL rendezvous (src/distributed/distributed.cc:106-120,145). */
B200_API int b200_comm_set_wait_limit_ns(b200_comm* comm, uint64_t nanoseconds);
/* Failure-path testing on ONE GPU, no counterpart in the reference: instead of b200_comm_connect,
 * map every peer onto this rank's own buffers.  A peer's announcement then never arrives by
 * itself, so a call runs into the wait limit and returns — unless the host plays the peers' part
 * first with b200_comm_loopback_announce(call_number), call numbers counting from 1 per
 * communicator (failed calls count too).  The all-reduce of such a communicator returns
 * world x this rank's partial. */
B200_API int b200_comm_connect_loopback(b200_comm* comm);
B200_API int b200_comm_loopback_announce(b200_comm* comm, uint32_t call_number, b200_stream_t stream);

/* tensor_model_parallel_all_reduce (src/distributed/distributed.cc:205-226): out[rows, hidden]
 * = bf16(sum over ranks, in rank order, fp32) of the partials in the exchange buffers of
 * `parity`.  One-shot: every rank reads every peer's partial over NVLink with plain loads.
 * Successive calls must alternate parity.  The wait for the peers is bounded; a time-out is
 * reported through the device status words. */
B200_API int b200_allreduce(b200_comm* comm, int parity, void* out, int rows, int hidden,
                            b200_stream_t stream);
/* The all-reduce above fused with the RMSNorm::fused_add_forward_inplace that the models run on
 * its result (src/models/qwen3.cc:24,31; src/layers/linear.cc:52-55,73-76):
 * residual <- bf16(all-reduce) + residual; x_out <- rmsnorm(sum) * weight. */
B200_API int b200_allreduce_fused_add_rmsnorm(b200_comm* comm, int parity, void* x_out,
                                              void* residual, const void* weight, int rows,
                                              int hidden, float eps, int round_sum_first,
                                              b200_stream_t stream);

/* ---- step runner (include/sglang/engine/engine.h:57-103) -------------------- */

/* The fields of ModelConfig the forward pass reads (include/sglang/models/config.h:15-42). */
typedef struct b200_model_config {
    int32_t num_layers;
    int32_t hidden_size;
    int32_t num_qo_heads;
    int32_t num_kv_heads;
    int32_t head_dim;
    int32_t intermediate_size;
    int32_t vocab_size;
    float rms_norm_eps;
    float rope_theta;
    int32_t max_position;
    int32_t tie_word_embeddings;
    int32_t qk_norm;        /* per-head q/k RMSNorm (Qwen3, Qwen3-MoE) */
    int32_t fused_residual; /* 1: Qwen3 wiring (src/models/qwen3.cc:21-35); 0: Llama wiring (src/models/llama.cc:15-29) */
    int32_t attention_bias; /* qkv bias (Qwen2) */
    int32_t hidden_act;     /* 0 = silu, 1 = gelu */
    int32_t num_experts;    /* 0 = dense MLP */
    int32_t num_experts_per_tok;
    int32_t moe_intermediate_size;
    int32_t norm_topk_prob;
} b200_model_config;

/* The fields of EngineConfig that size device state (include/sglang/engine/config.h:13-32). */
typedef struct b200_engine_config {
    int32_t page_size;         /* tokens per KV page (the reference Engine runs 1) */
    int32_t num_pages;         /* usable pages; one more is allocated as the dummy page */
    int32_t max_running_req;   /* page-table rows; row max_running_req is the dummy request's */
    int32_t max_seq_len;
    int32_t max_extend_tokens; /* most tokens one prefill step may carry */
    int32_t tp_rank;
    int32_t tp_size;
    int32_t expert_parallel;   /* MoE models under tp_size > 1: 0 = every rank holds a slice of every
                                  expert's intermediate dimension (the reference's layout), 1 = rank r
                                  holds whole experts [r*E/tp, (r+1)*E/tp) */
} b200_engine_config;

enum { B200_PHASE_PREFILL = 0, B200_PHASE_DECODE = 1 };

/* One scheduler step, as Scheduler::prepare_batch describes it on the host
 * (src/scheduler/scheduler.cc:275-358): all arrays are HOST memory and are copied
 * by the call.  Requests [num_reqs, num_padded_reqs) are padding (the dummy
 * request of GraphRunner::pad_batch, src/engine/engine.cc:628-645). */
typedef struct b200_step {
    int32_t phase;
    int32_t num_reqs;
    int32_t num_padded_reqs;
    const int32_t* table_idx;   /* [num_padded_reqs] page-table row (Req::table_idx) */
    const int32_t* cached_lens; /* [num_padded_reqs] keys already in the pool (Req::cached_len) */
    const int32_t* extend_lens; /* [num_padded_reqs] tokens run this step (Req::extend_len; 1 in decode) */
    const int32_t* write_pos;   /* [num_reqs] token-pool column that receives the sampled token, < 0 = none */
    const float* temperatures;  /* [num_reqs] or NULL = every request greedy (BatchSamplingArgs, engine.h:22-26) */
    const int32_t* top_k;       /* [num_reqs] or NULL */
    const float* top_p;         /* [num_reqs] or NULL */
    const uint64_t* seeds;      /* [num_reqs] or NULL: per-request RNG seed (no counterpart in the reference) */
    uint64_t step_index;        /* offsets the per-request random stream */
} b200_step;

typedef struct b200_engine b200_engine;

/* Models whose layers are listed one by one (no counterpart in the reference, whose models repeat one
 * layer): every layer names its mixer and its feed-forward with their own sizes.  The residual stream
 * of such a model is fp32.  All matrices are stored [out, in] with both sides padded with zeros to a
 * multiple of 64 (b200_pad_width; head and value dimensions up to 128 are padded to 128, latent widths
 * to a multiple of 128), vectors likewise; norms divide by the true width. */
enum { B200_DTYPE_BF16 = 0, B200_DTYPE_F32 = 1 };
enum {
    B200_MIXER_LATENT_ATTENTION = 0,
    B200_MIXER_WINDOW_ATTENTION = 1,
    B200_MIXER_LINEAR_ATTENTION = 2,
    B200_MIXER_STATE_SPACE = 3,   /* b200_recurrence, either rule */
    B200_MIXER_DELTA_RULE = 4,
    B200_MIXER_LIGHTNING = 5,     /* b200_recurrence as well */
    B200_MIXER_MATRIX_MEMORY = 6
};
/* Norms on queries and keys: none, RMS norms with a weight, or division by the root mean square alone. */
enum { B200_HEAD_NORM_NONE = 0, B200_HEAD_NORM_WEIGHTED = 1, B200_HEAD_NORM_UNIT = 2 };
enum { B200_GATE_NONE = 0, B200_GATE_ELEMENT = 1, B200_GATE_HEAD = 2 };
/* How the outputs of two mixers side by side become one. */
enum {
    B200_JOIN_SUM = 0,      /* added, each times its out_scale, by one output projection */
    B200_JOIN_NORMED = 1    /* each RMS-normalised with its own weight, then half of their sum */
};
enum { B200_NORM_INPUT = 0, B200_NORM_OUTPUT = 1, B200_NORM_BOTH = 2 };
/* The norms around blocks and before the output head: RMS norms, or layer norms with a weight and a bias. */
enum { B200_NORM_RMS = 0, B200_NORM_LAYER = 1 };
enum { B200_MLP_NONE = 0, B200_MLP_DENSE = 1, B200_MLP_TABLE_MOE = 2, B200_MLP_SCORED_MOE = 3 };

typedef struct b200_layer_config {
    int32_t mixer;         /* B200_MIXER_* */
    int32_t heads;
    int32_t head_dim;      /* query / key dimensions per head */
    int32_t value_dim;
    int32_t q_rank;        /* latent attention: width of the query latent */
    int32_t kv_rank;       /* latent attention: width of the key / value latent, what the cache holds per token */
    float score_scale;
    int32_t mlp;           /* B200_MLP_* */
    int32_t intermediate;  /* of the dense layer, or of each expert */
    int32_t epilogue;      /* B200_EPILOGUE_*: what is between the up and the down projection; a gated one
                              has gate and up stacked in "mlp_up" */
    int32_t num_experts;
    int32_t experts_per_tok; /* table: width of the token-id -> experts table, each chosen expert weighs 1 / that;
                                scored: experts with the largest scores */
    /* window attention */
    int32_t kv_heads;
    int32_t window;          /* the query at position i sees key j <= i if i - j < window ... */
    int32_t keep_first;      /* ... or j < keep_first */
    int32_t rotary_dim;
    double rope_base;
    int32_t value_mix;       /* values mixed with those of the first layer that has this set */
    /* linear attention */
    int32_t decay_rank;
    float decay_tau;
    /* scored experts */
    int32_t router_groups;
    int32_t router_keep;     /* groups whose experts can be chosen */
    float router_scale;
    int32_t shared_intermediate; /* of the expert every token uses; 0: none */
    /* limits of B200_EPILOGUE_CLAMPED_SWIGLU */
    float act_limit;
    float shared_act_limit;
    /* window attention */
    int32_t head_norm;       /* B200_HEAD_NORM_* on queries and keys */
    int32_t gate;            /* B200_GATE_* on the output */
    int32_t qkv_bias;
    int32_t sink;            /* a score per head that joins the softmax's denominator */
    int32_t chunk;           /* > 0, instead of the window: keys of the query's own chunk of the sequence */
    /* rotations (latent attention: of the rotary_dim key dimensions that all heads share, in neighbouring pairs):
     * frequencies divided by rope_factor where their wavelength exceeds rope_original / rope_low, kept below
     * rope_original / rope_high, blended between; rope_original 0: all of them divided; factor 0: none */
    double rope_factor, rope_low, rope_high, rope_original;
    int32_t kv_from;         /* latent and window attention: the layer whose cache this one reads, -1: its own */
    /* recurrences (head_dim: state rows; kv_heads: heads of k and q) */
    int32_t conv_taps;
    int32_t norm_groups;
    /* a second mixer that reads the same input */
    int32_t beside;          /* index into the stack's `beside`, -1: none */
    int32_t join;            /* B200_JOIN_* */
    float out_scale;         /* of this mixer's output (window attention, recurrences) */
    /* window attention */
    int32_t value_rotary;    /* cached values are rotated by their position over all of value_dim (base rope_base, no
                                stretching), and what a query at position i gets out is turned back by i */
    int32_t head_mix;        /* the softmax weights of every head become a sum over all heads' weights */
    /* matrix memory */
    float gate_cap;
    /* scored experts */
    int32_t score;           /* B200_SCORE_* */
    int32_t identity_experts; /* the last outputs of the router: experts that return their input */
} b200_layer_config;

typedef struct b200_stack_config {
    int32_t num_layers;
    const b200_layer_config* layers;
    int32_t dtype;       /* B200_DTYPE_*: bf16 matrices and activations, or everything in fp32 */
    float norm_offset;   /* added to the stored weights of the layer norms and the final norm (0 or 1) */
    float logit_scale;
    int32_t norm_output; /* B200_NORM_*: blocks read the normalised residual; or they read the residual, and what
                            they return is normalised before it is added; or both */
    int32_t num_beside;
    const b200_layer_config* beside;   /* mixers that run beside another one (only mixer fields are read) */
    int32_t norm_kind;   /* B200_NORM_RMS or B200_NORM_LAYER */
    float embed_scale;   /* a factor on the embedding rows; 0 means 1 */
} b200_stack_config;

/* The padded size of a width / of a per-head dimension / of a latent width (see above). */
B200_API int b200_pad_width(int n);
B200_API int b200_pad_head_dim(int n);
B200_API int b200_pad_latent(int n);
/* The column where the rotated part of a latent row starts (latents with one are kv_rank numbers, padding up to
 * there, and the rotated part, padded as a whole). */
B200_API int b200_latent_rope_at(int kv_rank);

/* Engine::Engine (src/engine/engine.cc:412-489): allocates weights (uninitialised), the KV
 * pool [2, L, (num_pages+1)*page_size, kv_heads/tp, head_dim], the page table and token pool
 * [max_running_req+1, align32(max_seq_len)] (dummy row filled with slot num_pages*page_size),
 * RoPE tables and activation buffers on the current device. */
B200_API int b200_engine_create(const b200_model_config* model, const b200_engine_config* config,
                                b200_engine** out);
/* The same for a model whose layers are listed one by one; of `model` only num_layers, hidden_size,
 * vocab_size, rms_norm_eps and tie_word_embeddings are read.  Per layer a latent pool
 * [(num_pages+1)*page_size, pad(kv_rank)], a K and a V pool, or a state per table row.  tp_size must be 1. */
B200_API int b200_engine_create_stack(const b200_model_config* model, const b200_stack_config* stack,
                                      const b200_engine_config* config, b200_engine** out);
B200_API int b200_engine_destroy(b200_engine* engine);

/* Device address and size of a named tensor: "embed", "lm_head", "final_norm", "rope_cos",
 * "rope_sin", "page_table", "token_pool", "kv_cache", "logits", "next_tokens", and per layer
 * "qkv", "qkv_bias", "o", "gate_up", "down", "input_norm", "post_norm", "q_norm", "k_norm",
 * "router", "experts_gate_up", "experts_down" (layouts: src/models/weight_loader.cc:27-33,455,497).
 * Layer stacks: per layer "norm1", "norm2", "down_qkv" [q latent + kv latent, hidden], "q_latent_norm",
 * "kv_latent_norm", "uq" [heads*dim, q latent], "uk" [heads*dim, kv latent], "uk_absorb" (per head the
 * transpose of its rows of uk: [heads, kv latent, dim]), "uv" [heads*vdim, kv latent], "o"
 * [hidden, heads*vdim], "mlp_up", "mlp_down" (experts stacked), "expert_table" int32 [vocab, experts
 * per token], "latent_cache".  Window attention: "qkvg" [heads*dim + kv_heads*dim + kv_heads*vdim + heads*vdim,
 * hidden], "q_head_norm", "k_head_norm" [dim], "value_mix" (one float), "o", "k_cache", "v_cache".  Linear
 * attention (dimensions padded to a multiple of 64): "qkvga" [2 heads*dim + 2 heads*vdim + rank, hidden],
 * "decay_up" [heads*dim, rank padded to 16], "decay_bias" fp32 [heads*dim], "head_norm" [vdim], "o",
 * "state" fp32 [max_running_req + 1, heads, dim, vdim].  Recurrences (dimensions padded the same way): "recurrence"
 * [the columns of b200_recurrence's joint rows, hidden], "conv" [taps, channels], "conv_bias" [channels], "decay_log",
 * "step_bias", "skip" [heads], all fp32, "head_norm", "o", "state", "conv_state".  Optional: "joint_bias" of the
 * input projection, "sinks" fp32 [heads], "norm1_out", "norm2_out".  Two mixers side by side share the input
 * projection "joint" [left columns + right columns, hidden], and under B200_JOIN_SUM "o" [hidden, left + right];
 * under B200_JOIN_NORMED there are "side_norm" [hidden] and the right one's "beside_o", "beside_side_norm".  The names
 * of the right one's other tensors start with "beside_".  Scored experts: "router" [experts, hidden],
 * "mlp_up", "mlp_down", "shared_up", "shared_down", and with B200_SCORE_SOFTMAX "router_correction" fp32.  Layer norms
 * add "norm1_bias", "norm2_bias", "norm1_out_bias", "norm2_out_bias" and "final_norm_bias".  "head_mix" fp32 [heads,
 * heads] (also, as the identity, where only the values are rotated); "memory" fp32, see b200_recurrence. */
B200_API int b200_engine_tensor(b200_engine* engine, const char* name, int layer, void** device_ptr,
                                int64_t* nbytes);
/* Synchronous host-to-device copy into a named tensor (nbytes must equal its size). */
B200_API int b200_engine_load(b200_engine* engine, const char* name, int layer, const void* host,
                              int64_t nbytes);

/* CacheManager::write_page_table / the token-pool fill (src/scheduler/prefill.cc:144-187):
 * table[rows[i], positions[i]] = values[i] from host arrays; which = 0 page table, 1 token pool. */
B200_API int b200_engine_write_table(b200_engine* engine, int which, const int32_t* rows,
                                     const int32_t* positions, const int32_t* values, int64_t count);

/* GraphRunner::capture_graphs (src/engine/engine.cc:670-730): captures CUDA graphs per padded decode
 * batch size — one that ends in argmax and one that ends in the sampling kernel (the reference
 * samples outside its graph, src/engine/engine.cc:504-523; here the sampling parameters and the
 * step index live in device memory, so the sampled step replays too).  batch_sizes NULL or count 0:
 * the reference's default list 1, 2, 4, 8, 16, ... and max_running_req (determine_batch_sizes,
 * :592-616).  A later decode step runs at the smallest captured size >= its num_padded_reqs
 * (GraphRunner::pad_batch, :628-645): the step runner adds dummy-request rows itself. */
B200_API int b200_engine_capture_graphs(b200_engine* engine, const int32_t* batch_sizes, int count);

/* Engine::forward_batch (src/engine/engine.cc:495-544) together with the device half of
 * Scheduler::prepare_batch (scheduler.cc:329-334: out_loc / input_ids gathers) and the token
 * write-back (scheduler.cc:403-412).  Asynchronous: next_tokens_host [num_reqs] (pinned memory
 * recommended) is valid after b200_engine_synchronize (ForwardOutput::synchronize). */
B200_API int b200_engine_step(b200_engine* engine, const b200_step* step, int32_t* next_tokens_host);
B200_API int b200_engine_synchronize(b200_engine* engine);

/* The same step reporting through the engine's result ring instead of a device-to-host copy and a
 * stream synchronisation: what ForwardOutput's pinned tensor + event (src/engine/engine.cc:526-531)
 * and the scheduler's per-request finish test (src/scheduler/scheduler.cc:449-455) are in the
 * reference.  The step's last kernel writes, into pinned host memory, the sampled tokens, one finish
 * flag per request (1 when write_pos[i] < 0, i.e. the request cannot decode further, or when the
 * token equals the end-of-sequence id and ignore_eos[i] is 0; a chunked prefill request also has
 * write_pos < 0 and its flag, like its token, means nothing), and the device status words.
 * b200_engine_wait blocks on that step's own event only - steps enqueued behind it keep running -
 * and returns pointers into the slot, valid until b200_engine_result_slots() further steps have
 * been enqueued; a ticket older than that is refused.  Its return code is the step's:
 * B200_ERR_TIMEOUT / B200_ERR_INVALID_ARGUMENT as b200_engine_synchronize reports them.
 * ignore_eos: [num_reqs] or NULL (nobody ignores).  b200_engine_set_eos_token: Engine::eos_token_id
 * (include/sglang/engine/engine.h:71); negative (the default) = the model has none. */
B200_API int b200_engine_set_eos_token(b200_engine* engine, int32_t eos_token_id);
B200_API int b200_engine_result_slots(void);
B200_API int b200_engine_step_async(b200_engine* engine, const b200_step* step, const uint8_t* ignore_eos,
                                    int64_t* ticket);
B200_API int b200_engine_wait(b200_engine* engine, int64_t ticket, const int32_t** tokens,
                              const uint8_t** finished);

/* Copies the logits [rows, vocab] of the last step to host memory (synchronous): bf16, or fp32 for a
 * layer stack that runs in fp32. */
B200_API int b200_engine_read_logits(b200_engine* engine, void* host, int rows);

/* Logits at any tokens of the last step, not only each request's last one (scoring a prompt): the final
 * hidden states stay on the device until the next step, and this applies the output head to the rows
 * `tokens` (HOST int32, places in the step's flattened token order) in slabs and copies fp32 logits
 * [count, vocab] to host memory.  Synchronous.  No counterpart in the reference. */
B200_API int b200_engine_token_logits(b200_engine* engine, const int32_t* tokens, int count, float* host);

/* Tests: from the next step on, layer stacks copy the fp32 residual stream after every layer to host
 * memory [num_layers, tokens of the step, hidden] (prefill steps only); NULL turns it off. */
B200_API int b200_engine_trace_residual(b200_engine* engine, float* host);

/* Tensor parallelism (engine created with tp_size > 1): export this rank's IPC handle
 * (b200_comm_handle_bytes bytes) and connect to all ranks' handles before the first step. */
B200_API int b200_engine_comm_export(b200_engine* engine, void* handle_out);
B200_API int b200_engine_comm_connect(b200_engine* engine, const void* all_handles);
/* The same over memory the host obtained elsewhere - a symmetric allocation whose peer addresses,
 * and the NVLink multicast address of the whole group where the fabric has one, the host already
 * knows (torch.distributed's symmetric memory in the tests; no counterpart in the reference, whose
 * all-reduce is NCCL's).  region: this rank's block of b200_engine_comm_region_bytes() zeroed bytes,
 * 256-byte aligned; peer_regions[tp_size]: every rank's block as this process addresses it;
 * multicast_region: the multicast address of the blocks or NULL.  With a multicast address the
 * all-reduce is reduced inside the switch (multimem.ld_reduce) and its result delivered to every
 * rank with one store (multimem.st); the sum's order of additions is then the switch's, not rank
 * order.  Replaces the communicator created with the engine; call before capturing graphs.  The
 * memory stays the caller's and must outlive the engine. */
B200_API int64_t b200_engine_comm_region_bytes(b200_engine* engine);
B200_API int b200_engine_comm_attach(b200_engine* engine, void* region, const void* const* peer_regions,
                                     const void* multicast_region);
/* The engine's communicator, for b200_comm_set_wait_limit_ns and the loop-back test hooks
 * (NULL when the engine was created with tp_size 1). */
B200_API b200_comm* b200_engine_comm(b200_engine* engine);

/* No counterpart in the reference.  With B200_DECODE_CHAIN=1 in the environment when the engine is
 * created, decode steps of at most 64 tokens of a dense, unsharded model run everything between two
 * attention launches (o_proj, add + norm, gate_up, activation, down, add + norm, the next layer's
 * qkv, QK-norm, RoPE, KV store) as one persistent kernel of 8-CTA clusters whose CTAs must all be
 * resident at once, instead of one kernel per operator (the default, and the faster of the two on
 * B200).  Returns the number of CTAs that kernel runs with on the current device, or 0 when the
 * device cannot hold it. */
B200_API int b200_decode_chain_grid(void);

/* The stream the engine enqueues on (Engine::stream_), as a cudaStream_t. */
B200_API b200_stream_t b200_engine_stream(b200_engine* engine);

/* Measurement aid with no counterpart in the reference (it profiles with steady_clock timers,
 * src/engine/engine.cc:36-87): while on, steps run eagerly (no graph replay) with a CUDA event
 * pair around each attention launch.  b200_engine_read_profile synchronises and returns the
 * summed attention time of the last step, how many attention launches that covers, and the
 * number of kernels the last step launched (also valid for graph replays, profiling or not). */
B200_API int b200_engine_set_profiling(b200_engine* engine, int on);
B200_API int b200_engine_read_profile(b200_engine* engine, float* attention_ms,
                                      int32_t* attention_launches, int32_t* kernel_launches);
/* The same for the fused all-reduce launches of the last profiled step (tensor parallelism). */
B200_API int b200_engine_read_profile_allreduce(b200_engine* engine, float* allreduce_ms,
                                                int32_t* launches);

/* Device time of the last step in milliseconds (CUDA events around it); synchronises. */
B200_API int b200_engine_last_step_ms(b200_engine* engine, float* ms);

#ifdef __cplusplus
}
#endif

#endif /* B200_TOKEN_LOOP_H_ */
