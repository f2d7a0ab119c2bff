// Device state of the step runner, shared by the driver (engine.cu) and the layer stack (layer_stack.cu).
#pragma once

#include <cuda.h>

#include <map>
#include <string>
#include <vector>

#include "common.cuh"
#include "kernels.h"

namespace b200 {

struct LayerStack;   // layers described one by one (layer_stack.cu)

struct LayerWeights {
    __nv_bfloat16 *qkv = nullptr, *qkv_bias = nullptr, *o = nullptr, *gate_up = nullptr, *down = nullptr;
    __nv_bfloat16 *input_norm = nullptr, *post_norm = nullptr, *q_norm = nullptr, *k_norm = nullptr;
    __nv_bfloat16 *router = nullptr, *experts_gate_up = nullptr, *experts_down = nullptr;
    // qkv and gate_up with the norm weight in front of them folded into their columns (decode steps
    // whose GEMMs carry the add + norm in their epilogues)
    __nv_bfloat16 *qkv_folded = nullptr, *gate_up_folded = nullptr;
    CUtensorMap tmap_k, tmap_v;
};

struct Tensor {
    void* ptr;
    int64_t bytes;
};

}  // namespace b200

struct b200_comm;

struct b200_engine {
    b200_model_config m;
    b200_engine_config c;
    int device = 0;
    int hq = 0, hkv = 0, inter = 0, qkv_dim = 0;  // per-rank sizes
    int moe_inter = 0, experts_local = 0, expert_begin = 0;  // per-rank expert layout
    int64_t num_slots = 0;
    int pt_rows = 0, pt_cols = 0;
    int max_tokens = 0, max_batch = 0;
    float sm_scale = 0.f;

    std::vector<void*> allocs;
    std::map<std::string, b200::Tensor> named;  // "name" or "name.<layer>"
    std::vector<b200::LayerWeights> layers;

    __nv_bfloat16 *embed = nullptr, *lm_head = nullptr, *final_norm = nullptr;
    float *rope_cos = nullptr, *rope_sin = nullptr;
    __nv_bfloat16* kv_cache = nullptr;
    int32_t *page_table = nullptr, *token_pool = nullptr;

    // activations
    __nv_bfloat16 *x = nullptr, *residual = nullptr, *qkv = nullptr, *attn_out = nullptr, *h = nullptr,
                  *sel = nullptr, *logits = nullptr;
    int32_t *positions = nullptr, *out_loc = nullptr, *input_ids = nullptr, *seq_lens = nullptr,
            *next_tokens = nullptr;
    void* logits_bf16 = nullptr;       // fp32 models: logits rounded for the sampler
    int32_t* row_ids_dev = nullptr;    // [max_batch] rows picked by b200_engine_token_logits
    int tokens_last_step = 0;
    bool trace_residual = false;
    void* attn_ws = nullptr;
    int64_t attn_ws_bytes = 0;
    __nv_bfloat16* router_logits = nullptr;
    void* moe_ws = nullptr;

    // per-step metadata: pinned staging + device mirror
    int32_t* meta_host = nullptr;
    int32_t* meta_dev = nullptr;
    int meta_ints = 0;
    int32_t *scatter_host = nullptr, *scatter_dev = nullptr;
    int64_t scatter_cap = 0;

    cudaStream_t stream = nullptr;
    cudaEvent_t ev_meta_done = nullptr, ev_step_begin = nullptr, ev_step_end = nullptr,
                ev_scatter_done = nullptr;
    bool meta_in_flight = false, scatter_in_flight = false;
    int* status = nullptr;

    std::map<int, cudaGraphExec_t> graphs;          // padded decode batch size -> graph ending in argmax
    std::map<int, cudaGraphExec_t> graphs_sampled;  // ... ending in the sampling kernel
    std::map<int, int> graph_launches;              // kernels inside each captured graph

    // Optional per-kernel timing of the attention launches of eager steps.
    bool profile_attention = false;
    bool capturing = false;
    std::vector<cudaEvent_t> prof_events;   // 2 per layer
    std::vector<cudaEvent_t> prof_events_ar;  // 2 per all-reduce call
    int prof_ar_recorded = 0;
    int prof_pairs_recorded = 0;
    int launches_last_step = 0;
    b200::LayerStack* stack = nullptr;  // set when the model lists its layers one by one
    b200_comm* comm = nullptr;  // tensor parallelism: exchange buffers for the fused all-reduce
    int64_t comm_buffer_bytes = 0;

    // Results of the steps in flight: a ring of pinned, device-mapped slots the last kernel of a step
    // writes straight into (tokens, finish flags, the device status words, the ticket), one event each.
    struct ResultSlot {
        int32_t* tokens = nullptr;         // [max_batch]
        uint8_t* finished = nullptr;       // [max_batch]
        uint8_t* ignore_eos = nullptr;     // [max_batch], written by the host before the launch
        int32_t* status = nullptr;         // [2] + 64-bit ticket behind them
        cudaEvent_t done = nullptr;
        int64_t ticket = -1;
        int num_reqs = 0;
    };
    static constexpr int kResultSlots = 4;
    ResultSlot ring[kResultSlots];
    uint8_t* ring_host = nullptr;
    int64_t next_ticket = 0;
    int32_t eos_token_id = -1;
    void* chain_scratch = nullptr;  // fp32 sums, partial sums of squares and barrier words of the decode layer chain
    // B200_DECODE_CHAIN=1: decode steps run everything between two attention launches as one
    // persistent kernel (decode_chain.cu).  Off by default: measured on B200 it is the slower of the
    // two paths (each of its phases pays several ~1 us round trips to L2 that separate launches hide
    // behind one another under programmatic dependent launch).
    bool use_chain = false;
    // Decode steps of a dense, unsharded model of at most 256 tokens: no add + norm kernels.  o_proj and
    // down_proj add the residual in their split-K epilogue and accumulate each row's sum of squares;
    // qkv_proj and gate_up_proj read the un-normalised residual against weights with the norm weight
    // folded in, and scale their accumulator by the row's 1 / rms.  B200_FOLD_NORM=0 turns it off.
    bool use_fold = true;
    bool use_fold_heads = true;         // B200_FOLD_HEADS=0: QK-norm + RoPE + K/V store stay a kernel of their own
    bool folded_valid = false;          // the folded copies match qkv / gate_up / the norm weights
    unsigned long long* ssq = nullptr;  // [2 * layers + 1, kSsqStride] sums of squares of the residual rows
    static constexpr int kSsqStride = 256;
    bool use_pdl = true;  // B200_PDL=0 turns programmatic dependent launches off
    bool kv_evict_first = true;  // B200_KV_EVICT_FIRST=0: K/V loads with the default L2 policy
    // Seeds are 64-bit: keep them 8-byte aligned inside the int32 staging block.  The 64-bit step
    // index follows them, so a captured graph reads a fresh one on every replay.
    static int seed_offset(int Bp) { return (7 * Bp + 1 + 1) & ~1; }
    static int step_index_offset(int Bp) { return seed_offset(Bp) + 2 * Bp; }
};

namespace b200 {

inline int dev_alloc(b200_engine* e, void** out, int64_t bytes, bool zero) {
    void* p = nullptr;
    if (bytes <= 0) bytes = 16;
    B200_CHECK_CUDA(cudaMalloc(&p, static_cast<size_t>(bytes)));
    e->allocs.push_back(p);
    if (zero) B200_CHECK_CUDA(cudaMemset(p, 0, static_cast<size_t>(bytes)));
    *out = p;
    return B200_OK;
}

template <typename T>
inline int named_alloc(b200_engine* e, T** out, const std::string& name, int64_t elems, bool zero = false) {
    void* p = nullptr;
    const int64_t bytes = elems * static_cast<int64_t>(sizeof(T));
    int err = dev_alloc(e, &p, bytes, zero);
    if (err != B200_OK) return err;
    *out = static_cast<T*>(p);
    e->named[name] = Tensor{p, bytes};
    return B200_OK;
}

#define B200_TRY(expr)                  \
    do {                                \
        int err__ = (expr);             \
        if (err__ != B200_OK) return err__; \
    } while (0)

// ---- the layer stack (layer_stack.cu) -------------------------------------------

// Validates the per-layer description and allocates weights, latent pools and activations.
int layer_stack_create(b200_engine* e, const b200_stack_config* sc);
void layer_stack_destroy(b200_engine* e);
// Decides, on the host, which requests of a prefill step attend in the latent space and which through
// expanded keys and values, and stages that plan behind the step's metadata copy.
int layer_stack_plan(b200_engine* e, const b200_step* st, int Bp);
// The layers on `T` tokens, as programmatic dependent launches if `pdl`; leaves the final-norm output in
// stack_hidden().
int layer_stack_enqueue(b200_engine* e, int phase, int Bp, int T, bool pdl);
// `count` rows of hidden states -> logits [count, stack_logits_ld].
int layer_stack_head(b200_engine* e, void* logits, const void* rows, int count);
int stack_dtype(const b200_engine* e);
int stack_logits_ld(const b200_engine* e);
int stack_row_bytes(const b200_engine* e);          // of one hidden-state row
const void* stack_hidden(const b200_engine* e);     // [T, padded hidden]
int32_t* stack_token_row(const b200_engine* e);     // [T] page-table row of every token of the step
int32_t* stack_token_len(const b200_engine* e);     // [T] keys it sees
void stack_set_trace(b200_engine* e, float* host);

}  // namespace b200
