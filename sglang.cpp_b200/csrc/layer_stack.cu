// Models whose layers are listed one by one: allocation of their weights, pools and states, the per-step
// plan, and the layer stack the step runner (engine.cu) enqueues between its token preparation and its
// output head.
//
// Per layer, on T tokens (fp32 residual stream r, everything else in the stack's dtype):
//     x = norm(r += previous block)       the norm on the input: one kernel, residual.cu
//     x = r += norm(previous block)       or on the output of a block, or both; one kernel as well (RMS or layer norms)
//     y = mixer(x)
//     x = ... once more
//     y = feed-forward(x)
//
// Mixers
//   latent attention:  [cq | c] = x W_down, both latents in one GEMM; cq, pool[slot] = norm(cq), norm(c)
//                      (latent_attention.cu); q = cq W_uq; o = attention in the latent space, or over expanded
//                      keys and values; y = o W_o.  A part of the key may turn with the position instead of being
//                      normalised; a layer may read the pool of another one
//   window attention:  [q | k | v | gate] = x W in one GEMM; norms, rotation, value mixing and the K/V store in
//                      one kernel; attention and its gate in the next (window_attention.cu); y = o W_o.  Heads may mix
//                      their weights (talking_heads.cu), values turn with the position, a layer read the pools of another
//   linear attention:  [q | k | v | gate | low-rank decay] = x W in one GEMM; recurrence, norm and gate
//                      (linear_attention.cu); y = o W_o
//   state space, delta rule, lightning, matrix memory:  [gate | v | k | q | steps] = x W in one GEMM; convolution,
//                      recurrence, norm and gate (recurrence.cu); y = o W_o
//   two of the last kinds (window attention, recurrences) side by side: one GEMM makes both rows; one output
//                      projection over both results adds them up, or each has its own and they meet, normalised, in
//                      the residual kernel
// Feed-forwards: dense; experts by token id, whose placement depends on token ids only and is laid out for all
// layers at once before the first; experts by score (router logits in fp32, routing and placement in two
// kernels, the weighted sum in the residual kernel that follows), beside one that every token uses.
//
// Latent attention has two forms.  In the latent space (decode steps, short extensions) the per-head projections
// are applied to the query and to the result.  Extensions of more than `expand_min` tokens expand keys and
// values of the whole request once (two GEMMs) into a scratch that the prefill kernel of the
// grouped-query models reads as if it were its paged pool.  A batch may hold both kinds of requests.
#include <math.h>
#include <stdlib.h>

#include <string>
#include <vector>

#include "common.cuh"
#include "engine_state.h"
#include "kernels.h"

namespace b200 {

namespace {
int pad_to(int n, int m) { return (n + m - 1) / m * m; }
int pad_width(int n) { return pad_to(n, 64); }
int pad_head_dim(int n) { return n <= 128 ? 128 : pad_to(n, 64); }
int pad_latent(int n) { return pad_to(n, 128); }
int latent_rope_at(int kv_rank) { return pad_to(kv_rank, 8); }   // where the rotated part of a latent row starts
int latent_width(int kv_rank, int rope_dim) { return pad_latent(rope_dim > 0 ? latent_rope_at(kv_rank) + rope_dim : kv_rank); }
bool is_recurrence(int mixer) {
    return mixer == B200_MIXER_STATE_SPACE || mixer == B200_MIXER_DELTA_RULE || mixer == B200_MIXER_LIGHTNING ||
           mixer == B200_MIXER_MATRIX_MEMORY;
}
int rule_of(int mixer) {
    return mixer == B200_MIXER_DELTA_RULE ? B200_RULE_DELTA : mixer == B200_MIXER_LIGHTNING ? B200_RULE_LIGHTNING
           : mixer == B200_MIXER_MATRIX_MEMORY ? B200_RULE_MATRIX_MEMORY : B200_RULE_STATE_SPACE;
}
}  // namespace

struct StackLayer {
    b200_layer_config c;
    int qp = 0, rp = 0, op = 0, dp = 0, vp = 0, ip = 0;   // padded sizes
    void *norm1_out = nullptr, *norm2_out = nullptr;       // of what the blocks return, where both sides have one
    void *norm1_bias = nullptr, *norm2_bias = nullptr, *norm1_out_bias = nullptr, *norm2_out_bias = nullptr;   // layer norms
    void *norm1 = nullptr, *norm2 = nullptr, *down_qkv = nullptr, *q_norm = nullptr, *kv_norm = nullptr, *uq = nullptr,
         *uk = nullptr, *uk_absorb = nullptr, *uv = nullptr, *o = nullptr, *up = nullptr, *down = nullptr;
    // the projection that a mixer's (or both mixers') rows come from, and this mixer's columns in them
    void *joint = nullptr, *joint_bias = nullptr;
    int64_t joint_ld = 0, joint_at = 0;
    // where this mixer's result goes: element offset in the result buffer, distance of its rows
    int64_t out_at = 0, out_ld = 0;
    StackLayer* beside = nullptr;
    void* side_norm = nullptr;    // of this mixer's result, under B200_JOIN_NORMED
    // window attention
    void *q_head_norm = nullptr, *k_head_norm = nullptr, *k_cache = nullptr, *v_cache = nullptr;
    float *value_mix = nullptr, *cos_t = nullptr, *sin_t = nullptr, *sinks = nullptr;
    float *value_cos = nullptr, *value_sin = nullptr, *head_mix = nullptr;
    int mix = HeadPrepare::kPlain;
    // linear attention
    void *decay_up = nullptr, *head_norm = nullptr;
    float *decay_bias = nullptr, *state = nullptr;
    int up_ld = 0;
    // recurrences
    float *conv = nullptr, *conv_bias = nullptr, *decay_log = nullptr, *step_bias = nullptr, *skip = nullptr;
    void* conv_state = nullptr;
    float* memory = nullptr;
    // scored experts
    void *router = nullptr, *shared_up = nullptr, *shared_down = nullptr;
    float* correction = nullptr;
    int isp = 0;
    int32_t* table = nullptr;
    void* cache = nullptr;
    int32_t *rows = nullptr, *counts = nullptr, *offsets = nullptr;   // expert placement of this step
    bool can_expand = false;
};

struct LayerStack {
    std::vector<StackLayer> layers, besides;
    struct RopeTable {
        b200_layer_config c;
        float *cos_t, *sin_t;
    };
    std::vector<RopeTable> ropes;
    int dtype = B200_DTYPE_BF16;
    int esz = 2;            // bytes per element
    int hp = 0, vocab_p = 0;
    float norm_offset = 0.f, logit_scale = 1.f;
    bool norm_input = true, norm_output = false, layer_norm = false;
    float embed_scale = 1.f;
    void *embed = nullptr, *head = nullptr, *final_norm = nullptr, *final_norm_bias = nullptr;
    float* residual = nullptr;
    void *x = nullptr, *joint = nullptr, *cq = nullptr, *q = nullptr, *attn = nullptr, *y = nullptr, *h = nullptr,
         *xp = nullptr, *ye = nullptr;
    // latent-space attention, in slabs of at most latent_rows query rows
    int latent_rows = 0;
    void *qa = nullptr, *ol = nullptr, *ws = nullptr;
    int64_t ws_bytes = 0;
    int32_t *token_row = nullptr, *token_len = nullptr;
    // expanded attention
    int expand_min = 32;
    int64_t expand_cap = 0;    // tokens the scratch holds
    void *xc = nullptr, *xk = nullptr, *xv = nullptr;
    int32_t* iota = nullptr;   // an identity page-table row
    // the plan of the current prefill step: x_len | x_base | gather_base | tokens in the latent space
    int32_t *plan_host = nullptr, *plan_dev = nullptr;
    int plan_expanded = 0, plan_latent = 0, plan_max_extend = 0, plan_max_len = 0;
    int64_t plan_rows = 0;     // scratch rows in use
    // the latent-space rows of a mixed step, compacted
    int32_t *compact_row = nullptr, *compact_len = nullptr;
    void *qc = nullptr, *ac = nullptr;
    int max_extend = 0;        // longest extension of the current step
    // window attention
    void *first_values = nullptr, *mixed_heads = nullptr;
    // recurrences
    void *mixed = nullptr, *chunks = nullptr;
    float *steps = nullptr, *units = nullptr;
    void* y2 = nullptr;        // the right one of two results under B200_JOIN_NORMED
    // scored experts: the routing of the layer that is running
    float *router_logits = nullptr, *route_weights = nullptr;
    int32_t *route_ids = nullptr, *route_rows = nullptr, *route_counts = nullptr, *route_offsets = nullptr;
    void *shared_h = nullptr, *shared_y = nullptr;
    std::vector<TableRouteLayer> routes;
    TableRouteLayer* routes_dev = nullptr;
    int max_experts = 0;
    float* trace = nullptr;    // host [layers, tokens, width]
};

namespace {

#define S_TRY(expr)                         \
    do {                                    \
        int err__ = (expr);                 \
        if (err__ != B200_OK) return err__; \
    } while (0)

int named_bytes(b200_engine* e, void** out, const std::string& name, int64_t bytes, bool zero = true) {
    S_TRY(dev_alloc(e, out, bytes, zero));
    e->named[name] = Tensor{*out, bytes};
    return B200_OK;
}

__global__ void iota_kernel(int32_t* p, int64_t n) {
    const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i < n) p[i] = static_cast<int32_t>(i);
}

__global__ void compact_rows_kernel(int32_t* __restrict__ row, int32_t* __restrict__ len,
                                    const int32_t* __restrict__ token_row, const int32_t* __restrict__ token_len,
                                    const int32_t* __restrict__ tokens, int n) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    row[i] = token_row[tokens[i]];
    len[i] = token_len[tokens[i]];
}

// A rotation whose frequencies may be stretched.
bool rope_ok(const b200_layer_config& c, int widest) {
    return c.rotary_dim >= 0 && c.rotary_dim % 2 == 0 && c.rotary_dim <= widest && (c.rotary_dim == 0 || c.rope_base > 0.0) &&
           (c.rope_factor == 0.0 || (c.rope_factor > 0.0 && c.rope_original == 0.0) ||
            (c.rope_factor > 0.0 && c.rope_low > 0.0 && c.rope_high > c.rope_low && c.rope_original > 0.0));
}
bool same_rope(const b200_layer_config& a, const b200_layer_config& b) {
    if (a.rotary_dim != b.rotary_dim || a.rope_base != b.rope_base || a.rope_factor != b.rope_factor) return false;
    if (a.rope_factor == 0.0 || a.rope_original != b.rope_original) return a.rope_factor == 0.0;
    return a.rope_original == 0.0 || (a.rope_low == b.rope_low && a.rope_high == b.rope_high);
}

int check_mixer(const b200_layer_config& c, int l) {
    B200_CHECK_ARG(c.heads > 0 && c.heads <= 65535 && c.head_dim > 0 && c.value_dim > 0,
                   "layer %d: head count and sizes must be positive", l);
    if (c.mixer == B200_MIXER_LATENT_ATTENTION) {
        B200_CHECK_ARG(c.q_rank > 0 && c.kv_rank > 0, "layer %d: latent attention needs positive ranks", l);
        B200_CHECK_ARG(rope_ok(c, c.head_dim), "layer %d: bad rotation", l);
    } else if (c.mixer == B200_MIXER_WINDOW_ATTENTION) {
        B200_CHECK_ARG(c.kv_heads > 0 && c.heads % c.kv_heads == 0, "layer %d: %d heads over %d key/value heads", l, c.heads,
                       c.kv_heads);
        B200_CHECK_ARG(c.window > 0 && c.keep_first >= 0 && c.chunk >= 0, "layer %d: bad window", l);
        B200_CHECK_ARG(c.gate >= B200_GATE_NONE && c.gate <= B200_GATE_HEAD, "layer %d: unknown gate", l);
        B200_CHECK_ARG(rope_ok(c, c.head_dim), "layer %d: bad rotation", l);
        B200_CHECK_ARG(c.value_dim <= 1024 && c.head_dim <= 2048, "layer %d: heads are too wide", l);
        B200_CHECK_ARG(c.head_norm >= B200_HEAD_NORM_NONE && c.head_norm <= B200_HEAD_NORM_UNIT, "layer %d: unknown head norm", l);
        B200_CHECK_ARG(!(c.head_mix || c.value_rotary) || (!c.sink && c.heads <= 128), "layer %d: mixing heads take no sinks, and at most 128 heads", l);
        B200_CHECK_ARG(!c.value_rotary || (c.value_dim % 2 == 0 && c.rope_base > 0.0 && !c.value_mix),
                       "layer %d: bad value rotation", l);
        B200_CHECK_ARG(c.kv_from < 0 || (!c.value_mix && !c.qkv_bias), "layer %d: no projections of its own to mix or bias", l);
    } else if (c.mixer == B200_MIXER_LINEAR_ATTENTION) {
        B200_CHECK_ARG(c.decay_rank > 0 && c.decay_tau > 0.f, "layer %d: bad decay", l);
        B200_CHECK_ARG(linear_attention_supported(pad_width(c.value_dim), pad_width(c.head_dim)),
                       "layer %d: heads are too wide", l);
    } else if (is_recurrence(c.mixer)) {
        B200_CHECK_ARG(c.kv_heads > 0 && c.heads % c.kv_heads == 0, "layer %d: %d heads over %d key heads", l, c.heads, c.kv_heads);
        const bool conv = c.mixer == B200_MIXER_STATE_SPACE || c.mixer == B200_MIXER_DELTA_RULE;
        B200_CHECK_ARG(recurrence_supported(pad_width(c.value_dim), pad_width(c.head_dim), conv ? c.conv_taps : 1),
                       "layer %d: heads or convolution too wide", l);
        B200_CHECK_ARG(conv || c.kv_heads == c.heads, "layer %d: every head has its own key head here", l);
        B200_CHECK_ARG(c.mixer != B200_MIXER_MATRIX_MEMORY || c.gate_cap > 0.f, "layer %d: bad gate cap", l);
        B200_CHECK_ARG(c.mixer == B200_MIXER_DELTA_RULE || (c.norm_groups > 0 && c.heads * c.value_dim % c.norm_groups == 0),
                       "layer %d: bad norm groups", l);
    } else {
        B200_CHECK_ARG(false, "layer %d: unknown mixer %d", l, c.mixer);
    }
    return B200_OK;
}

int check_layer(const b200_layer_config& c, int l) {
    S_TRY(check_mixer(c, l));
    B200_CHECK_ARG(c.mlp >= B200_MLP_NONE && c.mlp <= B200_MLP_SCORED_MOE, "layer %d: unknown feed-forward %d", l, c.mlp);
    if (c.mlp == B200_MLP_NONE) return B200_OK;
    B200_CHECK_ARG(c.intermediate > 0, "layer %d: feed-forward size must be positive", l);
    B200_CHECK_ARG(c.epilogue > B200_EPILOGUE_NONE && c.epilogue <= B200_EPILOGUE_CLAMPED_SWIGLU, "layer %d: unknown activation", l);
    const int outputs = c.num_experts + (c.mlp == B200_MLP_SCORED_MOE ? c.identity_experts : 0);
    if (c.mlp != B200_MLP_DENSE)
        B200_CHECK_ARG(c.num_experts > 0 && outputs >= c.num_experts && outputs <= kMaxTableExperts && c.experts_per_tok > 0 &&
                           c.experts_per_tok <= outputs,
                       "layer %d: %d of %d experts (at most %d)", l, c.experts_per_tok, outputs, kMaxTableExperts);
    if (c.mlp == B200_MLP_SCORED_MOE) {
        B200_CHECK_ARG(c.router_groups > 0 && outputs % c.router_groups == 0 && c.router_keep > 0 &&
                           c.router_keep <= c.router_groups &&
                           c.experts_per_tok <= outputs / c.router_groups * c.router_keep && c.shared_intermediate >= 0,
                       "layer %d: bad expert groups", l);
        B200_CHECK_ARG(c.score == B200_SCORE_SOFTMAX || (c.score == B200_SCORE_SIGMOID && c.identity_experts == 0),
                       "layer %d: identity experts come with softmax scores", l);
        B200_CHECK_ARG(c.identity_experts == 0 || c.shared_intermediate == 0, "layer %d: identity experts beside a shared one", l);
    }
    return B200_OK;
}

// Sizes of the activation buffers: the widest of any layer, in elements per token (workspaces: bytes).
struct Widths {
    int64_t joint = 0, cq = 0, q = 0, attn = 0, h = 0, pairs = 0, latent = 0, xk = 0, xv = 0, xc = 0, ws = 0, first = 0,
            experts = 0, router = 0, top = 0, shared = 0, mixed_heads = 0, mixed = 0, steps = 0, units = 0, chunks = 0;
    bool normed_pair = false;
    bool scored = false, any_expand = false;
    static void widest(int64_t& a, int64_t b) { if (b > a) a = b; }
};

// cos / sin of position * frequency, computed in double on the host; layers with the same rotation share a table.
int rope_table(b200_engine* e, const b200_layer_config& c, float*& cos_t, float*& sin_t) {
    LayerStack* S = e->stack;
    for (const LayerStack::RopeTable& t : S->ropes)
        if (same_rope(t.c, c)) {
            cos_t = t.cos_t;
            sin_t = t.sin_t;
            return B200_OK;
        }
    constexpr double kTwoPi = 6.283185307179586476925286766559;
    const int half = c.rotary_dim / 2;
    const int64_t n = static_cast<int64_t>(e->pt_cols) * half;
    std::vector<float> cs(n), sn(n);
    for (int i = 0; i < half; ++i) {
        double f = pow(c.rope_base, -2.0 * i / c.rotary_dim);
        if (c.rope_factor > 0.0 && c.rope_original == 0.0) {
            f /= c.rope_factor;
        } else if (c.rope_factor > 0.0) {
            const double wave = kTwoPi / f;
            const double s = (c.rope_original / wave - c.rope_low) / (c.rope_high - c.rope_low);
            if (wave > c.rope_original / c.rope_low)
                f /= c.rope_factor;
            else if (wave >= c.rope_original / c.rope_high)
                f = (1.0 - s) * f / c.rope_factor + s * f;
        }
        for (int64_t p = 0; p < e->pt_cols; ++p) {
            cs[p * half + i] = static_cast<float>(cos(static_cast<double>(p) * f));
            sn[p * half + i] = static_cast<float>(sin(static_cast<double>(p) * f));
        }
    }
    void* p = nullptr;
    S_TRY(dev_alloc(e, &p, n * 4, true));
    cos_t = static_cast<float*>(p);
    S_TRY(dev_alloc(e, &p, n * 4, true));
    sin_t = static_cast<float*>(p);
    S->ropes.push_back({c, cos_t, sin_t});
    if (n == 0) return B200_OK;
    B200_CHECK_CUDA(cudaMemcpy(cos_t, cs.data(), n * 4, cudaMemcpyHostToDevice));
    B200_CHECK_CUDA(cudaMemcpy(sin_t, sn.data(), n * 4, cudaMemcpyHostToDevice));
    return B200_OK;
}

int alloc_latent(b200_engine* e, StackLayer& L, int l, const std::string& sfx, Widths& w) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    L.qp = pad_width(c.q_rank);
    L.rp = latent_width(c.kv_rank, c.rotary_dim);
    L.op = pad_latent(c.kv_rank);
    L.dp = pad_head_dim(c.head_dim);
    L.vp = pad_head_dim(c.value_dim);
    const int64_t hp = S->hp, z = S->esz, H = c.heads, qp = L.qp, rp = L.rp, op = L.op, dp = L.dp, vp = L.vp;
    const bool own = c.kv_from < 0;
    if (!own) {
        B200_CHECK_ARG(c.kv_from < l && S->layers[c.kv_from].c.mixer == B200_MIXER_LATENT_ATTENTION &&
                           S->layers[c.kv_from].c.kv_from < 0, "layer %d: layer %d has no latents of its own", l, c.kv_from);
        const b200_layer_config& from = S->layers[c.kv_from].c;
        B200_CHECK_ARG(from.kv_rank == c.kv_rank && same_rope(from, c), "layer %d: its latents are not those of layer %d", l, c.kv_from);
        L.cache = S->layers[c.kv_from].cache;
    }
    S_TRY(named_bytes(e, &L.down_qkv, "down_qkv" + sfx, (qp + (own ? rp : 0)) * hp * z));
    S_TRY(named_bytes(e, &L.q_norm, "q_latent_norm" + sfx, qp * z));
    if (own) S_TRY(named_bytes(e, &L.kv_norm, "kv_latent_norm" + sfx, rp * z));
    S_TRY(rope_table(e, c, L.cos_t, L.sin_t));
    S_TRY(named_bytes(e, &L.uq, "uq" + sfx, H * dp * qp * z));
    S_TRY(named_bytes(e, &L.uk_absorb, "uk_absorb" + sfx, H * rp * dp * z));
    S_TRY(named_bytes(e, &L.uv, "uv" + sfx, H * vp * op * z));
    if (own) S_TRY(named_bytes(e, &L.cache, "latent_cache" + sfx, e->num_slots * rp * z));
    // what the prefill kernel of the grouped-query models takes (and its positive score scale)
    L.can_expand = S->dtype == B200_DTYPE_BF16 && dp == 128 && vp == 128 && c.score_scale > 0.f && H <= 65535;
    if (L.can_expand) S_TRY(named_bytes(e, &L.uk, "uk" + sfx, H * dp * rp * z));
    w.any_expand |= L.can_expand;
    Widths::widest(w.joint, qp + rp);
    Widths::widest(w.cq, qp);
    Widths::widest(w.q, H * dp);
    Widths::widest(w.latent, H * rp);
    Widths::widest(w.ws, latent_attention_workspace_bytes(S->latent_rows, c.heads, L.rp));
    if (L.can_expand) {
        Widths::widest(w.xk, H * dp);
        Widths::widest(w.xv, H * vp);
        Widths::widest(w.xc, rp);
    }
    return B200_OK;
}

// Columns of the joint projection's rows.
int64_t joint_width(const StackLayer& L) {
    const b200_layer_config& c = L.c;
    const int64_t H = c.heads, G = c.kv_heads, dp = L.dp, vp = L.vp;
    if (c.mixer == B200_MIXER_LINEAR_ATTENTION) return 2 * H * (dp + vp) + pad_width(c.decay_rank);
    if (c.mixer == B200_MIXER_WINDOW_ATTENTION)
        return H * dp + (c.kv_from < 0 ? G * (dp + vp) : 0) + (c.gate == B200_GATE_ELEMENT ? H * vp : c.gate == B200_GATE_HEAD ? pad_width(c.heads) : 0);
    const int steps = c.mixer == B200_MIXER_LIGHTNING ? 0 : c.mixer == B200_MIXER_STATE_SPACE ? 1 : 2;   // per head
    return 2 * H * vp + 2 * G * dp + pad_width(steps * c.heads);
}

// (names of a mixer's tensors start with `pre`)
int alloc_window(b200_engine* e, StackLayer& L, int l, const std::string& pre, const std::string& sfx, Widths& w) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    const int64_t z = S->esz, G = c.kv_heads, dp = L.dp, vp = L.vp;
    if (c.head_norm == B200_HEAD_NORM_WEIGHTED) {
        S_TRY(named_bytes(e, &L.q_head_norm, pre + "q_head_norm" + sfx, dp * z));
        S_TRY(named_bytes(e, &L.k_head_norm, pre + "k_head_norm" + sfx, dp * z));
    }
    if (c.kv_from < 0) {
        S_TRY(named_bytes(e, &L.k_cache, pre + "k_cache" + sfx, e->num_slots * G * dp * z));
        S_TRY(named_bytes(e, &L.v_cache, pre + "v_cache" + sfx, e->num_slots * G * vp * z));
    } else {
        B200_CHECK_ARG(pre.empty() && c.kv_from < l && S->layers[c.kv_from].c.mixer == B200_MIXER_WINDOW_ATTENTION &&
                           S->layers[c.kv_from].c.kv_from < 0, "layer %d: layer %d has no keys and values of its own", l, c.kv_from);
        const StackLayer& from = S->layers[c.kv_from];
        B200_CHECK_ARG(from.c.kv_heads == c.kv_heads && from.c.head_dim == c.head_dim && from.c.value_dim == c.value_dim &&
                           from.c.head_norm == c.head_norm && from.c.value_rotary == c.value_rotary && same_rope(from.c, c),
                       "layer %d: its keys and values are not those of layer %d", l, c.kv_from);
        L.k_cache = from.k_cache;
        L.v_cache = from.v_cache;
    }
    S_TRY(rope_table(e, c, L.cos_t, L.sin_t));
    void* p = nullptr;
    if (c.value_rotary) {
        b200_layer_config whole = c;
        whole.rotary_dim = c.value_dim;
        whole.rope_factor = 0.0;
        S_TRY(rope_table(e, whole, L.value_cos, L.value_sin));
    }
    if (c.head_mix || c.value_rotary) {
        S_TRY(named_bytes(e, &p, pre + "head_mix" + sfx, static_cast<int64_t>(c.heads) * c.heads * 4));
        L.head_mix = static_cast<float*>(p);
        Widths::widest(w.mixed_heads, static_cast<int64_t>(c.heads) * G * vp);
        if (talking_decode_supported(c.heads, c.kv_heads)) Widths::widest(w.ws, head_mix_workspace_bytes(e->max_batch, c.heads, c.kv_heads));
    }
    if (c.sink) {
        S_TRY(named_bytes(e, &p, pre + "sinks" + sfx, c.heads * 4ll));
        L.sinks = static_cast<float*>(p);
    }
    if (c.value_mix) {
        L.mix = HeadPrepare::kSave;
        for (int o = 0; o < l; ++o) {
            const b200_layer_config& f = S->layers[o].c;
            if (f.mixer != B200_MIXER_WINDOW_ATTENTION || !f.value_mix) continue;
            L.mix = HeadPrepare::kMix;
            B200_CHECK_ARG(f.kv_heads == c.kv_heads && f.value_dim == c.value_dim,
                           "layer %d: mixes %d x %d values with the %d x %d of layer %d", l, c.kv_heads, c.value_dim, f.kv_heads,
                           f.value_dim, o);
            break;
        }
        S_TRY(named_bytes(e, &p, pre + "value_mix" + sfx, 4));
        L.value_mix = static_cast<float*>(p);
        Widths::widest(w.first, G * vp);
    }
    if (c.kv_heads <= 8 && 8 % c.kv_heads == 0)
        Widths::widest(w.ws, decode_workspace_bytes(e->max_batch, c.heads, c.kv_heads));
    return B200_OK;
}

int alloc_linear(b200_engine* e, StackLayer& L, const std::string& pre, const std::string& sfx) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    L.up_ld = pad_to(c.decay_rank, 16);
    const int64_t z = S->esz, H = c.heads, dp = L.dp, vp = L.vp;
    void* p = nullptr;
    S_TRY(named_bytes(e, &L.decay_up, pre + "decay_up" + sfx, H * dp * L.up_ld * z));
    S_TRY(named_bytes(e, &p, pre + "decay_bias" + sfx, H * dp * 4));
    L.decay_bias = static_cast<float*>(p);
    S_TRY(named_bytes(e, &L.head_norm, pre + "head_norm" + sfx, vp * z));
    S_TRY(named_bytes(e, &p, pre + "state" + sfx, static_cast<int64_t>(e->pt_rows) * H * dp * vp * 4));
    L.state = static_cast<float*>(p);
    return B200_OK;
}

int alloc_recurrence(b200_engine* e, StackLayer& L, const std::string& pre, const std::string& sfx, Widths& w) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    const bool delta = c.mixer == B200_MIXER_DELTA_RULE, conv = delta || c.mixer == B200_MIXER_STATE_SPACE,
               memory = c.mixer == B200_MIXER_MATRIX_MEMORY;
    const int64_t z = S->esz, H = c.heads, dp = L.dp, vp = L.vp, channels = H * vp + 2 * c.kv_heads * dp;
    void* p = nullptr;
    auto floats = [&](float*& to, const char* name, int64_t n) -> int {
        S_TRY(named_bytes(e, &p, pre + name + sfx, n * 4));
        to = static_cast<float*>(p);
        return B200_OK;
    };
    if (conv) {
        S_TRY(floats(L.conv, "conv", c.conv_taps * channels));
        S_TRY(floats(L.conv_bias, "conv_bias", channels));
        S_TRY(named_bytes(e, &L.conv_state, pre + "conv_state" + sfx, static_cast<int64_t>(e->pt_rows) * c.conv_taps * channels * z));
    }
    if (!memory) S_TRY(floats(L.decay_log, "decay_log", H));
    if (conv || memory) S_TRY(floats(L.step_bias, "step_bias", memory ? 2 * H : H));
    if (c.mixer == B200_MIXER_STATE_SPACE) S_TRY(floats(L.skip, "skip", H));
    S_TRY(named_bytes(e, &L.head_norm, pre + "head_norm" + sfx, (delta ? vp : H * vp) * z));
    S_TRY(floats(L.state, "state", static_cast<int64_t>(e->pt_rows) * H * dp * vp));
    if (memory) S_TRY(floats(L.memory, "memory", e->pt_rows * H * recurrence_memory_floats(L.dp, L.vp)));
    const RecurrenceScratch need = recurrence_scratch(rule_of(c.mixer), e->max_tokens, e->max_batch,
                                                      c.heads, c.kv_heads, L.dp, L.vp, S->dtype);
    Widths::widest(w.mixed, need.mixed);
    Widths::widest(w.steps, need.steps);
    Widths::widest(w.units, need.units);
    Widths::widest(w.chunks, need.chunks);
    return B200_OK;
}

// What a mixer other than latent attention has beside its input and output projections.
int alloc_mixer(b200_engine* e, StackLayer& L, int l, const std::string& pre, const std::string& sfx, Widths& w) {
    const b200_layer_config& c = L.c;
    const bool window = c.mixer == B200_MIXER_WINDOW_ATTENTION;
    L.dp = window ? pad_head_dim(c.head_dim) : pad_width(c.head_dim);
    L.vp = window ? pad_head_dim(c.value_dim) : pad_width(c.value_dim);
    L.out_ld = static_cast<int64_t>(c.heads) * L.vp;
    L.joint_ld = joint_width(L);
    if (window) return alloc_window(e, L, l, pre, sfx, w);
    if (is_recurrence(c.mixer)) return alloc_recurrence(e, L, pre, sfx, w);
    return alloc_linear(e, L, pre, sfx);
}

// Mixer (or both mixers) of a layer: the projections around it, then the rest.
int alloc_layer_mixer(b200_engine* e, StackLayer& L, int l, const std::string& sfx, Widths& w) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    const int64_t hp = S->hp, z = S->esz;
    if (c.mixer == B200_MIXER_LATENT_ATTENTION) {
        B200_CHECK_ARG(c.beside < 0, "layer %d: nothing runs beside latent attention", l);
        S_TRY(alloc_latent(e, L, l, sfx, w));
        L.out_ld = static_cast<int64_t>(c.heads) * L.vp;
        Widths::widest(w.attn, L.out_ld);
        return named_bytes(e, &L.o, "o" + sfx, hp * L.out_ld * z);
    }
    S_TRY(alloc_mixer(e, L, l, "", sfx, w));
    StackLayer* R = L.beside;
    const char* name = c.mixer == B200_MIXER_WINDOW_ATTENTION ? "qkvg" : c.mixer == B200_MIXER_LINEAR_ATTENTION ? "qkvga" : "recurrence";
    const int64_t left_out = L.out_ld;
    if (R != nullptr) {
        B200_CHECK_ARG(c.mixer != B200_MIXER_LINEAR_ATTENTION && R->c.mixer != B200_MIXER_LINEAR_ATTENTION &&
                           R->c.mixer != B200_MIXER_LATENT_ATTENTION && !R->c.value_mix, "layer %d: mixers that do not run side by side", l);
        B200_CHECK_ARG(c.join == B200_JOIN_SUM || c.join == B200_JOIN_NORMED, "layer %d: unknown join", l);
        S_TRY(check_mixer(R->c, l));
        S_TRY(alloc_mixer(e, *R, l, "beside_", sfx, w));
        name = "joint";
        R->joint_at = L.joint_ld;
        L.joint_ld = R->joint_ld = L.joint_ld + R->joint_ld;
        Widths::widest(w.attn, left_out + R->out_ld);
        if (c.join == B200_JOIN_SUM) {
            R->out_at = left_out;
            L.out_ld = R->out_ld = left_out + R->out_ld;
        } else {
            w.normed_pair = true;
            R->out_at = static_cast<int64_t>(e->max_tokens) * left_out;
            S_TRY(named_bytes(e, &R->o, "beside_o" + sfx, hp * R->out_ld * z));
            S_TRY(named_bytes(e, &L.side_norm, "side_norm" + sfx, hp * z));
            S_TRY(named_bytes(e, &R->side_norm, "beside_side_norm" + sfx, hp * z));
        }
    }
    S_TRY(named_bytes(e, &L.joint, name + sfx, L.joint_ld * hp * z));
    if (c.qkv_bias || (R != nullptr && R->c.qkv_bias)) S_TRY(named_bytes(e, &L.joint_bias, "joint_bias" + sfx, L.joint_ld * z));
    S_TRY(named_bytes(e, &L.o, "o" + sfx, hp * L.out_ld * z));
    Widths::widest(w.joint, L.joint_ld);
    Widths::widest(w.attn, L.out_ld);
    return B200_OK;
}

int norm_of(b200_engine* e, const char* name, const std::string& sfx, void*& weight, void*& bias) {
    const LayerStack* S = e->stack;
    const int64_t bytes = static_cast<int64_t>(S->hp) * S->esz;
    S_TRY(named_bytes(e, &weight, name + sfx, bytes));
    return S->layer_norm ? named_bytes(e, &bias, std::string(name) + "_bias" + sfx, bytes) : B200_OK;
}

int alloc_feed_forward(b200_engine* e, StackLayer& L, const std::string& sfx, Widths& w) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    const int64_t hp = S->hp, z = S->esz, Tm = e->max_tokens;
    L.ip = pad_width(c.intermediate);
    const int64_t n_up = (epilogue_is_gated(c.epilogue) ? 2 : 1) * static_cast<int64_t>(L.ip);
    const int64_t E = c.mlp == B200_MLP_DENSE ? 1 : c.num_experts;
    S_TRY(norm_of(e, "norm2", sfx, L.norm2, L.norm2_bias));
    if (S->norm_input && S->norm_output) S_TRY(norm_of(e, "norm2_out", sfx, L.norm2_out, L.norm2_out_bias));
    S_TRY(named_bytes(e, &L.up, "mlp_up" + sfx, E * n_up * hp * z));
    S_TRY(named_bytes(e, &L.down, "mlp_down" + sfx, E * hp * L.ip * z));
    if (c.mlp == B200_MLP_DENSE) {
        Widths::widest(w.h, L.ip);
        return B200_OK;
    }
    const int64_t top = c.experts_per_tok;
    Widths::widest(w.h, top * L.ip);
    Widths::widest(w.pairs, top);
    void* p = nullptr;
    if (c.mlp == B200_MLP_SCORED_MOE) {
        w.scored = true;
        const int outputs = pad_width(c.num_experts + c.identity_experts);
        S_TRY(named_bytes(e, &L.router, "router" + sfx, outputs * hp * z));
        if (c.score == B200_SCORE_SOFTMAX) {
            S_TRY(named_bytes(e, &p, "router_correction" + sfx, (c.num_experts + c.identity_experts) * 4ll));
            L.correction = static_cast<float*>(p);
        }
        Widths::widest(w.experts, E);
        Widths::widest(w.router, outputs);
        Widths::widest(w.top, top);
        if (c.shared_intermediate > 0) {
            L.isp = pad_width(c.shared_intermediate);
            const int64_t n_shared = (epilogue_is_gated(c.epilogue) ? 2 : 1) * static_cast<int64_t>(L.isp);
            S_TRY(named_bytes(e, &L.shared_up, "shared_up" + sfx, n_shared * hp * z));
            S_TRY(named_bytes(e, &L.shared_down, "shared_down" + sfx, hp * L.isp * z));
            Widths::widest(w.shared, L.isp);
        }
        return B200_OK;
    }
    S_TRY(named_bytes(e, &p, "expert_table" + sfx, static_cast<int64_t>(e->m.vocab_size) * top * 4));
    L.table = static_cast<int32_t*>(p);
    S_TRY(dev_alloc(e, &p, (Tm * top + 2 * E + 1) * 4, true));
    L.rows = static_cast<int32_t*>(p);
    L.counts = L.rows + Tm * top;
    L.offsets = L.counts + E;
    if (c.num_experts > S->max_experts) S->max_experts = c.num_experts;
    S->routes.push_back(TableRouteLayer{L.table, L.rows, L.counts, L.offsets, c.experts_per_tok, c.num_experts});
    return B200_OK;
}

}  // namespace

int layer_stack_create(b200_engine* e, const b200_stack_config* sc) {
    B200_CHECK_ARG(sc->layers && sc->num_layers > 0, "layer stack: no layers");
    B200_CHECK_ARG(sc->dtype == B200_DTYPE_BF16 || sc->dtype == B200_DTYPE_F32, "layer stack: unknown dtype");
    LayerStack* S = new LayerStack();
    e->stack = S;
    S->dtype = sc->dtype;
    S->esz = sc->dtype == B200_DTYPE_F32 ? 4 : 2;
    S->norm_offset = sc->norm_offset;
    S->logit_scale = sc->logit_scale;
    B200_CHECK_ARG(sc->norm_output >= B200_NORM_INPUT && sc->norm_output <= B200_NORM_BOTH, "layer stack: unknown norm placement");
    B200_CHECK_ARG(sc->num_beside >= 0 && (sc->num_beside == 0 || sc->beside), "layer stack: no mixers to run beside others");
    S->norm_input = sc->norm_output != B200_NORM_OUTPUT;
    S->norm_output = sc->norm_output != B200_NORM_INPUT;
    B200_CHECK_ARG(sc->norm_kind == B200_NORM_RMS || sc->norm_kind == B200_NORM_LAYER, "layer stack: unknown norm");
    S->layer_norm = sc->norm_kind == B200_NORM_LAYER;
    B200_CHECK_ARG(!S->layer_norm || (sc->norm_offset == 0.f && sc->logit_scale == 1.f), "layer stack: layer norms take no offset or scale");
    S->embed_scale = sc->embed_scale == 0.f ? 1.f : sc->embed_scale;
    S->hp = pad_width(e->m.hidden_size);
    S->vocab_p = pad_width(e->m.vocab_size);
    if (const char* v = getenv("B200_LATENT_EXPAND_MIN")) S->expand_min = atoi(v);
    const int64_t hp = S->hp, z = S->esz, Tm = e->max_tokens;
    S_TRY(named_bytes(e, &S->embed, "embed", S->vocab_p * hp * z));
    if (e->m.tie_word_embeddings) {
        S->head = S->embed;
        e->named["lm_head"] = e->named["embed"];
    } else {
        S_TRY(named_bytes(e, &S->head, "lm_head", S->vocab_p * hp * z));
    }
    S_TRY(norm_of(e, "final_norm", "", S->final_norm, S->final_norm_bias));

    Widths w;
    S->latent_rows = e->max_batch > 1024 ? e->max_batch : 1024;
    if (S->latent_rows > e->max_tokens) S->latent_rows = e->max_tokens;
    S->layers.resize(sc->num_layers);
    S->besides.resize(sc->num_beside);
    for (int i = 0; i < sc->num_beside; ++i) S->besides[i].c = sc->beside[i];
    for (int l = 0; l < sc->num_layers; ++l) {
        StackLayer& L = S->layers[l];
        L.c = sc->layers[l];
        const b200_layer_config& c = L.c;
        S_TRY(check_layer(c, l));
        B200_CHECK_ARG(!((S->norm_output || S->layer_norm) && c.mlp == B200_MLP_TABLE_MOE),
                       "layer %d: experts by token id take the RMS norm on their input", l);
        B200_CHECK_ARG(c.mlp != B200_MLP_SCORED_MOE || c.identity_experts == 0 || S->layer_norm,
                       "layer %d: identity experts come with layer norms", l);
        B200_CHECK_ARG(!S->layer_norm || c.beside < 0 || c.join == B200_JOIN_SUM, "layer %d: layer norms do not join mixers", l);
        const std::string sfx = "." + std::to_string(l);
        S_TRY(norm_of(e, "norm1", sfx, L.norm1, L.norm1_bias));
        if (S->norm_input && S->norm_output) S_TRY(norm_of(e, "norm1_out", sfx, L.norm1_out, L.norm1_out_bias));
        B200_CHECK_ARG(c.beside < sc->num_beside, "layer %d: no mixer %d to run beside", l, c.beside);
        if (c.beside >= 0) L.beside = &S->besides[c.beside];
        S_TRY(alloc_layer_mixer(e, L, l, sfx, w));
        if (c.mlp != B200_MLP_NONE) S_TRY(alloc_feed_forward(e, L, sfx, w));
    }
    void* p = nullptr;
    S_TRY(dev_alloc(e, &p, Tm * hp * 4, true));
    S->residual = static_cast<float*>(p);
    S_TRY(dev_alloc(e, &S->x, Tm * hp * z, true));
    S_TRY(dev_alloc(e, &S->y, Tm * hp * z, true));
    S_TRY(dev_alloc(e, &S->joint, Tm * w.joint * z, true));
    S_TRY(dev_alloc(e, &S->cq, Tm * w.cq * z, true));
    S_TRY(dev_alloc(e, &S->q, Tm * w.q * z, true));
    S_TRY(dev_alloc(e, &S->attn, Tm * w.attn * z, true));
    S_TRY(dev_alloc(e, &S->h, Tm * w.h * z, true));
    S_TRY(dev_alloc(e, &S->xp, Tm * w.pairs * hp * z, true));
    S_TRY(dev_alloc(e, &S->ye, Tm * w.pairs * hp * z, true));
    S_TRY(dev_alloc(e, &S->qa, S->latent_rows * w.latent * z, true));
    S_TRY(dev_alloc(e, &S->ol, S->latent_rows * w.latent * z, true));
    S->ws_bytes = w.ws;
    S_TRY(dev_alloc(e, &S->ws, w.ws, true));
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->token_row = static_cast<int32_t*>(p);
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->token_len = static_cast<int32_t*>(p);
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->compact_row = static_cast<int32_t*>(p);
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->compact_len = static_cast<int32_t*>(p);
    if (w.steps > 0) {
        S_TRY(dev_alloc(e, &S->mixed, w.mixed, true));
        S_TRY(dev_alloc(e, &p, w.steps, true));
        S->steps = static_cast<float*>(p);
        S_TRY(dev_alloc(e, &p, w.units, true));
        S->units = static_cast<float*>(p);
        S_TRY(dev_alloc(e, &S->chunks, w.chunks, true));
    }
    if (w.normed_pair) S_TRY(dev_alloc(e, &S->y2, Tm * hp * z, true));
    if (w.mixed_heads > 0) S_TRY(dev_alloc(e, &S->mixed_heads, Tm * w.mixed_heads * z, true));
    if (w.first > 0) S_TRY(dev_alloc(e, &S->first_values, Tm * w.first * z, true));
    if (w.scored) {
        S_TRY(dev_alloc(e, &p, Tm * w.router * 4, true));
        S->router_logits = static_cast<float*>(p);
        S_TRY(dev_alloc(e, &p, Tm * w.top * 4, true));
        S->route_weights = static_cast<float*>(p);
        S_TRY(dev_alloc(e, &p, (2 * Tm * w.top + 3 * w.experts + 1) * 4, true));
        S->route_ids = static_cast<int32_t*>(p);
        S->route_rows = S->route_ids + Tm * w.top;
        S->route_counts = S->route_rows + Tm * w.top;
        S->route_offsets = S->route_counts + 2 * w.experts;
        if (w.shared > 0) {
            S_TRY(dev_alloc(e, &S->shared_h, Tm * w.shared * z, true));
            S_TRY(dev_alloc(e, &S->shared_y, Tm * hp * z, true));
        }
    }
    if (w.any_expand) {
        // room for the pool's tokens (each request rounded up to 64), at most 64 K of them, within 4 GB
        S->expand_cap = e->num_slots + 64ll * e->max_batch;
        if (S->expand_cap > 65536) S->expand_cap = 65536;
        while (S->expand_cap > 4096 && S->expand_cap * (w.xk + w.xv) * 2 > (4ll << 30)) S->expand_cap /= 2;
        S->expand_cap = S->expand_cap / 64 * 64 + 64;
        S_TRY(dev_alloc(e, &S->xc, S->expand_cap * w.xc * 2, true));
        S_TRY(dev_alloc(e, &S->xk, S->expand_cap * w.xk * 2, true));
        S_TRY(dev_alloc(e, &S->xv, S->expand_cap * w.xv * 2, true));
        S_TRY(dev_alloc(e, &p, S->expand_cap * 4, false));
        S->iota = static_cast<int32_t*>(p);
        iota_kernel<<<static_cast<unsigned>((S->expand_cap + 255) / 256), 256>>>(S->iota, S->expand_cap);
        B200_CHECK_LAUNCH();
        // compacted queries and outputs of the requests that stay in the latent space beside expanded ones
        S_TRY(dev_alloc(e, &S->qc, Tm * w.q * z, true));
        S_TRY(dev_alloc(e, &S->ac, Tm * w.attn * z, true));
    }
    const int64_t plan_ints = 3ll * e->max_batch + Tm;
    B200_CHECK_CUDA(cudaMallocHost(&S->plan_host, plan_ints * sizeof(int32_t)));
    S_TRY(dev_alloc(e, &p, plan_ints * 4, true));
    S->plan_dev = static_cast<int32_t*>(p);
    if (!S->routes.empty()) {
        const size_t bytes = S->routes.size() * sizeof(TableRouteLayer);
        S_TRY(dev_alloc(e, &p, static_cast<int64_t>(bytes), false));
        S->routes_dev = static_cast<TableRouteLayer*>(p);
        B200_CHECK_CUDA(cudaMemcpy(p, S->routes.data(), bytes, cudaMemcpyHostToDevice));
    }
    return B200_OK;
}

void layer_stack_destroy(b200_engine* e) {
    if (!e->stack) return;
    if (e->stack->plan_host) cudaFreeHost(e->stack->plan_host);
    delete e->stack;
    e->stack = nullptr;
}

int stack_dtype(const b200_engine* e) { return e->stack->dtype; }
int stack_logits_ld(const b200_engine* e) { return e->stack->vocab_p; }
int stack_row_bytes(const b200_engine* e) { return e->stack->hp * e->stack->esz; }
const void* stack_hidden(const b200_engine* e) { return e->stack->x; }
int32_t* stack_token_row(const b200_engine* e) { return e->stack->token_row; }
int32_t* stack_token_len(const b200_engine* e) { return e->stack->token_len; }
void stack_set_trace(b200_engine* e, float* host) { e->stack->trace = host; }

int layer_stack_plan(b200_engine* e, const b200_step* st, int Bp) {
    LayerStack* S = e->stack;
    S->plan_expanded = S->plan_latent = S->plan_max_extend = S->plan_max_len = 0;
    S->plan_rows = 0;
    S->max_extend = 1;
    if (st->phase != B200_PHASE_PREFILL) return B200_OK;
    int32_t* x_len = S->plan_host;
    int32_t* x_base = x_len + Bp;
    int32_t* g_base = x_base + Bp;
    int32_t* tokens = g_base + Bp;
    int at = 0;
    for (int b = 0; b < Bp; ++b) {
        const int ext = st->extend_lens[b], len = st->cached_lens[b] + ext;
        if (ext > S->max_extend) S->max_extend = ext;
        const int64_t need = (len + 63) / 64 * 64;
        if (ext > S->expand_min && S->plan_rows + need <= S->expand_cap) {
            x_len[b] = len;
            x_base[b] = g_base[b] = static_cast<int32_t>(S->plan_rows);
            S->plan_rows += need;
            ++S->plan_expanded;
            if (ext > S->plan_max_extend) S->plan_max_extend = ext;
            if (len > S->plan_max_len) S->plan_max_len = len;
        } else {
            x_len[b] = 0;      // nothing to do for the expanded kernels
            x_base[b] = 0;
            g_base[b] = -1;
            for (int i = 0; i < ext; ++i) tokens[S->plan_latent++] = at + i;
        }
        at += ext;
    }
    if (S->plan_expanded > 0)
        B200_CHECK_CUDA(cudaMemcpyAsync(S->plan_dev, S->plan_host, (3ll * Bp + S->plan_latent) * sizeof(int32_t),
                                        cudaMemcpyHostToDevice, e->stream));
    return B200_OK;
}

namespace {

int project(b200_engine* e, void* y, const void* x, const void* w, int M, int N, int K, int epilogue, float limit = 0.f,
            const void* bias = nullptr) {
    if (e->stack->dtype == B200_DTYPE_F32)
        return launch_linear_f32(static_cast<float*>(y), static_cast<const float*>(x), static_cast<const float*>(w), M, N, K,
                                 1, nullptr, nullptr, epilogue, e->stream, limit, static_cast<const float*>(bias));
    return launch_linear(y, x, w, bias, M, N, K, K, epilogue, e->status, e->stream, nullptr, limit);
}

int project_heads(b200_engine* e, void* y, const void* x, const void* w, int M, int heads, int N, int K) {
    if (e->stack->dtype == B200_DTYPE_F32)
        return launch_linear_f32(static_cast<float*>(y), static_cast<const float*>(x), static_cast<const float*>(w), M, N, K,
                                 heads, nullptr, nullptr, B200_EPILOGUE_NONE, e->stream);
    return launch_linear_heads(y, x, w, M, heads, N, K, e->status, e->stream);
}

int project_experts(b200_engine* e, void* y, const void* x, const void* w, const StackLayer& L, const int32_t* counts,
                    const int32_t* offsets, int T, int N, int K, int epilogue) {
    const int E = L.c.num_experts;
    if (e->stack->dtype == B200_DTYPE_F32)
        return launch_linear_f32(static_cast<float*>(y), static_cast<const float*>(x), static_cast<const float*>(w), T, N, K,
                                 E, counts, offsets, epilogue, e->stream, L.c.act_limit);
    return launch_grouped_gemm(y, x, w, counts, offsets, E, T, static_cast<int64_t>(T) * L.c.experts_per_tok, N, K,
                               epilogue, e->status, e->stream, L.c.act_limit);
}

// Latent-space attention of `rows` query rows (q and out [rows, heads * dim], tables per row).
int attend_latent(b200_engine* e, const StackLayer& L, void* out, const void* q, const int32_t* row_table,
                  const int32_t* row_len, int rows, bool decode) {
    LayerStack* S = e->stack;
    const int H = L.c.heads;
    for (int r0 = 0; r0 < rows; r0 += S->latent_rows) {
        const int n = rows - r0 < S->latent_rows ? rows - r0 : S->latent_rows;
        const char* qs = static_cast<const char*>(q) + static_cast<int64_t>(r0) * H * L.dp * S->esz;
        char* os = static_cast<char*>(out) + static_cast<int64_t>(r0) * H * L.vp * S->esz;
        S_TRY(project_heads(e, S->qa, qs, L.uk_absorb, n, H, L.rp, L.dp));
        LatentAttention a;
        a.out = S->ol;
        a.q = S->qa;
        a.cache = L.cache;
        a.num_slots = e->num_slots;
        a.page_table = e->page_table;
        a.pt_stride = e->pt_cols;
        a.row_table = row_table + r0;
        a.row_len = row_len + r0;
        a.rows = n;
        a.heads = H;
        a.width = L.rp;
        a.out_width = L.op;
        a.page_size = e->c.page_size;
        a.scale = L.c.score_scale;
        a.only_last_key_new = decode;
        a.workspace = S->ws;
        a.workspace_bytes = S->ws_bytes;
        if (S->dtype == B200_DTYPE_BF16 && latent_attention_tc_supported(a))
            S_TRY(launch_latent_attention_tc(a, e->status, e->stream));
        else
            S_TRY(launch_latent_attention_plain(a, S->dtype, e->status, e->stream));
        S_TRY(project_heads(e, os, S->ol, L.uv, n, H, L.vp, L.op));
    }
    return B200_OK;
}

int attend(b200_engine* e, const StackLayer& L, int phase, int Bp, int T) {
    LayerStack* S = e->stack;
    if (phase == B200_PHASE_DECODE || S->plan_expanded == 0 || !L.can_expand)
        return attend_latent(e, L, S->attn, S->q, S->token_row, S->token_len, T, phase == B200_PHASE_DECODE);
    const int H = L.c.heads;
    const int32_t* x_len = S->plan_dev;
    const int32_t* x_base = x_len + Bp;
    const int32_t* g_base = x_base + Bp;
    const int32_t* tokens = g_base + Bp;
    const int32_t* table_idx = e->meta_dev;
    const int32_t* qo = e->meta_dev + 2 * Bp;
    const int rows = static_cast<int>(S->plan_rows);
    S_TRY(launch_gather_latents(S->xc, L.cache, e->num_slots, e->page_table, e->pt_cols, table_idx, x_len, g_base, Bp,
                                S->plan_max_len, L.rp, e->status, e->stream));
    S_TRY(project(e, S->xk, S->xc, L.uk, rows, H * L.dp, L.rp, B200_EPILOGUE_NONE));
    S_TRY(launch_linear(S->xv, S->xc, L.uv, nullptr, rows, H * L.vp, L.op, L.rp, B200_EPILOGUE_NONE, e->status, e->stream));
    // request b's expanded rows start at x_base[b]: with the identity row as the page table and a row
    // stride of one, "table row x_base[b]" maps position p to x_base[b] + p
    S_TRY(launch_attention_prefill(S->attn, S->q, static_cast<int64_t>(H) * L.dp, L.dp, S->xk, S->xv, rows, S->iota, 1,
                                   x_base, x_len, qo, Bp, S->plan_max_extend, H, H, 64, L.c.score_scale, e->status,
                                   e->stream));
    const int n = S->plan_latent;
    if (n == 0) return B200_OK;
    S_TRY(launch_move_rows(S->qc, S->q, tokens, n, H * L.dp / 8, false, e->stream));
    S_TRY(attend_latent(e, L, S->ac, S->qc, S->compact_row, S->compact_len, n, false));
    return launch_move_rows(S->attn, S->ac, tokens, n, H * L.vp / 8, true, e->stream);
}

int latent_mixer(b200_engine* e, const StackLayer& L, int T) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    const bool own = c.kv_from < 0;
    LatentNorm n;
    n.q_latent = S->cq;
    n.cache = own ? L.cache : nullptr;
    n.joint = S->joint;
    n.q_weight = L.q_norm;
    n.kv_weight = L.kv_norm;
    n.out_loc = e->out_loc;
    n.positions = e->positions;
    n.tokens = T;
    n.q_rank = c.q_rank;
    n.qp = L.qp;
    n.kv_rank = c.kv_rank;
    n.rp = own ? L.rp : 0;
    n.rope_at = latent_rope_at(c.kv_rank);
    n.rope_dim = c.rotary_dim;
    n.max_pos = e->pt_cols;
    n.cos_t = L.cos_t;
    n.sin_t = L.sin_t;
    n.num_slots = e->num_slots;
    n.eps = e->m.rms_norm_eps;
    n.status = e->status;
    S_TRY(project(e, S->joint, S->x, L.down_qkv, T, n.qp + n.rp, S->hp, B200_EPILOGUE_NONE));
    S_TRY(launch_latent_norm_store(n, S->dtype, e->stream));
    S_TRY(project(e, S->q, S->cq, L.uq, T, c.heads * L.dp, L.qp, B200_EPILOGUE_NONE));
    return launch_rotate_pairs(S->q, T, c.heads, L.dp, c.rotary_dim, L.cos_t, L.sin_t, e->positions, e->pt_cols, S->dtype,
                               e->status, e->stream);
}

// A mixer's columns of the joint rows, and its place in the result buffer.
char* joint_of(const LayerStack* S, const StackLayer& L) { return static_cast<char*>(S->joint) + L.joint_at * S->esz; }
char* result_of(const LayerStack* S, const StackLayer& L) { return static_cast<char*>(S->attn) + L.out_at * S->esz; }

int window_prepare(b200_engine* e, const StackLayer& L, int T) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    HeadPrepare a;
    a.joint = joint_of(S, L);
    a.ld = L.joint_ld;
    a.tokens = T;
    a.heads = c.heads;
    a.kv_heads = c.kv_from < 0 ? c.kv_heads : 0;   // (another layer has prepared its keys and values)
    a.dim = c.head_dim;
    a.dp = L.dp;
    a.vp = L.vp;
    a.unit_norm = c.head_norm == B200_HEAD_NORM_UNIT;
    a.value_rotary = c.value_rotary ? c.value_dim : 0;
    a.value_cos = L.value_cos;
    a.value_sin = L.value_sin;
    a.q_weight = L.q_head_norm;
    a.k_weight = L.k_head_norm;
    a.eps = e->m.rms_norm_eps;
    a.rotary_dim = c.rotary_dim;
    a.max_pos = e->pt_cols;
    a.cos_t = L.cos_t;
    a.sin_t = L.sin_t;
    a.positions = e->positions;
    a.out_loc = e->out_loc;
    a.k_cache = L.k_cache;
    a.v_cache = L.v_cache;
    a.num_slots = e->num_slots;
    a.mix = L.mix;
    a.lambda = L.value_mix;
    a.first_values = S->first_values;
    a.status = e->status;
    return launch_head_prepare(a, S->dtype, e->stream);
}

int window_attend(b200_engine* e, const StackLayer& L, int phase, int Bp, int T) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    WindowAttention a;
    a.out = result_of(S, L);
    a.q = joint_of(S, L);
    a.q_st = L.joint_ld;
    a.k_cache = L.k_cache;
    a.v_cache = L.v_cache;
    a.num_slots = e->num_slots;
    a.page_table = e->page_table;
    a.pt_stride = e->pt_cols;
    a.table_idx = e->meta_dev;
    a.seq_lens = e->seq_lens;
    a.qo_indptr = e->meta_dev + 2 * Bp;
    a.row_table = S->token_row;
    a.row_len = S->token_len;
    a.tokens = T;
    a.batch = Bp;
    a.max_extend = S->max_extend;
    a.decode = phase == B200_PHASE_DECODE;
    a.heads = c.heads;
    a.kv_heads = c.kv_heads;
    a.dp = L.dp;
    a.vp = L.vp;
    a.page_size = e->c.page_size;
    a.scale = c.score_scale;
    a.window.size = c.window;
    a.window.keep_first = c.keep_first;
    a.window.chunk = c.chunk;
    a.window.sinks = L.sinks;
    if (c.gate != B200_GATE_NONE) {
        const int64_t own = c.kv_from < 0 ? static_cast<int64_t>(c.kv_heads) * (L.dp + L.vp) : 0;
        a.window.gate = joint_of(S, L) + (static_cast<int64_t>(c.heads) * L.dp + own) * S->esz;
        a.window.gate_st = a.q_st;
        a.window.gate_per_head = c.gate == B200_GATE_HEAD;
    }
    a.window.out_scale = c.out_scale;
    a.window.out_st = L.out_ld;
    if (L.head_mix != nullptr) {
        a.mix.weights = L.head_mix;
        a.mix.rotary = c.value_rotary ? c.value_dim : 0;
        a.mix.max_pos = e->pt_cols;
        a.mix.cos_t = L.value_cos;
        a.mix.sin_t = L.value_sin;
        a.mix.positions = e->positions;
        // vectors of root mean square 1, a little longer for having been rounded
        a.mix.score_bound = c.head_norm == B200_HEAD_NORM_UNIT ? 1.02f * static_cast<float>(c.head_dim) : 0.f;
        a.mix.scratch = S->mixed_heads;
    }
    a.workspace = S->ws;
    a.workspace_bytes = S->ws_bytes;
    a.status = e->status;
    return launch_window_attention(a, S->dtype, e->stream);
}

int linear_mixer(b200_engine* e, const StackLayer& L, int phase, int Bp, int T) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    LinearAttention a = {};
    a.out = S->attn;
    a.joint = S->joint;
    a.joint_ld = L.joint_ld;
    a.tokens = T;
    a.batch = Bp;
    a.decode = phase == B200_PHASE_DECODE ? 1 : 0;
    a.table_idx = e->meta_dev;
    a.cached = e->meta_dev + Bp;
    a.qo_indptr = e->meta_dev + 2 * Bp;
    a.state = L.state;
    a.heads = c.heads;
    a.dim = c.head_dim;
    a.padded_dim = L.dp;
    a.value_dim = c.value_dim;
    a.padded_value_dim = L.vp;
    a.rank = c.decay_rank;
    a.up_ld = L.up_ld;
    a.up = L.decay_up;
    a.bias = L.decay_bias;
    a.norm = L.head_norm;
    a.tau = c.decay_tau;
    a.eps = e->m.rms_norm_eps;
    a.q_scale = static_cast<float>(1.0 / sqrt(static_cast<double>(c.head_dim)));
    return launch_linear_attention(a, S->dtype, e->stream);
}

int recurrence_mixer(b200_engine* e, const StackLayer& L, int phase, int Bp, int T) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    Recurrence a = {};
    a.out = result_of(S, L);
    a.out_ld = L.out_ld;
    a.joint = joint_of(S, L);
    a.joint_ld = L.joint_ld;
    a.rule = rule_of(c.mixer);
    a.gate_cap = c.gate_cap;
    a.memory = L.memory;
    a.tokens = T;
    a.batch = Bp;
    a.max_extend = S->max_extend;
    a.decode = phase == B200_PHASE_DECODE ? 1 : 0;
    a.table_idx = e->meta_dev;
    a.cached = e->meta_dev + Bp;
    a.qo_indptr = e->meta_dev + 2 * Bp;
    a.state = L.state;
    a.conv_state = L.conv_state;
    a.heads = c.heads;
    a.kv_heads = c.kv_heads;
    a.dim = c.head_dim;
    a.padded_dim = L.dp;
    a.value_dim = c.value_dim;
    a.padded_value_dim = L.vp;
    a.taps = c.conv_taps;
    a.norm_groups = c.norm_groups;
    a.conv = L.conv;
    a.conv_bias = L.conv_bias;
    a.decay_log = L.decay_log;
    a.step_bias = L.step_bias;
    a.skip = L.skip;
    a.norm = L.head_norm;
    a.eps = e->m.rms_norm_eps;
    a.out_scale = c.out_scale;
    a.mixed = S->mixed;
    a.steps = S->steps;
    a.units = S->units;
    a.chunks = S->chunks;
    return launch_recurrence(a, S->dtype, e->stream);
}

// Attention launches bracketed by events while the engine is being profiled.
template <typename F>
int timed_attention(b200_engine* e, F launch) {
    const bool timed = e->profile_attention && !e->capturing;
    const int at = e->prof_pairs_recorded;
    if (timed) {
        while (static_cast<int>(e->prof_events.size()) < 2 * (at + 1)) {
            cudaEvent_t ev = nullptr;
            B200_CHECK_CUDA(cudaEventCreate(&ev));
            e->prof_events.push_back(ev);
        }
        B200_CHECK_CUDA(cudaEventRecord(e->prof_events[2 * at], e->stream));
    }
    S_TRY(launch());
    if (timed) {
        B200_CHECK_CUDA(cudaEventRecord(e->prof_events[2 * at + 1], e->stream));
        e->prof_pairs_recorded = at + 1;
    }
    return B200_OK;
}

// A mixer between the joint projection and the output projection.
int run_mixer(b200_engine* e, const StackLayer& L, int phase, int Bp, int T) {
    if (L.c.mixer == B200_MIXER_LINEAR_ATTENTION) return linear_mixer(e, L, phase, Bp, T);
    if (is_recurrence(L.c.mixer)) return recurrence_mixer(e, L, phase, Bp, T);
    S_TRY(window_prepare(e, L, T));
    return timed_attention(e, [&] { return window_attend(e, L, phase, Bp, T); });
}

// S->x through the layer's mixer, or both of them, to S->y (under B200_JOIN_NORMED the right one's result to S->y2).
int mix(b200_engine* e, int l, int phase, int Bp, int T) {
    LayerStack* S = e->stack;
    const StackLayer& L = S->layers[l];
    if (L.c.mixer == B200_MIXER_LATENT_ATTENTION) {
        S_TRY(latent_mixer(e, L, T));
        S_TRY(timed_attention(e, [&] { return attend(e, L, phase, Bp, T); }));
    } else {
        S_TRY(project(e, S->joint, S->x, L.joint, T, static_cast<int>(L.joint_ld), S->hp, B200_EPILOGUE_NONE, 0.f, L.joint_bias));
        S_TRY(run_mixer(e, L, phase, Bp, T));
        if (L.beside != nullptr) S_TRY(run_mixer(e, *L.beside, phase, Bp, T));
        if (L.side_norm != nullptr)
            S_TRY(project(e, S->y2, result_of(S, *L.beside), L.beside->o, T, S->hp, static_cast<int>(L.beside->out_ld),
                          B200_EPILOGUE_NONE));
    }
    return project(e, S->y, S->attn, L.o, T, S->hp, static_cast<int>(L.out_ld), B200_EPILOGUE_NONE);
}

// S->x through a dense layer to S->y, or through the experts its scores choose to S->ye (and the expert that
// every token uses to S->shared_y).
int feed_forward(b200_engine* e, const StackLayer& L, int T) {
    LayerStack* S = e->stack;
    const b200_layer_config& c = L.c;
    const int hp = S->hp, gated = epilogue_is_gated(c.epilogue) ? 2 : 1;
    if (c.mlp == B200_MLP_DENSE) {
        S_TRY(project(e, S->h, S->x, L.up, T, gated * L.ip, hp, c.epilogue, c.act_limit));
        return project(e, S->y, S->h, L.down, T, hp, L.ip, B200_EPILOGUE_NONE);
    }
    const int ep = pad_width(c.num_experts + c.identity_experts);
    S_TRY(project(e, S->router_logits, S->x, L.router, T, ep, hp,
                  S->dtype == B200_DTYPE_F32 ? B200_EPILOGUE_NONE : B200_EPILOGUE_F32));
    ScoreRoute r;
    r.logits = S->router_logits;
    r.ld = ep;
    r.tokens = T;
    r.experts = c.num_experts;
    r.top = c.experts_per_tok;
    r.groups = c.router_groups;
    r.keep = c.router_keep;
    r.scale = c.router_scale;
    r.score = c.score;
    r.identity = c.identity_experts;
    r.correction = L.correction;
    r.ids = S->route_ids;
    r.weights = S->route_weights;
    r.counts = S->route_counts;
    S_TRY(launch_score_route(r, e->stream));
    S_TRY(launch_score_place(S->xp, S->x, hp * S->esz, r, S->route_rows, S->route_counts + c.num_experts, S->route_offsets,
                             e->stream));
    S_TRY(project_experts(e, S->h, S->xp, L.up, L, r.counts, S->route_offsets, T, gated * L.ip, hp, c.epilogue));
    S_TRY(project_experts(e, S->ye, S->h, L.down, L, r.counts, S->route_offsets, T, hp, L.ip, B200_EPILOGUE_NONE));
    if (L.isp == 0) return B200_OK;
    S_TRY(project(e, S->shared_h, S->x, L.shared_up, T, gated * L.isp, hp, c.epilogue, c.shared_act_limit));
    return project(e, S->shared_y, S->shared_h, L.shared_down, T, hp, L.isp, B200_EPILOGUE_NONE);
}

// What a block has left behind for the residual kernel that follows it.
void take_block(LayerStack* S, const StackLayer* experts, const StackLayer* pair, int T, ResidualPostNorm& rn) {
    rn.init = false;
    rn.src = experts ? S->ye : S->y;
    rn.src_rows = experts ? S->route_rows : nullptr;
    rn.src_weights = experts ? S->route_weights : nullptr;
    rn.src_top = experts ? experts->c.experts_per_tok : 1;
    rn.src_count = static_cast<int64_t>(T) * rn.src_top;
    rn.self = S->x;    // of identity experts
    rn.src2 = pair ? S->y2 : experts && experts->isp > 0 ? S->shared_y : nullptr;
    rn.pair_weight = pair ? pair->side_norm : nullptr;
    rn.pair_weight2 = pair ? pair->beside->side_norm : nullptr;
    rn.pair_scale = 0.5f;
}

}  // namespace

int layer_stack_enqueue(b200_engine* e, int phase, int Bp, int T, bool pdl) {
    LayerStack* S = e->stack;
    cudaStream_t s = e->stream;
    const int hp = S->hp, width = e->m.hidden_size;
    const int num_layers = static_cast<int>(S->layers.size());
    e->prof_pairs_recorded = 0;
    if (!S->routes.empty())
        S_TRY(launch_table_route(S->routes_dev, static_cast<int>(S->routes.size()), S->max_experts, e->input_ids, T,
                                 e->m.vocab_size, e->status, s));
    if (S->plan_expanded > 0 && S->plan_latent > 0)
        B200_CHECK_CUDA(launch_kernel(compact_rows_kernel, dim3(div_ceil(S->plan_latent, 256)), dim3(256), 0, s,
                                      dim3(1, 1, 1), S->compact_row, S->compact_len,
                                      static_cast<const int32_t*>(S->token_row), static_cast<const int32_t*>(S->token_len),
                                      static_cast<const int32_t*>(S->plan_dev + 3 * Bp), S->plan_latent));
    // What the next residual update adds: at first the embedding rows of the tokens.  `rn` drives the kernel with
    // the norm on what is read, `post` the one with the norm on what is added (and with weighted sources).
    ResidualNorm rn;
    rn.residual = S->residual;
    rn.weight_offset = S->norm_offset;
    rn.tokens = T;
    rn.width = width;
    rn.padded = hp;
    rn.eps = e->m.rms_norm_eps;
    rn.src = S->embed;
    rn.src_rows = e->input_ids;
    rn.src_top = 1;
    rn.src_count = e->m.vocab_size;
    rn.init = true;
    ResidualPostNorm post;
    post.out = S->x;
    post.residual = S->residual;
    post.src = S->embed;
    post.src_rows = e->input_ids;
    post.src_count = e->m.vocab_size;
    post.layer = S->layer_norm;
    post.src_scale = rn.src_scale = S->embed_scale;
    post.init = true;
    post.weight_offset = S->norm_offset;
    post.tokens = T;
    post.width = width;
    post.padded = hp;
    post.eps = e->m.rms_norm_eps;
    const StackLayer* scored = nullptr;   // the last block was this layer's scored experts
    const StackLayer* pair = nullptr;     // the last block was this layer's two mixers, normalised each
    const void *own_norm = nullptr, *own_bias = nullptr;   // norm_output: the norm of the last block's output
    auto add_plain = [&]() {
        rn.src = S->y;
        rn.src_rows = nullptr;
        rn.src_top = 1;
        rn.src_count = T;
        rn.src_scale = 1.f;
        rn.init = false;
        scored = pair = nullptr;
    };
    // Adds the last block and leaves what the next one reads: normalised with `weight`, or as it is.
    auto advance = [&](const void* weight, const void* bias, void* out, const int32_t* rows, int top, float out_scale,
                       const StackLayer* next_scored) -> int {
        post.clear = next_scored ? S->route_counts : nullptr;
        post.clear_count = next_scored ? 2 * next_scored->c.num_experts : 0;
        if (!S->norm_output && !S->layer_norm && scored == nullptr && pair == nullptr && next_scored == nullptr) {
            rn.weight = weight;
            rn.out = out;
            rn.out_rows = rows;
            rn.out_top = top;
            rn.out_scale = out_scale;
            return launch_residual_norm(rn, S->dtype, e->status, s);
        }
        if (!rn.init) take_block(S, scored, pair, T, post);
        post.add_weight = own_norm;
        post.add_bias = own_bias;
        post.out_weight = weight;
        post.out_bias = bias;
        post.out_scale = out_scale;
        return launch_residual_post_norm(post, S->dtype, e->status, s);
    };
    // (the residual after layer l is complete once the kernel that opens what follows it has run)
    auto traced = [&](int layers_done) -> int {
        if (S->trace == nullptr || phase != B200_PHASE_PREFILL || layers_done == 0) return B200_OK;
        B200_CHECK_CUDA(cudaMemcpy2DAsync(S->trace + static_cast<int64_t>(layers_done - 1) * T * width, width * 4ull,
                                          S->residual, hp * 4ull, width * 4ull, T, cudaMemcpyDeviceToHost, s));
        return B200_OK;
    };
    for (int l = 0; l < num_layers; ++l) {
        const StackLayer& L = S->layers[l];
        const b200_layer_config& c = L.c;
        // The first norm is launched as an ordinary dependent of what prepares the step, so that every
        // kernel after it finds positions, slots and lengths complete even ahead of its own wait.
        S_TRY(advance(S->norm_input ? L.norm1 : nullptr, L.norm1_bias, S->x, nullptr, 1, 1.f, nullptr));
        if (l == 0) set_pdl_launches(pdl);
        S_TRY(traced(l));
        S_TRY(mix(e, l, phase, Bp, T));
        add_plain();
        if (L.side_norm != nullptr) pair = &L;
        if (S->norm_output) {
            own_norm = S->norm_input ? L.norm1_out : L.norm1;
            own_bias = S->norm_input ? L.norm1_out_bias : L.norm1_bias;
        }
        if (c.mlp == B200_MLP_NONE) continue;
        if (c.mlp == B200_MLP_TABLE_MOE) {
            const int n_up = (epilogue_is_gated(c.epilogue) ? 2 : 1) * L.ip;
            S_TRY(advance(L.norm2, nullptr, S->xp, L.rows, c.experts_per_tok, 1.f, nullptr));
            S_TRY(project_experts(e, S->h, S->xp, L.up, L, L.counts, L.offsets, T, n_up, hp, c.epilogue));
            S_TRY(project_experts(e, S->ye, S->h, L.down, L, L.counts, L.offsets, T, hp, L.ip, B200_EPILOGUE_NONE));
            pair = nullptr;
            rn.src = S->ye;
            rn.src_rows = L.rows;
            rn.src_top = c.experts_per_tok;
            rn.src_count = static_cast<int64_t>(T) * c.experts_per_tok;
            rn.src_scale = 1.f / static_cast<float>(c.experts_per_tok);
            rn.init = false;
            continue;
        }
        S_TRY(advance(S->norm_input ? L.norm2 : nullptr, L.norm2_bias, S->x, nullptr, 1, 1.f, c.mlp == B200_MLP_SCORED_MOE ? &L : nullptr));
        S_TRY(feed_forward(e, L, T));
        add_plain();
        if (c.mlp == B200_MLP_SCORED_MOE) scored = &L;
        if (S->norm_output) {
            own_norm = S->norm_input ? L.norm2_out : L.norm2;
            own_bias = S->norm_input ? L.norm2_out_bias : L.norm2_bias;
        }
    }
    S_TRY(advance(S->final_norm, S->final_norm_bias, S->x, nullptr, 1, S->logit_scale, nullptr));
    return traced(num_layers);
}

int layer_stack_head(b200_engine* e, void* logits, const void* rows, int count) {
    LayerStack* S = e->stack;
    return project(e, logits, rows, S->head, count, S->vocab_p, S->hp, B200_EPILOGUE_NONE);
}

}  // namespace b200

extern "C" {

int b200_pad_width(int n) { return b200::pad_width(n); }
int b200_pad_head_dim(int n) { return b200::pad_head_dim(n); }
int b200_pad_latent(int n) { return b200::pad_latent(n); }
int b200_latent_rope_at(int kv_rank) { return b200::latent_rope_at(kv_rank); }

}  // extern "C"
