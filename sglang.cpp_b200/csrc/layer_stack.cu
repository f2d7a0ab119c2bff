// Models whose layers are listed one by one: allocation of their weights and latent pools, the per-step
// plan, and the layer stack the step runner (engine.cu) enqueues between its token preparation and its
// output head.
//
// Per layer, on T tokens (fp32 residual stream r, everything else in the stack's dtype):
//     x  = norm(r += previous block)              one kernel, residual.cu
//     [cq | c] = x W_down                         both latents in one GEMM
//     cq, pool[slot] = norm(cq), norm(c)          latent_attention.cu
//     q  = cq W_uq
//     o  = attention(q, pool)                     in the latent space, or over expanded keys and values
//     y  = o W_o
//     x  = norm(r += y), to the expert-sorted rows when the feed-forward is a mixture of experts
//     y  = feed-forward(x)
// The placement of tokens on experts depends on token ids only and is laid out for all layers at once
// before the first.
//
// Attention has two forms.  In the latent space (decode steps, short extensions) the per-head projections
// are applied to the query and to the result.  Extensions of more than `expand_min` tokens expand keys and
// values of the whole request once (two GEMMs) into a scratch that the prefill kernel of the
// grouped-query models reads as if it were its paged pool.  A batch may hold both kinds of requests.
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
}  // namespace

struct StackLayer {
    b200_layer_config c;
    int qp = 0, rp = 0, dp = 0, vp = 0, ip = 0;   // padded sizes
    void *norm1 = nullptr, *norm2 = nullptr, *down_qkv = nullptr, *q_norm = nullptr, *kv_norm = nullptr, *uq = nullptr,
         *uk = nullptr, *uk_absorb = nullptr, *uv = nullptr, *o = nullptr, *up = nullptr, *down = nullptr;
    int32_t* table = nullptr;
    void* cache = nullptr;
    int32_t *rows = nullptr, *counts = nullptr, *offsets = nullptr;   // expert placement of this step
    bool can_expand = false;
};

struct LayerStack {
    std::vector<StackLayer> layers;
    int dtype = B200_DTYPE_BF16;
    int esz = 2;            // bytes per element
    int hp = 0, vocab_p = 0;
    float norm_offset = 0.f, logit_scale = 1.f;
    void *embed = nullptr, *head = nullptr, *final_norm = nullptr;
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

int check_layer(const b200_layer_config& c, int l) {
    B200_CHECK_ARG(c.mixer == B200_MIXER_LATENT_ATTENTION, "layer %d: unknown mixer %d", l, c.mixer);
    B200_CHECK_ARG(c.heads > 0 && c.head_dim > 0 && c.value_dim > 0 && c.q_rank > 0 && c.kv_rank > 0,
                   "layer %d: latent attention needs positive sizes", l);
    B200_CHECK_ARG(c.mlp >= B200_MLP_NONE && c.mlp <= B200_MLP_TABLE_MOE, "layer %d: unknown feed-forward %d", l, c.mlp);
    if (c.mlp == B200_MLP_NONE) return B200_OK;
    B200_CHECK_ARG(c.intermediate > 0, "layer %d: feed-forward size must be positive", l);
    B200_CHECK_ARG(c.epilogue > B200_EPILOGUE_NONE && c.epilogue <= B200_EPILOGUE_RELU2, "layer %d: unknown activation", l);
    if (c.mlp == B200_MLP_TABLE_MOE)
        B200_CHECK_ARG(c.num_experts > 0 && c.num_experts <= kMaxTableExperts && c.experts_per_tok > 0 &&
                           c.experts_per_tok <= c.num_experts,
                       "layer %d: %d of %d experts (at most %d)", l, c.experts_per_tok, c.num_experts, kMaxTableExperts);
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
    S_TRY(named_bytes(e, &S->final_norm, "final_norm", hp * z));

    int64_t joint = 0, cq = 0, q = 0, attn = 0, h = 0, pairs = 0, latent = 0, xk = 0, xv = 0, xc = 0, ws = 0;
    S->latent_rows = e->max_batch > 1024 ? e->max_batch : 1024;
    if (S->latent_rows > e->max_tokens) S->latent_rows = e->max_tokens;
    bool any_expand = false;
    auto widest = [](int64_t& a, int64_t b) { if (b > a) a = b; };
    S->layers.resize(sc->num_layers);
    for (int l = 0; l < sc->num_layers; ++l) {
        StackLayer& L = S->layers[l];
        L.c = sc->layers[l];
        const b200_layer_config& c = L.c;
        S_TRY(check_layer(c, l));
        L.qp = pad_width(c.q_rank);
        L.rp = pad_latent(c.kv_rank);
        L.dp = pad_head_dim(c.head_dim);
        L.vp = pad_head_dim(c.value_dim);
        const std::string sfx = "." + std::to_string(l);
        const int64_t H = c.heads, qp = L.qp, rp = L.rp, dp = L.dp, vp = L.vp;
        S_TRY(named_bytes(e, &L.norm1, "norm1" + sfx, hp * z));
        S_TRY(named_bytes(e, &L.down_qkv, "down_qkv" + sfx, (qp + rp) * hp * z));
        S_TRY(named_bytes(e, &L.q_norm, "q_latent_norm" + sfx, qp * z));
        S_TRY(named_bytes(e, &L.kv_norm, "kv_latent_norm" + sfx, rp * z));
        S_TRY(named_bytes(e, &L.uq, "uq" + sfx, H * dp * qp * z));
        S_TRY(named_bytes(e, &L.uk_absorb, "uk_absorb" + sfx, H * rp * dp * z));
        S_TRY(named_bytes(e, &L.uv, "uv" + sfx, H * vp * rp * z));
        S_TRY(named_bytes(e, &L.o, "o" + sfx, hp * H * vp * z));
        S_TRY(named_bytes(e, &L.cache, "latent_cache" + sfx, e->num_slots * rp * z));
        // what the prefill kernel of the grouped-query models takes (and its positive score scale)
        L.can_expand = S->dtype == B200_DTYPE_BF16 && dp == 128 && vp == 128 && c.score_scale > 0.f && H <= 65535;
        if (L.can_expand) S_TRY(named_bytes(e, &L.uk, "uk" + sfx, H * dp * rp * z));
        any_expand |= L.can_expand;
        widest(joint, qp + rp);
        widest(cq, qp);
        widest(q, H * dp);
        widest(attn, H * vp);
        widest(latent, H * rp);
        widest(ws, latent_attention_workspace_bytes(S->latent_rows, c.heads, L.rp));
        if (L.can_expand) {
            widest(xk, H * dp);
            widest(xv, H * vp);
            widest(xc, rp);
        }
        if (c.mlp == B200_MLP_NONE) continue;
        L.ip = pad_width(c.intermediate);
        const int64_t n_up = (epilogue_is_gated(c.epilogue) ? 2 : 1) * static_cast<int64_t>(L.ip);
        const int64_t E = c.mlp == B200_MLP_TABLE_MOE ? c.num_experts : 1;
        S_TRY(named_bytes(e, &L.norm2, "norm2" + sfx, hp * z));
        S_TRY(named_bytes(e, &L.up, "mlp_up" + sfx, E * n_up * hp * z));
        S_TRY(named_bytes(e, &L.down, "mlp_down" + sfx, E * hp * L.ip * z));
        if (c.mlp == B200_MLP_DENSE) {
            widest(h, L.ip);
            continue;
        }
        const int64_t top = c.experts_per_tok;
        void* p = nullptr;
        S_TRY(named_bytes(e, &p, "expert_table" + sfx, static_cast<int64_t>(e->m.vocab_size) * top * 4));
        L.table = static_cast<int32_t*>(p);
        S_TRY(dev_alloc(e, &p, (Tm * top + 2 * E + 1) * 4, true));
        L.rows = static_cast<int32_t*>(p);
        L.counts = L.rows + Tm * top;
        L.offsets = L.counts + E;
        widest(h, top * L.ip);
        widest(pairs, top);
        if (c.num_experts > S->max_experts) S->max_experts = c.num_experts;
        S->routes.push_back(TableRouteLayer{L.table, L.rows, L.counts, L.offsets, c.experts_per_tok, c.num_experts});
    }
    void* p = nullptr;
    S_TRY(dev_alloc(e, &p, Tm * hp * 4, true));
    S->residual = static_cast<float*>(p);
    S_TRY(dev_alloc(e, &S->x, Tm * hp * z, true));
    S_TRY(dev_alloc(e, &S->y, Tm * hp * z, true));
    S_TRY(dev_alloc(e, &S->joint, Tm * joint * z, true));
    S_TRY(dev_alloc(e, &S->cq, Tm * cq * z, true));
    S_TRY(dev_alloc(e, &S->q, Tm * q * z, true));
    S_TRY(dev_alloc(e, &S->attn, Tm * attn * z, true));
    S_TRY(dev_alloc(e, &S->h, Tm * h * z, true));
    S_TRY(dev_alloc(e, &S->xp, Tm * pairs * hp * z, true));
    S_TRY(dev_alloc(e, &S->ye, Tm * pairs * hp * z, true));
    S_TRY(dev_alloc(e, &S->qa, S->latent_rows * latent * z, true));
    S_TRY(dev_alloc(e, &S->ol, S->latent_rows * latent * z, true));
    S->ws_bytes = ws;
    S_TRY(dev_alloc(e, &S->ws, ws, true));
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->token_row = static_cast<int32_t*>(p);
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->token_len = static_cast<int32_t*>(p);
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->compact_row = static_cast<int32_t*>(p);
    S_TRY(dev_alloc(e, &p, Tm * 4, true));
    S->compact_len = static_cast<int32_t*>(p);
    if (any_expand) {
        // room for the pool's tokens (each request rounded up to 64), at most 64 K of them, within 4 GB
        S->expand_cap = e->num_slots + 64ll * e->max_batch;
        if (S->expand_cap > 65536) S->expand_cap = 65536;
        while (S->expand_cap > 4096 && S->expand_cap * (xk + xv) * 2 > (4ll << 30)) S->expand_cap /= 2;
        S->expand_cap = S->expand_cap / 64 * 64 + 64;
        S_TRY(dev_alloc(e, &S->xc, S->expand_cap * xc * 2, true));
        S_TRY(dev_alloc(e, &S->xk, S->expand_cap * xk * 2, true));
        S_TRY(dev_alloc(e, &S->xv, S->expand_cap * xv * 2, true));
        S_TRY(dev_alloc(e, &p, S->expand_cap * 4, false));
        S->iota = static_cast<int32_t*>(p);
        iota_kernel<<<static_cast<unsigned>((S->expand_cap + 255) / 256), 256>>>(S->iota, S->expand_cap);
        B200_CHECK_LAUNCH();
        // compacted queries and outputs of the requests that stay in the latent space beside expanded ones
        S_TRY(dev_alloc(e, &S->qc, Tm * q * z, true));
        S_TRY(dev_alloc(e, &S->ac, Tm * attn * z, true));
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
    if (st->phase != B200_PHASE_PREFILL) return B200_OK;
    int32_t* x_len = S->plan_host;
    int32_t* x_base = x_len + Bp;
    int32_t* g_base = x_base + Bp;
    int32_t* tokens = g_base + Bp;
    int at = 0;
    for (int b = 0; b < Bp; ++b) {
        const int ext = st->extend_lens[b], len = st->cached_lens[b] + ext;
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

int project(b200_engine* e, void* y, const void* x, const void* w, int M, int N, int K, int epilogue) {
    if (e->stack->dtype == B200_DTYPE_F32)
        return launch_linear_f32(static_cast<float*>(y), static_cast<const float*>(x), static_cast<const float*>(w), M, N, K,
                                 1, nullptr, nullptr, epilogue, e->stream);
    return launch_linear(y, x, w, nullptr, M, N, K, K, epilogue, e->status, e->stream);
}

int project_heads(b200_engine* e, void* y, const void* x, const void* w, int M, int heads, int N, int K) {
    if (e->stack->dtype == B200_DTYPE_F32)
        return launch_linear_f32(static_cast<float*>(y), static_cast<const float*>(x), static_cast<const float*>(w), M, N, K,
                                 heads, nullptr, nullptr, B200_EPILOGUE_NONE, e->stream);
    return launch_linear_heads(y, x, w, M, heads, N, K, e->status, e->stream);
}

int project_experts(b200_engine* e, void* y, const void* x, const void* w, const StackLayer& L, int T, int N, int K,
                    int epilogue) {
    const int E = L.c.num_experts;
    if (e->stack->dtype == B200_DTYPE_F32)
        return launch_linear_f32(static_cast<float*>(y), static_cast<const float*>(x), static_cast<const float*>(w), T, N, K,
                                 E, L.counts, L.offsets, epilogue, e->stream);
    return launch_grouped_gemm(y, x, w, L.counts, L.offsets, E, T, static_cast<int64_t>(T) * L.c.experts_per_tok, N, K,
                               epilogue, e->status, e->stream);
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
        a.page_size = e->c.page_size;
        a.scale = L.c.score_scale;
        a.only_last_key_new = decode;
        a.workspace = S->ws;
        a.workspace_bytes = S->ws_bytes;
        if (S->dtype == B200_DTYPE_BF16 && latent_attention_tc_supported(a))
            S_TRY(launch_latent_attention_tc(a, e->status, e->stream));
        else
            S_TRY(launch_latent_attention_plain(a, S->dtype, e->status, e->stream));
        S_TRY(project_heads(e, os, S->ol, L.uv, n, H, L.vp, L.rp));
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
    S_TRY(project(e, S->xv, S->xc, L.uv, rows, H * L.vp, L.rp, B200_EPILOGUE_NONE));
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

}  // namespace

int layer_stack_enqueue(b200_engine* e, int phase, int Bp, int T, bool pdl) {
    LayerStack* S = e->stack;
    cudaStream_t s = e->stream;
    const int hp = S->hp, width = e->m.hidden_size;
    const int num_layers = static_cast<int>(S->layers.size());
    if (!S->routes.empty())
        S_TRY(launch_table_route(S->routes_dev, static_cast<int>(S->routes.size()), S->max_experts, e->input_ids, T,
                                 e->m.vocab_size, e->status, s));
    if (S->plan_expanded > 0 && S->plan_latent > 0)
        B200_CHECK_CUDA(launch_kernel(compact_rows_kernel, dim3(div_ceil(S->plan_latent, 256)), dim3(256), 0, s,
                                      dim3(1, 1, 1), S->compact_row, S->compact_len,
                                      static_cast<const int32_t*>(S->token_row), static_cast<const int32_t*>(S->token_len),
                                      static_cast<const int32_t*>(S->plan_dev + 3 * Bp), S->plan_latent));
    // What the next residual update adds: at first the embedding rows of the tokens.
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
    auto add_plain = [&]() {
        rn.src = S->y;
        rn.src_rows = nullptr;
        rn.src_top = 1;
        rn.src_count = T;
        rn.src_scale = 1.f;
        rn.init = false;
    };
    auto norm_to = [&](const void* weight, void* out, const int32_t* rows, int top, float out_scale) -> int {
        rn.weight = weight;
        rn.out = out;
        rn.out_rows = rows;
        rn.out_top = top;
        rn.out_scale = out_scale;
        return launch_residual_norm(rn, S->dtype, e->status, s);
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
        S_TRY(norm_to(L.norm1, S->x, nullptr, 1, 1.f));
        if (l == 0) set_pdl_launches(pdl);
        S_TRY(traced(l));
        S_TRY(project(e, S->joint, S->x, L.down_qkv, T, L.qp + L.rp, hp, B200_EPILOGUE_NONE));
        S_TRY(launch_latent_norm_store(S->cq, L.cache, S->joint, L.q_norm, L.kv_norm, e->out_loc, T, c.q_rank, L.qp,
                                       c.kv_rank, L.rp, e->num_slots, e->m.rms_norm_eps, S->dtype, e->status, s));
        S_TRY(project(e, S->q, S->cq, L.uq, T, c.heads * L.dp, L.qp, B200_EPILOGUE_NONE));
        const bool timed = e->profile_attention && !e->capturing;
        if (timed) {
            while (static_cast<int>(e->prof_events.size()) < 2 * num_layers) {
                cudaEvent_t ev = nullptr;
                B200_CHECK_CUDA(cudaEventCreate(&ev));
                e->prof_events.push_back(ev);
            }
            B200_CHECK_CUDA(cudaEventRecord(e->prof_events[2 * l], s));
        }
        S_TRY(attend(e, L, phase, Bp, T));
        if (timed) {
            B200_CHECK_CUDA(cudaEventRecord(e->prof_events[2 * l + 1], s));
            e->prof_pairs_recorded = l + 1;
        }
        S_TRY(project(e, S->y, S->attn, L.o, T, hp, c.heads * L.vp, B200_EPILOGUE_NONE));
        add_plain();
        if (c.mlp == B200_MLP_NONE) continue;
        const int n_up = (epilogue_is_gated(c.epilogue) ? 2 : 1) * L.ip;
        if (c.mlp == B200_MLP_DENSE) {
            S_TRY(norm_to(L.norm2, S->x, nullptr, 1, 1.f));
            S_TRY(project(e, S->h, S->x, L.up, T, n_up, hp, c.epilogue));
            S_TRY(project(e, S->y, S->h, L.down, T, hp, L.ip, B200_EPILOGUE_NONE));
            add_plain();
        } else {
            S_TRY(norm_to(L.norm2, S->xp, L.rows, c.experts_per_tok, 1.f));
            S_TRY(project_experts(e, S->h, S->xp, L.up, L, T, n_up, hp, c.epilogue));
            S_TRY(project_experts(e, S->ye, S->h, L.down, L, T, hp, L.ip, B200_EPILOGUE_NONE));
            rn.src = S->ye;
            rn.src_rows = L.rows;
            rn.src_top = c.experts_per_tok;
            rn.src_count = static_cast<int64_t>(T) * c.experts_per_tok;
            rn.src_scale = 1.f / static_cast<float>(c.experts_per_tok);
            rn.init = false;
        }
    }
    S_TRY(norm_to(S->final_norm, S->x, nullptr, 1, S->logit_scale));
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

}  // extern "C"
