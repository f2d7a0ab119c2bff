// Mixture-of-experts layer: router top-k, token permute, grouped expert GEMMs, weighted combine.
//
// Stands where MoELayer::forward does (src/moe/moe.cc:36-96).  The reference walks
// top_k x num_experts host-synchronised iterations; here one step is six launches with no host
// involvement: route (softmax + top-k per token, expert histogram) -> scan -> scatter (rows
// grouped by expert) -> grouped gate_up GEMM with the gated activation in its epilogue ->
// grouped down GEMM -> combine in the reference's accumulation order (k ascending, bf16 after
// every multiply and add, as index_add_ on bf16 tensors does).
#include "common.cuh"
#include "kernels.h"

namespace b200 {
namespace {

constexpr int kMaxExpertsPerLane = 8;  // num_experts <= 256
constexpr int kMaxTopK = 16;

// One warp per token.
__global__ void __launch_bounds__(128)
moe_route_kernel(const __nv_bfloat16* __restrict__ logits, int tokens, int E, int top_k, int renorm,
                 int32_t* __restrict__ ids, float* __restrict__ weights, int32_t* __restrict__ counts) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int lane = threadIdx.x & 31;
    const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (t >= tokens) return;
    const __nv_bfloat16* row = logits + static_cast<int64_t>(t) * E;
    float v[kMaxExpertsPerLane];
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < kMaxExpertsPerLane; ++i) {
        const int e = lane + i * 32;
        v[i] = e < E ? __bfloat162float(row[e]) : -INFINITY;
        mx = fmaxf(mx, v[i]);
    }
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < kMaxExpertsPerLane; ++i) {
        v[i] = (lane + i * 32) < E ? __expf(v[i] - mx) : -1.f;  // -1 marks "not a candidate"
        if (v[i] > 0.f) sum += v[i];
    }
    sum = warp_sum(sum);
    const float inv = 1.f / sum;
    float wsel[kMaxTopK];
    int isel[kMaxTopK];
    float wsum = 0.f;
    for (int k = 0; k < top_k; ++k) {
        // Largest remaining probability; the lower expert index wins ties.
        float best = -1.f;
        int bi = 0x7fffffff;
#pragma unroll
        for (int i = 0; i < kMaxExpertsPerLane; ++i)
            if (v[i] > best) {
                best = v[i];
                bi = lane + i * 32;
            }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) {
                best = ob;
                bi = oi;
            }
        }
        if ((bi & 31) == lane) v[bi >> 5] = -1.f;
        wsel[k] = best * inv;
        isel[k] = bi;
        wsum += wsel[k];
    }
    if (lane == 0) {
        for (int k = 0; k < top_k; ++k) {
            float w = wsel[k];
            if (renorm) w = w / (wsum + 1e-8f);
            ids[t * top_k + k] = isel[k];
            weights[t * top_k + k] = round_bf16(w);  // the reference casts the weights to bf16
            atomicAdd(&counts[isel[k]], 1);
        }
    }
}

// Row ranges of the experts [e_begin, e_begin + e_count) this call computes (all of them unless
// the experts are partitioned over ranks); every other expert gets offset -1 = "not here".
__global__ void __launch_bounds__(256)
moe_scan_kernel(const int32_t* __restrict__ counts, int32_t* __restrict__ offsets,
                int32_t* __restrict__ cursor, int E, int e_begin, int e_count) {
    pdl_launch_dependents();
    pdl_wait_prior();
    __shared__ int s[256];
    const int e = threadIdx.x;
    const bool local = e >= e_begin && e < e_begin + e_count;
    s[e] = (e < E && local) ? counts[e] : 0;
    __syncthreads();
    if (threadIdx.x == 0) {
        int run = 0;
        for (int i = 0; i < E; ++i) {
            const int c = s[i];
            s[i] = run;
            run += c;
        }
        offsets[E] = run;
    }
    __syncthreads();
    if (e < E) {
        offsets[e] = local ? s[e] : -1;
        cursor[e] = 0;
    }
}

// One CTA per (token, k) pair: claim a row in the expert's range and copy the token there.
__global__ void __launch_bounds__(128)
moe_scatter_kernel(const uint4* __restrict__ hidden, uint4* __restrict__ xp,
                   const int32_t* __restrict__ ids, const int32_t* __restrict__ offsets,
                   int32_t* __restrict__ cursor, int32_t* __restrict__ pos, int top_k, int vec_per_row) {
    pdl_launch_dependents();
    pdl_wait_prior();
    __shared__ int s_row;
    const int pair = blockIdx.x;
    if (threadIdx.x == 0) {
        const int e = ids[pair];
        const int base = offsets[e];
        s_row = base < 0 ? -1 : base + atomicAdd(&cursor[e], 1);
        pos[pair] = s_row;
    }
    __syncthreads();
    if (s_row < 0) return;  // another rank's expert
    const uint4* src = hidden + static_cast<int64_t>(pair / top_k) * vec_per_row;
    uint4* dst = xp + static_cast<int64_t>(s_row) * vec_per_row;
    for (int v = threadIdx.x; v < vec_per_row; v += blockDim.x) dst[v] = src[v];
}

// out[t] = fold over k of bf16(acc + bf16(y[pos[t,k]] * w[t,k])), acc starting at 0.
__global__ void __launch_bounds__(128)
moe_combine_kernel(uint4* __restrict__ out, const uint4* __restrict__ y, const int32_t* __restrict__ pos,
                   const float* __restrict__ weights, int top_k, int vec_per_row) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int t = blockIdx.x;
    for (int v = threadIdx.x; v < vec_per_row; v += blockDim.x) {
        float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        for (int k = 0; k < top_k; ++k) {
            const float w = weights[t * top_k + k];
            const int row = pos[t * top_k + k];
            if (row < 0) continue;  // another rank's expert: its term arrives through the all-reduce
            const uint4 a = y[static_cast<int64_t>(row) * vec_per_row + v];
            const uint32_t aw[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                acc[2 * j] = round_bf16(acc[2 * j] + round_bf16(bf16_lo(aw[j]) * w));
                acc[2 * j + 1] = round_bf16(acc[2 * j + 1] + round_bf16(bf16_hi(aw[j]) * w));
            }
        }
        out[static_cast<int64_t>(t) * vec_per_row + v] =
            make_uint4(pack_bf16(acc[0], acc[1]), pack_bf16(acc[2], acc[3]), pack_bf16(acc[4], acc[5]),
                       pack_bf16(acc[6], acc[7]));
    }
}

// Table routing (experts by token id): the placement does not depend on the activations, so one launch at
// the start of a step lays out every table-routed layer of the model, one CTA per layer: histogram in
// shared memory, scan, then a row for every (token, choice) pair.
__global__ void __launch_bounds__(1024)
table_route_kernel(const TableRouteLayer* __restrict__ layers, const int32_t* __restrict__ token_ids, int tokens,
                   int vocab, int* status) {
    extern __shared__ int s_cnt[];
    __shared__ int s_warp[32];
    pdl_launch_dependents();
    pdl_wait_prior();
    const TableRouteLayer L = layers[blockIdx.x];
    const int E = L.experts;
    auto expert_of = [&](int pair) {
        const int id = token_ids[pair / L.top];
        const int e = id >= 0 && id < vocab ? L.table[static_cast<int64_t>(id) * L.top + pair % L.top] : 0;
        if (e < 0 || e >= E) {
            atomicExch(&status[kStatusBadIndex], e + 1);
            return 0;
        }
        return e;
    };
    for (int e = threadIdx.x; e < E; e += blockDim.x) s_cnt[e] = 0;
    __syncthreads();
    const int pairs = tokens * L.top;
    for (int i = threadIdx.x; i < pairs; i += blockDim.x) atomicAdd(&s_cnt[expert_of(i)], 1);
    __syncthreads();
    // exclusive scan of the counts, each thread a contiguous piece; the counts become running cursors
    const int per = (E + static_cast<int>(blockDim.x) - 1) / static_cast<int>(blockDim.x);
    const int e0 = min(static_cast<int>(threadIdx.x) * per, E), e1 = min(e0 + per, E);
    int mine = 0;
    for (int e = e0; e < e1; ++e) mine += s_cnt[e];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int incl = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += up;
    }
    if (lane == 31) s_warp[warp] = incl;
    __syncthreads();
    if (warp == 0) {
        int v = lane < static_cast<int>(blockDim.x >> 5) ? s_warp[lane] : 0;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int up = __shfl_up_sync(0xffffffffu, v, o);
            if (lane >= o) v += up;
        }
        s_warp[lane] = v;
    }
    __syncthreads();
    int run = incl - mine + (warp > 0 ? s_warp[warp - 1] : 0);
    for (int e = e0; e < e1; ++e) {
        const int c = s_cnt[e];
        L.counts[e] = c;
        L.offsets[e] = run;
        s_cnt[e] = run;
        run += c;
    }
    if (threadIdx.x == 0) L.offsets[E] = pairs;
    __syncthreads();
    for (int i = threadIdx.x; i < pairs; i += blockDim.x) L.rows[i] = atomicAdd(&s_cnt[expert_of(i)], 1);
}

// Scored routing: sigmoid scores in fp32, optionally only inside the best groups of neighbouring experts (a
// group counts for the sum of its two best), the best `top` of them, weights = scores over their sum.  One
// warp per token; ties go to the lower index.
struct ScoreRouteArgs {
    const float* logits;     // [tokens, ld]
    int64_t ld;
    int tokens, experts, top, groups, keep;
    float scale;
    int32_t* ids;            // [tokens, top]
    float* weights;          // [tokens, top]
    int32_t* counts;         // [experts], zero before
    int smem_floats;         // per warp: scores | group scores | chosen scores (| softmax scores)
    int identity;            // outputs behind those of the experts
    const float* correction;
};

__device__ __forceinline__ void warp_argmax(float& best, int& at) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float b = __shfl_xor_sync(0xffffffffu, best, o);
        const int i = __shfl_xor_sync(0xffffffffu, at, o);
        if (b > best || (b == best && i < at)) {
            best = b;
            at = i;
        }
    }
}

__global__ void __launch_bounds__(128)
score_route_kernel(const ScoreRouteArgs a) {
    extern __shared__ float s_route[];
    pdl_launch_dependents();
    pdl_wait_prior();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int64_t t = static_cast<int64_t>(blockIdx.x) * (blockDim.x >> 5) + warp;
    if (t >= a.tokens) return;
    constexpr float kTaken = -2.f, kOut = -1.f;   // below every score
    float* score = s_route + static_cast<int64_t>(warp) * a.smem_floats;
    float* group = score + a.experts;
    float* chosen = group + a.groups;
    for (int e = lane; e < a.experts; e += 32) {
        const float s = 1.f / (1.f + expf(-a.logits[t * a.ld + e]));
        score[e] = s == s ? s : 0.f;   // NaN logits: a token's experts are valid and differ all the same
    }
    __syncwarp();
    if (a.keep < a.groups) {
        const int size = a.experts / a.groups;
        for (int g = lane; g < a.groups; g += 32) {
            float first = kOut, second = kOut;
            for (int i = 0; i < size; ++i) {
                const float s = score[g * size + i];
                if (s > first) {
                    second = first;
                    first = s;
                } else if (s > second) {
                    second = s;
                }
            }
            group[g] = first + (size > 1 ? second : 0.f);
        }
        __syncwarp();
        for (int k = 0; k < a.keep; ++k) {
            float best = kOut;
            int at = 0x7fffffff;
            for (int g = lane; g < a.groups; g += 32)
                if (group[g] > best) {
                    best = group[g];
                    at = g;
                }
            warp_argmax(best, at);
            if (lane == 0 && at < a.groups) group[at] = kTaken;
            __syncwarp();
        }
        for (int e = lane; e < a.experts; e += 32)
            if (group[e / size] != kTaken) score[e] = kOut;
        __syncwarp();
    }
    float sum = 0.f;
    for (int k = 0; k < a.top; ++k) {
        float best = kOut;
        int at = 0x7fffffff;
        for (int e = lane; e < a.experts; e += 32)
            if (score[e] > best) {
                best = score[e];
                at = e;
            }
        warp_argmax(best, at);
        sum += best;
        if (lane == 0) {
            score[at] = kTaken;
            chosen[k] = best;
            a.ids[t * a.top + k] = at;
            atomicAdd(&a.counts[at], 1);
        }
        __syncwarp();
    }
    for (int k = lane; k < a.top; k += 32) a.weights[t * a.top + k] = chosen[k] / (sum + 1e-20f) * a.scale;
}

// The same with softmax scores over experts and identity experts.  Groups and choice go by score + correction, which may
// be negative; a group counts for its best.
__global__ void __launch_bounds__(128)
softmax_route_kernel(const ScoreRouteArgs a) {
    extern __shared__ float s_route[];
    pdl_launch_dependents();
    pdl_wait_prior();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, outputs = a.experts + a.identity;
    const int64_t t = static_cast<int64_t>(blockIdx.x) * (blockDim.x >> 5) + warp;
    if (t >= a.tokens) return;
    float* choice = s_route + static_cast<int64_t>(warp) * a.smem_floats;
    float* group = choice + outputs;
    float* score = group + a.groups;
    const float* z = a.logits + t * a.ld;
    float top = -INFINITY, sum = 0.f;
    for (int e = lane; e < outputs; e += 32) top = fmaxf(top, z[e]);
    top = warp_max(top);
    for (int e = lane; e < outputs; e += 32) {
        score[e] = expf(z[e] - top);
        sum += score[e];
    }
    sum = warp_sum(sum);
    for (int e = lane; e < outputs; e += 32) {
        const float s = score[e] / sum, c = s + (a.correction != nullptr ? a.correction[e] : 0.f);
        score[e] = s == s ? s : 0.f;   // NaN logits: a token's experts are valid and differ all the same
        choice[e] = c == c ? c : 0.f;
    }
    __syncwarp();
    const int size = outputs / a.groups;
    // the best of n numbers, lowest index first; n when all of them are out
    auto best_of = [&](const float* x, int n) {
        float best = -INFINITY;
        int at = n;
        for (int i = lane; i < n; i += 32)
            if (x[i] > best) {
                best = x[i];
                at = i;
            }
        warp_argmax(best, at);
        return at;
    };
    if (a.keep < a.groups) {
        for (int g = lane; g < a.groups; g += 32) {
            float best = -INFINITY;
            for (int i = 0; i < size; ++i) best = fmaxf(best, choice[g * size + i]);
            group[g] = best;
        }
        __syncwarp();
        constexpr float kKept = INFINITY;
        for (int k = 0; k < a.keep; ++k) {
            float best = -INFINITY;
            int at = a.groups;
            for (int g = lane; g < a.groups; g += 32)
                if (group[g] != kKept && group[g] > best) {
                    best = group[g];
                    at = g;
                }
            warp_argmax(best, at);
            if (lane == 0 && at < a.groups) group[at] = kKept;
            __syncwarp();
        }
        for (int e = lane; e < outputs; e += 32)
            if (group[e / size] != kKept) choice[e] = -INFINITY;
        __syncwarp();
    }
    for (int k = 0; k < a.top; ++k) {
        const int at = best_of(choice, outputs);
        if (lane == 0 && at < outputs) {
            choice[at] = -INFINITY;
            a.ids[t * a.top + k] = at;
            a.weights[t * a.top + k] = score[at] * a.scale;
            if (at < a.experts) atomicAdd(&a.counts[at], 1);
        }
        __syncwarp();
    }
}

// A row among its expert's for every choice of a token, and the token's activations copied there.  The first
// rows of the experts follow from the counts, so no scan runs in between; one CTA per token.
__global__ void __launch_bounds__(128)
score_place_kernel(uint4* __restrict__ xp, const uint4* __restrict__ x, int32_t* __restrict__ rows,
                   const int32_t* __restrict__ ids, const int32_t* __restrict__ counts, int32_t* __restrict__ cursor,
                   int32_t* __restrict__ offsets, int experts, int top, int vec_per_row) {
    extern __shared__ int s_place[];
    pdl_launch_dependents();
    pdl_wait_prior();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int64_t t = blockIdx.x;
    for (int k = warp; k < top; k += warps) {
        const int e = ids[t * top + k];
        if (e >= experts) {   // an identity expert: the token keeps its row where it is
            if (lane == 0) s_place[k] = rows[t * top + k] = -1;
            continue;
        }
        int before = 0;
        for (int i = lane; i < e; i += 32) before += counts[i];
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
        if (lane == 0) {
            const int row = before + atomicAdd(&cursor[e], 1);
            s_place[k] = row;
            rows[t * top + k] = row;
        }
    }
    if (t == 0 && warp == warps - 1) {
        int carry = 0;
        for (int base = 0; base < experts; base += 32) {
            const int e = base + lane;
            const int n = e < experts ? counts[e] : 0;
            int incl = n;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int up = __shfl_up_sync(0xffffffffu, incl, o);
                if (lane >= o) incl += up;
            }
            if (e < experts) offsets[e] = carry + incl - n;
            carry += __shfl_sync(0xffffffffu, incl, 31);
        }
        if (lane == 0) offsets[experts] = carry;
    }
    __syncthreads();
    for (int v = threadIdx.x; v < vec_per_row; v += blockDim.x) {
        const uint4 u = x[t * vec_per_row + v];
        for (int k = 0; k < top; ++k)
            if (s_place[k] >= 0) xp[static_cast<int64_t>(s_place[k]) * vec_per_row + v] = u;
    }
}

struct MoeWorkspace {
    int32_t *ids, *counts, *offsets, *cursor, *pos;
    float* weights;
    __nv_bfloat16 *xp, *hact, *y2;
};

int64_t align256(int64_t x) { return (x + 255) / 256 * 256; }

int64_t carve(MoeWorkspace* w, uint8_t* base, int tokens, int E, int top_k, int H, int I) {
    const int64_t pairs = static_cast<int64_t>(tokens) * top_k;
    int64_t off = 0;
    auto take = [&](int64_t bytes) {
        uint8_t* p = base ? base + off : nullptr;
        off += align256(bytes);
        return p;
    };
    w->ids = reinterpret_cast<int32_t*>(take(pairs * 4));
    w->weights = reinterpret_cast<float*>(take(pairs * 4));
    w->pos = reinterpret_cast<int32_t*>(take(pairs * 4));
    w->counts = reinterpret_cast<int32_t*>(take((E + 1) * 4));
    w->offsets = reinterpret_cast<int32_t*>(take((E + 1) * 4));
    w->cursor = reinterpret_cast<int32_t*>(take((E + 1) * 4));
    w->xp = reinterpret_cast<__nv_bfloat16*>(take(pairs * H * 2));
    w->hact = reinterpret_cast<__nv_bfloat16*>(take(pairs * I * 2));
    w->y2 = reinterpret_cast<__nv_bfloat16*>(take(pairs * H * 2));
    return off;
}

}  // namespace

int64_t moe_workspace_bytes(int tokens, int E, int top_k, int H, int I) {
    MoeWorkspace w;
    return carve(&w, nullptr, tokens, E, top_k, H, I);
}

int launch_table_route(const TableRouteLayer* layers_dev, int num_layers, int max_experts, const int32_t* token_ids,
                       int tokens, int vocab, int* status, cudaStream_t stream) {
    if (tokens == 0 || num_layers == 0) return B200_OK;
    B200_CHECK_CUDA(launch_kernel(table_route_kernel, dim3(num_layers), dim3(1024), max_experts * sizeof(int), stream,
                                  dim3(1, 1, 1), layers_dev, token_ids, tokens, vocab, status));
    return B200_OK;
}

int launch_score_route(const ScoreRoute& r, cudaStream_t stream) {
    if (r.tokens == 0) return B200_OK;
    ScoreRouteArgs a;
    a.logits = r.logits;
    a.ld = r.ld;
    a.tokens = r.tokens;
    a.experts = r.experts;
    a.top = r.top;
    a.groups = r.groups;
    a.keep = r.keep;
    a.scale = r.scale;
    a.ids = r.ids;
    a.weights = r.weights;
    a.counts = r.counts;
    a.identity = r.identity;
    a.correction = r.correction;
    const bool softmax = r.score == B200_SCORE_SOFTMAX;
    const int outputs = r.experts + r.identity;
    a.smem_floats = softmax ? 2 * outputs + r.groups : r.experts + r.groups + r.top;
    // few tokens: one warp per CTA, spread over the SMs
    const int warps = r.tokens >= 1024 && outputs <= 1024 ? 4 : 1;
    B200_CHECK_CUDA(launch_kernel(softmax ? softmax_route_kernel : score_route_kernel, dim3(div_ceil(r.tokens, warps)), dim3(32 * warps),
                                  static_cast<size_t>(warps) * a.smem_floats * 4, stream, dim3(1, 1, 1), a));
    return B200_OK;
}

int launch_score_place(void* xp, const void* x, int row_bytes, const ScoreRoute& r, int32_t* rows, int32_t* cursor,
                       int32_t* offsets, cudaStream_t stream) {
    if (r.tokens == 0) return B200_OK;
    B200_CHECK_CUDA(launch_kernel(score_place_kernel, dim3(r.tokens), dim3(128), static_cast<size_t>(r.top) * 4, stream,
                                  dim3(1, 1, 1), static_cast<uint4*>(xp), static_cast<const uint4*>(x), rows,
                                  static_cast<const int32_t*>(r.ids), static_cast<const int32_t*>(r.counts), cursor,
                                  offsets, r.experts, r.top, row_bytes / 16));
    return B200_OK;
}

int launch_moe_route(int32_t* ids, float* weights, int32_t* counts, const void* logits, int tokens, int E,
                     int top_k, int renorm, cudaStream_t stream) {
    B200_CHECK_CUDA(cudaMemsetAsync(counts, 0, (E + 1) * sizeof(int32_t), stream));
    const bool pdl = pdl_launches_enabled();
    set_pdl_launches(false);  // follows a memset
    cudaError_t ce = launch_kernel(moe_route_kernel, dim3(div_ceil(tokens, 4)), dim3(128), 0, stream, dim3(1, 1, 1),
                                   static_cast<const __nv_bfloat16*>(logits), tokens, E, top_k, renorm, ids,
                                   weights, counts);
    set_pdl_launches(pdl);
    B200_CHECK_CUDA(ce);
    return B200_OK;
}

int launch_moe_forward(void* out, const void* hidden, const void* router_logits, const void* gate_up,
                       const void* down, int tokens, int E, int top_k, int H, int I, int renorm,
                       int activation, int expert_begin, int num_local_experts, void* workspace,
                       int* status, cudaStream_t stream) {
    if (tokens == 0) return B200_OK;
    MoeWorkspace w;
    carve(&w, static_cast<uint8_t*>(workspace), tokens, E, top_k, H, I);
    const int pairs = tokens * top_k;
    int err = launch_moe_route(w.ids, w.weights, w.counts, router_logits, tokens, E, top_k, renorm, stream);
    if (err != B200_OK) return err;
    B200_CHECK_CUDA(launch_kernel(moe_scan_kernel, dim3(1), dim3(256), 0, stream, dim3(1, 1, 1),
                                  static_cast<const int32_t*>(w.counts), w.offsets, w.cursor, E, expert_begin,
                                  num_local_experts));
    B200_CHECK_CUDA(launch_kernel(moe_scatter_kernel, dim3(pairs), dim3(128), 0, stream, dim3(1, 1, 1),
                                  static_cast<const uint4*>(hidden), reinterpret_cast<uint4*>(w.xp),
                                  static_cast<const int32_t*>(w.ids), static_cast<const int32_t*>(w.offsets),
                                  w.cursor, w.pos, top_k, H / 8));
    const int epi = activation == 1 ? B200_EPILOGUE_GEGLU_ERF : B200_EPILOGUE_SWIGLU;
    // A token picks distinct experts, so no expert gets more rows than there are tokens.
    // gate_up / down hold the local experts only, so group g is expert expert_begin + g.
    const int32_t* counts = w.counts + expert_begin;
    const int32_t* offsets = w.offsets + expert_begin;
    err = launch_grouped_gemm(w.hact, w.xp, gate_up, counts, offsets, num_local_experts, tokens, pairs, 2 * I, H,
                              epi, status, stream);
    if (err != B200_OK) return err;
    err = launch_grouped_gemm(w.y2, w.hact, down, counts, offsets, num_local_experts, tokens, pairs, H, I,
                              B200_EPILOGUE_NONE, status, stream);
    if (err != B200_OK) return err;
    B200_CHECK_CUDA(launch_kernel(moe_combine_kernel, dim3(tokens), dim3(128), 0, stream, dim3(1, 1, 1),
                                  static_cast<uint4*>(out), reinterpret_cast<const uint4*>(w.y2),
                                  static_cast<const int32_t*>(w.pos), static_cast<const float*>(w.weights),
                                  top_k, H / 8));
    return B200_OK;
}

}  // namespace b200

extern "C" {

int64_t b200_moe_workspace_bytes(int tokens, int num_experts, int top_k, int hidden_size, int intermediate_size) {
    if (tokens < 0 || num_experts <= 0 || top_k <= 0 || hidden_size <= 0 || intermediate_size <= 0) return -1;
    return b200::moe_workspace_bytes(tokens, num_experts, top_k, hidden_size, intermediate_size);
}

int b200_moe_route(int32_t* topk_ids, float* topk_weights, int32_t* expert_counts, const void* router_logits,
                   int tokens, int num_experts, int top_k, int renormalize, b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0, "moe_route: tokens must be >= 0");
    B200_CHECK_ARG(num_experts > 0 && num_experts <= 256, "MoELayer requires 0 < num_experts <= 256");
    B200_CHECK_ARG(top_k > 0 && top_k <= b200::kMaxTopK, "MoELayer requires 0 < top_k <= 16");
    B200_CHECK_ARG(top_k <= num_experts, "MoELayer top_k must be <= num_experts");
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(topk_ids && topk_weights && expert_counts && router_logits, "moe_route: NULL tensor");
    return b200::launch_moe_route(topk_ids, topk_weights, expert_counts, router_logits, tokens, num_experts,
                                  top_k, renormalize, static_cast<cudaStream_t>(stream));
}

int b200_table_route(int32_t* rows, int32_t* counts, int32_t* offsets, const int32_t* table,
                     const int32_t* token_ids, int tokens, int vocab, int top, int experts, b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0 && vocab > 0 && top > 0 && experts >= top, "table_route: bad shape");
    B200_CHECK_ARG(experts <= b200::kMaxTableExperts, "table_route: at most %d experts", b200::kMaxTableExperts);
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(rows && counts && offsets && table && token_ids, "table_route: NULL tensor");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    // the kernel reads its layer descriptions from device memory; a caller of the single-layer form pays
    // for a small allocation
    const b200::TableRouteLayer layer{table, rows, counts, offsets, top, experts};
    void* dev = nullptr;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    B200_CHECK_CUDA(cudaMalloc(&dev, sizeof(layer)));
    cudaError_t ce = cudaMemcpyAsync(dev, &layer, sizeof(layer), cudaMemcpyHostToDevice, s);
    if (ce == cudaSuccess)
        err = b200::launch_table_route(static_cast<const b200::TableRouteLayer*>(dev), 1, experts, token_ids, tokens, vocab,
                                       status, s);
    if (ce == cudaSuccess) ce = cudaStreamSynchronize(s);
    cudaFree(dev);
    B200_CHECK_CUDA(ce);
    return err;
}

int b200_score_route(int32_t* ids, float* weights, int32_t* rows, int32_t* counts, int32_t* offsets, void* xp,
                     const void* x, int row_bytes, const float* logits, int64_t logits_ld, int tokens, int experts,
                     int top, int groups, int keep_groups, float scale, int score, int identity_experts,
                     const float* correction, b200_stream_t stream) {
    const int outputs = experts + identity_experts;
    B200_CHECK_ARG(tokens >= 0 && experts > 0 && identity_experts >= 0 && outputs <= b200::kMaxTableExperts && top > 0 && groups > 0 &&
                       outputs % groups == 0 && keep_groups > 0 && keep_groups <= groups &&
                       top <= outputs / groups * keep_groups, "score_route: bad shape");
    B200_CHECK_ARG(score == B200_SCORE_SOFTMAX || (score == B200_SCORE_SIGMOID && identity_experts == 0 && !correction),
                   "score_route: identity experts and corrections come with softmax scores");
    B200_CHECK_ARG(row_bytes > 0 && row_bytes % 16 == 0 && logits_ld >= outputs, "score_route: bad row size");
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(ids && weights && rows && counts && offsets && xp && x && logits, "score_route: NULL tensor");
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    B200_CHECK_CUDA(cudaMemsetAsync(counts, 0, 2ll * experts * 4, s));
    b200::ScoreRoute r;
    r.logits = logits;
    r.ld = logits_ld;
    r.tokens = tokens;
    r.experts = experts;
    r.top = top;
    r.groups = groups;
    r.keep = keep_groups;
    r.scale = scale;
    r.score = score;
    r.identity = identity_experts;
    r.correction = correction;
    r.ids = ids;
    r.weights = weights;
    r.counts = counts;
    int err = b200::launch_score_route(r, s);
    if (err != B200_OK) return err;
    return b200::launch_score_place(xp, x, row_bytes, r, rows, counts + experts, offsets, s);
}

int b200_moe_forward_local(void* out, const void* hidden_states, const void* router_logits,
                           const void* gate_up_proj, const void* down_proj, int tokens, int num_experts,
                           int top_k, int hidden_size, int intermediate_size, int renormalize,
                           int activation, int expert_begin, int num_local_experts, void* workspace,
                           int64_t workspace_bytes, b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0, "MoELayer token count must be >= 0");
    B200_CHECK_ARG(num_experts > 0 && num_experts <= 256, "MoELayer requires 0 < num_experts <= 256");
    B200_CHECK_ARG(top_k > 0 && top_k <= b200::kMaxTopK, "MoELayer requires 0 < top_k <= 16");
    B200_CHECK_ARG(top_k <= num_experts, "MoELayer top_k must be <= num_experts");
    B200_CHECK_ARG(hidden_size > 0 && hidden_size % 64 == 0, "MoELayer hidden size must be a positive multiple of 64");
    B200_CHECK_ARG(intermediate_size > 0 && intermediate_size % 64 == 0,
                   "MoELayer intermediate size must be a positive multiple of 64");
    B200_CHECK_ARG(activation == 0 || activation == 1, "Unsupported MoE activation function");
    B200_CHECK_ARG(expert_begin >= 0 && num_local_experts > 0 && expert_begin + num_local_experts <= num_experts,
                   "moe_forward: local expert range outside [0, num_experts)");
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(out && hidden_states && router_logits && gate_up_proj && down_proj && workspace,
                   "moe_forward: NULL tensor");
    B200_CHECK_ARG(workspace_bytes >= b200::moe_workspace_bytes(tokens, num_experts, top_k, hidden_size, intermediate_size),
                   "moe_forward: workspace too small");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    return b200::launch_moe_forward(out, hidden_states, router_logits, gate_up_proj, down_proj, tokens,
                                    num_experts, top_k, hidden_size, intermediate_size, renormalize, activation,
                                    expert_begin, num_local_experts, workspace, status,
                                    static_cast<cudaStream_t>(stream));
}

int b200_moe_forward(void* out, const void* hidden_states, const void* router_logits, const void* gate_up_proj,
                     const void* down_proj, int tokens, int num_experts, int top_k, int hidden_size,
                     int intermediate_size, int renormalize, int activation, void* workspace,
                     int64_t workspace_bytes, b200_stream_t stream) {
    return b200_moe_forward_local(out, hidden_states, router_logits, gate_up_proj, down_proj, tokens, num_experts,
                                  top_k, hidden_size, intermediate_size, renormalize, activation, 0,
                                  num_experts > 0 ? num_experts : 1, workspace, workspace_bytes, stream);
}

}  // extern "C"
