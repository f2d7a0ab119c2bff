// y = x W^T for few rows (decode batches, M <= 256): a weight-streaming GEMM on
// the tcgen05 tensor cores.
//
// The kernel is bound by reading W once from HBM, so the layout is chosen for
// bytes in flight rather than for tensor-core occupancy:
//   * swap-AB: the MMA "A" operand is a 128-row tile of W (output features run
//     along the TMEM lanes), the "B" operand is the whole activation block
//     x[0:NT, k-slice] (tokens run along TMEM columns).  A stage of shared
//     memory is then 2/3 weight bytes instead of mostly padding rows of x.
//   * split-K across a thread-block cluster: (feature tiles) x (K slices) CTAs
//     so that about one CTA per SM issues TMA loads at once; each CTA usually
//     holds its whole K slice in shared memory, i.e. the entire weight matrix
//     is requested at t=0.
//   * partial sums are exchanged through distributed shared memory in fixed
//     rank order (deterministic), then bias / gated activation / bf16 rounding
//     are applied by the CTA that owns that slice of features.
//   * weight tiles do not depend on the previous kernel, so they are requested
//     before griddepcontrol.wait; only the x loads wait for the producer of x.
//
// Gated epilogue (gate_up projection + SwiGLU): two accumulators share the x
// operand, one fed by a gate-row tile of W and one by the matching up-row tile,
// so a thread holds gate[n][m] and up[n][m] for the same (n, m).
#include "common.cuh"
#include "kernels.h"
#include "tensormap.cuh"
#include "tcgen05.cuh"

namespace b200 {
namespace {

constexpr int kTileN = 128;  // output features per CTA (UMMA M)
constexpr int kBlockK = 64;  // bf16 elements per k-block (one 128-byte swizzle row)
constexpr int kMaxStages = 8;
constexpr int kThreads = 192;  // warp 0: TMA, warp 1: MMA + TMEM owner, warps 2-5: epilogue
constexpr int kChunkCols = 32;  // token columns per tcgen05.ld
constexpr int kRoundCols = 64;  // token columns exchanged per cluster round

// ---- cluster helpers ----------------------------------------------------------

__device__ __forceinline__ uint32_t cluster_ctarank() {
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}
__device__ __forceinline__ uint32_t cluster_nctarank() {
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_nctarank;" : "=r"(r));
    return r;
}
__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float ld_dsmem_f32(uint32_t local_addr, uint32_t rank) {
    uint32_t remote;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
    return v;
}

__device__ __forceinline__ void st_dsmem_f32(uint32_t cluster_addr, float v) {
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(cluster_addr), "f"(v) : "memory");
}
__device__ __forceinline__ float4 ld_dsmem_f32x4(uint32_t local_addr, uint32_t rank) {
    uint32_t remote;
    float4 v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
    asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];"
                 : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w)
                 : "r"(remote)
                 : "memory");
    return v;
}

__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + __expf(-x)); }
__device__ __forceinline__ float gelu_erf_f(float x) { return 0.5f * x * (1.0f + erff(x * 0.70710678118654752f)); }
// The activation is a template parameter: a run-time switch makes the compiler keep all three
// bodies (erff and tanhf are long) in the epilogue of every gated GEMM.
template <int EPI>
__device__ __forceinline__ float gated_act(float g) {
    if (EPI == B200_EPILOGUE_SWIGLU) return __fdividef(g, 1.0f + __expf(-g));  // 2 ulp in fp32, far below the bf16 step
    if (EPI == B200_EPILOGUE_GEGLU_ERF) return gelu_erf_f(g);
    return 0.5f * g * (1.0f + tanhf(0.7978845608f * (g + 0.044715f * g * g * g)));
}
template <int EPI>
__device__ __forceinline__ float gated_pair(float g, float u, float limit) {
    if (EPI == B200_EPILOGUE_CLAMPED_SWIGLU) return clamped_swiglu<false>(g, u, limit);
    return gated_act<EPI>(g) * u;
}
__device__ __forceinline__ float gelu_tanh_f(float x) {
    return 0.5f * x * (1.0f + tanhf(0.7978845608f * (x + 0.044715f * x * x * x)));
}

struct SkinnyParams {
    __nv_bfloat16* y;          // [M, n_out]
    const __nv_bfloat16* bias; // [n_out] or NULL (plain epilogue only)
    int M;                     // rows of x / y
    int n_out;                 // output features (N, or N/2 with a gated epilogue)
    int up_row_offset;         // row of W where the "up" half starts (gated only)
    int kb_total;              // K / 64
    int nt;                    // token columns of the accumulator (multiple of 32, >= M)
    int stages;                // shared-memory stages in the ring
    int epilogue;              // B200_EPILOGUE_*
    int* status;
    // Grouped mode (expert GEMMs): blockIdx.z = group, blockIdx.y = 256-row slab of the group.
    // Group g multiplies rows [offsets[g], offsets[g] + counts[g]) of x by rows
    // [g * w_rows_per_group, ...) of w; counts / offsets live in device memory.
    const int32_t* group_counts;
    const int32_t* group_offsets;
    int w_rows_per_group;
    // Per-head mode: blockIdx.z = head; it reads columns [z * head_k, ...) of x and writes columns
    // [z * n_out, ...) of y with the weights of its own w_rows_per_group rows.
    int head_k;          // 0 = off
    float act_limit;     // B200_EPILOGUE_CLAMPED_SWIGLU
    int64_t y_pitch;     // row pitch of y (n_out, or heads * n_out)
    // Fusions with the residual stream (split-K launches of the decode step; see SkinnyFusion in kernels.h).
    const unsigned long long* ssq_in;   // "normalised input": accumulator x rsqrt(ssq_in[m] / 2^24 / norm_width + eps)
    float norm_eps;
    int norm_width;
    __nv_bfloat16* residual;            // "residual output": residual[m, n] = bf16(bf16(acc) + residual[m, n]), y unused
    unsigned long long* ssq_out;        // ... and ssq_out[m] += (that sum)^2 in 2^-24 fixed point
    int ssq_of_rounded;                 // square the stored (bf16) sum instead of the fp32 one
    // "attention heads": every 128-feature tile is one head of a packed qkv projection; the epilogue
    // applies the per-head RMS norm and the NeoX rotation and stores K / V into the pool.
    int head_mode;
    const __nv_bfloat16* q_norm_w;      // [128] or NULL
    const __nv_bfloat16* k_norm_w;
    const float* cos_t;                 // [max_pos, 64]
    const float* sin_t;
    const int32_t* positions;           // [M]
    const int32_t* out_loc;             // [M]
    __nv_bfloat16* k_cache;             // [num_slots, kv_heads, 128]
    __nv_bfloat16* v_cache;
    int q_heads, kv_heads, max_pos;
    long long num_slots;
    float qk_eps;
};
constexpr float kSsqScale = 16777216.0f;   // 2^24

// HEADS: the attention-head epilogue (plain projections only) is compiled into an instance of its own;
// it needs about 90 registers more than the rest, which would cost lm_head its second CTA per SM.
template <int EPI, bool HEADS = false>
__global__ void __launch_bounds__(kThreads, 1)
skinny_gemm_kernel(const __grid_constant__ CUtensorMap tmap_w,
                   const __grid_constant__ CUtensorMap tmap_x,
                   const __grid_constant__ CUtensorMap tmap_x64,
                   const __grid_constant__ CUtensorMap tmap_x128,
                   const __grid_constant__ CUtensorMap tmap_x256, const SkinnyParams p) {
    constexpr int NUM_A = epilogue_is_gated(EPI) ? 2 : 1;
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t full_bar[kMaxStages];
    __shared__ __align__(8) uint64_t empty_bar[kMaxStages];
    __shared__ __align__(8) uint64_t tmem_full_bar;
    __shared__ uint32_t tmem_base_slot;
    __shared__ float s_rstd[256];   // per token column, "normalised input" launches only

    // Let the next kernel in the stream become resident right away: its set-up and weight loads
    // then overlap this kernel (it still waits for this grid to finish before touching its input).
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t smem_base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    int nt = p.nt;          // accumulator columns = rows of the x box
    int rows = p.M;         // valid rows of x / y handled by this CTA
    int x_row0 = 0;         // first row of x and of y
    int w_row0 = 0;         // first row of this group's weights
    int x_col0 = 0;         // per-head mode: first column of x / of y
    int y_col0 = 0;
    if (p.head_k > 0) {
        w_row0 = static_cast<int>(blockIdx.z) * p.w_rows_per_group;
        x_col0 = static_cast<int>(blockIdx.z) * p.head_k;
        y_col0 = static_cast<int>(blockIdx.z) * p.n_out;
    }
    const CUtensorMap* tx = &tmap_x;
    if (p.group_counts != nullptr) {
        pdl_wait_prior();   // the group table comes from the kernel before this one
        const int grp = blockIdx.z;
        const int cnt = p.group_counts[grp];
        const int m0 = static_cast<int>(blockIdx.y) * 256;
        if (m0 >= cnt) return;  // whole CTA, before any barrier or TMEM use
        rows = min(256, cnt - m0);
        if (rows <= 32) { nt = 32; tx = &tmap_x; }
        else if (rows <= 64) { nt = 64; tx = &tmap_x64; }
        else if (rows <= 128) { nt = 128; tx = &tmap_x128; }
        else { nt = 256; tx = &tmap_x256; }
        x_row0 = p.group_offsets[grp] + m0;
        w_row0 = grp * p.w_rows_per_group;
    }
    const uint32_t a_bytes = kTileN * kBlockK * 2;            // 16 KB per weight tile
    const uint32_t b_bytes = static_cast<uint32_t>(nt) * kBlockK * 2;
    const uint32_t stage_bytes = NUM_A * a_bytes + b_bytes;

    const uint32_t rank = cluster_ctarank();
    const uint32_t split = cluster_nctarank();
    const int kbp = (p.kb_total + static_cast<int>(split) - 1) / static_cast<int>(split);
    const int kb_begin = static_cast<int>(rank) * kbp;
    const int my_kb = max(0, min(kb_begin + kbp, p.kb_total) - kb_begin);
    const int n0 = blockIdx.x * kTileN;
    const int F = kTileN / static_cast<int>(split);     // features owned by one rank
    const int cpr = nt < kRoundCols ? nt : kRoundCols;  // token columns per exchange round
    // Head epilogue: the exchange is by token instead of by feature - a rank owns cpr / split token
    // columns of a round with all 128 features, so a head's sum of squares and both elements of every
    // rotation pair are in one CTA.  Its scratch sits behind the exchange buffers: cos | sin
    // [nt / split][64] for the owned tokens, then their pool slots [nt / split].
    const int cpl = cpr / static_cast<int>(split);      // token columns of a round owned by one rank
    const int head_kind = !HEADS ? -1 : (static_cast<int>(blockIdx.x) < p.q_heads ? 0
                          : static_cast<int>(blockIdx.x) < p.q_heads + p.kv_heads ? 1 : 2);   // q, k, v
    const __nv_bfloat16* head_w = head_kind == 0 ? p.q_norm_w : head_kind == 1 ? p.k_norm_w : nullptr;
    const uint32_t head_off = static_cast<uint32_t>(p.stages) * (NUM_A * kTileN * kBlockK * 2 + static_cast<uint32_t>(nt) * kBlockK * 2) +
                              (nt > cpr ? 2u : 1u) * NUM_A * cpr * kTileN * 4u;
    const int owned_tokens = nt / static_cast<int>(split);
    float* s_cos = reinterpret_cast<float*>(smem_raw + (smem_base - smem_u32(smem_raw)) + head_off);
    float* s_sin = s_cos + owned_tokens * (kTileN / 2);
    int* s_slot = reinterpret_cast<int*>(s_sin + owned_tokens * (kTileN / 2));

    // TMEM columns: NUM_A accumulators of nt columns, rounded up to a power of two >= 32.
    uint32_t tmem_cols = 32;
    while (tmem_cols < static_cast<uint32_t>(NUM_A * nt)) tmem_cols <<= 1;

    if (threadIdx.x == 0) {
        for (int s = 0; s < p.stages; ++s) {
            mbar_init(smem_u32(&full_bar[s]), 1);
            mbar_init(smem_u32(&empty_bar[s]), 1);
        }
        mbar_init(smem_u32(&tmem_full_bar), 1);
        fence_mbar_init();
        // Weight tiles first, from the thread that has just initialised the barriers: they do not
        // depend on the kernel before this one, nor on the TMEM allocation and the block-wide
        // barrier below, so the requests leave about half a microsecond earlier.
        const int early = min(my_kb, p.stages);
        for (int i = 0; i < early; ++i) {
            const uint32_t bar = smem_u32(&full_bar[i]);
            const uint32_t dst = smem_base + i * stage_bytes;
            const int kc = (kb_begin + i) * kBlockK;
            mbar_arrive_expect_tx(bar, stage_bytes);
            tma_load_2d(dst, &tmap_w, kc, w_row0 + n0, bar);
            if (NUM_A == 2) tma_load_2d(dst + a_bytes, &tmap_w, kc, w_row0 + p.up_row_offset + n0, bar);
        }
        tma_prefetch_desc(tx);
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(&tmem_base_slot), tmem_cols);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = tmem_base_slot;

    bool failed = false;

    if (warp == 0) {
        if (lane == 0) {
            // (the first ring-full of weight tiles was requested during set-up)
            auto load_w = [&](uint32_t dst, int kc, int row, uint32_t bar) { tma_load_2d(dst, &tmap_w, kc, row, bar); };
            pdl_wait_prior();
            for (int i = 0; i < my_kb && !failed; ++i) {
                const int s = i % p.stages;
                const uint32_t bar = smem_u32(&full_bar[s]);
                const uint32_t dst = smem_base + s * stage_bytes;
                const int kc = (kb_begin + i) * kBlockK;
                if (i >= p.stages) {
                    const uint32_t par = static_cast<uint32_t>((i / p.stages) - 1) & 1u;
                    if (!mbar_wait_bounded(smem_u32(&empty_bar[s]), par, p.status, 101)) {
                        failed = true;
                        break;
                    }
                    mbar_arrive_expect_tx(bar, stage_bytes);
                    load_w(dst, kc, w_row0 + n0, bar);
                    if (NUM_A == 2) load_w(dst + a_bytes, kc, w_row0 + p.up_row_offset + n0, bar);
                }
                tma_load_2d(dst + NUM_A * a_bytes, tx, x_col0 + kc, x_row0, bar);
            }
        }
    } else if (warp == 1) {
        pdl_wait_prior();
        if (lane == 0) {
            const uint32_t idesc = idesc_bf16_m128(nt);
            for (int i = 0; i < my_kb; ++i) {
                const int s = i % p.stages;
                const uint32_t par = static_cast<uint32_t>(i / p.stages) & 1u;
                if (!mbar_wait_bounded(smem_u32(&full_bar[s]), par, p.status, 102)) {
                    failed = true;
                    break;
                }
                tc_fence_after();
                const uint32_t a0 = smem_base + s * stage_bytes;
                const uint32_t b0 = a0 + NUM_A * a_bytes;
#pragma unroll
                for (int k = 0; k < kBlockK / 16; ++k) {
                    const uint32_t acc = (i > 0 || k > 0) ? 1u : 0u;
                    const uint64_t bdesc = kmajor_sw128_desc(b0 + k * 32);
                    tc_mma_bf16(tmem_base, kmajor_sw128_desc(a0 + k * 32), bdesc, idesc, acc);
                    if (NUM_A == 2)
                        tc_mma_bf16(tmem_base + nt, kmajor_sw128_desc(a0 + a_bytes + k * 32), bdesc,
                                    idesc, acc);
                }
                tc_commit(smem_u32(&empty_bar[s]));
            }
            if (my_kb > 0 && !failed)
                tc_commit(smem_u32(&tmem_full_bar));
            else
                mbar_arrive(smem_u32(&tmem_full_bar));
        }
    } else {
        if (head_kind >= 0) {
            // positions, slots and the rotation table are complete before the layer stack starts:
            // fetched ahead of the wait, under the weight stream
            const int te = static_cast<int>(threadIdx.x) - 64;
            // owned token lm of round r is column r * cpr + rank * cpl + lm % cpl of the accumulator
            auto token_of = [&](int lm) { return (lm / cpl) * cpr + static_cast<int>(rank) * cpl + lm % cpl; };
            if (head_kind < 2) {
                for (int idx = te; idx < owned_tokens * (kTileN / 8); idx += kThreads - 64) {
                    const int lm = idx / (kTileN / 8), j4 = idx % (kTileN / 8) * 4;
                    const int m = token_of(lm);
                    int pos = m < rows ? p.positions[x_row0 + m] : 0;
                    if (pos < 0 || pos >= p.max_pos) {
                        if (j4 == 0) atomicExch(&p.status[kStatusBadIndex], pos + 1);
                        pos = min(max(pos, 0), p.max_pos - 1);
                    }
                    const int64_t at = static_cast<int64_t>(pos) * (kTileN / 2) + j4;
                    *reinterpret_cast<float4*>(s_cos + lm * (kTileN / 2) + j4) = *reinterpret_cast<const float4*>(p.cos_t + at);
                    *reinterpret_cast<float4*>(s_sin + lm * (kTileN / 2) + j4) = *reinterpret_cast<const float4*>(p.sin_t + at);
                }
            }
            if (head_kind > 0) {
                for (int lm = te; lm < owned_tokens; lm += kThreads - 64) {
                    const int m = token_of(lm);
                    int slot = m < rows ? p.out_loc[x_row0 + m] : -1;
                    if (m < rows && (slot < 0 || slot >= p.num_slots)) {
                        atomicExch(&p.status[kStatusBadIndex], slot + 1);
                        slot = -1;
                    }
                    s_slot[lm] = slot;
                }
            }
        }
        pdl_wait_prior();
        if (p.ssq_in != nullptr) {
            // the row statistics come from the kernel before this one; the cluster barrier of the first
            // exchange round orders these writes before their first use
            for (int m = static_cast<int>(threadIdx.x) - 64; m < nt; m += kThreads - 64)
                s_rstd[m] = m < rows ? rsqrtf(static_cast<float>(p.ssq_in[x_row0 + m]) * (1.0f / kSsqScale) /
                                                  static_cast<float>(p.norm_width) + p.norm_eps)
                                     : 0.f;
        }
    }
    __syncwarp();

    // ---- epilogue: every warp walks the same sequence of cluster barriers ----
    // Split-K exchange is PUSH based: rank r owns F = 128/split features of the tile.  Every CTA
    // stores its partial sums for those features straight into rank r's exchange buffer (remote
    // shared-memory stores do not stall the sender), one cluster barrier makes them visible, and
    // the owner reduces from its own shared memory in rank order.  Nobody reads or writes a
    // peer's memory after the last barrier, so CTAs leave independently.  The exchange buffer is
    // a region of its own behind the operand stages: a peer may push while this CTA's MMAs still
    // read the stages.
    const bool is_epi = warp >= 2;
    const int q = warp & 3;                       // TMEM lane quarter this warp may read
    const int feat_local = q * 32 + lane;         // feature row inside the tile
    const int nrounds = nt / cpr;
    const uint32_t round_bytes = static_cast<uint32_t>(NUM_A) * cpr * kTileN * 4u;
    const uint32_t xbuf_addr = smem_base + static_cast<uint32_t>(p.stages) * stage_bytes;
    const float* xbuf = reinterpret_cast<const float*>(smem_raw + (xbuf_addr - smem_u32(smem_raw)));
    // Where this thread's feature lives: owner rank and the base of that rank's buffer.
    const uint32_t owner = static_cast<uint32_t>(feat_local / F);
    const uint32_t fl = static_cast<uint32_t>(feat_local % F);
    uint32_t remote_base = 0;
    if (split > 1) asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote_base) : "r"(xbuf_addr), "r"(owner));

    if (is_epi) {
        if (!mbar_wait_bounded(smem_u32(&tmem_full_bar), 0, p.status, 103)) failed = true;
        tc_fence_after();
    }

    for (int r = 0; r < nrounds; ++r) {
        const uint32_t buf_off = static_cast<uint32_t>(r & 1) * round_bytes;
        if (is_epi) {
            for (int cc = 0; cc < cpr / kChunkCols; ++cc) {
                const int c = r * (cpr / kChunkCols) + cc;
                uint32_t g[32], u[32];
                if (my_kb > 0 && !failed) {
                    const uint32_t taddr = tmem_base + (static_cast<uint32_t>(q * 32) << 16) +
                                           static_cast<uint32_t>(c * kChunkCols);
                    tmem_ld_32x32b_x32(taddr, g);
                    if (NUM_A == 2) tmem_ld_32x32b_x32(taddr + nt, u);
                    tmem_ld_wait();
                } else {
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        g[j] = 0u;
                        u[j] = 0u;
                    }
                }
                if (split == 1) {
                    const int n = n0 + feat_local;
                    if (n < p.n_out) {
                        const float bias = p.bias ? __bfloat162float(p.bias[n]) : 0.f;
#pragma unroll
                        for (int j = 0; j < 32; ++j) {
                            const int m = c * kChunkCols + j;
                            if (m < rows) {
                                float v;
                                if (NUM_A == 2) {
                                    const float gv = round_bf16(__uint_as_float(g[j]));
                                    const float uv = round_bf16(__uint_as_float(u[j]));
                                    v = gated_pair<EPI>(gv, uv, p.act_limit);
                                } else {
                                    v = __uint_as_float(g[j]) + bias;
                                    if (EPI == B200_EPILOGUE_RELU2) v = fmaxf(v, 0.f) * fmaxf(v, 0.f);
                                    if (EPI == B200_EPILOGUE_GELU_ERF) v = gelu_erf_f(v);
                                }
                                const int64_t at = static_cast<int64_t>(x_row0 + m) * p.y_pitch + y_col0 + n;
                                if (EPI == B200_EPILOGUE_F32)
                                    reinterpret_cast<float*>(p.y)[at] = v;
                                else
                                    p.y[at] = __float2bfloat16_rn(v);
                            }
                        }
                    }
                } else if (head_kind >= 0) {
                    // owner layout: [source rank][owned column][feature]; the owner changes every cpl columns
                    const int cpl_shift = 31 - __clz(cpl);
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        const int col = cc * kChunkCols + j;
                        const uint32_t local = xbuf_addr + buf_off +
                                               ((rank * cpl + (col & (cpl - 1))) * kTileN + feat_local) * 4u;
                        uint32_t remote;
                        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local), "r"(col >> cpl_shift));
                        st_dsmem_f32(remote, __uint_as_float(g[j]));
                    }
                } else {
                    // owner layout: [source rank][accumulator][column][owned feature]
                    const uint32_t dst0 = remote_base + buf_off +
                                          ((rank * NUM_A * cpr + cc * kChunkCols) * F + fl) * 4u;
#pragma unroll
                    for (int j = 0; j < 32; ++j) {
                        st_dsmem_f32(dst0 + static_cast<uint32_t>(j * F) * 4u, __uint_as_float(g[j]));
                        if (NUM_A == 2)
                            st_dsmem_f32(dst0 + static_cast<uint32_t>((cpr + j) * F) * 4u, __uint_as_float(u[j]));
                    }
                }
            }
        }
        if (split == 1) continue;

        cluster_sync_all();
        if (head_kind >= 0) {
            // ---- head epilogue (plain projection only): eight lanes per owned token, lane `sub` holds
            // features [8 sub, 8 sub + 8) of each half of the head, so a rotation pair is in one lane ----
            if (is_epi) {
                const int te = (warp - 2) * 32 + lane;
                const float* rb = xbuf + buf_off / 4u;
                for (int base = 0; base < cpl * 8; base += 128) {
                    const int i = base + te;
                    const bool active = i < cpl * 8;          // (whole groups of eight lanes)
                    const int tl = active ? i >> 3 : 0, sub = i & 7;
                    const int m = r * cpr + static_cast<int>(rank) * cpl + tl;
                    const int lm = r * cpl + tl;
                    float x1[8], x2[8];
#pragma unroll
                    for (int e = 0; e < 8; ++e) x1[e] = x2[e] = 0.f;
#pragma unroll
                    for (uint32_t rr = 0; rr < 8; ++rr) {
                        if (rr < split) {
                            const float* src = rb + (rr * cpl + tl) * kTileN + sub * 8;
                            const float4 a0 = *reinterpret_cast<const float4*>(src), a1 = *reinterpret_cast<const float4*>(src + 4);
                            const float4 b0 = *reinterpret_cast<const float4*>(src + 64), b1 = *reinterpret_cast<const float4*>(src + 68);
                            x1[0] += a0.x; x1[1] += a0.y; x1[2] += a0.z; x1[3] += a0.w;
                            x1[4] += a1.x; x1[5] += a1.y; x1[6] += a1.z; x1[7] += a1.w;
                            x2[0] += b0.x; x2[1] += b0.y; x2[2] += b0.z; x2[3] += b0.w;
                            x2[4] += b1.x; x2[5] += b1.y; x2[6] += b1.z; x2[7] += b1.w;
                        }
                    }
                    // the projection's own output, as the unfused path stores it: bf16(acc * rstd + bias)
                    const float rs = p.ssq_in != nullptr ? s_rstd[m] : 1.0f;
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        x1[e] *= rs;
                        x2[e] *= rs;
                        if (p.bias) {
                            x1[e] += __bfloat162float(p.bias[n0 + sub * 8 + e]);
                            x2[e] += __bfloat162float(p.bias[n0 + 64 + sub * 8 + e]);
                        }
                        x1[e] = round_bf16(x1[e]);
                        x2[e] = round_bf16(x2[e]);
                    }
                    const bool live = active && m < rows;
                    __nv_bfloat16* dst = nullptr;
                    if (head_kind == 0) {
                        dst = p.y + static_cast<int64_t>(x_row0 + m) * p.n_out + n0;
                    } else if (live && s_slot[lm] >= 0) {
                        const int kvh = static_cast<int>(blockIdx.x) - p.q_heads - (head_kind == 2 ? p.kv_heads : 0);
                        dst = (head_kind == 1 ? p.k_cache : p.v_cache) +
                              (static_cast<int64_t>(s_slot[lm]) * p.kv_heads + kvh) * kTileN;
                    }
                    if (head_kind < 2) {
                        if (head_w != nullptr) {
                            float ss = 0.f;
#pragma unroll
                            for (int e = 0; e < 8; ++e) ss += x1[e] * x1[e] + x2[e] * x2[e];
                            ss += __shfl_xor_sync(0xffffffffu, ss, 4);
                            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
                            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
                            const float scale = rsqrtf(ss / static_cast<float>(kTileN) + p.qk_eps);
                            const uint4 wa = *reinterpret_cast<const uint4*>(head_w + sub * 8);
                            const uint4 wb = *reinterpret_cast<const uint4*>(head_w + 64 + sub * 8);
                            const uint32_t wa4[4] = {wa.x, wa.y, wa.z, wa.w}, wb4[4] = {wb.x, wb.y, wb.z, wb.w};
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                x1[2 * e] = round_bf16(x1[2 * e] * scale * bf16_lo(wa4[e]));
                                x1[2 * e + 1] = round_bf16(x1[2 * e + 1] * scale * bf16_hi(wa4[e]));
                                x2[2 * e] = round_bf16(x2[2 * e] * scale * bf16_lo(wb4[e]));
                                x2[2 * e + 1] = round_bf16(x2[2 * e + 1] * scale * bf16_hi(wb4[e]));
                            }
                        }
                        const float* cs = s_cos + lm * (kTileN / 2) + sub * 8;
                        const float* sn = s_sin + lm * (kTileN / 2) + sub * 8;
#pragma unroll
                        for (int e = 0; e < 8; ++e) {
                            const float a = x1[e], b = x2[e];
                            x1[e] = a * cs[e] - b * sn[e];
                            x2[e] = b * cs[e] + a * sn[e];
                        }
                    }
                    if (live && dst != nullptr) {
                        *reinterpret_cast<uint4*>(dst + sub * 8) = make_uint4(pack_bf16(x1[0], x1[1]), pack_bf16(x1[2], x1[3]),
                                                                            pack_bf16(x1[4], x1[5]), pack_bf16(x1[6], x1[7]));
                        *reinterpret_cast<uint4*>(dst + 64 + sub * 8) = make_uint4(pack_bf16(x2[0], x2[1]), pack_bf16(x2[2], x2[3]),
                                                                                 pack_bf16(x2[4], x2[5]), pack_bf16(x2[6], x2[7]));
                    }
                }
            }
            continue;
        }
        if (is_epi) {
            // F / 4 is a power of two (split is 2, 4 or 8): shifts instead of divisions.
            const int f4_shift = 31 - __clz(F / 4);
            const int te = (warp - 2) * 32 + lane;  // 0..127
            const float* rb = xbuf + buf_off / 4u;
            for (int i = te; i < (cpr << f4_shift); i += 128) {
                const int col = i >> f4_shift;
                const int f = (i & ((1 << f4_shift) - 1)) * 4;   // owned-feature index
                // All partials first (independent loads), then the sum in rank order.
                float4 pg[8], pu[8];
#pragma unroll
                for (uint32_t rr = 0; rr < 8; ++rr) {
                    if (rr < split) {
                        pg[rr] = *reinterpret_cast<const float4*>(rb + ((rr * NUM_A * cpr + col) * F + f));
                        if (NUM_A == 2)
                            pu[rr] = *reinterpret_cast<const float4*>(rb + ((rr * NUM_A * cpr + cpr + col) * F + f));
                    }
                }
                float4 sg = make_float4(0.f, 0.f, 0.f, 0.f), su = sg;
#pragma unroll
                for (uint32_t rr = 0; rr < 8; ++rr) {
                    if (rr < split) {
                        sg.x += pg[rr].x; sg.y += pg[rr].y; sg.z += pg[rr].z; sg.w += pg[rr].w;
                        if (NUM_A == 2) {
                            su.x += pu[rr].x; su.y += pu[rr].y; su.z += pu[rr].z; su.w += pu[rr].w;
                        }
                    }
                }
                const int m = r * cpr + col;
                const int n = n0 + static_cast<int>(rank) * F + f;
                const bool valid = m < rows && n < p.n_out;
                float v[4] = {sg.x, sg.y, sg.z, sg.w};
                float uu[4] = {su.x, su.y, su.z, su.w};
                if (p.ssq_in != nullptr) {
                    const float rs = s_rstd[m];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        v[e] *= rs;
                        uu[e] *= rs;
                    }
                }
                if (p.residual != nullptr) {
                    // the residual stream ends here: add, store, and hand the row's sum of squares to the next GEMM
                    float part = 0.f;
                    if (valid) {
                        __nv_bfloat16* rp = p.residual + static_cast<int64_t>(x_row0 + m) * p.n_out + n;
                        const uint2 rr = *reinterpret_cast<const uint2*>(rp);
                        const float r4[4] = {bf16_lo(rr.x), bf16_hi(rr.x), bf16_lo(rr.y), bf16_hi(rr.y)};
                        float s4[4];
#pragma unroll
                        for (int e = 0; e < 4; ++e) s4[e] = round_bf16(v[e]) + r4[e];
                        const uint2 packed = make_uint2(pack_bf16(s4[0], s4[1]), pack_bf16(s4[2], s4[3]));
                        *reinterpret_cast<uint2*>(rp) = packed;
                        if (p.ssq_of_rounded) {
                            s4[0] = bf16_lo(packed.x); s4[1] = bf16_hi(packed.x);
                            s4[2] = bf16_lo(packed.y); s4[3] = bf16_hi(packed.y);
                        }
                        part = s4[0] * s4[0] + s4[1] * s4[1] + s4[2] * s4[2] + s4[3] * s4[3];
                    }
                    // the F / 4 neighbouring lanes hold the other features of the same token column
                    for (int o = F / 8; o > 0; o >>= 1) part += __shfl_xor_sync(0xffffffffu, part, o);
                    if ((i & (F / 4 - 1)) == 0 && m < rows)
                        atomicAdd(p.ssq_out + x_row0 + m, static_cast<unsigned long long>(part * kSsqScale));
                    continue;
                }
                if (valid) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        if (NUM_A == 2) {
                            const float gv = round_bf16(v[e]), uv = round_bf16(uu[e]);
                            v[e] = gated_pair<EPI>(gv, uv, p.act_limit);
                        } else if (p.bias) {
                            v[e] += __bfloat162float(p.bias[n + e]);
                        }
                        if (EPI == B200_EPILOGUE_RELU2) v[e] = fmaxf(v[e], 0.f) * fmaxf(v[e], 0.f);
                        if (EPI == B200_EPILOGUE_GELU_ERF) v[e] = gelu_erf_f(v[e]);
                    }
                    const int64_t at = static_cast<int64_t>(x_row0 + m) * p.y_pitch + y_col0 + n;
                    if (EPI == B200_EPILOGUE_F32) {
                        *reinterpret_cast<float4*>(reinterpret_cast<float*>(p.y) + at) = make_float4(v[0], v[1], v[2], v[3]);
                        continue;
                    }
                    uint2 packed = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
                    *reinterpret_cast<uint2*>(p.y + at) = packed;
                }
            }
        }
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base, tmem_cols);
}

using SkinnyKernel = void (*)(CUtensorMap, CUtensorMap, CUtensorMap, CUtensorMap, CUtensorMap, SkinnyParams);
SkinnyKernel skinny_kernel_for(int epilogue, bool heads = false) {
    if (heads) return skinny_gemm_kernel<B200_EPILOGUE_NONE, true>;
    switch (epilogue) {
        case B200_EPILOGUE_SWIGLU: return skinny_gemm_kernel<B200_EPILOGUE_SWIGLU>;
        case B200_EPILOGUE_GEGLU: return skinny_gemm_kernel<B200_EPILOGUE_GEGLU>;
        case B200_EPILOGUE_GEGLU_ERF: return skinny_gemm_kernel<B200_EPILOGUE_GEGLU_ERF>;
        case B200_EPILOGUE_RELU2: return skinny_gemm_kernel<B200_EPILOGUE_RELU2>;
        case B200_EPILOGUE_GELU_ERF: return skinny_gemm_kernel<B200_EPILOGUE_GELU_ERF>;
        case B200_EPILOGUE_CLAMPED_SWIGLU: return skinny_gemm_kernel<B200_EPILOGUE_CLAMPED_SWIGLU>;
        case B200_EPILOGUE_F32: return skinny_gemm_kernel<B200_EPILOGUE_F32>;
        default: return skinny_gemm_kernel<B200_EPILOGUE_NONE>;
    }
}

}  // namespace

struct TmapCacheEntry {
    const void* base;
    uint64_t inner, outer, pitch;
    uint32_t box_inner, box_outer;
    CUtensorMap map;
};

// Small per-thread cache: the same weights and activation buffers come back
// every layer and every step, and encoding a tensor map costs about a microsecond.
int cached_tmap(CUtensorMap* out, const void* base, uint64_t inner, uint64_t outer, uint64_t pitch,
                uint32_t box_inner, uint32_t box_outer) {
    constexpr int kEntries = 1024;
    thread_local TmapCacheEntry cache[kEntries];
    thread_local bool used[kEntries] = {};
    uint64_t h = reinterpret_cast<uintptr_t>(base) * 0x9E3779B97F4A7C15ull;
    h ^= (outer * 0x100000001B3ull) ^ (inner << 20) ^ (static_cast<uint64_t>(box_outer) << 44);
    const int idx = static_cast<int>((h >> 17) % kEntries);
    TmapCacheEntry& e = cache[idx];
    if (used[idx] && e.base == base && e.inner == inner && e.outer == outer && e.pitch == pitch &&
        e.box_inner == box_inner && e.box_outer == box_outer) {
        *out = e.map;
        return B200_OK;
    }
    int err = make_tmap_2d_bf16_sw128(out, base, inner, outer, pitch, box_inner, box_outer);
    if (err != B200_OK) return err;
    e = TmapCacheEntry{base, inner, outer, pitch, box_inner, box_outer, *out};
    used[idx] = true;
    return B200_OK;
}

static void set_fusion(SkinnyParams* p, const SkinnyFusion* f) {
    p->ssq_in = f ? f->ssq_in : nullptr;
    p->norm_eps = f ? f->eps : 0.f;
    p->norm_width = f ? f->norm_width : 1;
    p->residual = f ? static_cast<__nv_bfloat16*>(f->residual) : nullptr;
    p->ssq_out = f ? f->ssq_out : nullptr;
    p->ssq_of_rounded = f && f->ssq_of_rounded ? 1 : 0;
    const HeadEpilogue* h = f ? f->heads : nullptr;
    p->head_mode = h ? 1 : 0;
    p->q_norm_w = h ? static_cast<const __nv_bfloat16*>(h->q_norm_w) : nullptr;
    p->k_norm_w = h ? static_cast<const __nv_bfloat16*>(h->k_norm_w) : nullptr;
    p->cos_t = h ? h->cos_t : nullptr;
    p->sin_t = h ? h->sin_t : nullptr;
    p->positions = h ? h->positions : nullptr;
    p->out_loc = h ? h->out_loc : nullptr;
    p->k_cache = h ? static_cast<__nv_bfloat16*>(h->k_cache) : nullptr;
    p->v_cache = h ? static_cast<__nv_bfloat16*>(h->v_cache) : nullptr;
    p->q_heads = h ? h->q_heads : 0;
    p->kv_heads = h ? h->kv_heads : 0;
    p->max_pos = h ? h->max_pos : 1;
    p->num_slots = h ? h->num_slots : 0;
    p->qk_eps = h ? h->eps : 0.f;
}

static int env_int(const char* name, int dflt) {
    const char* v = getenv(name);
    return (v && *v) ? atoi(v) : dflt;
}

// Split of `tiles` output tiles along K: at most one CTA per SM, and clusters of 8 only as many as the GPCs
// hold at once with one CTA per SM (14 on B200; 16 of them ran in two waves: a [2048, 2048] projection took
// 18 us with a split of 8 and 14 us with 4).
static int cluster_split(int tiles, int kb_total) {
    constexpr int kMaxClusters8 = 14;
    int split = 1;
    while (split < 8 && tiles * split * 2 <= sm_count() && split * 2 <= kb_total &&
           (split < 4 || tiles <= kMaxClusters8))
        split *= 2;
    return split;
}

// K split of a slab: up to one CTA per SM in total, at most 8 ranks (portable cluster size).
int skinny_gemm_split(int M, int N, int K, int epilogue) {
    (void)M;
    const int n_out = epilogue_is_gated(epilogue) ? N / 2 : N;
    const int kb_total = K / kBlockK;
    const int n_tiles = div_ceil(n_out, kTileN);
    const int forced = env_int("B200_GEMM_SPLIT", 0);
    if (forced > 0) return forced;
    // One CTA per SM at most: a CTA holds its whole K slice plus the exchange buffer, so two
    // rarely fit on an SM, and a second wave would double the kernel's time.
    return cluster_split(n_tiles, kb_total);
}

// One slab of at most 256 rows.
int launch_skinny_gemm(void* y, const void* x, const void* w, const void* bias, int M, int N,
                       int K, int64_t ldx, int epilogue, int* status, cudaStream_t stream,
                       const SkinnyFusion* fuse = nullptr, float act_limit = 0.f) {
    const bool gated = epilogue_is_gated(epilogue);
    const int n_out = gated ? N / 2 : N;
    // accumulator columns: 32, or a multiple of the 64-column exchange round (the epilogue walks whole rounds)
    const int nt = M <= 32 ? 32 : div_ceil(M, kRoundCols) * kRoundCols;
    const int kb_total = K / kBlockK;
    const int n_tiles = div_ceil(n_out, kTileN);
    const int num_a = gated ? 2 : 1;
    const int split = skinny_gemm_split(M, N, K, epilogue);
    if (fuse != nullptr && split == 1) {
        set_last_error("linear: the residual-stream fusions live in the split-K epilogue; this shape does not split");
        return B200_ERR_UNSUPPORTED;
    }
    const int kbp = div_ceil(kb_total, split);

    const uint32_t stage_bytes = num_a * kTileN * kBlockK * 2 + nt * kBlockK * 2;
    const int cpr = nt < kRoundCols ? nt : kRoundCols;
    uint32_t exch_bytes = split > 1 ? (nt > cpr ? 2u : 1u) * num_a * cpr * kTileN * 4u : 0u;
    if (fuse != nullptr && fuse->heads != nullptr) {
        if (gated || N != (fuse->heads->q_heads + 2 * fuse->heads->kv_heads) * kTileN) {
            set_last_error("linear: the head epilogue wants a plain projection of (q_heads + 2 kv_heads) x 128 features");
            return B200_ERR_INVALID_ARGUMENT;
        }
        if (cpr % split != 0) {
            set_last_error("linear: the head epilogue needs the K split (%d) to divide the %d token columns of a round", split, cpr);
            return B200_ERR_UNSUPPORTED;
        }
        // cos | sin [nt / split][64] and the slots [nt / split] of the tokens a rank owns
        exch_bytes += static_cast<uint32_t>(nt / split) * (kTileN * 4u + 4u) + 16u;
    }
    const uint32_t smem_limit = 200 * 1024;
    int stages = kbp < kMaxStages ? kbp : kMaxStages;
    // More tiles than SMs (lm_head): keep the ring small enough for two CTAs per SM, so one CTA's
    // start-up and epilogue overlap the other's streaming.
    if (n_tiles * split > sm_count())
        while (stages > 2 && stages * stage_bytes + exch_bytes > 100 * 1024) --stages;
    while (stages > 1 && stages * stage_bytes > smem_limit) --stages;
    while (stages > 1 && stages * stage_bytes + exch_bytes > smem_limit) --stages;
    uint32_t smem_bytes = stages * stage_bytes + exch_bytes;
    smem_bytes += 1024;  // alignment slack
    if (stage_bytes + exch_bytes > smem_limit) {
        set_last_error("linear: one pipeline stage (%u bytes) does not fit in shared memory",
                       stage_bytes);
        return B200_ERR_UNSUPPORTED;
    }

    CUtensorMap tmap_w, tmap_x;
    int err = cached_tmap(&tmap_w, w, static_cast<uint64_t>(K), static_cast<uint64_t>(N),
                          static_cast<uint64_t>(K) * 2, kBlockK, kTileN);
    if (err != B200_OK) return err;
    err = cached_tmap(&tmap_x, x, static_cast<uint64_t>(K), static_cast<uint64_t>(M),
                      static_cast<uint64_t>(ldx) * 2, kBlockK, static_cast<uint32_t>(nt));
    if (err != B200_OK) return err;

    SkinnyParams p;
    p.y = static_cast<__nv_bfloat16*>(y);
    p.bias = static_cast<const __nv_bfloat16*>(bias);
    p.M = M;
    p.n_out = n_out;
    p.up_row_offset = N / 2;
    p.kb_total = kb_total;
    p.nt = nt;
    p.stages = stages;
    p.epilogue = epilogue;
    p.status = status;
    p.group_counts = nullptr;
    p.group_offsets = nullptr;
    p.w_rows_per_group = 0;
    p.head_k = 0;
    p.act_limit = act_limit;
    p.y_pitch = n_out;
    set_fusion(&p, fuse);

    auto kernel = skinny_kernel_for(epilogue, p.head_mode != 0);
    B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem_bytes)));
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(n_tiles, split, 1), dim3(kThreads), smem_bytes, stream,
                                  dim3(1, split, 1), tmap_w, tmap_x, tmap_x, tmap_x, tmap_x, p));
    return B200_OK;
}

// Grouped GEMM for expert layers: group g multiplies rows [offsets[g], offsets[g] + counts[g]) of
// x [total_rows, K] by w[g] ([N, K], groups stacked) into the same rows of y.  counts / offsets
// are device arrays (no host synchronisation); max_rows_per_group bounds any count.
int launch_grouped_gemm(void* y, const void* x, const void* w, const int32_t* counts,
                        const int32_t* offsets, int num_groups, int max_rows_per_group,
                        int64_t total_rows, int N, int K, int epilogue, int* status,
                        cudaStream_t stream, float act_limit) {
    const bool gated = epilogue_is_gated(epilogue);
    const int n_out = gated ? N / 2 : N;
    const int num_a = gated ? 2 : 1;
    const int kb_total = K / kBlockK;
    const int n_tiles = div_ceil(n_out, kTileN);
    const int slabs = div_ceil(max_rows_per_group, 256);
    if (num_groups == 0 || slabs == 0 || total_rows == 0) return B200_OK;
    // Many rows per group on average (prefill batches): tensor-bound, take the tile kernel.
    if (total_rows >= static_cast<int64_t>(num_groups) * env_int("B200_GROUPED_TILE_MIN_ROWS", 128) && num_groups <= 256)
        return launch_grouped_tile_gemm(y, x, w, counts, offsets, num_groups, total_rows, N, K, epilogue, status,
                                        stream, act_limit);
    int nt_max = 32;
    while (nt_max < 256 && nt_max < max_rows_per_group) nt_max *= 2;
    const uint32_t stage_bytes = num_a * kTileN * kBlockK * 2 + nt_max * kBlockK * 2;
    const uint32_t smem_limit = 200 * 1024;
    int stages = kb_total < kMaxStages ? kb_total : kMaxStages;
    // Many more CTAs than SMs (every expert active): keep the ring small enough for two CTAs per
    // SM, so one CTA's start-up and epilogue overlap the other's streaming.
    const int ring_cap_kb = env_int("B200_GROUPED_RING_KB", 100);
    if (static_cast<int64_t>(n_tiles) * num_groups > 2 * sm_count())
        while (stages > 2 && stages * stage_bytes > static_cast<uint32_t>(ring_cap_kb) * 1024u) --stages;
    while (stages > 1 && stages * stage_bytes > smem_limit) --stages;
    const uint32_t smem_bytes = stages * stage_bytes + 1024;

    CUtensorMap tmap_w, tx[4];
    int err = cached_tmap(&tmap_w, w, static_cast<uint64_t>(K), static_cast<uint64_t>(num_groups) * N,
                          static_cast<uint64_t>(K) * 2, kBlockK, kTileN);
    if (err != B200_OK) return err;
    const uint32_t boxes[4] = {32, 64, 128, 256};
    for (int i = 0; i < 4; ++i) {
        err = cached_tmap(&tx[i], x, static_cast<uint64_t>(K), static_cast<uint64_t>(total_rows),
                          static_cast<uint64_t>(K) * 2, kBlockK, boxes[i]);
        if (err != B200_OK) return err;
    }
    SkinnyParams p;
    p.y = static_cast<__nv_bfloat16*>(y);
    p.bias = nullptr;
    p.M = 0;
    p.n_out = n_out;
    p.up_row_offset = N / 2;
    p.kb_total = kb_total;
    p.nt = nt_max;
    p.stages = stages;
    p.epilogue = epilogue;
    p.status = status;
    p.group_counts = counts;
    p.group_offsets = offsets;
    p.w_rows_per_group = N;
    p.head_k = 0;
    p.act_limit = act_limit;
    p.y_pitch = n_out;
    set_fusion(&p, nullptr);
    auto kernel = skinny_kernel_for(epilogue);
    B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         static_cast<int>(smem_bytes)));
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(n_tiles, slabs, num_groups), dim3(kThreads), smem_bytes, stream,
                                  dim3(1, 1, 1), tmap_w, tx[0], tx[1], tx[2], tx[3], p));
    return B200_OK;
}

// y[m, h*N + n] = sum_k x[m, h*K + k] w[h*N + n, k]: one projection per head, slabs of 256 rows.
int launch_linear_heads(void* y, const void* x, const void* w, int M, int heads, int N, int K, int* status,
                        cudaStream_t stream) {
    const int kb_total = K / kBlockK;
    const int n_tiles = div_ceil(N, kTileN);
    // the K split of the plain form, over all heads' tiles
    const int split = cluster_split(n_tiles * heads, kb_total);
    const int kbp = div_ceil(kb_total, split);
    for (int m0 = 0; m0 < M; m0 += 256) {
        const int rows = M - m0 < 256 ? M - m0 : 256;
        const int nt = rows <= 32 ? 32 : div_ceil(rows, kRoundCols) * kRoundCols;
        const uint32_t stage_bytes = kTileN * kBlockK * 2 + nt * kBlockK * 2;
        const int cpr = nt < kRoundCols ? nt : kRoundCols;
        const uint32_t exch_bytes = split > 1 ? (nt > cpr ? 2u : 1u) * cpr * kTileN * 4u : 0u;
        int stages = kbp < kMaxStages ? kbp : kMaxStages;
        // more CTAs than SMs: small rings, two CTAs per SM
        const uint32_t limit = n_tiles * heads * split > sm_count() ? 100 * 1024 : 200 * 1024;
        while (stages > 1 && stages * stage_bytes + exch_bytes > limit) --stages;
        const uint32_t smem_bytes = stages * stage_bytes + exch_bytes + 1024;
        const __nv_bfloat16* xs = static_cast<const __nv_bfloat16*>(x) + static_cast<int64_t>(m0) * heads * K;
        CUtensorMap tmap_w, tmap_x;
        int err = cached_tmap(&tmap_w, w, static_cast<uint64_t>(K), static_cast<uint64_t>(heads) * N,
                              static_cast<uint64_t>(K) * 2, kBlockK, kTileN);
        if (err != B200_OK) return err;
        err = cached_tmap(&tmap_x, xs, static_cast<uint64_t>(heads) * K, static_cast<uint64_t>(rows),
                          static_cast<uint64_t>(heads) * K * 2, kBlockK, static_cast<uint32_t>(nt));
        if (err != B200_OK) return err;
        SkinnyParams p;
        p.y = static_cast<__nv_bfloat16*>(y) + static_cast<int64_t>(m0) * heads * N;
        p.bias = nullptr;
        p.M = rows;
        p.n_out = N;
        p.up_row_offset = 0;
        p.kb_total = kb_total;
        p.nt = nt;
        p.stages = stages;
        p.epilogue = B200_EPILOGUE_NONE;
        p.status = status;
        p.group_counts = nullptr;
        p.group_offsets = nullptr;
        p.w_rows_per_group = N;
        p.head_k = K;
        p.act_limit = 0.f;
        p.y_pitch = static_cast<int64_t>(heads) * N;
        set_fusion(&p, nullptr);
        auto kernel = skinny_kernel_for(B200_EPILOGUE_NONE);
        B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             static_cast<int>(smem_bytes)));
        B200_CHECK_CUDA(launch_kernel(kernel, dim3(n_tiles, split, heads), dim3(kThreads), smem_bytes, stream,
                                      dim3(1, split, 1), tmap_w, tmap_x, tmap_x, tmap_x, tmap_x, p));
    }
    return B200_OK;
}

int launch_linear(void* y, const void* x, const void* w, const void* bias, int M, int N, int K,
                  int64_t ldx, int epilogue, int* status, cudaStream_t stream, const SkinnyFusion* fuse,
                  float act_limit) {
    // Few rows: stream the weights once (swap-AB, split-K).  Many rows: tensor-bound tiles.
    if (M >= env_int("B200_GEMM_TILE_MIN_M", 257)) {
        if (fuse != nullptr) {
            set_last_error("linear: the residual-stream fusions need at most 256 rows");
            return B200_ERR_UNSUPPORTED;
        }
        return launch_tile_gemm(y, x, w, bias, M, N, K, ldx, epilogue, status, stream, act_limit);
    }
    const int n_out = epilogue_is_gated(epilogue) ? N / 2 : N;
    const __nv_bfloat16* xp = static_cast<const __nv_bfloat16*>(x);
    char* yp = static_cast<char*>(y);
    const int64_t y_row_bytes = static_cast<int64_t>(n_out) * (epilogue == B200_EPILOGUE_F32 ? 4 : 2);
    for (int m0 = 0; m0 < M; m0 += 256) {
        const int rows = (M - m0) < 256 ? (M - m0) : 256;
        int err = launch_skinny_gemm(yp + m0 * y_row_bytes,
                                     xp + static_cast<int64_t>(m0) * ldx, w, bias, rows, N, K, ldx,
                                     epilogue, status, stream, fuse, act_limit);
        if (err != B200_OK) return err;
    }
    return B200_OK;
}

}  // namespace b200

extern "C" {

int b200_linear_heads(void* y, const void* x, const void* w, int M, int heads, int N, int K, b200_stream_t stream) {
    B200_CHECK_ARG(M >= 0 && heads > 0 && N > 0 && K > 0, "linear_heads: bad shape");
    B200_CHECK_ARG(M == 0 || (y && x && w), "linear_heads: NULL tensor");
    B200_CHECK_ARG(K % 64 == 0 && N % 8 == 0, "linear_heads: K must be a multiple of 64, N of 8");
    B200_CHECK_ARG(heads <= 65535, "linear_heads: too many heads");
    if (M == 0) return B200_OK;
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    return b200::launch_linear_heads(y, x, w, M, heads, N, K, status, static_cast<cudaStream_t>(stream));
}

int b200_linear_act(void* y, const void* x, const void* w, int M, int N, int K, int epilogue, float act_limit, int dtype,
                    b200_stream_t stream) {
    B200_CHECK_ARG(M >= 0 && N > 0 && K > 0, "linear_act: bad shape");
    B200_CHECK_ARG(M == 0 || (y && x && w), "linear_act: NULL tensor");
    B200_CHECK_ARG(K % 64 == 0 && N % 16 == 0, "linear_act: K must be a multiple of 64, N of 16");
    B200_CHECK_ARG(epilogue >= B200_EPILOGUE_NONE && epilogue <= B200_EPILOGUE_F32, "linear_act: unknown epilogue");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "linear_act: unknown dtype");
    if (M == 0) return B200_OK;
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == B200_DTYPE_F32)
        return b200::launch_linear_f32(static_cast<float*>(y), static_cast<const float*>(x), static_cast<const float*>(w), M,
                                       N, K, 1, nullptr, nullptr, epilogue, s, act_limit);
    return b200::launch_linear(y, x, w, nullptr, M, N, K, K, epilogue, status, s, nullptr, act_limit);
}

int b200_linear(void* y, const void* x, const void* w, const void* bias, int M, int N, int K,
                int64_t ldx, int epilogue, b200_stream_t stream) {
    B200_CHECK_ARG(M >= 0 && N > 0 && K > 0, "linear: bad shape");
    B200_CHECK_ARG(M == 0 || (y && x && w), "linear: NULL tensor");
    B200_CHECK_ARG(K % 64 == 0, "linear: K must be a multiple of 64");
    B200_CHECK_ARG(ldx >= K && ldx % 8 == 0, "linear: ldx must be >= K and a multiple of 8");
    B200_CHECK_ARG(epilogue >= B200_EPILOGUE_NONE && epilogue <= B200_EPILOGUE_RELU2,
                   "linear: unknown epilogue");
    const bool gated = b200::epilogue_is_gated(epilogue);
    B200_CHECK_ARG(!gated || (N % 2 == 0), "linear: a gated epilogue needs an even N");
    B200_CHECK_ARG(!gated || bias == nullptr, "linear: bias is not supported with a gated epilogue");
    B200_CHECK_ARG((gated ? N / 2 : N) % 8 == 0, "linear: output width must be a multiple of 8");
    if (M == 0) return B200_OK;
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    return b200::launch_linear(y, x, w, bias, M, N, K, ldx, epilogue, status,
                               static_cast<cudaStream_t>(stream));
}

}  // extern "C"
