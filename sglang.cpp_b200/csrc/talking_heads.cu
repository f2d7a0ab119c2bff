// Paged attention whose heads mix their softmax weights before they meet the values (head_mix.cuh): prompts, and the
// choice of the kernels.  Decode steps run on attention_decode.cu.
//
//   * prefill_kernel leaves O_gc, what the weights of head g make of the values of key / value head c, for all pairs.
//     One CTA owns (request, key head, 128 / group query tokens, two value heads): a tile of 128 rows, each a (token,
//     head in the group) pair, against the window's keys.  Per K/V tile of 128 keys
//         S = Q K^T                  accumulator in TMEM
//         P = exp(S)                 as bf16 in TMEM, in two places in turn; S is free once its threads have read it
//         O_c += P V_c               for both value heads in one product, accumulators in TMEM for the whole row
//     Queries and keys are bounded (they are unit vectors up to a factor), so the exponentials need no running maximum:
//     nothing is rescaled, and the two groups of softmax warps take K/V tiles in turn without waiting for one another.
//     No product waits for the one before it: S of the next tile runs ahead of P V of this one.  Warp 0 loads tiles
//     through rings of two TMA buffers, keys a tile ahead of values; warp 1 issues the products.
//   * mix_kernel sums O_gc over the heads.
//   * fp32, other head sizes and counts, unbounded scores: the plain attention kernel in place of the first one.
#include "common.cuh"
#include "head_mix.cuh"
#include "kernels.h"
#include "tcgen05.cuh"
#include "tensormap.cuh"

namespace b200 {
namespace {

constexpr int kD = 128;
constexpr int kTile = 128;                  // keys per K/V tile and rows per query tile
constexpr int kSoftmaxThreads = 2 * 256;
constexpr int kThreads = 64 + kSoftmaxThreads;
constexpr uint32_t kAtomBytes = 128 * 128;  // 128 rows x 64 bf16: one swizzle atom column
constexpr int kStages = 2;
constexpr uint32_t kQOff = 0, kKOff = 2 * kAtomBytes, kKBytes = 2 * kAtomBytes;   // per stage: keys 64 columns wide each
constexpr uint32_t kVOff = kKOff + kStages * kKBytes, kVBytes = 4 * kAtomBytes;   // per stage: both value heads
constexpr uint32_t kSmemBytes = kVOff + kStages * kVBytes;
constexpr uint32_t kColS = 0, kColP = 128, kColO = 256;   // TMEM columns: S; P of even and odd tiles (64 each); O of the value heads
constexpr float kMaxExponent = 100.f;       // log2 of the largest exponential

struct PrefillParams {
    __nv_bfloat16* raw;     // [tokens, heads, kv heads, 128]
    const __nv_bfloat16* q;
    int64_t q_st;
    const int32_t* page_table;
    int64_t pt_stride;
    const int32_t *table_idx, *seq_lens, *qo_indptr;
    int q_heads, kv_heads, group, value_pairs;
    int kpc;                // keys per TMA copy = min(page_size, 128)
    int whole_tile_boxes;
    int64_t num_slots;
    float scale_log2;
    int* status;
    AttentionWindow w;
};

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__global__ void __launch_bounds__(kThreads, 1)
prefill_kernel(const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_v,
               const __grid_constant__ CUtensorMap tmap_k_tile, const __grid_constant__ CUtensorMap tmap_v_tile,
               const PrefillParams p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t k_full[kStages], k_empty[kStages], v_full[kStages], v_empty[kStages];
    __shared__ __align__(8) uint64_t s_full[2], s_free[2], p_full[2], pv_done[2];   // per tile parity
    __shared__ __align__(8) uint64_t all_done;   // (of its own: a group that skips phases of pv_done cannot wait for a later one)
    __shared__ uint32_t tmem_base_slot;

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t smem_base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t* smem_gen = smem_raw + (smem_base - smem_u32(smem_raw));
    const int G = p.group, QB = kTile / G;
    const int b = blockIdx.z, h = blockIdx.y / p.value_pairs, c0 = blockIdx.y % p.value_pairs * 2;
    const int nv = min(2, p.kv_heads - c0);

    pdl_launch_dependents();
    pdl_wait_prior();

    const int q_begin = p.qo_indptr[b], ext = p.qo_indptr[b + 1] - q_begin, len = p.seq_lens[b], table = p.table_idx[b];
    const int nqb = (ext + QB - 1) / QB;
    const int qb = nqb - 1 - static_cast<int>(blockIdx.x);   // heaviest blocks first
    if (qb < 0 || ext <= 0 || len <= 0) return;              // whole CTA, before any barrier or TMEM use
    const int t0 = qb * QB, t_end = min(t0 + QB, ext);
    const int pos0 = len - ext, kv_end = min(len, pos0 + t_end);
    const int head_tiles = (min(p.w.keep_first, kv_end) + kTile - 1) / kTile;
    const int skip = max(0, p.w.oldest(pos0 + t0) / kTile - head_tiles);
    const int ntiles = (kv_end + kTile - 1) / kTile - skip;
    auto first_key = [&](int kt) { return (kt >= head_tiles ? kt + skip : kt) * kTile; };

    if (threadIdx.x == 0) {
        for (int s = 0; s < kStages; ++s) {
            mbar_init(smem_u32(&k_full[s]), 1);
            mbar_init(smem_u32(&k_empty[s]), 1);
            mbar_init(smem_u32(&v_full[s]), 1);
            mbar_init(smem_u32(&v_empty[s]), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&s_full[i]), 1);
            mbar_init(smem_u32(&s_free[i]), 8);   // likewise
            mbar_init(smem_u32(&p_full[i]), 8);   // one arrival per softmax warp of the tile
            mbar_init(smem_u32(&pv_done[i]), 1);
        }
        mbar_init(smem_u32(&all_done), 1);
        fence_mbar_init();
    }
    // Rows that no copy ever wrote must not hold NaN patterns: only the last tile has such rows, and only in buffers that
    // no tile before it has filled.
    const bool clear = kv_end % kTile != 0 && ntiles <= kStages;
    if (clear) {
        uint4* z = reinterpret_cast<uint4*>(smem_gen + kKOff);
        for (uint32_t i = threadIdx.x; i < (kSmemBytes - kKOff) / 16; i += kThreads) z[i] = make_uint4(0, 0, 0, 0);
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(&tmem_base_slot), 512);
        tmem_relinquish();
    }
    // Q rows in the swizzled K-major layout: row r = (token t0 + r / G, head h * G + r % G); rows past the request's
    // last token are zero.  Warps 2-17: 32 rows, a quarter of the columns each.
    if (warp >= 2) {
        const int sw = warp - 2, r = (sw & 3) * 32 + lane, tok = t0 + r / G;
        const uint4* src = reinterpret_cast<const uint4*>(p.q + static_cast<int64_t>(q_begin + tok) * p.q_st +
                                                          static_cast<int64_t>(h * G + r % G) * kD);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = (sw >> 2) * 4 + i;
            const uint4 v = tok < t_end ? src[c] : make_uint4(0, 0, 0, 0);
            const uint32_t a = swz128(smem_base + kQOff + (c >> 3) * kAtomBytes + r * 128, c & 7);
            asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(a), "r"(v.x), "r"(v.y), "r"(v.z), "r"(v.w) : "memory");
        }
    }
    fence_proxy_async_smem();
    tc_fence_before();
    // The producer does not wait for the others, unless they are clearing its buffers.
    if (warp == 0 && !clear)
        asm volatile("bar.arrive 2, %0;" ::"n"(kThreads) : "memory");
    else
        asm volatile("bar.sync 2, %0;" ::"n"(kThreads) : "memory");
    tc_fence_after();

    if (warp == 0) {
        // ================= producer =================
        __syncwarp();   // (one of its threads has set up the barriers)
        const int32_t* pt_row = p.page_table + static_cast<int64_t>(table) * p.pt_stride;
        const uint32_t copy_bytes = static_cast<uint32_t>(p.kpc) * 128u;
        // the first slots of a tile's pages, fetched a tile ahead of their use
        struct Pages {
            int at[4];
        };
        auto pages_of = [&](int kt) {
            Pages s = {{0, 0, 0, 0}};
            if (kt >= ntiles) return s;
            const int k0 = first_key(kt), ncopies = (min(kTile, kv_end - k0) + p.kpc - 1) / p.kpc;
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (i * 32 + lane < ncopies) s.at[i] = pt_row[k0 + (i * 32 + lane) * p.kpc];
            return s;
        };
        auto load = [&](int kt, const Pages& pages, bool values) {
            const int stage = kt % kStages, valid = min(kTile, kv_end - first_key(kt)), ncopies = (valid + p.kpc - 1) / p.kpc;
            const uint32_t bar = smem_u32(values ? &v_full[stage] : &k_full[stage]);
            if (kt >= kStages && !mbar_wait_bounded(smem_u32(values ? &v_empty[stage] : &k_empty[stage]),
                                                    static_cast<uint32_t>(kt / kStages - 1) & 1u, p.status, 341))
                return false;
            int sl[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                sl[i] = pages.at[i];
                if (sl[i] < 0 || static_cast<int64_t>(sl[i]) + p.kpc > p.num_slots) {
                    atomicExch(&p.status[kStatusBadIndex], sl[i] + 1);
                    sl[i] = 0;
                }
            }
            // A tile whose pages are consecutive slots is fetched with two 128-key boxes per head.
            bool mine = true;
            const int first = __shfl_sync(0xffffffffu, sl[0], 0);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int copy = i * 32 + lane;
                if (copy < ncopies && sl[i] != first + copy * p.kpc) mine = false;
            }
            const bool whole = __all_sync(0xffffffffu, mine) && valid == kTile && p.whole_tile_boxes;
            const int heads = values ? nv : 1;
            const uint32_t dst0 = smem_base + (values ? kVOff + stage * kVBytes : kKOff + stage * kKBytes);
            if (lane == 0) mbar_arrive_expect_tx(bar, static_cast<uint32_t>(heads * ncopies) * 2u * copy_bytes);
            __syncwarp();
            if (whole) {
                if (lane < 2 * heads)
                    tma_load_3d(dst0 + lane * kAtomBytes, values ? &tmap_v_tile : &tmap_k_tile, (lane & 1) * 64,
                                values ? c0 + (lane >> 1) : h, first, bar);
                return true;
            }
            for (int j = 0; j < heads; ++j) {
                const int head = values ? c0 + j : h;
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int copy = i * 32 + lane;
                    if (copy < ncopies) {
                        const uint32_t dst = dst0 + j * 2 * kAtomBytes + copy * copy_bytes;
                        tma_load_3d(dst, values ? &tmap_v : &tmap_k, 0, head, sl[i], bar);
                        tma_load_3d(dst + kAtomBytes, values ? &tmap_v : &tmap_k, 64, head, sl[i], bar);
                    }
                }
            }
            return true;
        };
        Pages now = pages_of(0), next = pages_of(1);
        bool going = load(0, now, false);
        for (int kt = 0; kt < ntiles && going; ++kt) {
            const Pages after = pages_of(kt + 2);
            going = (kt + 1 >= ntiles || load(kt + 1, next, false)) && load(kt, now, true);
            now = next;
            next = after;
        }
    } else if (warp == 1) {
        // ================= MMA issuer =================
        if (elect_one()) {
            const uint32_t tmem_base = tmem_base_slot;
            const uint32_t idesc_s = idesc_bf16_128x128(false), idesc_pv = idesc_bf16_128xn(nv * 128, true);
            auto issue_s = [&](int kt) {
                const int stage = kt % kStages;
                const uint32_t keys = smem_base + kKOff + stage * kKBytes;
                if (!mbar_wait_bounded(smem_u32(&k_full[stage]), static_cast<uint32_t>(kt / kStages) & 1u, p.status, 342)) return false;
                tc_fence_after();
#pragma unroll
                for (int ks = 0; ks < 8; ++ks) {
                    const uint32_t off = (ks >> 2) * kAtomBytes + (ks & 3) * 32;
                    tc_mma_bf16(tmem_base + kColS, kmajor_sw128_desc(smem_base + kQOff + off), kmajor_sw128_desc(keys + off), idesc_s,
                                ks > 0 ? 1u : 0u);
                }
                tc_commit(smem_u32(&s_full[kt & 1]));
                tc_commit(smem_u32(&k_empty[stage]));
                return true;
            };
            const bool begun = issue_s(0);
            for (int kt = 0; kt < ntiles && begun; ++kt) {
                const uint32_t i = kt & 1, turn = static_cast<uint32_t>(kt >> 1) & 1u;
                const int stage = kt % kStages;
                // S of the next tile as soon as this one's has been read
                if (kt + 1 < ntiles && (!mbar_wait_bounded(smem_u32(&s_free[i]), turn, p.status, 344) || !issue_s(kt + 1))) break;
                if (!mbar_wait_bounded(smem_u32(&v_full[stage]), static_cast<uint32_t>(kt / kStages) & 1u, p.status, 347) ||
                    !mbar_wait_bounded(smem_u32(&p_full[i]), turn, p.status, 343))
                    break;
                tc_fence_after();
                const uint32_t values = smem_base + kVOff + stage * kVBytes;
#pragma unroll
                for (int ks = 0; ks < 8; ++ks)   // keys ks*16 .. +15: eight packed columns of P; both value heads' columns
                    tc_mma_bf16_ts(tmem_base + kColO, tmem_base + kColP + i * 64u + ks * 8u, mnmajor_sw128_desc(values + ks * 2048),
                                   idesc_pv, (kt > 0 || ks > 0) ? 1u : 0u);
                tc_commit(smem_u32(&v_empty[stage]));
                tc_commit(smem_u32(&pv_done[i]));
                if (kt + 1 == ntiles) tc_commit(smem_u32(&all_done));
            }
        }
    } else {
        // ================= softmax / output rows =================
        const int sw = warp - 2;                  // 0..15
        const int turn = sw >> 3;                 // takes the tiles of this parity, then value head c0 + turn
        const int qtr = warp & 3;                 // TMEM lane quarter this warp may read
        const int half = (sw & 7) >> 2;           // keys / head-dim columns [64*half, 64*half + 64)
        const int r = qtr * 32 + lane;            // query row = TMEM lane
        const int tok = t0 + r / G;
        const int limit = min(pos0 + tok, len - 1);   // last visible key of this row
        const int oldest = p.w.oldest(limit);         // keys before it are seen below keep_first only
        // which of the 32 keys from `first` on this row sees, as bits
        auto below = [](int n) { return n <= 0 ? 0u : n >= 32 ? 0xffffffffu : (1u << n) - 1u; };
        auto seen = [&](int first) {
            return below(limit + 1 - first) & (~below(oldest - first) | below(p.w.keep_first - first));
        };
        const uint32_t lane_addr = tmem_base_slot + (static_cast<uint32_t>(qtr * 32) << 16);
        const uint32_t s_addr = lane_addr + kColS + static_cast<uint32_t>(half * 64);
        const uint32_t p_addr = lane_addr + kColP + static_cast<uint32_t>(turn * 64 + half * 32);
        const float sc = p.scale_log2;
        float sum0 = 0.f, sum1 = 0.f;
        bool failed = false;
        for (int kt = turn; kt < ntiles; kt += 2) {
            if (!failed && !mbar_wait_bounded(smem_u32(&s_full[turn]), static_cast<uint32_t>(kt >> 1) & 1u, p.status, 345))
                failed = true;
            tc_fence_after();
            const int k0 = first_key(kt) + half * 64;    // first key of this thread's columns
            const bool need_mask = __any_sync(0xffffffffu, k0 + 63 > limit || (k0 < oldest && k0 + 63 >= p.w.keep_first));
            uint32_t sv[2][32];
            tmem_ld_32x32b_x32(s_addr, sv[0]);
            tmem_ld_32x32b_x32(s_addr + 32, sv[1]);
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&s_free[turn]));
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                if (need_mask) {   // (an exponent of -inf: no weight)
                    const uint32_t bits = seen(k0 + c * 32);
#pragma unroll
                    for (int i = 0; i < 32; ++i)
                        if ((bits & (1u << i)) == 0) sv[c][i] = 0xff800000u;
                }
                uint32_t packed[16];
#pragma unroll
                for (int i = 0; i < 32; i += 2) {
                    const float p0 = ex2(__uint_as_float(sv[c][i]) * sc), p1 = ex2(__uint_as_float(sv[c][i + 1]) * sc);
                    sum0 += p0;
                    sum1 += p1;
                    packed[i >> 1] = pack_bf16(p0, p1);
                }
                if (c == 0 && kt >= 2) {   // P of this group's last tile has been read
                    if (!failed && !mbar_wait_bounded(smem_u32(&pv_done[turn]), static_cast<uint32_t>((kt >> 1) - 1) & 1u, p.status, 348))
                        failed = true;
                    tc_fence_after();
                }
                tmem_st_32x32b_x16(p_addr + c * 16, packed);
            }
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&p_full[turn]));
        }
        // all products, then O over the sum of the row's four partial sums
        if (!failed && !mbar_wait_bounded(smem_u32(&all_done), 0u, p.status, 346)) failed = true;
        tc_fence_after();
        float* s_sum = reinterpret_cast<float*>(smem_gen + kQOff);   // [4][128]: nobody reads Q any more
        s_sum[(turn * 2 + half) * kTile + r] = sum0 + sum1;
        asm volatile("bar.sync 1, %0;" ::"n"(kSoftmaxThreads) : "memory");
        const float l = (s_sum[r] + s_sum[kTile + r]) + (s_sum[2 * kTile + r] + s_sum[3 * kTile + r]);
        if (turn < nv) {
            const bool store = !failed && tok < t_end;
            const float inv = l > 0.f ? 1.f / l : 0.f;
            const int64_t row = (static_cast<int64_t>(q_begin + (store ? tok : 0)) * p.q_heads + h * G + r % G) * p.kv_heads + c0 + turn;
            uint4* dst = reinterpret_cast<uint4*>(p.raw + row * kD + half * 64);
            const uint32_t o_addr = lane_addr + kColO + static_cast<uint32_t>(turn) * 128u + static_cast<uint32_t>(half * 64);
            // (the TMEM loads are warp-wide: every lane takes part, only the stores are per row)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                uint32_t ov[32];
                tmem_ld_32x32b_x32(o_addr + c * 32, ov);
                tmem_ld_wait();
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    auto at = [&](int e) { return __uint_as_float(ov[j * 8 + e]) * inv; };
                    const uint4 w = make_uint4(pack_bf16(at(0), at(1)), pack_bf16(at(2), at(3)), pack_bf16(at(4), at(5)),
                                               pack_bf16(at(6), at(7)));
                    if (store) dst[c * 4 + j] = w;
                }
            }
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base_slot, 512);
}

// Half a warp per (token, key / value head), HC output heads and 64 pairs of elements at a time, four pairs per thread.
constexpr int kMixWarps = 4, kMixLanes = 16, kMixItems = kMixWarps * 32 / kMixLanes;

// VEC: the number of pairs is a multiple of four.
template <typename T, int HC, bool VEC>
__global__ void __launch_bounds__(kMixWarps * 32, 5)
mix_kernel(const MixOutput a, const T* __restrict__ raw, int tokens) {
    extern __shared__ __align__(16) float s_mix[];   // transposed, rows of a multiple of HC: [from head][to head]
    const int lane = threadIdx.x & (kMixLanes - 1);
    const int H = a.heads, group = H / a.kv_heads, steps = (group + HC - 1) / HC, row = a.kv_heads * steps * HC, pairs = a.pairs();
    pdl_launch_dependents();
    for (int i = threadIdx.x; i < H * row; i += kMixWarps * 32) {
        const int g = i / row, c = i % row / (steps * HC), j = i % (steps * HC);
        s_mix[i] = j < group ? a.weights[(c * group + j) * H + g] : 0.f;
    }
    __syncthreads();
    pdl_wait_prior();
    const int64_t items = static_cast<int64_t>(tokens) * a.kv_heads, from = static_cast<int64_t>(a.kv_heads) * a.vp;
    for (int64_t item = static_cast<int64_t>(blockIdx.x) * kMixItems + threadIdx.x / kMixLanes; item < items;
         item += static_cast<int64_t>(gridDim.x) * kMixItems) {
        const int64_t t = item / a.kv_heads;
        const int c = static_cast<int>(item - t * a.kv_heads);
        const T* src = raw + t * H * from + static_cast<int64_t>(c) * a.vp;
        for (int h0 = 0; h0 < group; h0 += HC) {
            for (int m = 4 * lane; m < pairs; m += 4 * kMixLanes) {
                float4 u[HC], v[HC];
#pragma unroll
                for (int i = 0; i < HC; ++i) u[i] = v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                const float* w = s_mix + c * steps * HC + h0;
#pragma unroll 4
                for (int g = 0; g < H; ++g, w += row) {
                    const T* o = src + g * from + m;
                    const float4 x = load_quad<VEC>(o, pairs - m), y = load_quad<VEC>(o + pairs, pairs - m);
                    float f[HC];
                    if (HC % 4 == 0) {
#pragma unroll
                        for (int i = 0; i < HC; i += 4) *reinterpret_cast<float4*>(f + i) = *reinterpret_cast<const float4*>(w + i);
                    } else {
#pragma unroll
                        for (int i = 0; i < HC; ++i) f[i] = w[i];
                    }
#pragma unroll
                    for (int i = 0; i < HC; ++i) {
                        u[i].x = fmaf(f[i], x.x, u[i].x);
                        u[i].y = fmaf(f[i], x.y, u[i].y);
                        u[i].z = fmaf(f[i], x.z, u[i].z);
                        u[i].w = fmaf(f[i], x.w, u[i].w);
                        v[i].x = fmaf(f[i], y.x, v[i].x);
                        v[i].y = fmaf(f[i], y.y, v[i].y);
                        v[i].z = fmaf(f[i], y.z, v[i].z);
                        v[i].w = fmaf(f[i], y.w, v[i].w);
                    }
                }
                const Turn r = turn_of<VEC>(a, t, m);
#pragma unroll
                for (int i = 0; i < HC; ++i) {
                    if (h0 + i >= group) break;
                    finish_mixed<T, VEC>(a, t, c * group + h0 + i, m, u[i], v[i], r);
                }
            }
        }
        if (2 * pairs < a.vp)
            for (int i = 0; i < group; ++i) clear_padding<T>(a, t, c * group + i, kMixLanes);
    }
}

template <typename T, bool VEC>
auto mix_kernel_for(int group) {
    return group <= 1 ? mix_kernel<T, 1, VEC> : group <= 2 ? mix_kernel<T, 2, VEC> : mix_kernel<T, 4, VEC>;
}

template <typename T>
int launch_mix(const WindowAttention& a, cudaStream_t stream) {
    const MixOutput m = mix_output(a);
    const int group = a.heads / a.kv_heads;
    auto kernel = m.pairs() % 4 == 0 ? mix_kernel_for<T, true>(group) : mix_kernel_for<T, false>(group);
    const int each = group <= 2 ? group : div_ceil(group, 4) * 4;   // (columns of a group in shared memory)
    const size_t smem = static_cast<size_t>(a.heads) * a.kv_heads * each * 4;
    B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    const int64_t ctas = div_ceil64(static_cast<int64_t>(a.tokens) * a.kv_heads, kMixItems);
    const int most = sm_count() * 12;
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(static_cast<unsigned>(ctas < most ? ctas : most)), dim3(kMixWarps * 32), smem, stream,
                                  dim3(1, 1, 1), m, static_cast<const T*>(a.mix.scratch), a.tokens));
    return B200_OK;
}

int launch_prefill(const WindowAttention& a, cudaStream_t stream) {
    PrefillParams p;
    p.raw = static_cast<__nv_bfloat16*>(a.mix.scratch);
    p.q = static_cast<const __nv_bfloat16*>(a.q);
    p.q_st = a.q_st;
    p.page_table = a.page_table;
    p.pt_stride = a.pt_stride;
    p.table_idx = a.table_idx;
    p.seq_lens = a.seq_lens;
    p.qo_indptr = a.qo_indptr;
    p.q_heads = a.heads;
    p.kv_heads = a.kv_heads;
    p.group = a.heads / a.kv_heads;
    p.value_pairs = div_ceil(a.kv_heads, 2);
    p.kpc = a.page_size < kTile ? a.page_size : kTile;
    p.num_slots = a.num_slots;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.status = a.status;
    p.w = a.window;
    const int tile_box = a.num_slots >= kTile ? kTile : p.kpc;
    p.whole_tile_boxes = (tile_box == kTile && p.kpc < kTile) ? 1 : 0;
    CUtensorMap tk, tv, tk_tile, tv_tile;
    int err = make_kv_tile_tmap(&tk, a.k_cache, a.num_slots, a.kv_heads, p.kpc);
    if (err == B200_OK) err = make_kv_tile_tmap(&tv, a.v_cache, a.num_slots, a.kv_heads, p.kpc);
    if (err == B200_OK) err = make_kv_tile_tmap(&tk_tile, a.k_cache, a.num_slots, a.kv_heads, tile_box);
    if (err == B200_OK) err = make_kv_tile_tmap(&tv_tile, a.v_cache, a.num_slots, a.kv_heads, tile_box);
    if (err != B200_OK) return err;
    const int smem = kSmemBytes + 1024;
    B200_CHECK_CUDA(cudaFuncSetAttribute(prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    const dim3 grid(div_ceil(a.max_extend, kTile / p.group), a.kv_heads * p.value_pairs, a.batch);
    B200_CHECK_CUDA(launch_kernel(prefill_kernel, grid, dim3(kThreads), smem, stream, dim3(1, 1, 1), tk, tv, tk_tile, tv_tile, p));
    return B200_OK;
}

}  // namespace

bool talking_heads_tc_supported(const WindowAttention& a, int dtype) {
    const int group = a.heads / a.kv_heads;
    if (dtype != B200_DTYPE_BF16 || a.plain || a.dp != 128 || a.vp != 128 || a.scale <= 0.f || group > 16) return false;
    if (!(a.mix.score_bound > 0.f) || a.mix.score_bound * a.scale * 1.4426950408889634f > kMaxExponent) return false;
    if (a.window.gate_st % 8 != 0 || a.window.out_st % 8 != 0 || !attention_prefill_tc_supported(a.q, a.q_st, a.dp, a.out)) return false;
    if (a.decode) return a.batch <= 1024 && talking_decode_supported(a.heads, a.kv_heads);
    return (group & (group - 1)) == 0 && a.kv_heads * div_ceil(a.kv_heads, 2) <= 65535;
}

int launch_talking_heads(const WindowAttention& a, int dtype, cudaStream_t stream) {
    const bool tc = talking_heads_tc_supported(a, dtype);
    if (tc && a.decode) return launch_talking_decode(a, stream);
    const int err = tc ? launch_prefill(a, stream) : launch_plain_all_values(a, dtype, stream);
    if (err != B200_OK) return err;
    return dtype == B200_DTYPE_F32 ? launch_mix<float>(a, stream) : launch_mix<__nv_bfloat16>(a, stream);
}

}  // namespace b200

extern "C" {

int64_t b200_head_mix_scratch_bytes(int tokens, int heads, int kv_heads, int padded_value_dim, int dtype) {
    if (tokens < 0 || heads <= 0 || kv_heads <= 0 || padded_value_dim <= 0) return -1;
    return static_cast<int64_t>(tokens) * heads * kv_heads * padded_value_dim * (dtype == B200_DTYPE_F32 ? 4 : 2);
}

int64_t b200_head_mix_workspace_bytes(int max_batch, int heads, int kv_heads) {
    if (max_batch <= 0 || heads <= 0 || kv_heads <= 0 || !b200::talking_decode_supported(heads, kv_heads)) return -1;
    return b200::head_mix_workspace_bytes(max_batch, heads, kv_heads);
}

}  // extern "C"
