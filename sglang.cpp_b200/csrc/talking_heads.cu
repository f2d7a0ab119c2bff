// Paged attention whose heads mix their softmax weights before they meet the values (head_mix.cuh): prompts, and the
// choice of the kernels.  Decode steps run on attention_decode.cu.
//
//   * prefill_kernel leaves O_gc, what the weights of head g make of the values of key / value head c, for all pairs.
//     One CTA per SM walks over work items (request, key head, 128 / group query tokens, two value heads): a tile of 128
//     rows, each a (token, head in the group) pair, against the window's keys.  Per K/V tile of 128 keys
//         S = Q K^T                  accumulator in TMEM
//         P = exp(S)                 as bf16 in TMEM, in two places in turn; S is free once its threads have read it
//         O_c += P V_c               for both value heads in one product, accumulators in TMEM for the whole row
//     Queries and keys are bounded (they are unit vectors up to a factor), so the exponentials need no running maximum:
//     nothing is rescaled, and the two groups of softmax warps take K/V tiles in turn without waiting for one another.
//     No product waits for the one before it: S of the next tile runs ahead of P V of this one.  Warp 0 loads queries
//     and, through rings of two TMA buffers, keys a tile ahead of values, into the next items as well; warp 1 issues
//     the products.
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
constexpr uint32_t kQOff = 0, kKOff = 2 * kAtomBytes, kKBytes = 2 * kAtomBytes;   // keys: columns 0-63, 64-127
constexpr uint32_t kVOff = kKOff + kStages * kKBytes, kVBytes = 4 * kAtomBytes;   // values: the same of either head
constexpr uint32_t kTileBytes = kVOff + kStages * kVBytes;
constexpr uint32_t kColS = 0, kColP = 128, kColO = 256;   // TMEM columns: S; P of even and odd tiles (64 each); O of the value heads
constexpr float kMaxExponent = 100.f;       // log2 of the largest exponential

// A work item.
struct PrefillItem {
    int q_begin, t0, t_end, pos0, len, table, h, c0;
    int kv_end, head_tiles, skip, ntiles;    // ntiles 0: nothing to do; handed to the other roles, the end
    __device__ __forceinline__ int first_key(int kt) const { return (kt >= head_tiles ? kt + skip : kt) * kTile; }
};
// Behind the tiles in shared memory.  Barriers in pairs: per stage, or for even and odd tiles.
struct PrefillSync {
    float sum[4][kTile];                    // a row's weights, added up by the four threads that share it
    uint64_t k_full[kStages], k_empty[kStages], v_full[kStages], v_empty[kStages];
    uint64_t s_full[2], s_free[2], p_full[2], pv_done[2];
    uint64_t q_full, q_free, o_full, o_free;   // once per item
    uint64_t item_seen;
    PrefillItem item[2];                    // in place with q_full
    uint32_t tmem;
};
constexpr uint32_t kMaxSmem = 227 * 1024;   // (tiles start on a multiple of 1024, as the array itself should)
static_assert(kTileBytes + sizeof(PrefillSync) <= kMaxSmem, "");

struct PrefillParams {
    __nv_bfloat16* raw;     // [tokens, heads, kv heads, 128]
    const int32_t* page_table;
    int64_t pt_stride;
    const int32_t *table_idx, *seq_lens, *qo_indptr;
    int q_heads, kv_heads, group, value_pairs;
    int blocks, items;      // query blocks of the longest request; blocks * kv heads * value pairs * requests
    int kpc;                // keys per TMA copy = min(page_size, 128)
    int tile_boxes;         // the *_tile maps may be used (a pool of at least 128 slots)
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
__device__ __forceinline__ void tma_load_4d(uint32_t dst, const void* tmap, int c0, int c1, int c2, int c3, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes"
        " [%0], [%1, {%2, %3, %4, %5}], [%6];" ::"r"(dst),
        "l"(reinterpret_cast<uint64_t>(tmap)), "r"(c0), "r"(c1), "r"(c2), "r"(c3), "r"(bar)
        : "memory");
}
// 32 bytes, a whole sector.
__device__ __forceinline__ void store_32b(void* p, const uint32_t (&v)[8]) {
    asm volatile("st.global.v8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"l"(p), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]),
                 "r"(v[5]), "r"(v[6]), "r"(v[7])
                 : "memory");
}

// Whether any of the softmax threads says so; all of them meet here.
__device__ __forceinline__ bool softmax_any(bool mine) {
    int any;
    asm volatile(
        "{\n\t.reg .pred p, q;\n\t"
        "setp.ne.b32 p, %1, 0;\n\t"
        "bar.red.or.pred q, 1, %2, p;\n\t"
        "selp.b32 %0, 1, 0, q;\n\t}"
        : "=r"(any)
        : "r"(static_cast<int>(mine)), "n"(kSoftmaxThreads)
        : "memory");
    return any != 0;
}

__device__ __forceinline__ PrefillItem item_of(const PrefillParams& p, int index) {
    PrefillItem it = {};
    if (index >= p.items) return it;
    const int x = index % p.blocks, y = index / p.blocks % (p.kv_heads * p.value_pairs), b = index / p.blocks / (p.kv_heads * p.value_pairs);
    const int q_begin = p.qo_indptr[b], q_end = p.qo_indptr[b + 1], len = p.seq_lens[b], table = p.table_idx[b];
    const int QB = kTile / p.group, ext = q_end - q_begin, qb = (ext + QB - 1) / QB - 1 - x;   // heaviest blocks first
    if (qb < 0 || ext <= 0 || len <= 0) return it;
    it.q_begin = q_begin;
    it.t0 = qb * QB;
    it.t_end = min(it.t0 + QB, ext);
    it.pos0 = len - ext;
    it.len = len;
    it.table = table;
    it.h = y / p.value_pairs;
    it.c0 = y % p.value_pairs * 2;
    it.kv_end = min(len, it.pos0 + it.t_end);
    it.head_tiles = (min(p.w.keep_first, it.kv_end) + kTile - 1) / kTile;
    it.skip = max(0, p.w.oldest(it.pos0 + it.t0) / kTile - it.head_tiles);
    it.ntiles = (it.kv_end + kTile - 1) / kTile - it.skip;
    return it;
}

__global__ void __launch_bounds__(kThreads, 1)
prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
               const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_k_tile,
               const __grid_constant__ CUtensorMap tmap_v_tile, const PrefillParams p) {
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t smem_base = smem_u32(smem_raw);
    PrefillSync& S = *reinterpret_cast<PrefillSync*>(smem_raw + kTileBytes);
    const int G = p.group, step = static_cast<int>(gridDim.x), heads_per_box = min(2, p.kv_heads);
    if ((smem_base & 1023u) != 0) {   // (never: the swizzle counts on it)
        if (threadIdx.x == 0) atomicExch(&p.status[kStatusTimeout], 349);
        return;
    }
    pdl_launch_dependents();
    if (threadIdx.x == 0) {
        for (int s = 0; s < kStages; ++s) {
            mbar_init(smem_u32(&S.k_full[s]), 1);
            mbar_init(smem_u32(&S.k_empty[s]), 1);
            mbar_init(smem_u32(&S.v_full[s]), 1);
            mbar_init(smem_u32(&S.v_empty[s]), 1);
        }
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&S.s_full[i]), 1);
            mbar_init(smem_u32(&S.s_free[i]), 8);   // one arrival per softmax warp of the tile
            mbar_init(smem_u32(&S.p_full[i]), 8);
            mbar_init(smem_u32(&S.pv_done[i]), 1);
        }
        mbar_init(smem_u32(&S.q_full), 1);
        mbar_init(smem_u32(&S.q_free), 1);
        mbar_init(smem_u32(&S.o_full), 1);
        mbar_init(smem_u32(&S.item_seen), 1);
        mbar_init(smem_u32(&S.o_free), kSoftmaxThreads / 32);
        fence_mbar_init();
    }
    // Rows that no copy of this launch has written yet must not hold NaN patterns.
    {
        uint4* z = reinterpret_cast<uint4*>(smem_raw + kKOff);
        for (uint32_t i = threadIdx.x; i < (kTileBytes - kKOff) / 16; i += kThreads) z[i] = make_uint4(0, 0, 0, 0);
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(&S.tmem), 512);
        tmem_relinquish();
    }
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    pdl_wait_prior();

    if (warp == 0) {
        // ================= producer =================
        const uint32_t copy_bytes = static_cast<uint32_t>(p.kpc) * 128u;
        int n = 0, items = 0;   // tiles, items so far
        bool going = true;
        // (the whole warp gives up together)
        auto wait = [&](uint64_t& bar, int phase, int site) {
            return __all_sync(0xffffffffu, mbar_wait_bounded(smem_u32(&bar), static_cast<uint32_t>(phase) & 1u, p.status, site)) != 0;
        };
        PrefillItem it = item_of(p, blockIdx.x);
        for (int index = blockIdx.x; index < p.items && going; index += step) {
            const PrefillItem next = item_of(p, index + step);
            if (it.ntiles > 0) {
                if (items > 0 && !(wait(S.q_free, items - 1, 340) && wait(S.item_seen, items - 1, 354))) break;
                if (lane == 0) {
                    S.item[items & 1] = it;
                    mbar_arrive_expect_tx(smem_u32(&S.q_full), 2 * kAtomBytes);
                    tma_load_4d(smem_base + kQOff, &tmap_q, 0, it.h * G, it.q_begin + it.t0, 0, smem_u32(&S.q_full));
                }
                ++items;
                const int32_t* pt_row = p.page_table + static_cast<int64_t>(it.table) * p.pt_stride;
                // Full tiles whose pages are consecutive slots are fetched by one copy: the first slot of 32 tiles, one
                // per lane, or -1.
                auto look_up = [&](int base) {
                    const int kt = base + lane;
                    if (kt >= it.ntiles || !p.tile_boxes || p.kpc < 16) return -1;
                    const int k0 = it.first_key(kt);
                    if (it.kv_end - k0 < kTile) return -1;
                    const int first = pt_row[k0];
                    bool ok = first >= 0 && first + kTile <= p.num_slots;
                    for (int i = p.kpc; i < kTile; i += p.kpc) ok = pt_row[k0 + i] == first + i && ok;
                    return ok ? first : -1;
                };
                int firsts = look_up(0);
                auto load = [&](int kt, int first, bool values) {
                    const int g = n + kt, stage = g % kStages;
                    const uint32_t bar = smem_u32(values ? &S.v_full[stage] : &S.k_full[stage]);
                    if (g >= kStages && !wait(values ? S.v_empty[stage] : S.k_empty[stage], g / kStages - 1, 341)) return false;
                    const int heads = values ? heads_per_box : 1, head0 = values ? it.c0 : it.h;
                    const uint32_t dst0 = smem_base + (values ? kVOff + stage * kVBytes : kKOff + stage * kKBytes);
                    if (first >= 0) {
                        if (lane == 0) {
                            mbar_arrive_expect_tx(bar, heads * 2 * kAtomBytes);   // (a head that is not there is zeros)
                            tma_load_4d(dst0, values ? &tmap_v_tile : &tmap_k_tile, 0, first, 0, head0, bar);
                        }
                        __syncwarp();
                        return true;
                    }
                    const int k0 = it.first_key(kt), ncopies = (min(kTile, it.kv_end - k0) + p.kpc - 1) / p.kpc;
                    if (lane == 0) mbar_arrive_expect_tx(bar, static_cast<uint32_t>(heads * ncopies) * 2u * copy_bytes);
                    __syncwarp();
                    for (int copy = lane; copy < ncopies; copy += 32) {
                        int slot = pt_row[k0 + copy * p.kpc];
                        if (slot < 0 || static_cast<int64_t>(slot) + p.kpc > p.num_slots) {
                            atomicExch(&p.status[kStatusBadIndex], slot + 1);
                            slot = 0;
                        }
                        for (int j = 0; j < heads; ++j) {
                            const uint32_t dst = dst0 + j * 2 * kAtomBytes + copy * copy_bytes;
                            tma_load_3d(dst, values ? &tmap_v : &tmap_k, 0, head0 + j, slot, bar);
                            tma_load_3d(dst + kAtomBytes, values ? &tmap_v : &tmap_k, 64, head0 + j, slot, bar);
                        }
                    }
                    return true;
                };
                int first = __shfl_sync(0xffffffffu, firsts, 0);
                going = load(0, first, false);
                for (int kt = 0; kt < it.ntiles && going; ++kt) {
                    int following = -1;
                    if (kt + 1 < it.ntiles) {
                        if ((kt + 1) % 32 == 0) firsts = look_up(kt + 1);
                        following = __shfl_sync(0xffffffffu, firsts, (kt + 1) % 32);
                        going = load(kt + 1, following, false);
                    }
                    going = going && load(kt, first, true);
                    first = following;
                }
                n += it.ntiles;
            }
            it = next;
        }
        if (going && (items == 0 || (wait(S.q_free, items - 1, 352) && wait(S.item_seen, items - 1, 355))) && lane == 0) {
            S.item[items & 1].ntiles = 0;
            mbar_arrive(smem_u32(&S.q_full));
        }
    } else if (warp == 1) {
        // ================= MMA issuer =================
        if (elect_one()) {
            const uint32_t tmem = S.tmem, idesc_s = idesc_bf16_128x128(false), idesc_pv = idesc_bf16_128xn(heads_per_box * 128, true);
            int n = 0, items = 0;
            bool going = true;
            while (going) {
                if (!mbar_wait_bounded(smem_u32(&S.q_full), static_cast<uint32_t>(items) & 1u, p.status, 345)) break;
                const int ntiles = S.item[items & 1].ntiles;
                if (ntiles == 0) break;
                auto issue_s = [&](int kt) {
                    const int g = n + kt, stage = g % kStages;
                    const uint32_t keys = smem_base + kKOff + stage * kKBytes;
                    // S of the tile before has been read
                    if (g > 0 && !mbar_wait_bounded(smem_u32(&S.s_free[(g - 1) & 1]), static_cast<uint32_t>((g - 1) >> 1) & 1u, p.status, 344))
                        return false;
                    if (!mbar_wait_bounded(smem_u32(&S.k_full[stage]), static_cast<uint32_t>(g / kStages) & 1u, p.status, 342)) return false;
                    tc_fence_after();
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks) {
                        const uint32_t off = (ks >> 2) * kAtomBytes + (ks & 3) * 32;
                        tc_mma_bf16(tmem + kColS, kmajor_sw128_desc(smem_base + kQOff + off), kmajor_sw128_desc(keys + off), idesc_s,
                                    ks > 0 ? 1u : 0u);
                    }
                    tc_commit(smem_u32(&S.s_full[g & 1]));
                    tc_commit(smem_u32(&S.k_empty[stage]));
                    if (kt + 1 == ntiles) tc_commit(smem_u32(&S.q_free));
                    return true;
                };
                going = issue_s(0);
                for (int kt = 0; kt < ntiles && going; ++kt) {
                    const int g = n + kt, stage = g % kStages;
                    going = (kt + 1 >= ntiles || issue_s(kt + 1)) &&
                            mbar_wait_bounded(smem_u32(&S.v_full[stage]), static_cast<uint32_t>(g / kStages) & 1u, p.status, 347) &&
                            // O of the item before has been read
                            (kt > 0 || items == 0 ||
                             mbar_wait_bounded(smem_u32(&S.o_free), static_cast<uint32_t>(items - 1) & 1u, p.status, 350)) &&
                            mbar_wait_bounded(smem_u32(&S.p_full[g & 1]), static_cast<uint32_t>(g >> 1) & 1u, p.status, 343);
                    if (!going) break;
                    tc_fence_after();
                    const uint32_t values = smem_base + kVOff + stage * kVBytes;
#pragma unroll
                    for (int ks = 0; ks < 8; ++ks)   // keys ks*16 .. +15: eight packed columns of P; both heads' columns
                        tc_mma_bf16_ts(tmem + kColO, tmem + kColP + (g & 1) * 64u + ks * 8u, mnmajor_sw128_desc(values + ks * 2048),
                                       idesc_pv, (kt > 0 || ks > 0) ? 1u : 0u);
                    tc_commit(smem_u32(&S.v_empty[stage]));
                    tc_commit(smem_u32(&S.pv_done[g & 1]));
                    if (kt + 1 == ntiles) tc_commit(smem_u32(&S.o_full));
                }
                n += ntiles;
                ++items;
            }
        }
    } else {
        // ================= softmax / output rows =================
        const int sw = warp - 2;                  // 0..15
        const int turn = sw >> 3;                 // takes the tiles of this parity, and value head c0 + turn
        const int qtr = warp & 3;                 // TMEM lane quarter this warp may read
        const int half = (sw & 7) >> 2;           // keys / head-dim columns [64*half, 64*half + 64)
        const int r = qtr * 32 + lane;            // query row = TMEM lane
        const uint32_t lane_addr = S.tmem + (static_cast<uint32_t>(qtr * 32) << 16);
        const uint32_t s_addr = lane_addr + kColS + static_cast<uint32_t>(half * 64);
        const uint32_t p_addr = lane_addr + kColP + static_cast<uint32_t>(turn * 64 + half * 32);
        const uint32_t o_addr = lane_addr + kColO + static_cast<uint32_t>(turn * 128 + half * 64);
        const float sc = p.scale_log2;
        int n = 0, items = 0, mine = 0;           // tiles, items and this group's tiles so far
        bool failed = false;
        auto wait = [&](uint64_t& bar, int phase, int site) {
            if (!failed && !mbar_wait_bounded(smem_u32(&bar), static_cast<uint32_t>(phase) & 1u, p.status, site)) failed = true;
            tc_fence_after();
        };
        while (true) {
            wait(S.q_full, items, 353);
            const PrefillItem it = S.item[items & 1];
            if (softmax_any(failed || it.ntiles == 0)) break;   // (everybody has read the last item's sums as well)
            if (threadIdx.x == 64) mbar_arrive(smem_u32(&S.item_seen));
            const int tok = it.t0 + r / G;
            const int limit = min(it.pos0 + tok, it.len - 1);   // last visible key of this row
            const int oldest = p.w.oldest(limit);               // keys before it are seen below keep_first only
            // which of the 32 keys from `first` on this row sees, as bits
            auto below = [](int m) { return m <= 0 ? 0u : m >= 32 ? 0xffffffffu : (1u << m) - 1u; };
            auto seen = [&](int first) {
                return below(limit + 1 - first) & (~below(oldest - first) | below(p.w.keep_first - first));
            };
            float sum0 = 0.f, sum1 = 0.f;
            for (int kt = (n & 1) ^ turn; kt < it.ntiles; kt += 2, ++mine) {
                wait(S.s_full[turn], mine, 346);
                const int k0 = it.first_key(kt) + half * 64;    // first key of this thread's columns
                const bool need_mask = __any_sync(0xffffffffu, k0 + 63 > limit || (k0 < oldest && k0 + 63 >= p.w.keep_first));
                uint32_t sv[2][32];
                tmem_ld_32x32b_x32(s_addr, sv[0]);
                tmem_ld_32x32b_x32(s_addr + 32, sv[1]);
                tmem_ld_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&S.s_free[turn]));
                if (mine > 0) wait(S.pv_done[turn], mine - 1, 348);   // P of this group's last tile has been read
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
                    tmem_st_32x32b_x16(p_addr + c * 16, packed);
                }
                tmem_st_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(smem_u32(&S.p_full[turn]));
            }
            // O over the sum of the row's four partial sums
            S.sum[turn * 2 + half][r] = sum0 + sum1;
            asm volatile("bar.sync 1, %0;" ::"n"(kSoftmaxThreads) : "memory");
            const float l = (S.sum[0][r] + S.sum[1][r]) + (S.sum[2][r] + S.sum[3][r]);
            wait(S.o_full, items, 351);
            uint32_t ov[2][32];
            tmem_ld_32x32b_x32(o_addr, ov[0]);
            tmem_ld_32x32b_x32(o_addr + 32, ov[1]);
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&S.o_free));   // (the sums have been read as well)
            if (it.c0 + turn < p.kv_heads) {
                // Four neighbouring threads exchange quarters of their rows (16 columns, 32 bytes), so that they store
                // whole ones: of the row of thread `row` of the four, this thread gets its own quarter.
                const float inv = l > 0.f ? 1.f / l : 0.f;
                const int me = lane & 3;
                uint32_t w[4][8];   // [quarter]
#pragma unroll
                for (int c = 0; c < 4; ++c)
#pragma unroll
                    for (int j = 0; j < 8; ++j)
                        w[c][j] = pack_bf16(__uint_as_float(ov[c >> 1][(c & 1) * 16 + 2 * j]) * inv,
                                            __uint_as_float(ov[c >> 1][(c & 1) * 16 + 2 * j + 1]) * inv);
#pragma unroll
                for (int bit = 1; bit < 4; bit <<= 1)   // rows and quarters trade places, a bit of their numbers at a time
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        if (c & bit) continue;
#pragma unroll
                        for (int j = 0; j < 8; ++j) {
                            const bool upper = (me & bit) != 0;
                            const uint32_t give = upper ? w[c][j] : w[c | bit][j];
                            const uint32_t got = __shfl_xor_sync(0xffffffffu, give, bit);
                            if (upper) w[c][j] = got;
                            else w[c | bit][j] = got;
                        }
                    }
#pragma unroll
                for (int c = 0; c < 4; ++c) {
                    const int row = (r & ~3) + c, tok_c = it.t0 + row / G;
                    const int64_t at = (static_cast<int64_t>(it.q_begin + tok_c) * p.q_heads + it.h * G + row % G) * p.kv_heads + it.c0 + turn;
                    if (tok_c < it.t_end && !failed) store_32b(p.raw + at * kD + half * 64 + me * 16, w[c]);
                }
            }
            n += it.ntiles;
            ++items;
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(S.tmem, 512);
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

// A 4-D map of bf16 with the 128-byte swizzle.
int make_map_4d(CUtensorMap* out, const void* base, const cuuint64_t (&dims)[4], const cuuint64_t (&strides)[3], const cuuint32_t (&box)[4]) {
    EncodeTiledFn fn = encode_tiled_fn();
    if (!fn) {
        set_last_error("cuTensorMapEncodeTiled is not available from this driver");
        return B200_ERR_CUDA;
    }
    const cuuint32_t es[4] = {1, 1, 1, 1};
    const CUresult r = fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, es,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        set_last_error("cuTensorMapEncodeTiled (4-D map) failed with CUresult %d", static_cast<int>(r));
        return B200_ERR_CUDA;
    }
    return B200_OK;
}

int launch_prefill(const WindowAttention& a, cudaStream_t stream) {
    PrefillParams p;
    p.raw = static_cast<__nv_bfloat16*>(a.mix.scratch);
    p.page_table = a.page_table;
    p.pt_stride = a.pt_stride;
    p.table_idx = a.table_idx;
    p.seq_lens = a.seq_lens;
    p.qo_indptr = a.qo_indptr;
    p.q_heads = a.heads;
    p.kv_heads = a.kv_heads;
    p.group = a.heads / a.kv_heads;
    p.value_pairs = div_ceil(a.kv_heads, 2);
    p.blocks = div_ceil(a.max_extend, kTile / p.group);
    p.items = p.blocks * p.kv_heads * p.value_pairs * a.batch;
    p.kpc = a.page_size < kTile ? a.page_size : kTile;
    p.num_slots = a.num_slots;
    p.tile_boxes = a.num_slots >= kTile ? 1 : 0;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.status = a.status;
    p.w = a.window;
    // columns 0-63 of a tile's rows, then columns 64-127: of the (token, head) rows of a query block, of the slots of a tile,
    // of one or two heads
    const cuuint64_t head = kD * 2, half = 128, slot = static_cast<cuuint64_t>(a.kv_heads) * head;
    const cuuint32_t two = p.kv_heads < 2 ? 1u : 2u, rows = p.tile_boxes ? kTile : 8u;
    CUtensorMap tq, tk, tv, tk_tile, tv_tile;
    int err = make_map_4d(&tq, a.q, {64, static_cast<cuuint64_t>(a.heads), static_cast<cuuint64_t>(a.tokens), 2},
                          {head, static_cast<cuuint64_t>(a.q_st) * 2, half},
                          {64, static_cast<cuuint32_t>(p.group), static_cast<cuuint32_t>(kTile / p.group), 2});
    const cuuint64_t pool[4] = {64, static_cast<cuuint64_t>(a.num_slots), 2, static_cast<cuuint64_t>(a.kv_heads)}, strides[3] = {slot, half, head};
    if (err == B200_OK) err = make_map_4d(&tk_tile, a.k_cache, pool, strides, {64, rows, 2, 1});
    if (err == B200_OK) err = make_map_4d(&tv_tile, a.v_cache, pool, strides, {64, rows, 2, two});
    if (err == B200_OK) err = make_kv_tile_tmap(&tk, a.k_cache, a.num_slots, a.kv_heads, p.kpc);
    if (err == B200_OK) err = make_kv_tile_tmap(&tv, a.v_cache, a.num_slots, a.kv_heads, p.kpc);
    if (err != B200_OK) return err;
    const int smem = static_cast<int>(kTileBytes + sizeof(PrefillSync));
    B200_CHECK_CUDA(cudaFuncSetAttribute(prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    const int grid = p.items < sm_count() ? p.items : sm_count();
    B200_CHECK_CUDA(launch_kernel(prefill_kernel, dim3(grid), dim3(kThreads), smem, stream, dim3(1, 1, 1), tq, tk, tv, tk_tile, tv_tile, p));
    return B200_OK;
}

}  // namespace

bool talking_heads_tc_supported(const WindowAttention& a, int dtype) {
    const int group = a.heads / a.kv_heads;
    if (dtype != B200_DTYPE_BF16 || a.plain || a.dp != 128 || a.vp != 128 || a.scale <= 0.f || group > 16) return false;
    if (!(a.mix.score_bound > 0.f) || a.mix.score_bound * a.scale * 1.4426950408889634f > kMaxExponent) return false;
    if (a.window.gate_st % 8 != 0 || a.window.out_st % 8 != 0 || !attention_prefill_tc_supported(a.q, a.q_st, a.dp, a.out)) return false;
    if (a.decode) return a.batch <= 1024 && talking_decode_supported(a.heads, a.kv_heads);
    const int64_t items = static_cast<int64_t>(div_ceil(a.max_extend, kTile / group)) * a.kv_heads * div_ceil(a.kv_heads, 2) * a.batch;
    return (group & (group - 1)) == 0 && items < (1ll << 30);
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
