// Split-KV attention in the latent space on the tcgen05 tensor cores (decode steps, short extensions).
//
// Every query row (one token) has H heads that all read the same latents, so one latent tile is loaded
// once for all heads.  The products are turned around so that the long dimension, not the few heads, fills
// the 128 rows of the MMA:
//     S^T = C Q^T      KT keys x N heads, K = latent width: A is the latent tile as TMA delivers it
//     O^T += C^T P^T   128 latent elements x N heads, K = KT keys: A is the SAME tile read MN-major, so it
//                      is fetched from HBM once and never moved again (columns from out_width on, which only
//                      take part in the scores, are left out)
// with N = 16, 32 or 64 heads per block (more heads run as further blocks of the same row) and S^T, O^T
// accumulating in TMEM.
//
// A tile is KT keys - 128, or 64 for wide latents, whose tiles stay in shared memory so long (until the softmax
// of the whole tile is done) that 128 keys would leave no room to load ahead.  It lives in shared memory as
// width / 128 units of KT keys x 128 elements, a ring of which the producer keeps full; a unit is free again
// as soon as its O^T product has read it.
// Softmax: one thread per key (= TMEM lane), all heads of the block in its registers.  The reference
// maximum of a head only moves when some score exceeds it by more than 2^8, which a single block-wide vote
// finds out; the running sum stays per thread until a row is finished.  Everything about scores and weights
// is fp32; the weights are rounded to bf16 only as the operand of the second product.
//
// Work split: the tiles of all (row, head block) items form one sequence that is cut into equal contiguous
// runs, one per CTA (one CTA per SM).  An item that spans CTAs leaves fp32 partials, combined by the merge
// kernel.  No host plan: lengths are read from device memory, so a captured graph replays at any lengths.
//
// Roles: warp 0 producer, warp 1 issues S^T, warps 2-5 softmax and output, warp 6 issues O^T.  S^T and (where
// shared memory allows) P are double-buffered, so the two products and the softmax of neighbouring tiles
// overlap.
#include <math.h>

#include "common.cuh"
#include "kernels.h"
#include "tcgen05.cuh"
#include "tensormap.cuh"

namespace b200 {
namespace {

constexpr int kUnitElems = 128;                            // latent elements per unit
constexpr int kMaxUnits = 12;                              // units in the ring
constexpr int kThreads = 224;
constexpr int kMaxWidth = 640, kMaxOutWidth = 512;
constexpr uint32_t kColO = 0, kColS = 256;                 // TMEM columns: O^T (4 x 64), S^T (2 x 64)
constexpr float kLazyLog2 = 8.0f;
constexpr int kLens = 64;

struct LatentParams {
    __nv_bfloat16* out;         // [rows, heads, out_width]
    float* part_o;              // [2 * grid][N][out_width] un-normalised
    float* part_m;              // [2 * grid][N]
    float* part_l;
    int32_t* item_cta;          // [2 * items]: first and last CTA of an item
    const int32_t* page_table;
    int64_t pt_stride;
    const int32_t* row_table;
    const int32_t* row_len;
    int rows, heads, width, out_width;
    int blocks, per_block;      // head blocks per row, heads per block (<= N)
    int nb, no;                 // units per tile, and those of them that are averaged
    int ring;                   // units in the ring (>= nb)
    int p_bufs;                 // buffers of P, 1 or 2
    int kpc;                    // keys per TMA copy
    int64_t num_slots;
    float scale_log2;
    int early;                  // only the last key of a row is new in this step: everything else may be read
                                // ahead of the previous kernel's completion
    int* status;
};

// MN-major operand under the 128-byte swizzle (rows are keys, 64 latent elements per 128-byte row): the
// next 64 elements one atom further, the next 8 keys 1024 bytes further.
template <int KT>
__device__ __forceinline__ uint64_t mnmajor_desc(uint32_t smem_addr) {
    uint64_t d = 0;
    d |= static_cast<uint64_t>((smem_addr >> 4) & 0x3FFFu);
    d |= static_cast<uint64_t>((KT * 128) >> 4) << 16;
    d |= static_cast<uint64_t>(1024 >> 4) << 32;
    d |= static_cast<uint64_t>(1) << 46;
    d |= static_cast<uint64_t>(2) << 61;
    return d;
}

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
__device__ __forceinline__ bool softmax_any(bool v) {
    uint32_t r;
    asm volatile(
        "{\n\t"
        ".reg .pred p, q;\n\t"
        "setp.ne.u32 p, %1, 0;\n\t"
        "bar.red.or.pred q, 2, 128, p;\n\t"
        "selp.u32 %0, 1, 0, q;\n\t"
        "}\n"
        : "=r"(r)
        : "r"(v ? 1u : 0u)
        : "memory");
    return r != 0;
}

// Sums N per-lane vectors over the 32 lanes of a warp: each halving step swaps half of what is left with
// the lane `off` away.  Afterwards v[j] holds the total of column `col0 + j`, j < max(N / 32, 1).
template <int N>
__device__ __forceinline__ int warp_transpose_sum(float (&v)[N]) {
    const int lane = threadIdx.x & 31;
    int n = N, col0 = 0;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
        if (n > 1) {
            const int half = n / 2;
            const bool upper = (lane & off) != 0;
#pragma unroll
            for (int j = 0; j < N / 2; ++j) {
                if (j < half) {
                    const float send = upper ? v[j] : v[j + half];
                    const float keep = upper ? v[j + half] : v[j];
                    v[j] = keep + __shfl_xor_sync(0xffffffffu, send, off);
                }
            }
            if (upper) col0 += half;
            n = half;
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
        }
    }
    return col0;
}

// The run of tiles a CTA owns, walked item by item by every role in the same order.
struct Walk {
    int row, block, tile;   // current item and first tile of it that belongs to this CTA
    int left;               // tiles this CTA still has to do
    int row0;               // first row of the run: the lengths of the next kLens rows are in shared memory
    const int* lens;
};
struct Segment {
    int row, block, t0, t1, len;   // tiles [t0, t1) of an item whose row has len keys
    bool starts, ends;             // the item starts / ends inside this segment
};
template <int KT>
__device__ __forceinline__ bool next_segment(Walk& w, const LatentParams& p, Segment& s) {
    if (w.left <= 0) return false;
    auto len_of = [&](int row) { return row - w.row0 < kLens ? w.lens[row - w.row0] : p.row_len[row]; };
    int len = len_of(w.row);
    while (len <= 0) {   // rows without keys own no tile
        ++w.row;
        w.block = 0;
        if (w.row >= p.rows) return false;
        len = len_of(w.row);
    }
    const int nt = (len + KT - 1) / KT;
    s.row = w.row;
    s.block = w.block;
    s.len = len;
    s.t0 = w.tile;
    s.t1 = min(nt, w.tile + w.left);
    s.starts = s.t0 == 0;
    s.ends = s.t1 == nt;
    w.left -= s.t1 - s.t0;
    w.tile = 0;
    if (++w.block == p.blocks) {
        w.block = 0;
        if (++w.row >= p.rows) w.left = 0;
    }
    return true;
}

template <int N, int KT>
__global__ void __launch_bounds__(kThreads, 1)
latent_attention_tc_kernel(const __grid_constant__ CUtensorMap tmap_c, const __grid_constant__ CUtensorMap tmap_q,
                           const LatentParams p) {
    constexpr uint32_t kAtomBytes = KT * 128;        // KT keys x 64 elements, 128-byte rows
    constexpr uint32_t kUnitBytes = 2 * kAtomBytes;
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t unit_full[kMaxUnits];
    __shared__ __align__(8) uint64_t unit_empty[kMaxUnits];
    __shared__ __align__(8) uint64_t q_full, q_empty, s_full[2], s_empty[2], p_full[2], pv_done[2], o_free;
    __shared__ uint32_t tmem_base_slot;
    __shared__ int s_scan[kThreads / 32 + 1];
    __shared__ int s_total, s_row, s_block, s_tile;
    __shared__ __align__(16) float s_ref[N];     // reference maximum per head, log2 units
    __shared__ __align__(16) float s_alpha[N];
    __shared__ float s_warp[4][N];
    __shared__ volatile int s_failed[2];
    __shared__ int s_len[kLens];
    __shared__ int s_slot[128];     // the producer's current group of page-table look-ups

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t smem_base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const uint32_t q_base = smem_base + static_cast<uint32_t>(p.ring) * kUnitBytes;
    const uint32_t p_base = q_base + static_cast<uint32_t>(N) * static_cast<uint32_t>(p.width) * 2u;
    constexpr uint32_t kPBytes = KT / 64 * N * 128u;
    const uint32_t stage_off = p_base + static_cast<uint32_t>(p.p_bufs) * kPBytes - smem_u32(smem_raw);   // output staging [16][128] fp32
    // The weights are the B operand of the second product: keys contiguous (one 2-byte store per head), or for
    // a full 64 heads heads contiguous, so that a thread stores its key's row in 16-byte pieces.
    constexpr bool kHeadsContiguous = N == 64;

    pdl_launch_dependents();
    if (threadIdx.x == 0) {
        for (int i = 0; i < p.ring; ++i) {
            mbar_init(smem_u32(&unit_full[i]), 1);
            mbar_init(smem_u32(&unit_empty[i]), 1);
        }
        mbar_init(smem_u32(&q_full), 1);
        mbar_init(smem_u32(&q_empty), 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(smem_u32(&s_full[i]), 1);
            mbar_init(smem_u32(&s_empty[i]), 4);
            mbar_init(smem_u32(&p_full[i]), 4);
            mbar_init(smem_u32(&pv_done[i]), 1);
        }
        mbar_init(smem_u32(&o_free), 4);
        fence_mbar_init();
        tma_prefetch_desc(&tmap_c);
        tma_prefetch_desc(&tmap_q);
        s_row = p.rows;
        s_failed[0] = s_failed[1] = 0;
    }
    if (warp == 1) {
        tmem_alloc(smem_u32(&tmem_base_slot), 512);
        tmem_relinquish();
    }
    if (!p.early) pdl_wait_prior();

    // ---- where this CTA's run starts: a scan of the rows' tile counts ----
    {
        const int per = (p.rows + kThreads - 1) / kThreads;
        const int r0 = min(static_cast<int>(threadIdx.x) * per, p.rows), r1 = min(r0 + per, p.rows);
        int mine = 0;
        for (int r = r0; r < r1; ++r) mine += (max(p.row_len[r], 0) + KT - 1) / KT * p.blocks;
        int incl = mine;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int up = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += up;
        }
        if (lane == 31) s_scan[warp] = incl;
        __syncthreads();
        int before = 0, total = 0;
        for (int w = 0; w < kThreads / 32; ++w) {
            if (w < warp) before += s_scan[w];
            total += s_scan[w];
        }
        const int begin = before + incl - mine;
        const int run = (total + static_cast<int>(gridDim.x) - 1) / static_cast<int>(gridDim.x);
        const int g0 = static_cast<int>(blockIdx.x) * run;
        if (g0 >= begin && g0 < begin + mine) {
            int at = begin;
            for (int r = r0; r < r1; ++r) {
                const int nt = (max(p.row_len[r], 0) + KT - 1) / KT;
                if (g0 < at + nt * p.blocks) {
                    s_row = r;
                    s_block = (g0 - at) / nt;
                    s_tile = (g0 - at) % nt;
                    break;
                }
                at += nt * p.blocks;
            }
        }
        if (threadIdx.x == 0) s_total = total;
    }
    __syncthreads();
    if (threadIdx.x < kLens && s_row + static_cast<int>(threadIdx.x) < p.rows)
        s_len[threadIdx.x] = p.row_len[s_row + threadIdx.x];
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = tmem_base_slot;
    const int run = (s_total + static_cast<int>(gridDim.x) - 1) / static_cast<int>(gridDim.x);
    const int g0 = static_cast<int>(blockIdx.x) * run;
    Walk walk;
    walk.row = s_row;
    walk.block = s_block;
    walk.tile = s_tile;
    walk.row0 = s_row;
    walk.lens = s_len;
    walk.left = s_row < p.rows ? min(run, s_total - g0) : 0;
    bool failed = false;
    Segment seg;

    if (warp == 0) {
        // ================= producer =================
        // Page-table look-ups run a group of 128 copies ahead of the loads: the whole warp fetches the next
        // group while one elected lane issues the copies of this one (copies issued lane by lane cost 250
        // cycles each).  A copy past the last key reads a row outside the tensor, which the copy engine fills
        // with zeros.
        const int copies = KT / p.kpc, group_tiles = 128 / copies;
        const bool whole_unit = p.kpc == KT;      // one copy brings both halves of a unit
        auto slots_of = [&](const Segment& g, int t0, int (&sl)[4]) {
            const int32_t* pt = p.page_table + static_cast<int64_t>(p.row_table[g.row]) * p.pt_stride;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int key = t0 * KT + (i * 32 + lane) * p.kpc;
                sl[i] = static_cast<int>(p.num_slots);
                if (key < min(g.len, g.t1 * KT)) {
                    const int64_t v = pt[key];
                    if (v < 0 || v + p.kpc > p.num_slots)
                        atomicExch(&p.status[kStatusBadIndex], static_cast<int>(v) + 1);
                    else
                        sl[i] = static_cast<int>(v);
                }
            }
        };
        int next[4];
        int ring_at = 0, unit = 0, nseg = 0;
        uint32_t ring_parity = 1;          // of the slot's previous use
        bool waited = !p.early;
        bool have = next_segment<KT>(walk, p, seg);
        if (have) slots_of(seg, seg.t0, next);
        int t = have ? seg.t0 : 0;
        while (have && !failed) {
            __syncwarp();
#pragma unroll
            for (int i = 0; i < 4; ++i) s_slot[i * 32 + lane] = next[i];
            __syncwarp();
            // the group's tiles are [t, t_end); what comes behind them is looked up meanwhile
            const int t_end = min(t + group_tiles, seg.t1);
            const Segment cur = seg;
            if (t_end < seg.t1) {
                slots_of(seg, t_end, next);
            } else {
                have = next_segment<KT>(walk, p, seg);
                if (have) slots_of(seg, seg.t0, next);
            }
            const bool lead = elect_one();
            for (int tt = t; tt < t_end && !failed; ++tt) {
                if (!waited && (tt + 1) * KT >= cur.len) {   // this tile holds the newest key
                    pdl_wait_prior();
                    waited = true;
                }
                bool ok = true;
                if (lead) {
                    for (int u = 0; u < p.nb && ok; ++u, ++unit) {
                        if (unit >= p.ring &&
                            !mbar_wait_bounded(smem_u32(&unit_empty[ring_at]), ring_parity, p.status, 601)) {
                            ok = false;
                            break;
                        }
                        const uint32_t bar = smem_u32(&unit_full[ring_at]);
                        const uint32_t dst = smem_base + static_cast<uint32_t>(ring_at) * kUnitBytes;
                        mbar_arrive_expect_tx(bar, kUnitBytes);
                        if (whole_unit) {
                            tma_load_3d(dst, &tmap_c, 0, s_slot[tt - t], 2 * u, bar);
                        } else {
                            for (int c = 0; c < copies; ++c) {
                                const int sl = s_slot[(tt - t) * copies + c];
                                const uint32_t to = dst + static_cast<uint32_t>(c * p.kpc) * 128u;
                                tma_load_3d(to, &tmap_c, 0, sl, 2 * u, bar);
                                tma_load_3d(to + kAtomBytes, &tmap_c, 0, sl, 2 * u + 1, bar);
                            }
                        }
                        if (++ring_at == p.ring) {
                            ring_at = 0;
                            ring_parity ^= 1u;
                        }
                    }
                }
                if (tt == cur.t0) {
                    // the queries of this item, behind the first tile's latents
                    __syncwarp();
                    if (!waited) {
                        pdl_wait_prior();
                        waited = true;
                    }
                    if (lead && ok) {
                        if (nseg > 0 && !mbar_wait_bounded(smem_u32(&q_empty), static_cast<uint32_t>(nseg - 1) & 1u, p.status, 602)) {
                            ok = false;
                        } else {
                            const uint32_t bar = smem_u32(&q_full);
                            mbar_arrive_expect_tx(bar, static_cast<uint32_t>(N) * p.width * 2u);
                            for (int a = 0; a < p.width / 64; ++a)
                                tma_load_2d(q_base + static_cast<uint32_t>(a) * N * 128u, &tmap_q, a * 64,
                                            cur.row * p.heads + cur.block * p.per_block, bar);
                        }
                    }
                    ++nseg;
                }
                failed = !__all_sync(0xffffffffu, ok);
            }
            t = t_end < cur.t1 ? t_end : seg.t0;
        }
        if (!waited) pdl_wait_prior();
    } else if (warp == 1) {
        // ================= S^T = C Q^T =================
        pdl_wait_prior();
        if (elect_one()) {
            const uint32_t idesc = idesc_bf16(KT, N);
            int slot = 0, tiles = 0, nseg = 0;
            uint32_t parity = 0;
            while (!failed && next_segment<KT>(walk, p, seg)) {
                if (!mbar_wait_bounded(smem_u32(&q_full), static_cast<uint32_t>(nseg) & 1u, p.status, 603)) break;
                for (int t = seg.t0; t < seg.t1 && !failed; ++t, ++tiles) {
                    const int buf = tiles & 1;
                    if (tiles >= 2 && !mbar_wait_bounded(smem_u32(&s_empty[buf]), static_cast<uint32_t>((tiles >> 1) - 1) & 1u,
                                                         p.status, 604)) {
                        failed = true;
                        break;
                    }
                    const uint32_t d = tmem_base + kColS + static_cast<uint32_t>(buf) * 64u;
                    uint64_t b = kmajor_sw128_desc(q_base);
                    for (int u = 0; u < p.nb; ++u) {
                        if (!mbar_wait_bounded(smem_u32(&unit_full[slot]), parity, p.status, 605)) {
                            failed = true;
                            break;
                        }
                        tc_fence_after();
                        const uint64_t a = kmajor_sw128_desc(smem_base + static_cast<uint32_t>(slot) * kUnitBytes);
#pragma unroll
                        for (int ks = 0; ks < 8; ++ks)
                            tc_mma_bf16(d, a + ((ks >> 2) * kAtomBytes + (ks & 3) * 32) / 16,
                                        b + ((ks >> 2) * N * 128 + (ks & 3) * 32) / 16, idesc, (u > 0 || ks > 0) ? 1u : 0u);
                        b += 2 * N * 128 / 16;
                        if (u >= p.no) tc_commit(smem_u32(&unit_empty[slot]));   // nobody else reads it
                        if (++slot == p.ring) {
                            slot = 0;
                            parity ^= 1u;
                        }
                    }
                    if (failed) break;
                    tc_commit(smem_u32(&s_full[buf]));
                }
                tc_commit(smem_u32(&q_empty));
                ++nseg;
            }
        }
    } else if (warp == 6) {
        // ================= O^T += C^T P^T =================
        pdl_wait_prior();
        if (elect_one()) {
            // A is MN-major; B is too where the heads of a key are contiguous
            const uint32_t idesc = idesc_bf16_m128(N) | (1u << 15) | (kHeadsContiguous ? 1u << 16 : 0u);
            int slot = 0, tiles = 0, nseg = 0;
            while (!failed && next_segment<KT>(walk, p, seg)) {
                for (int t = seg.t0; t < seg.t1; ++t, ++tiles) {
                    if (!mbar_wait_bounded(smem_u32(&p_full[tiles & 1]), static_cast<uint32_t>(tiles >> 1) & 1u, p.status, 606) ||
                        (t == seg.t0 && nseg > 0 &&
                         !mbar_wait_bounded(smem_u32(&o_free), static_cast<uint32_t>(nseg - 1) & 1u, p.status, 610))) {
                        failed = true;
                        break;
                    }
                    tc_fence_after();
                    const uint32_t pb = p_base + (p.p_bufs == 2 ? static_cast<uint32_t>(tiles & 1) * kPBytes : 0u);
                    const uint64_t b = kHeadsContiguous ? mnmajor_desc<KT>(pb) : kmajor_sw128_desc(pb);
                    uint32_t d = tmem_base + kColO;
                    for (int u = 0; u < p.no; ++u, d += N) {
                        const uint64_t a = mnmajor_desc<KT>(smem_base + static_cast<uint32_t>(slot) * kUnitBytes);
#pragma unroll
                        for (int ks = 0; ks < KT / 16; ++ks)
                            tc_mma_bf16(d, a + ks * 2048 / 16,
                                        b + (kHeadsContiguous ? ks * 2048 : (ks >> 2) * N * 128 + (ks & 3) * 32) / 16, idesc,
                                        (t > seg.t0 || ks > 0) ? 1u : 0u);
                        tc_commit(smem_u32(&unit_empty[slot]));
                        if (++slot == p.ring) slot = 0;
                    }
                    slot += p.nb - p.no;
                    if (slot >= p.ring) slot -= p.ring;
                    tc_commit(smem_u32(&pv_done[tiles & 1]));
                }
                ++nseg;
            }
        }
    } else {
        // ================= softmax and output =================
        const int q = warp & 3;                 // TMEM lane quarter this warp may read
        const int elem = q * 32 + lane;         // latent element inside a unit = TMEM lane of O^T
        // key inside the tile: a 64-row product sits in the first 16 lanes of every quarter
        const int key = KT == 128 ? elem : q * 16 + (lane & 15);
        const bool has_key = KT == 128 || lane < 16;
        const int st = static_cast<int>(threadIdx.x) - 64;   // 0..127
        const uint32_t lane_addr = tmem_base + (static_cast<uint32_t>(q * 32) << 16);
        const uint32_t p_key = p_base + static_cast<uint32_t>(key >> 6) * N * 128u + static_cast<uint32_t>(key & 7) * 2u;
        const uint32_t p_chunk = static_cast<uint32_t>((key & 63) >> 3);
        float* stage = reinterpret_cast<float*>(smem_raw + stage_off);
        int tiles = 0;
        float l[N];
        pdl_wait_prior();
        while (!failed && next_segment<KT>(walk, p, seg)) {
#pragma unroll
            for (int h = 0; h < N; ++h) l[h] = 0.f;
            if (st < N) s_ref[st] = -INFINITY;
            softmax_sync();
            for (int t = seg.t0; t < seg.t1; ++t, ++tiles) {
                const int buf = tiles & 1;
                if (!mbar_wait_bounded(smem_u32(&s_full[buf]), static_cast<uint32_t>(tiles >> 1) & 1u, p.status, 607)) failed = true;
                tc_fence_after();
                const uint32_t s_addr = lane_addr + kColS + static_cast<uint32_t>(buf) * 64u;
                const uint32_t p_buf = p.p_bufs == 2 ? static_cast<uint32_t>(buf) * kPBytes : 0u;
                const bool valid = has_key && t * KT + key < seg.len;
                // does any score outgrow its head's reference?
                bool over = false;
#pragma unroll
                for (int c = 0; c < N / 16; ++c) {
                    uint32_t sv[16];
                    tmem_ld_32x32b_x16(s_addr + c * 16, sv);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 16; j += 4) {
                        const float4 ref = *reinterpret_cast<const float4*>(&s_ref[c * 16 + j]);
                        over |= __uint_as_float(sv[j]) * p.scale_log2 > ref.x + kLazyLog2;
                        over |= __uint_as_float(sv[j + 1]) * p.scale_log2 > ref.y + kLazyLog2;
                        over |= __uint_as_float(sv[j + 2]) * p.scale_log2 > ref.z + kLazyLog2;
                        over |= __uint_as_float(sv[j + 3]) * p.scale_log2 > ref.w + kLazyLog2;
                    }
                }
                // the product that last read this buffer of P is done
                const int read_by = tiles - p.p_bufs;
                if (t - seg.t0 >= p.p_bufs && !failed &&
                    !mbar_wait_bounded(smem_u32(&pv_done[read_by & 1]), static_cast<uint32_t>(read_by >> 1) & 1u, p.status, 608))
                    failed = true;
                // a wait that ran out in one warp ends all four at the same place (two flags in turn: a
                // warp may be one tile behind the one that sets the next)
                if (failed) s_failed[tiles & 1] = 1;
                const bool moved = softmax_any(over && valid);
                if (s_failed[tiles & 1] != 0) {
                    failed = true;
                    break;
                }
                tc_fence_after();
                if (moved) {
#pragma unroll
                    for (int c = 0; c < N / 16; ++c) {
                        uint32_t sv[16];
                        tmem_ld_32x32b_x16(s_addr + c * 16, sv);
                        tmem_ld_wait();
#pragma unroll
                        for (int j = 0; j < 16; ++j) {
                            const float mx = warp_max(valid ? __uint_as_float(sv[j]) * p.scale_log2 : -INFINITY);
                            if (lane == 0) s_warp[q][c * 16 + j] = mx;
                        }
                    }
                    softmax_sync();
                    if (st < N) {
                        const float old = s_ref[st];
                        const float mx = fmaxf(fmaxf(fmaxf(s_warp[0][st], s_warp[1][st]), fmaxf(s_warp[2][st], s_warp[3][st])), old);
                        s_alpha[st] = old == -INFINITY ? 1.f : ex2(old - mx);
                        s_ref[st] = mx;
                    }
                    softmax_sync();
                    if (t > seg.t0) {
                        // every product so far has added to O
                        if (!mbar_wait_bounded(smem_u32(&pv_done[(tiles - 1) & 1]), static_cast<uint32_t>((tiles - 1) >> 1) & 1u,
                                               p.status, 611))
                            failed = true;
                        tc_fence_after();
#pragma unroll
                        for (int h = 0; h < N; ++h) l[h] *= s_alpha[h];
                        for (int u = 0; u < p.no; ++u)
#pragma unroll
                            for (int c = 0; c < N / 16; ++c) {
                                const uint32_t o_addr = lane_addr + kColO + static_cast<uint32_t>(u * N + c * 16);
                                uint32_t ov[16];
                                tmem_ld_32x32b_x16(o_addr, ov);
                                tmem_ld_wait();
#pragma unroll
                                for (int j = 0; j < 16; ++j)
                                    ov[j] = __float_as_uint(__uint_as_float(ov[j]) * s_alpha[c * 16 + j]);
                                tmem_st_32x32b_x16(o_addr, ov);
                            }
                        tmem_st_wait();
                    }
                }
#pragma unroll
                for (int c = 0; c < N / 16; ++c) {
                    uint32_t sv[16];
                    tmem_ld_32x32b_x16(s_addr + c * 16, sv);
                    tmem_ld_wait();
                    float w[16];
#pragma unroll
                    for (int j = 0; j < 16; j += 4) {
                        const float4 ref = *reinterpret_cast<const float4*>(&s_ref[c * 16 + j]);
                        w[j] = ex2(fmaf(__uint_as_float(sv[j]), p.scale_log2, -ref.x));
                        w[j + 1] = ex2(fmaf(__uint_as_float(sv[j + 1]), p.scale_log2, -ref.y));
                        w[j + 2] = ex2(fmaf(__uint_as_float(sv[j + 2]), p.scale_log2, -ref.z));
                        w[j + 3] = ex2(fmaf(__uint_as_float(sv[j + 3]), p.scale_log2, -ref.w));
                    }
                    if (!valid) {
#pragma unroll
                        for (int j = 0; j < 16; ++j) w[j] = 0.f;
                    }
#pragma unroll
                    for (int j = 0; j < 16; ++j) l[c * 16 + j] += w[j];
                    if (has_key) {
                        if (kHeadsContiguous) {
#pragma unroll
                            for (int j = 0; j < 16; j += 8) {
                                const uint32_t addr = swz128(p_base + p_buf + static_cast<uint32_t>(key) * 128u, c * 2 + j / 8);
                                asm volatile("st.shared.v4.b32 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(pack_bf16(w[j], w[j + 1])),
                                             "r"(pack_bf16(w[j + 2], w[j + 3])), "r"(pack_bf16(w[j + 4], w[j + 5])),
                                             "r"(pack_bf16(w[j + 6], w[j + 7]))
                                             : "memory");
                            }
                        } else {
#pragma unroll
                            for (int j = 0; j < 16; ++j) {
                                const int h = c * 16 + j;
                                const __nv_bfloat16 b = __float2bfloat16_rn(w[j]);
                                const uint32_t addr = p_key + p_buf + static_cast<uint32_t>(h) * 128u + ((p_chunk ^ (h & 7)) << 4);
                                asm volatile("st.shared.b16 [%0], %1;" ::"r"(addr), "h"(*reinterpret_cast<const uint16_t*>(&b))
                                             : "memory");
                            }
                        }
                    }
                    __syncwarp();
                }
                fence_proxy_async_smem();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) {
                    mbar_arrive(smem_u32(&s_empty[buf]));
                    mbar_arrive(smem_u32(&p_full[buf]));
                }
            }
            if (failed) break;
            if (!mbar_wait_bounded(smem_u32(&pv_done[(tiles - 1) & 1]), static_cast<uint32_t>((tiles - 1) >> 1) & 1u, p.status, 609)) failed = true;
            tc_fence_after();
            {
                const int col = warp_transpose_sum<N>(l);
                constexpr int kCols = N >= 32 ? N / 32 : 1;
#pragma unroll
                for (int j = 0; j < kCols; ++j) s_warp[q][col + j] = l[j];
            }
            if (softmax_any(failed)) {
                failed = true;
                break;
            }
            const int item = seg.row * p.blocks + seg.block;
            const int cut = seg.starts ? 1 : 0;      // partial slot: 1 = goes on in the next CTA, 0 = came from the one before
            const bool whole = seg.starts && seg.ends;
            const int64_t slot = static_cast<int64_t>(blockIdx.x) * 2 + cut;
            if (st < N) {
                const float tot = s_warp[0][st] + s_warp[1][st] + s_warp[2][st] + s_warp[3][st];
                s_alpha[st] = whole ? 1.f / tot : 1.f;
                if (!whole) {
                    p.part_m[slot * N + st] = s_ref[st];
                    p.part_l[slot * N + st] = tot;
                }
            }
            if (st == 0 && seg.starts) {
                // the CTAs that share this item follow from its first tile's place in the sequence
                const int nt = (seg.len + KT - 1) / KT;
                const int first = g0 + tiles - (seg.t1 - seg.t0);
                p.item_cta[2 * item] = static_cast<int>(blockIdx.x);
                p.item_cta[2 * item + 1] = (first + nt - 1) / run;
            }
            softmax_sync();
            const int h0 = seg.block * p.per_block;
            const int nh = min(p.per_block, p.heads - h0);
            for (int u = 0; u < p.no; ++u) {
#pragma unroll
                for (int c = 0; c < N / 16; ++c) {
                    if (c * 16 >= nh) break;
                    uint32_t ov[16];
                    tmem_ld_32x32b_x16(lane_addr + kColO + static_cast<uint32_t>(u * N + c * 16), ov);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 16; ++j) stage[j * kUnitElems + elem] = __uint_as_float(ov[j]) * s_alpha[c * 16 + j];
                    softmax_sync();
                    // 16 heads x 128 elements, whole rows of a head at a time
                    if (whole) {
#pragma unroll
                        for (int i = st; i < 16 * kUnitElems / 8; i += 128) {
                            const int h = c * 16 + i / (kUnitElems / 8), e = i % (kUnitElems / 8) * 8;
                            if (h < nh) {
                                const float* v = stage + (i / (kUnitElems / 8)) * kUnitElems + e;
                                const float4 a = *reinterpret_cast<const float4*>(v), b = *reinterpret_cast<const float4*>(v + 4);
                                *reinterpret_cast<uint4*>(p.out + (static_cast<int64_t>(seg.row) * p.heads + h0 + h) * p.out_width +
                                                          u * kUnitElems + e) =
                                    make_uint4(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w), pack_bf16(b.x, b.y), pack_bf16(b.z, b.w));
                            }
                        }
                    } else {
#pragma unroll
                        for (int i = st; i < 16 * kUnitElems / 4; i += 128) {
                            const int h = c * 16 + i / (kUnitElems / 4), e = i % (kUnitElems / 4) * 4;
                            if (h < nh)
                                *reinterpret_cast<float4*>(p.part_o + (slot * N + h) * p.out_width + u * kUnitElems + e) =
                                    *reinterpret_cast<const float4*>(stage + (i / (kUnitElems / 4)) * kUnitElems + e);
                        }
                    }
                    softmax_sync();
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(smem_u32(&o_free));
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base, 512);
}

// One CTA per (item, head): weighs the partials of an item that was cut over several CTAs.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const LatentParams p, int N) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int row = blockIdx.x / p.heads, head = blockIdx.x - row * p.heads;
    const int block = head / p.per_block, h = head - block * p.per_block;
    const int item = row * p.blocks + block;
    __nv_bfloat16* out = p.out + (static_cast<int64_t>(row) * p.heads + head) * p.out_width;
    if (p.row_len[row] <= 0) {   // no keys: zeros
        for (int i = threadIdx.x; i < p.out_width; i += blockDim.x) out[i] = __float2bfloat16_rn(0.f);
        return;
    }
    const int c0 = p.item_cta[2 * item], c1 = p.item_cta[2 * item + 1];
    if (c0 == c1) return;   // written whole
    auto slot_of = [&](int c) { return (static_cast<int64_t>(c) * 2 + (c == c0 ? 1 : 0)) * N + h; };
    float mx = -INFINITY;
    for (int c = c0; c <= c1; ++c) mx = fmaxf(mx, p.part_m[slot_of(c)]);
    float tot = 0.f;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    const int e = static_cast<int>(threadIdx.x) * 4;
#pragma unroll 4
    for (int c = c0; c <= c1; ++c) {
        const int64_t s = slot_of(c);
        const float f = ex2(p.part_m[s] - mx);
        tot += f * p.part_l[s];
        if (e < p.out_width) {
            const float4 v = *reinterpret_cast<const float4*>(p.part_o + s * p.out_width + e);
            acc.x += f * v.x;
            acc.y += f * v.y;
            acc.z += f * v.z;
            acc.w += f * v.w;
        }
    }
    const float inv = tot > 0.f ? 1.f / tot : 0.f;
    if (e < p.out_width)
        *reinterpret_cast<uint2*>(out + e) = make_uint2(pack_bf16(acc.x * inv, acc.y * inv), pack_bf16(acc.z * inv, acc.w * inv));
}

// The pool as [width / 64][num_slots][64], copied kpc slots and `halves` 64-element columns at a time.
int make_latent_tmap(CUtensorMap* out, const void* cache, int width, int64_t num_slots, int kpc, int halves) {
    EncodeTiledFn fn = encode_tiled_fn();
    if (!fn) {
        set_last_error("cuTensorMapEncodeTiled is not available from this driver");
        return B200_ERR_CUDA;
    }
    const cuuint64_t dims[3] = {64, static_cast<cuuint64_t>(num_slots), static_cast<cuuint64_t>(width / 64)};
    const cuuint64_t strides[2] = {static_cast<cuuint64_t>(width) * 2, 128};
    const cuuint32_t box[3] = {64, static_cast<cuuint32_t>(kpc), static_cast<cuuint32_t>(halves)};
    const cuuint32_t es[3] = {1, 1, 1};
    CUresult r = fn(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(cache), dims, strides, box, es,
                    CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                    CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        set_last_error("cuTensorMapEncodeTiled (latent pool) failed with CUresult %d", static_cast<int>(r));
        return B200_ERR_CUDA;
    }
    return B200_OK;
}

struct Shape {
    int n, blocks, per_block;
};
Shape shape_of(int heads) {
    Shape s;
    s.blocks = div_ceil(heads, 64);
    s.per_block = div_ceil(heads, s.blocks);
    s.n = s.per_block <= 16 ? 16 : s.per_block <= 32 ? 32 : 64;
    return s;
}

int64_t align256(int64_t x) { return (x + 255) / 256 * 256; }

}  // namespace

int64_t latent_attention_workspace_bytes(int rows, int heads, int width) {
    const Shape s = shape_of(heads);
    const int64_t slots = 2ll * 160;   // two per CTA, at most one CTA per SM (148)
    return align256(slots * s.n * width * 4) + 2 * align256(slots * s.n * 4) + align256(static_cast<int64_t>(rows) * s.blocks * 8);
}

bool latent_attention_tc_supported(const LatentAttention& a) {
    const int out_width = a.out_width > 0 ? a.out_width : a.width;
    return a.width % kUnitElems == 0 && a.width <= kMaxWidth && out_width % kUnitElems == 0 && out_width <= kMaxOutWidth && a.scale > 0.f && sm_count() <= 160 &&
           (reinterpret_cast<uintptr_t>(a.cache) & 15u) == 0 && (reinterpret_cast<uintptr_t>(a.q) & 15u) == 0;
}

int launch_latent_attention_tc(const LatentAttention& a, int* status, cudaStream_t stream) {
    if (a.rows == 0) return B200_OK;
    const Shape sh = shape_of(a.heads);
    const int grid = sm_count();
    LatentParams p;
    p.out = static_cast<__nv_bfloat16*>(a.out);
    uint8_t* ws = static_cast<uint8_t*>(a.workspace);
    const int64_t slots = 2ll * 160;
    p.part_o = reinterpret_cast<float*>(ws);
    ws += align256(slots * sh.n * a.width * 4);
    p.part_m = reinterpret_cast<float*>(ws);
    ws += align256(slots * sh.n * 4);
    p.part_l = reinterpret_cast<float*>(ws);
    ws += align256(slots * sh.n * 4);
    p.item_cta = reinterpret_cast<int32_t*>(ws);
    p.page_table = a.page_table;
    p.pt_stride = a.pt_stride;
    p.row_table = a.row_table;
    p.row_len = a.row_len;
    p.rows = a.rows;
    p.heads = a.heads;
    p.width = a.width;
    p.out_width = a.out_width > 0 ? a.out_width : a.width;
    p.blocks = sh.blocks;
    p.per_block = sh.per_block;
    p.nb = a.width / kUnitElems;
    p.no = p.out_width / kUnitElems;
    const int kt = a.width > 256 ? 64 : 128;
    p.kpc = a.page_size < kt ? a.page_size : kt;
    p.num_slots = a.num_slots;
    p.scale_log2 = a.scale * 1.4426950408889634f;
    p.early = a.only_last_key_new && pdl_launches_enabled() ? 1 : 0;
    p.status = status;
    const uint32_t unit_bytes = static_cast<uint32_t>(kt) * 256u;
    const uint32_t p_bytes = kt / 64 * sh.n * 128u;
    const uint32_t fixed = static_cast<uint32_t>(sh.n) * a.width * 2u + p_bytes + 16u * kUnitElems * 4u + 1024u;
    constexpr uint32_t kBudget = 224u * 1024u;
    int ring = kMaxUnits;
    while (ring > p.nb && static_cast<uint32_t>(ring) * unit_bytes + fixed > kBudget) --ring;
    p.ring = ring;
    uint32_t smem = static_cast<uint32_t>(ring) * unit_bytes + fixed;
    p.p_bufs = smem + p_bytes <= kBudget ? 2 : 1;
    if (p.p_bufs == 2) smem += p_bytes;

    CUtensorMap tc, tq;
    int err = make_latent_tmap(&tc, a.cache, a.width, a.num_slots, p.kpc, p.kpc == kt ? 2 : 1);
    if (err != B200_OK) return err;
    err = cached_tmap(&tq, a.q, static_cast<uint64_t>(a.width), static_cast<uint64_t>(a.rows) * a.heads,
                      static_cast<uint64_t>(a.width) * 2, 64, static_cast<uint32_t>(sh.n));
    if (err != B200_OK) return err;
    auto kernel = kt == 64 ? (sh.n == 16   ? latent_attention_tc_kernel<16, 64>
                              : sh.n == 32 ? latent_attention_tc_kernel<32, 64>
                                           : latent_attention_tc_kernel<64, 64>)
                           : (sh.n == 16   ? latent_attention_tc_kernel<16, 128>
                              : sh.n == 32 ? latent_attention_tc_kernel<32, 128>
                                           : latent_attention_tc_kernel<64, 128>);
    B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(grid), dim3(kThreads), smem, stream, dim3(1, 1, 1), tc, tq, p));
    B200_CHECK_CUDA(launch_kernel(latent_merge_kernel, dim3(a.rows * a.heads), dim3(128), 0, stream, dim3(1, 1, 1), p, sh.n));
    return B200_OK;
}

}  // namespace b200
