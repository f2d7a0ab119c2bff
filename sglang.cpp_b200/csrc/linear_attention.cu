// Gated linear attention: a matrix state per request and head whose rows (key channels) decay one by one,
//     S <- diag(alpha_t) S + k_t v_t^T,   o_t = S^T q_t,   log alpha_t = log sigmoid(z_t) / tau,
// z from a low-rank projection that is finished here, in fp32.  The state is fp32 and lives in a slot per
// page-table row.  Three kernels:
//
//   * decode: one CTA per (request, head) streams the state once - read, decayed, updated, read out, written -
//     and applies the head's norm and the output gate.  The first reads run ahead of griddepcontrol.wait: only
//     the projections come from the kernel before.
//   * chunked (bf16 prefill): one CTA per (request, head, 64 value columns) walks the request's tokens in
//     segments of up to 64.  With b_t the decay logarithms summed up inside a segment and r a reference per
//     channel half way between the first and the last of them,
//         q~_t = q_t exp(b_t - r),   k~_s = k_s exp(r - b_s)
//         o_t  = sum_{s <= t} (q~_t . k~_s) v_s + q~_t . (exp(r) S)
//         S   <- exp(b_n) S + exp(b_n - r) sum_s k~_s v_s^T
//     are matrix products.  A segment ends where some channel has decayed by 2^-80 since its first token, so that
//     neither factor leaves the range of a float, however steep the decay is (a single token always fits).
//     Everything derived from decays or the state enters the products as the sum of two bf16 numbers.
//   * plain: token after token in fp32, for fp32 models and sizes the chunked kernel does not take.
//
// The last two leave the heads' raw outputs to a kernel that applies norm and gate.
#include "common.cuh"
#include "kernels.h"

namespace b200 {
namespace {

template <typename T>
__device__ __forceinline__ float to_f32(T x) { return static_cast<float>(x); }
template <>
__device__ __forceinline__ float to_f32(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T>
__device__ __forceinline__ T from_f32(float x) { return static_cast<T>(x); }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32(float x) { return __float2bfloat16_rn(x); }
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf16_lo(u.x), bf16_hi(u.x), bf16_lo(u.y), bf16_hi(u.y));
}
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }

// Where the parts of a row of the joint projection start.
struct Parts {
    int64_t k, v, gate, low;
};
__device__ __forceinline__ Parts parts_of(const LinearAttention& a) {
    Parts p;
    p.k = static_cast<int64_t>(a.heads) * a.padded_dim;
    p.v = 2 * p.k;
    p.gate = p.v + static_cast<int64_t>(a.heads) * a.padded_value_dim;
    p.low = p.gate + static_cast<int64_t>(a.heads) * a.padded_value_dim;
    return p;
}

// log sigmoid(z) / tau of channel `c` (of heads * padded_dim) for the low-rank row `low`.
template <typename T>
__device__ __forceinline__ float log_decay(const LinearAttention& a, const T* low, int64_t c) {
    const T* up = static_cast<const T*>(a.up) + c * a.up_ld;
    float z = a.bias[c];
    for (int r = 0; r < a.rank; r += 8) {   // both sides are zero from rank on
        const Vec8 x = load8(low + r), y = load8(up + r);
#pragma unroll
        for (int j = 0; j < 8; ++j) z = fmaf(x.v[j], y.v[j], z);
    }
    return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) / a.tau;
}

// ---- decode ---------------------------------------------------------------------

constexpr int kDecodeThreads = 256;
constexpr int kAhead = 16;   // state rows per thread in flight

template <typename T>
__global__ void __launch_bounds__(kDecodeThreads)
linear_attention_decode_kernel(const LinearAttention a) {
    extern __shared__ float smem[];
    __shared__ float s_red[kDecodeThreads / 32];
    const int dk = a.padded_dim, vp = a.padded_value_dim;
    float *s_q = smem, *s_k = s_q + dk, *s_alpha = s_k + dk, *s_o = s_alpha + dk;   // s_o [groups][vp]
    const int h = blockIdx.x, b = blockIdx.y;
    const int nv4 = vp >> 2;                         // float4 columns
    const int groups = kDecodeThreads / nv4;         // state rows handled at a time
    const int group = threadIdx.x / nv4, col = (threadIdx.x - group * nv4) * 4;
    const bool active = group < groups;
    float* state = a.state + ((static_cast<int64_t>(a.table_idx[b]) * a.heads + h) * dk) * vp + col;
    const bool fresh = a.cached[b] == 0;
    pdl_launch_dependents();
    float4 s[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
        const int r = group + i * groups;
        s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (active && !fresh && r < dk) s[i] = load4(state + static_cast<int64_t>(r) * vp);
    }
    pdl_wait_prior();
    const Parts at = parts_of(a);
    const T* row = static_cast<const T*>(a.joint) + b * a.joint_ld;
    for (int c = threadIdx.x; c < dk; c += kDecodeThreads) {
        s_q[c] = to_f32(row[static_cast<int64_t>(h) * dk + c]) * a.q_scale;
        s_k[c] = to_f32(row[at.k + static_cast<int64_t>(h) * dk + c]);
        s_alpha[c] = expf(log_decay(a, row + at.low, static_cast<int64_t>(h) * dk + c));
    }
    __syncthreads();
    if (active) {
        const float4 v = load4(row + at.v + static_cast<int64_t>(h) * vp + col);
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
        auto step = [&](int r, float4 x) {
            const float al = s_alpha[r], k = s_k[r], q = s_q[r];
            x.x = al * x.x + k * v.x;
            x.y = al * x.y + k * v.y;
            x.z = al * x.z + k * v.z;
            x.w = al * x.w + k * v.w;
            o.x += q * x.x;
            o.y += q * x.y;
            o.z += q * x.z;
            o.w += q * x.w;
            *reinterpret_cast<float4*>(state + static_cast<int64_t>(r) * vp) = x;
        };
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const int r = group + i * groups;
            if (r < dk) step(r, s[i]);
        }
        for (int r = group + kAhead * groups; r < dk; r += groups)
            step(r, fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(state + static_cast<int64_t>(r) * vp));
        *reinterpret_cast<float4*>(s_o + group * vp + col) = o;
    }
    __syncthreads();
    // the head's output: sum over the row groups, norm, gate
    float ss = 0.f;
    for (int c = threadIdx.x; c < vp; c += kDecodeThreads) {
        float o = s_o[c];
        for (int g = 1; g < groups; ++g) o += s_o[g * vp + c];
        s_o[c] = o;
        ss += o * o;
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    ss = warp_sum(ss);
    if (lane == 0) s_red[warp] = ss;
    __syncthreads();
    ss = warp_sum(lane < kDecodeThreads / 32 ? s_red[lane] : 0.f);
    const float scale = rsqrtf(ss / static_cast<float>(a.value_dim) + a.eps);
    T* out = static_cast<T*>(a.out) + (static_cast<int64_t>(b) * a.heads + h) * vp;
    for (int c = threadIdx.x; c < vp; c += kDecodeThreads) {
        const float g = to_f32(row[at.gate + static_cast<int64_t>(h) * vp + c]);
        out[c] = from_f32<T>(s_o[c] * scale * to_f32(static_cast<const T*>(a.norm)[c]) * silu(g));
    }
}

// ---- plain ----------------------------------------------------------------------

constexpr int kPlainThreads = 128;
constexpr int kPlainCols = 32;

template <typename T>
__global__ void __launch_bounds__(kPlainThreads)
linear_attention_plain_kernel(const LinearAttention a) {
    extern __shared__ float smem[];
    __shared__ float s_part[kPlainThreads / 32][kPlainCols];
    const int dk = a.padded_dim, vp = a.padded_value_dim;
    float *s_q = smem, *s_k = s_q + dk, *s_alpha = s_k + dk, *s_state = s_alpha + dk;   // s_state [dk][kPlainCols]
    const int h = blockIdx.y, b = blockIdx.z, v0 = blockIdx.x * kPlainCols;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    pdl_launch_dependents();
    pdl_wait_prior();
    const int begin = a.qo_indptr[b], end = a.qo_indptr[b + 1];
    if (begin >= end) return;
    const Parts at = parts_of(a);
    float* state = a.state + ((static_cast<int64_t>(a.table_idx[b]) * a.heads + h) * dk) * vp + v0;
    const bool fresh = a.cached[b] == 0;
    for (int r = warp; r < dk; r += kPlainThreads / 32)
        s_state[r * kPlainCols + lane] = fresh ? 0.f : state[static_cast<int64_t>(r) * vp + lane];
    for (int t = begin; t < end; ++t) {
        const T* row = static_cast<const T*>(a.joint) + t * a.joint_ld;
        for (int c = threadIdx.x; c < dk; c += kPlainThreads) {
            s_q[c] = to_f32(row[static_cast<int64_t>(h) * dk + c]) * a.q_scale;
            s_k[c] = to_f32(row[at.k + static_cast<int64_t>(h) * dk + c]);
            s_alpha[c] = expf(log_decay(a, row + at.low, static_cast<int64_t>(h) * dk + c));
        }
        const float v = to_f32(row[at.v + static_cast<int64_t>(h) * vp + v0 + lane]);
        __syncthreads();
        float o = 0.f;
        for (int r = warp; r < dk; r += kPlainThreads / 32) {
            const float s = s_alpha[r] * s_state[r * kPlainCols + lane] + s_k[r] * v;
            s_state[r * kPlainCols + lane] = s;
            o += s_q[r] * s;
        }
        s_part[warp][lane] = o;
        __syncthreads();
        if (warp == 0) {
            o = s_part[0][lane];
#pragma unroll
            for (int w = 1; w < kPlainThreads / 32; ++w) o += s_part[w][lane];
            static_cast<T*>(a.out)[(static_cast<int64_t>(t) * a.heads + h) * vp + v0 + lane] = from_f32<T>(o);
        }
    }
    for (int r = warp; r < dk; r += kPlainThreads / 32)
        state[static_cast<int64_t>(r) * vp + lane] = s_state[r * kPlainCols + lane];
}

// Norm and gate of the raw head outputs, in place; one warp per (token, head).
constexpr int kFinishWarps = 8;

template <typename T>
__global__ void __launch_bounds__(kFinishWarps * 32)
linear_attention_finish_kernel(const LinearAttention a) {
    const int lane = threadIdx.x & 31, vp = a.padded_value_dim;
    const int64_t row = static_cast<int64_t>(blockIdx.x) * kFinishWarps + (threadIdx.x >> 5);
    pdl_launch_dependents();
    pdl_wait_prior();
    if (row >= static_cast<int64_t>(a.tokens) * a.heads) return;
    const int64_t t = row / a.heads;
    const int h = static_cast<int>(row - t * a.heads);
    T* out = static_cast<T*>(a.out) + row * vp;
    const T* gate = static_cast<const T*>(a.joint) + t * a.joint_ld + parts_of(a).gate + static_cast<int64_t>(h) * vp;
    const T* norm = static_cast<const T*>(a.norm);
    float ss = 0.f;
    for (int c = lane * 4; c < vp; c += 128) {
        const float4 o = load4(out + c);
        ss += o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;
    }
    const float scale = rsqrtf(warp_sum(ss) / static_cast<float>(a.value_dim) + a.eps);
    for (int c = lane * 4; c < vp; c += 128) {
        const float4 o = load4(out + c), g = load4(gate + c), w = load4(norm + c);
        out[c] = from_f32<T>(o.x * scale * w.x * silu(g.x));
        out[c + 1] = from_f32<T>(o.y * scale * w.y * silu(g.y));
        out[c + 2] = from_f32<T>(o.z * scale * w.z * silu(g.z));
        out[c + 3] = from_f32<T>(o.w * scale * w.w * silu(g.w));
    }
}

// ---- chunked ----------------------------------------------------------------------

constexpr int kChunk = 64;            // tokens per segment at most
constexpr int kSlice = 64;            // value columns per CTA
constexpr int kChunkThreads = 256;
constexpr float kRangeLog2 = 80.f;    // a channel may decay by 2^-80 inside a segment
constexpr int kMaxLow = 64;           // padded rank of the decay projection
constexpr int kPad = 8;               // bf16 elements behind every shared row (conflict-free ldmatrix)
constexpr float kLog2e = 1.4426950408889634f;

template <int DK>
struct ChunkSmem {
    static constexpr int kRow = DK + kPad, kVRow = kSlice + kPad, kLowRow = kMaxLow + kPad;
    __nv_bfloat16 q[kChunk * kRow], k[kChunk * kRow];                 // as loaded
    __nv_bfloat16 v[2][kChunk * kVRow];                               // this segment's and the next one's
    __nv_bfloat16 low[kChunk * kLowRow];
    __nv_bfloat16 qh[kChunk * kRow], ql[kChunk * kRow];               // q~ in two parts
    __nv_bfloat16 kh[kChunk * kRow], kl[kChunk * kRow];               // k~
    __nv_bfloat16 sh[DK * kVRow], sl[DK * kVRow];                     // exp(r) S
    float b[kChunk * (DK + 4)];                                       // decay logarithms (base 2), then their sums
    float part[kChunkThreads];                                        // sums of the pieces of a column of b
    int n;                                                            // tokens of this segment
};

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;   // 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// x as the sum of two bf16 numbers.
__device__ __forceinline__ void split2(float x0, float x1, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x0, x1);
    lo = pack_bf16(x0 - bf16_lo(hi), x1 - bf16_hi(hi));
}

template <int DK>
__global__ void __launch_bounds__(kChunkThreads, 1)
linear_attention_chunk_kernel(const LinearAttention a) {
    using Smem = ChunkSmem<DK>;
    constexpr int ROW = Smem::kRow, VROW = Smem::kVRow, LROW = Smem::kLowRow, BROW = DK + 4;
    constexpr int kParts = kChunkThreads / DK;          // threads per column of b
    constexpr int kPartLen = kChunk / kParts;
    constexpr int kColSplit = 128 / DK;                 // warps that share 16 state rows
    constexpr int kStateTiles = kSlice / 8 / kColSplit; // 8-column tiles of state per warp
    constexpr int kZTiles = DK / 64;                    // 8-channel tiles of z per warp
    extern __shared__ uint8_t smem_raw[];
    Smem& S = *reinterpret_cast<Smem*>(smem_raw);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, r8 = lane & 7;
    const int h = blockIdx.y, req = blockIdx.z, v0 = blockIdx.x * kSlice;
    const int vp = a.padded_value_dim;
    pdl_launch_dependents();
    pdl_wait_prior();
    const int begin = a.qo_indptr[req], ext = a.qo_indptr[req + 1] - begin;
    if (ext <= 0) return;
    const Parts at = parts_of(a);
    const __nv_bfloat16* joint = static_cast<const __nv_bfloat16*>(a.joint) + static_cast<int64_t>(begin) * a.joint_ld;
    const int low_vec = a.up_ld / 8;

    auto load_segment = [&](int s0, int buf) {
        const int n = min(kChunk, ext - s0);
        for (int i = threadIdx.x; i < kChunk * (DK / 8); i += kChunkThreads) {
            const int t = i / (DK / 8), c = (i % (DK / 8)) * 8;
            const __nv_bfloat16* row = joint + static_cast<int64_t>(t < n ? s0 + t : s0) * a.joint_ld + static_cast<int64_t>(h) * DK + c;
            cp_async16(smem_u32(&S.q[t * ROW + c]), row, t < n);
            cp_async16(smem_u32(&S.k[t * ROW + c]), row + at.k, t < n);
        }
        for (int i = threadIdx.x; i < kChunk * (kSlice / 8); i += kChunkThreads) {
            const int t = i / (kSlice / 8), c = (i % (kSlice / 8)) * 8;
            const __nv_bfloat16* row = joint + static_cast<int64_t>(t < n ? s0 + t : s0) * a.joint_ld;
            cp_async16(smem_u32(&S.v[buf][t * VROW + c]), row + at.v + static_cast<int64_t>(h) * vp + v0 + c, t < n);
        }
        for (int i = threadIdx.x; i < kChunk * low_vec; i += kChunkThreads) {
            const int t = i / low_vec, c = (i - t * low_vec) * 8;
            const __nv_bfloat16* row = joint + static_cast<int64_t>(t < n ? s0 + t : s0) * a.joint_ld;
            cp_async16(smem_u32(&S.low[t * LROW + c]), row + at.low + c, t < n);
        }
    };
    load_segment(0, 0);

    // This warp's part of the state: 16 channels from row0, kStateTiles tiles of 8 columns from col0; the layout is
    // that of an MMA accumulator (element 0, 1: row g; 2, 3: row g + 8; columns 2 tq, 2 tq + 1).
    const int row0 = warp / kColSplit * 16, col0 = warp % kColSplit * (kSlice / kColSplit);
    float* state = a.state + ((static_cast<int64_t>(a.table_idx[req]) * a.heads + h) * DK) * vp + v0;
    float st[kStateTiles][4];
    const bool fresh = a.cached[req] == 0;
#pragma unroll
    for (int j = 0; j < kStateTiles; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const float2 x = fresh ? make_float2(0.f, 0.f)
                                   : *reinterpret_cast<const float2*>(state + static_cast<int64_t>(row0 + g + half * 8) * vp +
                                                                      col0 + j * 8 + 2 * tq);
            st[j][2 * half] = x.x;
            st[j][2 * half + 1] = x.y;
        }

    const int zc0 = warp * (DK / 8);                  // this warp's channels of z
    const int bc = threadIdx.x % DK, bpart = threadIdx.x / DK;   // this thread's column and piece of b
    // 16 tokens x 32 columns of the output per warp; the two warps of a scheduler take an early and a late tile
    const int mt = warp < 4 ? warp : 7 - warp, oc0 = (warp >> 2) * 32;
    const float log2e_tau = kLog2e / a.tau;
    const __nv_bfloat16* up = static_cast<const __nv_bfloat16*>(a.up) + static_cast<int64_t>(h) * DK * a.up_ld;
    const float* bias = a.bias + static_cast<int64_t>(h) * DK;

    int buf = 0;
    for (int s0 = 0; s0 < ext;) {
        const int n_max = min(kChunk, ext - s0);
        cp_async_wait_all();
        if (threadIdx.x == 0) S.n = n_max;
        __syncthreads();
        // ---- z = low up^T + bias, and its decay logarithm ----
        {
            float z[4][kZTiles][4];
#pragma unroll
            for (int m = 0; m < 4; ++m)
#pragma unroll
                for (int j = 0; j < kZTiles; ++j) z[m][j][0] = z[m][j][1] = z[m][j][2] = z[m][j][3] = 0.f;
            for (int r = 0; r < a.up_ld; r += 16) {
                uint32_t bf[kZTiles][2];
#pragma unroll
                for (int j = 0; j < kZTiles; ++j) {
                    const __nv_bfloat16* u = up + static_cast<int64_t>(zc0 + j * 8 + g) * a.up_ld + r + 2 * tq;
                    bf[j][0] = *reinterpret_cast<const uint32_t*>(u);
                    bf[j][1] = *reinterpret_cast<const uint32_t*>(u + 8);
                }
#pragma unroll
                for (int m = 0; m < 4; ++m) {
                    uint32_t af[4];
                    ldmatrix_x4(smem_u32(&S.low[(m * 16 + (mi & 1) * 8 + r8) * LROW + r + (mi >> 1) * 8]), af[0], af[1], af[2], af[3]);
#pragma unroll
                    for (int j = 0; j < kZTiles; ++j) mma_bf16_16816(z[m][j], af, bf[j][0], bf[j][1]);
                }
            }
#pragma unroll
            for (int j = 0; j < kZTiles; ++j) {
                const int c = zc0 + j * 8 + 2 * tq;
                const float b0 = bias[c], b1 = bias[c + 1];
#pragma unroll
                for (int m = 0; m < 4; ++m)
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        const float x = z[m][j][2 * half] + b0, y = z[m][j][2 * half + 1] + b1;
                        float2 ls;
                        ls.x = (fminf(x, 0.f) - __logf(1.f + __expf(-fabsf(x)))) * log2e_tau;
                        ls.y = (fminf(y, 0.f) - __logf(1.f + __expf(-fabsf(y)))) * log2e_tau;
                        *reinterpret_cast<float2*>(&S.b[(m * 16 + g + half * 8) * BROW + c]) = ls;
                    }
            }
        }
        __syncthreads();
        // ---- sums over the tokens, and how many of them fit ----
        float* column = S.b + bpart * kPartLen * BROW + bc;
        {
            float run = 0.f;
#pragma unroll 8
            for (int t = 0; t < kPartLen; ++t) run += column[t * BROW];
            S.part[bpart * DK + bc] = run;
        }
        const float first = S.b[bc];   // (row 0 is already its own sum)
        __syncthreads();
        {
            float run = 0.f;
            for (int i = 0; i < bpart; ++i) run += S.part[i * DK + bc];
            int fit = kChunk;
#pragma unroll 8
            for (int t = 0; t < kPartLen; ++t) {
                run += column[t * BROW];
                column[t * BROW] = run;
                if (first - run > kRangeLog2) fit = min(fit, bpart * kPartLen + t);
            }
            if (fit < n_max) atomicMin(&S.n, fit);
        }
        __syncthreads();
        const int n = S.n;
        const float* last = S.b + (n - 1) * BROW;
        // ---- q~, k~ and exp(r) S ----
        for (int i = threadIdx.x; i < kChunk * (DK / 2); i += kChunkThreads) {
            const int t = i / (DK / 2), c = (i % (DK / 2)) * 2;
            uint32_t qh = 0, ql = 0, kh = 0, kl = 0;
            if (t < n) {
                const uint32_t qv = *reinterpret_cast<const uint32_t*>(&S.q[t * ROW + c]);
                const uint32_t kv = *reinterpret_cast<const uint32_t*>(&S.k[t * ROW + c]);
                const float2 bt = *reinterpret_cast<const float2*>(&S.b[t * BROW + c]);
                const float d0 = bt.x - 0.5f * (S.b[c] + last[c]), d1 = bt.y - 0.5f * (S.b[c + 1] + last[c + 1]);
                split2(bf16_lo(qv) * a.q_scale * ex2(d0), bf16_hi(qv) * a.q_scale * ex2(d1), qh, ql);
                split2(bf16_lo(kv) * ex2(-d0), bf16_hi(kv) * ex2(-d1), kh, kl);
            }
            *reinterpret_cast<uint32_t*>(&S.qh[t * ROW + c]) = qh;
            *reinterpret_cast<uint32_t*>(&S.ql[t * ROW + c]) = ql;
            *reinterpret_cast<uint32_t*>(&S.kh[t * ROW + c]) = kh;
            *reinterpret_cast<uint32_t*>(&S.kl[t * ROW + c]) = kl;
        }
        float decay[2], rest[2];   // exp(b_n) and exp(b_n - r) of this thread's two state rows
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int c = row0 + g + half * 8;
            const float ref = 0.5f * (S.b[c] + last[c]), into = ex2(ref);
            decay[half] = ex2(last[c]);
            rest[half] = ex2(last[c] - ref);
#pragma unroll
            for (int j = 0; j < kStateTiles; ++j) {
                uint32_t hi, lo;
                split2(st[j][2 * half] * into, st[j][2 * half + 1] * into, hi, lo);
                *reinterpret_cast<uint32_t*>(&S.sh[c * VROW + col0 + j * 8 + 2 * tq]) = hi;
                *reinterpret_cast<uint32_t*>(&S.sl[c * VROW + col0 + j * 8 + 2 * tq]) = lo;
            }
        }
        __syncthreads();
        // what was loaded has been used up, but for the values
        if (s0 + n < ext) load_segment(s0 + n, buf ^ 1);
        const __nv_bfloat16* V = S.v[buf];

        // ---- output rows [16 mt, 16 mt + 16), columns [oc0, oc0 + 32) ----
        if (mt * 16 < n) {
            float o[4][4];
#pragma unroll
            for (int j = 0; j < 4; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
            float p[8][4];   // scores of these rows and all keys up to the last of them
#pragma unroll
            for (int j = 0; j < 8; ++j) p[j][0] = p[j][1] = p[j][2] = p[j][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < DK / 16; ++ks) {
                uint32_t ah[4], al[4];
                const int aoff = (mt * 16 + (mi & 1) * 8 + r8) * ROW + ks * 16 + (mi >> 1) * 8;
                ldmatrix_x4(smem_u32(&S.qh[aoff]), ah[0], ah[1], ah[2], ah[3]);
                ldmatrix_x4(smem_u32(&S.ql[aoff]), al[0], al[1], al[2], al[3]);
#pragma unroll
                for (int np = 0; np < 2; ++np) {   // the state from before the segment
                    uint32_t b0, b1, b2, b3;
                    const int soff = (ks * 16 + (mi & 1) * 8 + r8) * VROW + oc0 + np * 16 + (mi >> 1) * 8;
                    ldmatrix_x4_trans(smem_u32(&S.sh[soff]), b0, b1, b2, b3);
                    mma_bf16_16816(o[2 * np], ah, b0, b1);
                    mma_bf16_16816(o[2 * np + 1], ah, b2, b3);
                    mma_bf16_16816(o[2 * np], al, b0, b1);
                    mma_bf16_16816(o[2 * np + 1], al, b2, b3);
                    ldmatrix_x4_trans(smem_u32(&S.sl[soff]), b0, b1, b2, b3);
                    mma_bf16_16816(o[2 * np], ah, b0, b1);
                    mma_bf16_16816(o[2 * np + 1], ah, b2, b3);
                }
#pragma unroll
                for (int kt = 0; kt < 4; ++kt) {   // 16 keys at a time
                    if (kt > mt) continue;
                    uint32_t b0, b1, b2, b3;
                    const int koff = (kt * 16 + (mi >> 1) * 8 + r8) * ROW + ks * 16 + (mi & 1) * 8;
                    ldmatrix_x4(smem_u32(&S.kh[koff]), b0, b1, b2, b3);
                    mma_bf16_16816(p[2 * kt], ah, b0, b1);
                    mma_bf16_16816(p[2 * kt + 1], ah, b2, b3);
                    mma_bf16_16816(p[2 * kt], al, b0, b1);
                    mma_bf16_16816(p[2 * kt + 1], al, b2, b3);
                    ldmatrix_x4(smem_u32(&S.kl[koff]), b0, b1, b2, b3);
                    mma_bf16_16816(p[2 * kt], ah, b0, b1);
                    mma_bf16_16816(p[2 * kt + 1], ah, b2, b3);
                }
            }
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) {
                if (kt > mt) continue;
                if (kt == mt) {   // keys after the query
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        const int key = (e >> 2) * 8 + 2 * tq + (e & 1), row = g + (e & 2) * 4;
                        if (key > row) p[2 * kt + (e >> 2)][e & 3] = 0.f;
                    }
                }
                uint32_t ph[4], pl[4];
                split2(p[2 * kt][0], p[2 * kt][1], ph[0], pl[0]);
                split2(p[2 * kt][2], p[2 * kt][3], ph[1], pl[1]);
                split2(p[2 * kt + 1][0], p[2 * kt + 1][1], ph[2], pl[2]);
                split2(p[2 * kt + 1][2], p[2 * kt + 1][3], ph[3], pl[3]);
#pragma unroll
                for (int np = 0; np < 2; ++np) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(smem_u32(&V[(kt * 16 + (mi & 1) * 8 + r8) * VROW + oc0 + np * 16 + (mi >> 1) * 8]), b0, b1, b2, b3);
                    mma_bf16_16816(o[2 * np], ph, b0, b1);
                    mma_bf16_16816(o[2 * np + 1], ph, b2, b3);
                    mma_bf16_16816(o[2 * np], pl, b0, b1);
                    mma_bf16_16816(o[2 * np + 1], pl, b2, b3);
                }
            }
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + static_cast<int64_t>(h) * vp + v0 + oc0;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int t = mt * 16 + g + half * 8;
                if (t >= n) continue;
                __nv_bfloat16* dst = out + static_cast<int64_t>(begin + s0 + t) * a.heads * vp;
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    *reinterpret_cast<uint32_t*>(dst + j * 8 + 2 * tq) = pack_bf16(o[j][2 * half], o[j][2 * half + 1]);
            }
        }
        // ---- the state after the segment ----
        {
            float u[kStateTiles][4];
#pragma unroll
            for (int j = 0; j < kStateTiles; ++j) u[j][0] = u[j][1] = u[j][2] = u[j][3] = 0.f;
#pragma unroll
            for (int kt = 0; kt < kChunk / 16; ++kt) {
                uint32_t ah[4], al[4];
                const int aoff = (kt * 16 + (mi >> 1) * 8 + r8) * ROW + row0 + (mi & 1) * 8;
                ldmatrix_x4_trans(smem_u32(&S.kh[aoff]), ah[0], ah[1], ah[2], ah[3]);
                ldmatrix_x4_trans(smem_u32(&S.kl[aoff]), al[0], al[1], al[2], al[3]);
#pragma unroll
                for (int np = 0; np < kStateTiles / 2; ++np) {
                    uint32_t b0, b1, b2, b3;
                    ldmatrix_x4_trans(smem_u32(&V[(kt * 16 + (mi & 1) * 8 + r8) * VROW + col0 + np * 16 + (mi >> 1) * 8]), b0, b1, b2, b3);
                    mma_bf16_16816(u[2 * np], ah, b0, b1);
                    mma_bf16_16816(u[2 * np + 1], ah, b2, b3);
                    mma_bf16_16816(u[2 * np], al, b0, b1);
                    mma_bf16_16816(u[2 * np + 1], al, b2, b3);
                }
            }
#pragma unroll
            for (int j = 0; j < kStateTiles; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) st[j][e] = decay[e >> 1] * st[j][e] + rest[e >> 1] * u[j][e];
        }
        s0 += n;
        buf ^= 1;
        __syncthreads();   // q~, k~, S and b are written again
    }
#pragma unroll
    for (int j = 0; j < kStateTiles; ++j)
#pragma unroll
        for (int half = 0; half < 2; ++half)
            *reinterpret_cast<float2*>(state + static_cast<int64_t>(row0 + g + half * 8) * vp + col0 + j * 8 + 2 * tq) =
                make_float2(st[j][2 * half], st[j][2 * half + 1]);
}

bool chunked_supported(const LinearAttention& a, int dtype) {
    return dtype == B200_DTYPE_BF16 && !a.plain && (a.padded_dim == 64 || a.padded_dim == 128) &&
           a.padded_value_dim % kSlice == 0 && a.up_ld % 16 == 0 && a.up_ld <= kMaxLow;
}

int max_smem(const void* kernel, size_t bytes) {
    B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
    return B200_OK;
}

}  // namespace

// Value rows the decode kernel covers with one CTA, and channels whose vectors and state slice fit.
bool linear_attention_supported(int padded_value_dim, int padded_dim) {
    return padded_value_dim <= 4 * kDecodeThreads && padded_dim <= 1024;
}

int launch_linear_attention(const LinearAttention& a, int dtype, cudaStream_t stream) {
    if (a.tokens == 0 || a.batch == 0) return B200_OK;
    const bool f32 = dtype == B200_DTYPE_F32;
    if (a.decode) {
        const int groups = kDecodeThreads / (a.padded_value_dim / 4);
        const size_t smem = (3ull * a.padded_dim + static_cast<size_t>(groups) * a.padded_value_dim) * 4;
        auto kernel = f32 ? linear_attention_decode_kernel<float> : linear_attention_decode_kernel<__nv_bfloat16>;
        B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.heads, a.batch), dim3(kDecodeThreads), smem, stream, dim3(1, 1, 1), a));
        return B200_OK;
    }
    if (chunked_supported(a, dtype)) {
        auto kernel = a.padded_dim == 64 ? linear_attention_chunk_kernel<64> : linear_attention_chunk_kernel<128>;
        const size_t smem = a.padded_dim == 64 ? sizeof(ChunkSmem<64>) : sizeof(ChunkSmem<128>);
        int err = max_smem(reinterpret_cast<const void*>(kernel), smem);
        if (err != B200_OK) return err;
        B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.padded_value_dim / kSlice, a.heads, a.batch), dim3(kChunkThreads), smem,
                                      stream, dim3(1, 1, 1), a));
    } else {
        auto kernel = f32 ? linear_attention_plain_kernel<float> : linear_attention_plain_kernel<__nv_bfloat16>;
        const size_t smem = static_cast<size_t>(a.padded_dim) * (3 + kPlainCols) * 4;
        int err = max_smem(reinterpret_cast<const void*>(kernel), smem);
        if (err != B200_OK) return err;
        B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.padded_value_dim / kPlainCols, a.heads, a.batch), dim3(kPlainThreads), smem,
                                      stream, dim3(1, 1, 1), a));
    }
    const int64_t rows = static_cast<int64_t>(a.tokens) * a.heads;
    auto kernel = f32 ? linear_attention_finish_kernel<float> : linear_attention_finish_kernel<__nv_bfloat16>;
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(static_cast<unsigned>((rows + kFinishWarps - 1) / kFinishWarps)),
                                  dim3(kFinishWarps * 32), 0, stream, dim3(1, 1, 1), a));
    return B200_OK;
}

}  // namespace b200

extern "C" {

int b200_linear_attention(const b200_linear_attention_args* p, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(p, "linear_attention: NULL argument");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "linear_attention: unknown dtype");
    B200_CHECK_ARG(p->tokens >= 0 && p->batch >= 0 && p->batch <= 65535 && p->heads > 0 && p->heads <= 65535,
                   "linear_attention: bad sizes");
    B200_CHECK_ARG(p->dim > 0 && p->padded_dim >= p->dim && p->padded_dim % 64 == 0 && p->value_dim > 0 &&
                       p->padded_value_dim >= p->value_dim && p->padded_value_dim % 64 == 0 &&
                       b200::linear_attention_supported(p->padded_value_dim, p->padded_dim), "linear_attention: bad head sizes");
    B200_CHECK_ARG(p->rank > 0 && p->up_ld >= p->rank && p->up_ld % 16 == 0 && p->joint_ld % 8 == 0 && p->tau > 0.f,
                   "linear_attention: bad decay projection");
    B200_CHECK_ARG(!p->decode || p->tokens == p->batch, "linear_attention: a decode step brings one token per request");
    if (p->tokens == 0 || p->batch == 0) return B200_OK;
    B200_CHECK_ARG(p->out && p->joint && p->table_idx && p->cached && (p->decode || p->qo_indptr) && p->state && p->up &&
                       p->bias && p->norm, "linear_attention: NULL tensor");
    return b200::launch_linear_attention(*p, dtype, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
