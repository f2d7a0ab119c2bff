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
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
template <typename T>
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
template <>
__device__ __forceinline__ float silu<__nv_bfloat16>(float x) { return x * sigmoid_f(x); }

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
        out[c] = from_f32<T>(s_o[c] * scale * to_f32(static_cast<const T*>(a.norm)[c]) * silu<T>(g));
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
    const unsigned row = blockIdx.x * kFinishWarps + (threadIdx.x >> 5);
    pdl_launch_dependents();
    pdl_wait_prior();
    if (row >= static_cast<unsigned>(a.tokens) * a.heads) return;
    const int64_t t = row / a.heads;
    const int h = static_cast<int>(row - t * a.heads);
    T* out = static_cast<T*>(a.out) + static_cast<int64_t>(row) * vp;
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
        store4(out + c, make_float4(o.x * scale * w.x * silu<T>(g.x), o.y * scale * w.y * silu<T>(g.y),
                                    o.z * scale * w.z * silu<T>(g.z), o.w * scale * w.w * silu<T>(g.w)));
    }
}

// ---- chunked ----------------------------------------------------------------------

constexpr int kChunk = 64;            // tokens per segment at most
constexpr int kSlice = 64;            // value columns per CTA
constexpr int kChunkThreads = 512;
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
    __nv_bfloat16 ph[kChunk * kVRow], pl[kChunk * kVRow];             // scores
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
__device__ __forceinline__ float lg2(float x) {
    float y;
    asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
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
    constexpr int kColSplit = 256 / DK;                 // warps that share 16 state rows
    constexpr int kStateTiles = kSlice / 8 / kColSplit; // 8-column tiles of state per warp
    constexpr int kZTokens = DK / 32;                   // 16-token tiles of z per warp, 8 channels each
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

    const int zc0 = warp % (DK / 8) * 8, zm0 = warp / (DK / 8) * kZTokens;   // this warp's channels and token tiles of z
    const int bc = threadIdx.x % DK, bpart = threadIdx.x / DK;   // this thread's column and piece of b
    // 16 tokens x 16 columns of the output per warp; the four warps of a scheduler take four different token tiles
    const int mt = (warp + (warp >> 2)) & 3, oc0 = (warp >> 2) * 16;
    // warps 0 to 9 compute a 16 x 16 tile of scores each: (0,0) (1,0) (1,1) (2,0) ...
    const int smt = warp < 1 ? 0 : warp < 3 ? 1 : warp < 6 ? 2 : 3, skt = warp - smt * (smt + 1) / 2;
    const float inv_tau = 1.f / a.tau, log2e_tau = kLog2e / a.tau, q_shift = log2f(a.q_scale);
    const __nv_bfloat16* up = static_cast<const __nv_bfloat16*>(a.up) + static_cast<int64_t>(h) * DK * a.up_ld;
    const float* bias = a.bias + static_cast<int64_t>(h) * DK;

    // the first 16 ranks of this warp's channels and their bias, fetched a segment ahead (shared memory leaves no
    // room for them to stay in L1)
    uint32_t up0, up1;
    float bias0, bias1;
    auto fetch_up = [&](int r, uint32_t& b0, uint32_t& b1) {
        const __nv_bfloat16* u = up + static_cast<int64_t>(zc0 + g) * a.up_ld + r + 2 * tq;
        b0 = *reinterpret_cast<const uint32_t*>(u);
        b1 = *reinterpret_cast<const uint32_t*>(u + 8);
    };
    auto fetch_decay = [&]() {
        fetch_up(0, up0, up1);
        bias0 = bias[zc0 + 2 * tq];
        bias1 = bias[zc0 + 2 * tq + 1];
    };
    fetch_decay();

    int buf = 0;
    for (int s0 = 0; s0 < ext;) {
        const int n_max = min(kChunk, ext - s0);
        cp_async_wait_all();
        if (threadIdx.x == 0) S.n = n_max;
        __syncthreads();
        // ---- z = low up^T + bias, and its decay logarithm ----
        {
            float z[kZTokens][4];
#pragma unroll
            for (int m = 0; m < kZTokens; ++m) z[m][0] = z[m][1] = z[m][2] = z[m][3] = 0.f;
            for (int r = 0; r < a.up_ld; r += 16) {
                uint32_t b0 = up0, b1 = up1;
                if (r > 0) fetch_up(r, b0, b1);
#pragma unroll
                for (int m = 0; m < kZTokens; ++m) {
                    uint32_t af[4];
                    ldmatrix_x4(smem_u32(&S.low[((zm0 + m) * 16 + (mi & 1) * 8 + r8) * LROW + r + (mi >> 1) * 8]), af[0], af[1],
                                af[2], af[3]);
                    mma_bf16_16816(z[m], af, b0, b1);
                }
            }
            const int c = zc0 + 2 * tq;
#pragma unroll
            for (int m = 0; m < kZTokens; ++m)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const float x = z[m][2 * half] + bias0, y = z[m][2 * half + 1] + bias1;
                    float2 ls;
                    ls.x = fminf(x, 0.f) * log2e_tau - lg2(1.f + ex2(-kLog2e * fabsf(x))) * inv_tau;
                    ls.y = fminf(y, 0.f) * log2e_tau - lg2(1.f + ex2(-kLog2e * fabsf(y))) * inv_tau;
                    *reinterpret_cast<float2*>(&S.b[((zm0 + m) * 16 + g + half * 8) * BROW + c]) = ls;
                }
        }
        __syncthreads();
        // ---- sums over the tokens, and how many of them fit ----
        float* column = S.b + bpart * kPartLen * BROW + bc;
        {
            float run[kPartLen];
#pragma unroll
            for (int t = 0; t < kPartLen; ++t) run[t] = column[t * BROW];
#pragma unroll
            for (int t = 1; t < kPartLen; ++t) run[t] += run[t - 1];
            S.part[bpart * DK + bc] = run[kPartLen - 1];
            const float first = S.b[bc];   // (row 0 is already its own sum)
            __syncthreads();
            float before = 0.f;
            for (int i = 0; i < bpart; ++i) before += S.part[i * DK + bc];
#pragma unroll
            for (int t = 0; t < kPartLen; ++t) {
                run[t] += before;
                column[t * BROW] = run[t];
            }
            if (first - run[kPartLen - 1] > kRangeLog2) {   // (the sums only fall)
                int fit = 0;
#pragma unroll
                for (int t = 0; t < kPartLen; ++t) fit += first - run[t] > kRangeLog2 ? 0 : 1;
                fit += bpart * kPartLen;
                if (fit < n_max) atomicMin(&S.n, fit);
            }
        }
        __syncthreads();
        const int n = S.n;
        const float* last = S.b + (n - 1) * BROW;
        // ---- q~, k~ and exp(r) S ----
        {
            constexpr int kQuads = DK / 4, kRows = kChunkThreads / kQuads;   // a thread keeps to four channels
            const int c = threadIdx.x % kQuads * 4;
            const float4 b0 = load4(S.b + c), b1 = load4(last + c);
            const float r[4] = {0.5f * (b0.x + b1.x), 0.5f * (b0.y + b1.y), 0.5f * (b0.z + b1.z), 0.5f * (b0.w + b1.w)};
#pragma unroll 2
            for (int t = threadIdx.x / kQuads; t < kChunk; t += kRows) {
                uint2 qh = make_uint2(0, 0), ql = qh, kh = qh, kl = qh;
                if (t < n) {
                    const float4 q = load4(&S.q[t * ROW + c]), k = load4(&S.k[t * ROW + c]), b = load4(&S.b[t * BROW + c]);
                    const float d0 = b.x - r[0], d1 = b.y - r[1], d2 = b.z - r[2], d3 = b.w - r[3];
                    split2(q.x * ex2(d0 + q_shift), q.y * ex2(d1 + q_shift), qh.x, ql.x);
                    split2(q.z * ex2(d2 + q_shift), q.w * ex2(d3 + q_shift), qh.y, ql.y);
                    split2(k.x * ex2(-d0), k.y * ex2(-d1), kh.x, kl.x);
                    split2(k.z * ex2(-d2), k.w * ex2(-d3), kh.y, kl.y);
                }
                *reinterpret_cast<uint2*>(&S.qh[t * ROW + c]) = qh;
                *reinterpret_cast<uint2*>(&S.ql[t * ROW + c]) = ql;
                *reinterpret_cast<uint2*>(&S.kh[t * ROW + c]) = kh;
                *reinterpret_cast<uint2*>(&S.kl[t * ROW + c]) = kl;
            }
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

        // ---- scores of 16 queries and 16 keys ----
        if (warp < 10 && smt * 16 < n) {
            float p[2][4] = {};
#pragma unroll
            for (int ks = 0; ks < DK / 16; ++ks) {
                uint32_t ah[4], al[4], b0, b1, b2, b3;
                const int aoff = (smt * 16 + (mi & 1) * 8 + r8) * ROW + ks * 16 + (mi >> 1) * 8;
                const int koff = (skt * 16 + (mi >> 1) * 8 + r8) * ROW + ks * 16 + (mi & 1) * 8;
                ldmatrix_x4(smem_u32(&S.qh[aoff]), ah[0], ah[1], ah[2], ah[3]);
                ldmatrix_x4(smem_u32(&S.ql[aoff]), al[0], al[1], al[2], al[3]);
                ldmatrix_x4(smem_u32(&S.kh[koff]), b0, b1, b2, b3);
                mma_bf16_16816(p[0], ah, b0, b1);
                mma_bf16_16816(p[1], ah, b2, b3);
                mma_bf16_16816(p[0], al, b0, b1);
                mma_bf16_16816(p[1], al, b2, b3);
                ldmatrix_x4(smem_u32(&S.kl[koff]), b0, b1, b2, b3);
                mma_bf16_16816(p[0], ah, b0, b1);
                mma_bf16_16816(p[1], ah, b2, b3);
            }
#pragma unroll
            for (int tile = 0; tile < 2; ++tile)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int row = g + half * 8, key = tile * 8 + 2 * tq;
                    float x = p[tile][2 * half], y = p[tile][2 * half + 1];
                    if (skt == smt && key > row) x = 0.f;       // keys after the query
                    if (skt == smt && key + 1 > row) y = 0.f;
                    uint32_t hi, lo;
                    split2(x, y, hi, lo);
                    *reinterpret_cast<uint32_t*>(&S.ph[(smt * 16 + row) * VROW + skt * 16 + key]) = hi;
                    *reinterpret_cast<uint32_t*>(&S.pl[(smt * 16 + row) * VROW + skt * 16 + key]) = lo;
                }
        }
        // ---- what the state from before the segment adds to output rows [16 mt, +16), columns [oc0, +16) ----
        float o[2][4] = {};
        if (mt * 16 < n) {
#pragma unroll
            for (int ks = 0; ks < DK / 16; ++ks) {
                uint32_t ah[4], al[4], b0, b1, b2, b3;
                const int aoff = (mt * 16 + (mi & 1) * 8 + r8) * ROW + ks * 16 + (mi >> 1) * 8;
                const int soff = (ks * 16 + (mi & 1) * 8 + r8) * VROW + oc0 + (mi >> 1) * 8;
                ldmatrix_x4(smem_u32(&S.qh[aoff]), ah[0], ah[1], ah[2], ah[3]);
                ldmatrix_x4(smem_u32(&S.ql[aoff]), al[0], al[1], al[2], al[3]);
                ldmatrix_x4_trans(smem_u32(&S.sh[soff]), b0, b1, b2, b3);
                mma_bf16_16816(o[0], ah, b0, b1);
                mma_bf16_16816(o[1], ah, b2, b3);
                mma_bf16_16816(o[0], al, b0, b1);
                mma_bf16_16816(o[1], al, b2, b3);
                ldmatrix_x4_trans(smem_u32(&S.sl[soff]), b0, b1, b2, b3);
                mma_bf16_16816(o[0], ah, b0, b1);
                mma_bf16_16816(o[1], ah, b2, b3);
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
        __syncthreads();   // the scores are complete
        fetch_decay();
        if (mt * 16 < n) {
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) {
                if (kt > mt) continue;
                uint32_t ah[4], al[4], b0, b1, b2, b3;
                const int poff = (mt * 16 + (mi & 1) * 8 + r8) * VROW + kt * 16 + (mi >> 1) * 8;
                ldmatrix_x4(smem_u32(&S.ph[poff]), ah[0], ah[1], ah[2], ah[3]);
                ldmatrix_x4(smem_u32(&S.pl[poff]), al[0], al[1], al[2], al[3]);
                ldmatrix_x4_trans(smem_u32(&V[(kt * 16 + (mi & 1) * 8 + r8) * VROW + oc0 + (mi >> 1) * 8]), b0, b1, b2, b3);
                mma_bf16_16816(o[0], ah, b0, b1);
                mma_bf16_16816(o[1], ah, b2, b3);
                mma_bf16_16816(o[0], al, b0, b1);
                mma_bf16_16816(o[1], al, b2, b3);
            }
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + static_cast<int64_t>(h) * vp + v0 + oc0;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int t = mt * 16 + g + half * 8;
                if (t >= n) continue;
                __nv_bfloat16* dst = out + static_cast<int64_t>(begin + s0 + t) * a.heads * vp;
#pragma unroll
                for (int j = 0; j < 2; ++j)
                    *reinterpret_cast<uint32_t*>(dst + j * 8 + 2 * tq) = pack_bf16(o[j][2 * half], o[j][2 * half + 1]);
            }
        }
        s0 += n;
        buf ^= 1;
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
    B200_CHECK_ARG(static_cast<int64_t>(p->tokens) * p->heads < (1ll << 31), "linear_attention: too many tokens");
    B200_CHECK_ARG(!p->decode || p->tokens == p->batch, "linear_attention: a decode step brings one token per request");
    if (p->tokens == 0 || p->batch == 0) return B200_OK;
    B200_CHECK_ARG(p->out && p->joint && p->table_idx && p->cached && (p->decode || p->qo_indptr) && p->state && p->up &&
                       p->bias && p->norm, "linear_attention: NULL tensor");
    return b200::launch_linear_attention(*p, dtype, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
