// Recurrences with one decay per head and step.  Behind a short causal convolution, a scalar-decay state space
//     S <- g S + dt k v^T,                    o = S^T q + skip v
// and the gated delta rule (k and q unit vectors)
//     S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,    o = S^T q.
// Without one, lightning attention, whose decay is constant (k, q, v behind a silu)
//     S <- g S + k v^T,                       o = S^T q
// and the matrix memory, whose exponential gates (logarithms i and f) refer to a running maximum
//     m' = max(f + m, i),  S <- exp(f + m - m') S + exp(i - m') k v^T,  n likewise with k alone
//     o = S^T q / (max(|n . q|, exp(-m')) + 1e-6).
// The matrix state is fp32 and lives in a slot per page-table row, as do the convolution's last inputs (a ring: the
// input of position p is at p mod taps, so that a step writes a place that nobody reads in the same step).
//
//   * decode: one CTA per (request, head) convolves its channels, streams the state once - read, decayed, updated,
//     read out, written, in registers between its first and its last use - and, for the delta rule, applies the
//     head's norm and gate.  Everything that the projection before it does not write is read ahead of
//     griddepcontrol.wait.
//   * prefill: mix_kernel convolves all channels and leaves steps (decay logarithm, weight of what is written) and
//     unit factors in fp32; the recurrence itself follows in chunks of 64 tokens (bf16) or token by token.
//   * chunked: with B_t the decay logarithms summed up inside a chunk, G_t = exp(B_t), and S the state before it,
//         P_ts = exp(B_t - B_s) q_t . k_s  (s <= t),     A_ts = beta_t exp(B_t - B_s) k_t . k_s  (s < t)
//         U = (I + A)^-1 diag(beta) (V - diag(G) K S)     (state space: U = diag(dt) V)
//         O = diag(G) Q S + P U
//         S <- G_n S + K^T diag(exp(B_n - B_s)) U
//     (lightning: dt = 1).  The matrix memory, with m the maximum before the chunk and c_t = max_{s <= t} (i_s - B_s):
//         P_ts = exp(i_s - B_s - c_t) q_t . k_s  (s <= t),           m_t = B_t + max(m, c_t)
//         O = diag(exp(m - max(m, c))) Q S + diag(exp(c - max(m, c))) P V,   the same for n with 1 in the place of V
//         S <- exp(m - max(m, c_n)) S + K^T diag(exp(i_s - B_s - max(m, c_n))) V
//     No exponent is positive, however steep the decay.  P and the inverse do not depend on the state: prepare_kernel
//     makes them for all chunks at once (the inverse by substitution in fp32) and stores them in the order in which
//     chunk_kernel's threads hold MMA operands.  chunk_kernel walks a request's chunks, one CTA per head and 64
//     value columns.  k, q and v enter the products as the bf16 numbers the convolution returned, unit factors, steps
//     and decays being applied to fp32 results; everything derived from those or from the state enters as the
//     sum of two bf16 numbers.
//   * a last kernel applies norm and gate where the recurrence did not.
#include <math.h>

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
template <typename T>
__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
template <>
__device__ __forceinline__ float sigmoid<__nv_bfloat16>(float x) { return sigmoid_f(x); }

constexpr float kLog2e = 1.4426950408889634f;
constexpr float kUnitEps = 1e-6f, kMemoryEps = 1e-6f;
constexpr int kStepThreads = 512;
constexpr int kMaxAhead = 8;   // state rows per thread of the step kernel, in registers
constexpr int kMaxTaps = 16;
constexpr int kStateSpace = B200_RULE_STATE_SPACE, kDelta = B200_RULE_DELTA, kLightning = B200_RULE_LIGHTNING,
              kMemory = B200_RULE_MATRIX_MEMORY;
constexpr bool has_convolution(int rule) { return rule == kStateSpace || rule == kDelta; }

// Channel c of [v | k | q] is column values() + c of a row of the joint projection.
__device__ __forceinline__ int64_t values(const Recurrence& a) { return static_cast<int64_t>(a.heads) * a.padded_value_dim; }
__device__ __forceinline__ int64_t channels(const Recurrence& a) { return values(a) + 2ll * a.kv_heads * a.padded_dim; }

// What the recurrence reads channels from: what mix_kernel has left, or (matrix memory) the projection itself.
template <typename T>
__device__ __forceinline__ const T* mixed_rows(const Recurrence& a) {
    return a.rule == kMemory ? static_cast<const T*>(a.joint) + values(a) : static_cast<const T*>(a.mixed);
}
__device__ __forceinline__ int64_t mixed_ld(const Recurrence& a) { return a.rule == kMemory ? a.joint_ld : channels(a); }

// The matrix memory keeps n and m once per this many value columns: what one CTA writes no other one reads.
__host__ __device__ inline int memory_columns(int padded_dim) {
    const int most = kMaxAhead * kStepThreads / padded_dim;   // groups of four columns that a step CTA has room for
    int cols = 64;
    while (cols > 4 && cols > 4 * most) cols /= 2;
    return cols;
}
__host__ __device__ inline int memory_copies(int padded_dim, int padded_value_dim) { return padded_value_dim / memory_columns(padded_dim); }
__host__ __device__ inline int memory_width(int padded_dim) { return padded_dim + 4; }   // n, then m in units of log 2
__device__ __forceinline__ float* memory_of(const Recurrence& a, int64_t row, int h, int col0) {
    const int copy = col0 / memory_columns(a.padded_dim);
    return a.memory + ((row * a.heads + h) * memory_copies(a.padded_dim, a.padded_value_dim) + copy) * memory_width(a.padded_dim);
}

// log2 of a step's decay and the weight of what it writes (matrix memory: log2 of that), from a head's columns of the
// joint projection.
__device__ __forceinline__ float2 make_step(int rule, float za, float zb, float step_bias, float decay_log, float cap) {
    if (rule == kLightning) return make_float2(decay_log * kLog2e, 1.f);
    if (rule == kMemory) {
        const float f = cap * tanhf((zb + decay_log) / cap);
        return make_float2((fminf(f, 0.f) - log1pf(expf(-fabsf(f)))) * kLog2e, cap * tanhf((za + step_bias) / cap) * kLog2e);
    }
    const float x = za + step_bias, dt = fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
    return make_float2(-expf(decay_log) * dt * kLog2e, rule == kStateSpace ? dt : 1.f / (1.f + expf(-zb)));
}

// ---- convolution, steps, unit factors ------------------------------------------------

// Eight elements as they are in memory.
template <typename T>
struct Packed8;
template <>
struct __align__(16) Packed8<__nv_bfloat16> {
    uint4 u;
};
template <>
struct __align__(16) Packed8<float> {
    float4 a, b;
};
template <typename T>
__device__ __forceinline__ Packed8<T> pack8(const Vec8& x);
template <>
__device__ __forceinline__ Packed8<float> pack8(const Vec8& x) {
    return {make_float4(x.v[0], x.v[1], x.v[2], x.v[3]), make_float4(x.v[4], x.v[5], x.v[6], x.v[7])};
}
template <>
__device__ __forceinline__ Packed8<__nv_bfloat16> pack8(const Vec8& x) {
    return {make_uint4(pack_bf16(x.v[0], x.v[1]), pack_bf16(x.v[2], x.v[3]), pack_bf16(x.v[4], x.v[5]), pack_bf16(x.v[6], x.v[7]))};
}
__device__ __forceinline__ Vec8 unpack8(const Packed8<float>& p) { return {{p.a.x, p.a.y, p.a.z, p.a.w, p.b.x, p.b.y, p.b.z, p.b.w}}; }
__device__ __forceinline__ Vec8 unpack8(const Packed8<__nv_bfloat16>& p) {
    return {{bf16_lo(p.u.x), bf16_hi(p.u.x), bf16_lo(p.u.y), bf16_hi(p.u.y), bf16_lo(p.u.z), bf16_hi(p.u.z), bf16_lo(p.u.w),
             bf16_hi(p.u.w)}};
}

constexpr int kMixThreads = 128;
constexpr int kMixTokens = 16;
constexpr int kMixAhead = 2;   // tokens whose inputs are in flight

// Grid: blocks of tokens, blocks of channels (8 per thread; those of k and q cover whole heads) and one for the
// steps, requests.  TAPS 0: any number of them.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kMixThreads)
mix_kernel(const Recurrence a, int v_blocks, int heads_per_block) {
    __shared__ float s_part[kMixTokens][kMixThreads];
    pdl_launch_dependents();
    pdl_wait_prior();
    const int b = blockIdx.z, begin = a.qo_indptr[b], ext = a.qo_indptr[b + 1] - begin;
    const int t0 = blockIdx.x * kMixTokens;
    if (t0 >= ext) return;
    const int n = min(kMixTokens, ext - t0);
    const T* joint = static_cast<const T*>(a.joint) + static_cast<int64_t>(begin) * a.joint_ld;
    if (blockIdx.y == gridDim.y - 1) {
        for (int i = threadIdx.x; i < n * a.heads; i += kMixThreads) {
            const int t = t0 + i / a.heads, h = i % a.heads;
            const T* tail = joint + t * a.joint_ld + values(a) + channels(a) + h;
            const bool pair = a.rule == kDelta || a.rule == kMemory;
            reinterpret_cast<float2*>(a.steps)[static_cast<int64_t>(begin + t) * a.heads + h] =
                make_step(a.rule, a.rule == kLightning ? 0.f : to_f32(tail[0]), pair ? to_f32(tail[a.heads]) : 0.f,
                          a.rule == kLightning ? 0.f : a.step_bias[h], a.rule == kMemory ? a.step_bias[a.heads + h] : a.decay_log[h],
                          a.gate_cap);
        }
        return;
    }
    const int64_t nv = values(a), nc = channels(a);
    const bool heads = static_cast<int>(blockIdx.y) >= v_blocks;
    const int per_head = a.padded_dim >> 3, head0 = (static_cast<int>(blockIdx.y) - v_blocks) * heads_per_block;
    int64_t c;
    bool active;
    if (heads) {
        const int head = static_cast<int>(threadIdx.x) / per_head;
        active = head < heads_per_block && head0 + head < 2 * a.kv_heads;
        c = nv + static_cast<int64_t>(head0) * a.padded_dim + threadIdx.x * 8;
    } else {
        c = (static_cast<int64_t>(blockIdx.y) * kMixThreads + threadIdx.x) * 8;
        active = c < nv;
    }
    const int taps = TAPS > 0 ? TAPS : a.taps, cached = a.cached[b];
    T* ring = static_cast<T*>(a.conv_state) + static_cast<int64_t>(a.table_idx[b]) * taps * nc + c;
    const T* in = joint + nv + c;
    // the input of token r of this step, or of one before it
    auto input = [&](int r) {
        if (r >= 0) return load8(in + r * a.joint_ld);
        Vec8 x;
#pragma unroll
        for (int j = 0; j < 8; ++j) x.v[j] = 0.f;
        return cached + r >= 0 ? load8(ring + (cached + r) % taps * nc) : x;
    };
    if (active) {
        constexpr int kWindow = TAPS > 0 ? TAPS : 1;
        Vec8 w[kWindow], x[kWindow], bias;
#pragma unroll
        for (int j = 0; j < 8; ++j) bias.v[j] = 0.f;
        if (a.conv_bias != nullptr) bias = load8(a.conv_bias + c);
        if (TAPS > 0) {
#pragma unroll
            for (int i = 0; i < kWindow; ++i) {
                if (a.conv != nullptr) w[i] = load8(a.conv + i * nc + c);
                else for (int j = 0; j < 8; ++j) w[i].v[j] = 1.f;
                if (i + 1 < kWindow) x[i + 1] = input(t0 - (kWindow - 1) + i);
            }
        }
        T* out = static_cast<T*>(a.mixed) + static_cast<int64_t>(begin) * nc + c;
        const bool units = heads && a.rule == kDelta;
        auto emit = [&](int t, Vec8 y) {
#pragma unroll
            for (int j = 0; j < 8; ++j) y.v[j] = silu<T>(y.v[j]);
            const auto packed = pack8<T>(y);
            *reinterpret_cast<Packed8<T>*>(out + t * nc) = packed;
            if (!units) return;
            y = unpack8(packed);
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j) ss += y.v[j] * y.v[j];
            s_part[t - t0][threadIdx.x] = ss;
        };
        if (TAPS > 0) {
            for (int t = t0; t < t0 + n; t += kMixAhead) {
                Packed8<T> next[kMixAhead];
#pragma unroll
                for (int e = 0; e < kMixAhead; ++e)
                    next[e] = *reinterpret_cast<const Packed8<T>*>(in + min(t + e, t0 + n - 1) * a.joint_ld);
#pragma unroll
                for (int e = 0; e < kMixAhead; ++e) {
                    if (t + e >= t0 + n) break;
                    Vec8 y = bias;
#pragma unroll
                    for (int i = 0; i + 1 < kWindow; ++i) x[i] = x[i + 1];
                    x[kWindow - 1] = unpack8(next[e]);
#pragma unroll
                    for (int i = 0; i < kWindow; ++i)
#pragma unroll
                        for (int j = 0; j < 8; ++j) y.v[j] = fmaf(w[i].v[j], x[i].v[j], y.v[j]);
                    emit(t + e, y);
                }
            }
        } else {
            for (int t = t0; t < t0 + n; ++t) {
                Vec8 y = bias;
                for (int i = 0; i < taps; ++i) {
                    const Vec8 wi = load8(a.conv + i * nc + c), xi = input(t - (taps - 1) + i);
#pragma unroll
                    for (int j = 0; j < 8; ++j) y.v[j] = fmaf(wi.v[j], xi.v[j], y.v[j]);
                }
                emit(t, y);
            }
        }
        // (a request's first block is the only one that reads the ring)
        if (blockIdx.x == 0 && a.conv != nullptr)
            for (int r = max(0, ext - (taps - 1)); r < ext; ++r) store8(ring + (cached + r) % taps * nc, load8(in + r * a.joint_ld));
    }
    if (!heads || a.rule != kDelta) return;
    __syncthreads();
    const int here = min(heads_per_block, 2 * a.kv_heads - head0);
    for (int i = threadIdx.x; i < n * here; i += kMixThreads) {
        const int t = i / here, head = i - t * here;
        float ss = 0.f;
        for (int j = 0; j < per_head; ++j) ss += s_part[t][head * per_head + j];
        float f = rsqrtf(ss + kUnitEps);
        if (head0 + head >= a.kv_heads) f *= rsqrtf(static_cast<float>(a.dim));
        a.units[static_cast<int64_t>(begin + t0 + t) * 2 * a.kv_heads + head0 + head] = f;
    }
}

// ---- token by token: decode, and prompts that the chunked kernels do not take ------------

constexpr int kTapsAhead = 3;   // earlier inputs of a channel fetched together

// Grid: heads, requests, blocks of 4 << log_cols value columns (at most kStepThreads).
template <typename T, int RULE, bool DECODE, int AHEAD>
__global__ void __launch_bounds__(kStepThreads, 2)
step_kernel(const Recurrence a, int log_cols, bool finish) {
    extern __shared__ __align__(16) float smem[];
    __shared__ float s_ss[kStepThreads / 32], s_den[kStepThreads / 32];
    __shared__ float2 s_step;
    constexpr bool CONV = has_convolution(RULE);
    const int dk = a.padded_dim, vp = a.padded_value_dim;
    const int nv4 = 1 << log_cols, cols = nv4 * 4, groups = kStepThreads >> log_cols;
    float *s_v = smem, *s_k = s_v + cols, *s_q = s_k + dk, *s_red = s_q + dk, *s_n = s_red + kStepThreads * 4;   // s_n: kMemory
    const int h = blockIdx.x, b = blockIdx.y, col0 = blockIdx.z * cols;
    const int kvh = h / (a.heads / a.kv_heads);
    const int group = threadIdx.x >> log_cols, col = (threadIdx.x & (nv4 - 1)) * 4;
    const bool active = col0 + col < vp;
    const int64_t nv = values(a), nc = channels(a);
    const int64_t row_state = static_cast<int64_t>(a.table_idx[b]);
    // this thread's rows: group, group + groups, ...
    float* state = a.state + ((row_state * a.heads + h) * dk + group) * vp + col0 + col;
    const int rows = group < dk ? (dk - group + groups - 1) >> (31 - __clz(groups)) : 0, row_step = groups * vp;
    const int cached = a.cached[b];
    pdl_launch_dependents();
    float4 x[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
        x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (active && cached > 0 && i < rows) x[i] = load4(state + i * row_step);
    }
    // this CTA's channels: its value columns, the head's k and q
    const int own_v = min(cols, vp - col0), own = own_v + 2 * dk;
    auto channel = [&](int i) -> int64_t {
        if (i < own_v) return static_cast<int64_t>(h) * vp + col0 + i;
        i -= own_v;
        return nv + (i < dk ? static_cast<int64_t>(kvh) * dk + i : static_cast<int64_t>(a.kv_heads + kvh) * dk + i - dk);
    };
    auto place = [&](int i) -> float& { return i < own_v ? s_v[i] : s_k[i - own_v]; };   // (s_q follows s_k)
    T* ring = CONV ? static_cast<T*>(a.conv_state) + row_state * a.taps * nc : nullptr;
    const int now = DECODE && CONV ? cached % a.taps : 0;
    const bool steps = threadIdx.x == kStepThreads - 1;   // this thread works out the step
    float step_bias = 0.f, decay = 0.f, norm = 0.f, top = 0.f;   // top: the running maximum of kMemory
    if (RULE == kMemory) {   // (a thread works on the same elements of n all the way)
        const float* memory = memory_of(a, row_state, h, col0);
        for (int i = threadIdx.x; i < dk; i += kStepThreads) s_n[i] = cached > 0 ? memory[i] : 0.f;
        if (cached > 0) top = memory[dk];
    }
    if (DECODE && !CONV) {
        if (steps && RULE == kMemory) step_bias = a.step_bias[h], decay = a.step_bias[a.heads + h];
        if (steps && RULE == kLightning) decay = a.decay_log[h];
        if (finish && threadIdx.x < own_v) norm = to_f32(static_cast<const T*>(a.norm)[static_cast<int64_t>(h) * vp + threadIdx.x]);
    }
    if constexpr (DECODE && CONV) {
        // what the inputs before this one add to the channels, two of them at a time
        for (int i0 = threadIdx.x; i0 < own; i0 += 2 * kStepThreads) {
            float y[2] = {0.f, 0.f}, w[2][kTapsAhead], in[2][kTapsAhead];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int i = i0 + e * kStepThreads;
                const int64_t c = channel(i < own ? i : 0);
                if (a.conv_bias != nullptr) y[e] = a.conv_bias[c];
#pragma unroll
                for (int m = 0; m < kTapsAhead; ++m) {
                    const bool there = m + 1 < a.taps && cached > m;
                    const int slot = now - 1 - m + (now - 1 - m < 0 ? a.taps : 0);
                    w[e][m] = there ? a.conv[(a.taps - 2 - m) * nc + c] : 0.f;
                    in[e][m] = there ? to_f32(ring[slot * nc + c]) : 0.f;
                }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int i = i0 + e * kStepThreads;
                if (i >= own) continue;
                const int64_t c = channel(i);
                for (int m = a.taps - 2; m >= kTapsAhead; --m)
                    if (cached > m) y[e] = fmaf(a.conv[(a.taps - 2 - m) * nc + c], to_f32(ring[(cached - 1 - m) % a.taps * nc + c]), y[e]);
#pragma unroll
                for (int m = kTapsAhead - 1; m >= 0; --m) y[e] = fmaf(w[e][m], in[e][m], y[e]);
                place(i) = y[e];
            }
        }
        if (steps) {
            step_bias = a.step_bias[h];
            decay = a.decay_log[h];
        }
        if (finish && threadIdx.x < own_v) norm = to_f32(static_cast<const T*>(a.norm)[threadIdx.x]);
    }
    const float skip = RULE == kStateSpace ? a.skip[h] : 0.f;
    pdl_wait_prior();
    const int begin = DECODE ? b : a.qo_indptr[b], end = DECODE ? b + 1 : a.qo_indptr[b + 1];
    for (int64_t t = begin; t < end; ++t) {
        const T* row = static_cast<const T*>(a.joint) + t * a.joint_ld;
        float2 step;
        float gate = 0.f;
        if (DECODE) {
            const T* tail = row + nv + nc;
            float za = 0.f, zb = 0.f;
            if (steps) {
                if (RULE != kLightning) za = to_f32(tail[h]);
                if (RULE == kDelta || RULE == kMemory) zb = to_f32(tail[a.heads + h]);
            }
            if (finish && threadIdx.x < own_v) gate = to_f32(row[static_cast<int64_t>(h) * vp + threadIdx.x]);
            T* keep = CONV ? ring + static_cast<int64_t>(now) * nc : nullptr;
            const bool keeps = h % (a.heads / a.kv_heads) == 0 && blockIdx.z == 0;   // k and q are shared
            if constexpr (!CONV) {
                for (int i = threadIdx.x; i < own; i += kStepThreads) {
                    const float x = to_f32(row[nv + channel(i)]);
                    place(i) = RULE == kLightning ? to_f32(from_f32<T>(silu<T>(x))) : x;
                }
            } else {
                for (int i0 = threadIdx.x; i0 < own; i0 += 2 * kStepThreads) {
                    T in[2];
                    float w[2];
    #pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int i = i0 + e * kStepThreads;
                        const int64_t c = channel(i < own ? i : 0);
                        in[e] = row[nv + c];
                        w[e] = a.conv[(a.taps - 1) * nc + c];
                    }
    #pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int i = i0 + e * kStepThreads;
                        if (i >= own) continue;
                        place(i) = to_f32(from_f32<T>(silu<T>(fmaf(w[e], to_f32(in[e]), place(i)))));
                        if (i < own_v || keeps) keep[channel(i)] = in[e];
                    }
                }
            }
            if (steps) s_step = make_step(RULE, za, zb, step_bias, decay, a.gate_cap);
        } else {
            const T* mixed = mixed_rows<T>(a) + t * mixed_ld(a);
            for (int i = threadIdx.x; i < own; i += kStepThreads) place(i) = to_f32(mixed[channel(i)]);
            step = reinterpret_cast<const float2*>(a.steps)[t * a.heads + h];
        }
        __syncthreads();
        if (DECODE) step = s_step;
        float kf = step.y, qf = 1.f;   // factors of k and q
        float g = exp2f(step.x);
        if (RULE == kMemory) {
            const float next = fmaxf(step.x + top, step.y);
            g = exp2f(step.x + top - next);
            kf = exp2f(step.y - next);
            qf = rsqrtf(static_cast<float>(a.dim));
            top = next;
            float den = 0.f;
            for (int i = threadIdx.x; i < dk; i += kStepThreads) {
                const float n = fmaf(kf, s_k[i], g * s_n[i]);
                s_n[i] = n;
                den = fmaf(n, s_q[i], den);
            }
            den = warp_sum(den);
            if ((threadIdx.x & 31) == 0) s_den[threadIdx.x >> 5] = den;   // (published by the barrier below)
        }
        if (RULE == kDelta) {
            if (DECODE) {
                const int lane = threadIdx.x & 31;
                float sk = 0.f, sq = 0.f;
                for (int i = lane; i < dk; i += 32) {
                    sk += s_k[i] * s_k[i];
                    sq += s_q[i] * s_q[i];
                }
                kf = rsqrtf(warp_sum(sk) + kUnitEps);
                qf = rsqrtf(warp_sum(sq) + kUnitEps) * rsqrtf(static_cast<float>(a.dim));
            } else {
                kf = a.units[t * 2 * a.kv_heads + kvh];
                qf = a.units[t * 2 * a.kv_heads + a.kv_heads + kvh];
            }
        }
        float4 u = active ? *reinterpret_cast<const float4*>(s_v + col) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (RULE == kDelta) {
            float4 p = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < AHEAD; ++i) {
                if (i < rows) {
                    const float k = s_k[group + i * groups];
                    p.x = fmaf(k, x[i].x, p.x);
                    p.y = fmaf(k, x[i].y, p.y);
                    p.z = fmaf(k, x[i].z, p.z);
                    p.w = fmaf(k, x[i].w, p.w);
                }
            }
            *reinterpret_cast<float4*>(s_red + group * cols + col) = p;
            __syncthreads();
            p = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int i = 0; i < groups; ++i) {
                const float4 y = load4(s_red + i * cols + col);
                p.x += y.x;
                p.y += y.y;
                p.z += y.z;
                p.w += y.w;
            }
            const float f = g * kf;
            u = make_float4(step.y * (u.x - f * p.x), step.y * (u.y - f * p.y), step.y * (u.z - f * p.z), step.y * (u.w - f * p.w));
            __syncthreads();
        }
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (i < rows) {
                const float k = kf * s_k[group + i * groups], q = s_q[group + i * groups];
                x[i].x = fmaf(k, u.x, g * x[i].x);
                x[i].y = fmaf(k, u.y, g * x[i].y);
                x[i].z = fmaf(k, u.z, g * x[i].z);
                x[i].w = fmaf(k, u.w, g * x[i].w);
                o.x = fmaf(q, x[i].x, o.x);
                o.y = fmaf(q, x[i].y, o.y);
                o.z = fmaf(q, x[i].z, o.z);
                o.w = fmaf(q, x[i].w, o.w);
                if (DECODE && active) *reinterpret_cast<float4*>(state + i * row_step) = x[i];
            }
        }
        *reinterpret_cast<float4*>(s_red + group * cols + col) = o;
        __syncthreads();
        T* out = static_cast<T*>(a.out) + t * a.out_ld + static_cast<int64_t>(h) * vp + col0;
        const int c = threadIdx.x;
        float y = 0.f;
        if (c < own_v) {
            for (int i = 0; i < groups; ++i) y += s_red[i * cols + c];
            y *= qf;
            if (RULE == kMemory) {
                float den = 0.f;
#pragma unroll
                for (int i = 0; i < kStepThreads / 32; ++i) den += s_den[i];
                y /= fmaxf(fabsf(den * qf), exp2f(-top)) + kMemoryEps;
            }
            if (RULE == kStateSpace) y = fmaf(skip, s_v[c], y);
            if (!finish) out[c] = from_f32<T>(y);
        }
        if (DECODE && (RULE == kDelta || RULE == kMemory) && finish) {   // the whole head is here: norm and gate
            const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
            float ss = warp_sum(y * y);
            if (lane == 0) s_ss[warp] = ss;
            __syncthreads();
            ss = warp_sum(lane < kStepThreads / 32 ? s_ss[lane] : 0.f);
            const float scale = rsqrtf(ss / static_cast<float>(a.value_dim) + a.eps) * a.out_scale;
            if (c < own_v) out[c] = from_f32<T>(y * scale * norm * (RULE == kMemory ? sigmoid<T>(gate) : silu<T>(gate)));
        }
        if (!DECODE) __syncthreads();   // everything in shared memory has been used
    }
    if (RULE == kMemory && begin < end) {
        const int each = memory_columns(dk);
        for (int at = col0; at < min(col0 + cols, vp); at += each) {
            float* memory = memory_of(a, row_state, h, at);
            for (int i = threadIdx.x; i < dk; i += kStepThreads) memory[i] = s_n[i];
            if (threadIdx.x == 0) memory[dk] = top;
        }
    }
    if (DECODE || !active || begin >= end) return;
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (i < rows) *reinterpret_cast<float4*>(state + i * row_step) = x[i];
}

// ---- norm and gate of raw outputs, in place ------------------------------------------------

// Delta rule, and matrix memory normed by head: one warp per (token, head), four elements per lane in registers (more, for
// wide heads, read again).  The first has one norm for all heads, the second one of all heads' size.
constexpr int kFinishWarps = 8;

template <typename T>
__global__ void __launch_bounds__(kFinishWarps * 32)
finish_heads_kernel(const Recurrence a) {
    const int lane = threadIdx.x & 31, vp = a.padded_value_dim;
    const unsigned row = blockIdx.x * kFinishWarps + (threadIdx.x >> 5);
    pdl_launch_dependents();
    pdl_wait_prior();
    if (row >= static_cast<unsigned>(a.tokens) * a.heads) return;
    const int64_t t = row / a.heads;
    const int h = static_cast<int>(row - t * a.heads), c0 = lane * 4;
    T* out = static_cast<T*>(a.out) + t * a.out_ld + static_cast<int64_t>(h) * vp;
    const T* gate = static_cast<const T*>(a.joint) + t * a.joint_ld + static_cast<int64_t>(h) * vp;
    const bool memory = a.rule == kMemory;
    const T* norm = static_cast<const T*>(a.norm) + (memory ? static_cast<int64_t>(h) * vp : 0);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f), g = o, w = o;
    if (c0 < vp) {
        o = load4(out + c0);
        g = load4(gate + c0);
        w = load4(norm + c0);
    }
    float ss = o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;
    for (int c = c0 + 128; c < vp; c += 128) {
        const float4 y = load4(out + c);
        ss += y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
    }
    const float scale = rsqrtf(warp_sum(ss) / static_cast<float>(a.value_dim) + a.eps) * a.out_scale;
    auto emit = [&](int c, const float4& y, const float4& z, const float4& n) {
        auto open = [&](float x) { return memory ? sigmoid<T>(x) : silu<T>(x); };
        store4(out + c, make_float4(y.x * scale * n.x * open(z.x), y.y * scale * n.y * open(z.y), y.z * scale * n.z * open(z.z),
                                    y.w * scale * n.w * open(z.w)));
    };
    if (c0 < vp) emit(c0, o, g, w);
    for (int c = c0 + 128; c < vp; c += 128) emit(c, load4(out + c), load4(gate + c), load4(norm + c));
}

// The others: one CTA per (token, part of the norm); the state space's gate comes before the norm, the others' behind it.
// A part is a run of the concatenated heads without their
// padding, so it may begin and end inside one; VEC elements at a time.
constexpr int kPartThreads = 128;
constexpr int kPartKeep = 4;   // pieces of VEC elements a thread keeps in registers

template <typename T, int VEC>
__global__ void __launch_bounds__(kPartThreads)
finish_parts_kernel(const Recurrence a) {
    __shared__ float red[kPartThreads / 32];
    pdl_launch_dependents();
    pdl_wait_prior();
    const int64_t t = blockIdx.x;
    const int per = a.heads * a.value_dim / a.norm_groups, from = blockIdx.y * per;
    T* out = static_cast<T*>(a.out) + t * a.out_ld;
    const T* gate = static_cast<const T*>(a.joint) + t * a.joint_ld;
    const T* norm = static_cast<const T*>(a.norm);
    const bool before = a.rule == kStateSpace;
    auto place = [&](int i) { return (from + i) / a.value_dim * a.padded_value_dim + (from + i) % a.value_dim; };
    auto gated = [&](int at, float (&y)[VEC]) {
        if (VEC == 8) {
            const Vec8 o = load8(out + at);
#pragma unroll
            for (int j = 0; j < VEC; ++j) y[j] = o.v[j & 7];
            if (!before) return;
            const Vec8 z = load8(gate + at);
#pragma unroll
            for (int j = 0; j < VEC; ++j) y[j] *= silu<T>(z.v[j & 7]);
        } else {
            y[0] = to_f32(out[at]);
            if (before) y[0] *= silu<T>(to_f32(gate[at]));
        }
    };
    float kept[kPartKeep][VEC], ss = 0.f;
#pragma unroll
    for (int i = 0; i < kPartKeep; ++i) {
        const int e = (threadIdx.x + i * kPartThreads) * VEC;
        if (e >= per) continue;
        gated(place(e), kept[i]);
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += kept[i][j] * kept[i][j];
    }
    for (int e = (threadIdx.x + kPartKeep * kPartThreads) * VEC; e < per; e += kPartThreads * VEC) {
        float y[VEC];
        gated(place(e), y);
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += y[j] * y[j];
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = warp_sum(lane < kPartThreads / 32 ? red[lane] : 0.f);
    const float scale = rsqrtf(ss / static_cast<float>(per) + a.eps) * a.out_scale;
    auto emit = [&](int at, const float (&y)[VEC]) {
        if (VEC == 8) {
            const Vec8 w = load8(norm + at);
            Vec8 o;
#pragma unroll
            for (int j = 0; j < 8; ++j) o.v[j] = y[j % VEC] * scale * w.v[j];
            if (!before) {
                const Vec8 z = load8(gate + at);
#pragma unroll
                for (int j = 0; j < 8; ++j) o.v[j] *= sigmoid<T>(z.v[j]);
            }
            store8(out + at, o);
        } else {
            out[at] = from_f32<T>(y[0] * scale * to_f32(norm[at]) * (before ? 1.f : sigmoid<T>(to_f32(gate[at]))));
        }
    };
#pragma unroll
    for (int i = 0; i < kPartKeep; ++i) {
        const int e = (threadIdx.x + i * kPartThreads) * VEC;
        if (e < per) emit(place(e), kept[i]);
    }
    for (int e = (threadIdx.x + kPartKeep * kPartThreads) * VEC; e < per; e += kPartThreads * VEC) {
        float y[VEC];
        gated(place(e), y);
        emit(place(e), y);
    }
}

// ---- chunked ---------------------------------------------------------------------------------

constexpr int kChunk = 64;            // tokens per chunk
constexpr int kPad = 8;               // bf16 elements behind every shared row (conflict-free ldmatrix)
constexpr int kTiles = 10;            // 16 x 16 tiles on and below the diagonal
constexpr int kMatrixVecs = kTiles * 2 * 32;   // uint4 per matrix: [tile][upper / lower part][lane]

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
// Chunk i of request b, which brings the tokens from `begin` on: numbers that no two requests share.
__device__ __forceinline__ int64_t chunk_number(int begin, int b, int i) { return begin / kChunk + b + i; }

// Sums of a chunk's decay logarithms over its tokens: the calling warp's lane holds those of tokens 2 lane and
// 2 lane + 1.
__device__ __forceinline__ float2 running_sums(float2 x) {
    const int lane = threadIdx.x & 31;
    float s = x.x + x.y;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += up;
    }
    return make_float2(s - x.y, s);
}

constexpr int kPrepareThreads = 128;
constexpr int kPrepareHeads = 4;   // heads per CTA
constexpr int kARow = kChunk + 4;
struct PrepareSmem {
    union {
        struct {
            __nv_bfloat16 k[kChunk * (64 + kPad)], q[kChunk * (64 + kPad)];   // 64 columns at a time
        };
        float a[2][kChunk * kARow];   // two heads' A, then their inverses
    };
    float sum[2][kChunk], weight[2][kChunk], kf[kChunk], qf[kChunk];
};

// Running maxima of a chunk's numbers, held like running_sums.
__device__ __forceinline__ float2 running_maxima(float2 x) {
    const int lane = threadIdx.x & 31;
    float s = fmaxf(x.x, x.y);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s = fmaxf(s, up);
    }
    const float before = __shfl_up_sync(0xffffffffu, s, 1);
    return make_float2(lane > 0 ? fmaxf(before, x.x) : x.x, s);
}
// A token that is not there writes nothing.
template <int RULE>
__device__ __forceinline__ float2 no_step() { return make_float2(0.f, RULE == kMemory ? -INFINITY : 0.f); }


// Barrier of the two warps that work on one head.
__device__ __forceinline__ void pair_sync() {
    if (threadIdx.x < 64) asm volatile("bar.sync 1, 64;" ::: "memory");
    else asm volatile("bar.sync 2, 64;" ::: "memory");
}

// (I + A)^-1 of the 32 x 32 block at `a`, in its place: a column per lane, by forward substitution.
__device__ __forceinline__ void invert_block(float* a) {
    constexpr int N = kChunk / 2;
    const int lane = threadIdx.x & 31;
    float x[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {
        float acc[4] = {i == lane ? 1.f : 0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int s = 0; s < i; s += 4) {
            const float4 r = load4(a + i * kARow + s);
            acc[0] = fmaf(-r.x, x[s], acc[0]);
            if (s + 1 < i) acc[1] = fmaf(-r.y, x[s + 1], acc[1]);
            if (s + 2 < i) acc[2] = fmaf(-r.z, x[s + 2], acc[2]);
            if (s + 3 < i) acc[3] = fmaf(-r.w, x[s + 3], acc[3]);
        }
        x[i] = (acc[0] + acc[1]) + (acc[2] + acc[3]);
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < N; ++i) a[i * kARow + lane] = x[i];
}

// 16 rows of a product of 32 x 32 blocks in shared memory, every factor as the sum of two bf16 numbers.
__device__ __forceinline__ void multiply_block(float (&acc)[4][4], const float* left, const float* right) {
    const int lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int kt = 0; kt < 2; ++kt) {
        uint32_t ah[4], al[4];
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            const float2 v = *reinterpret_cast<const float2*>(left + (g + (p & 1) * 8) * kARow + kt * 16 + (p >> 1) * 8 + 2 * tq);
            split2(v.x, v.y, ah[p], al[p]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            uint32_t bh[2], bl[2];
#pragma unroll
            for (int p = 0; p < 2; ++p) {
                const float* r = right + (kt * 16 + p * 8 + 2 * tq) * kARow + j * 8 + g;
                split2(r[0], r[kARow], bh[p], bl[p]);
            }
            mma_bf16_16816(acc[j], ah, bh[0], bh[1]);
            mma_bf16_16816(acc[j], al, bh[0], bh[1]);
            mma_bf16_16816(acc[j], ah, bl[0], bl[1]);
        }
    }
}

// (I + A)^-1 of a head's chunk, in the place of A, by the pair of warps that works on it: the diagonal blocks by
// substitution, the block below them as -inverse(lower) A inverse(upper).
__device__ __forceinline__ void invert_chunk(float* a, int half) {
    constexpr int N = kChunk / 2;
    const int lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
    float *upper = a, *lower = a + N * kARow + N, *below = a + N * kARow, *spare = a + N;
    auto put = [&](float* to, const float (&acc)[4][4], float sign) {
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int p = 0; p < 2; ++p)
                *reinterpret_cast<float2*>(to + (half * 16 + g + p * 8) * kARow + j * 8 + 2 * tq) =
                    make_float2(sign * acc[j][2 * p], sign * acc[j][2 * p + 1]);
    };
    invert_block(half ? lower : upper);
    pair_sync();
    float acc[4][4];
    multiply_block(acc, below + half * 16 * kARow, upper);
    put(spare, acc, 1.f);
    pair_sync();
    multiply_block(acc, lower + half * 16 * kARow, spare);
    put(below, acc, -1.f);
    pair_sync();
}

// Grid: chunks of the longest request, k / q heads times the parts that their heads are dealt with in, requests.
template <int RULE>
__global__ void __launch_bounds__(kPrepareThreads, 4)
prepare_kernel(const Recurrence a, int parts) {
    extern __shared__ __align__(16) uint8_t smem_raw[];
    PrepareSmem& S = *reinterpret_cast<PrepareSmem*>(smem_raw);
    constexpr int ROW = 64 + kPad, kMatrices = RULE == kDelta ? 2 : 1;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, r8 = lane & 7;
    pdl_launch_dependents();
    pdl_wait_prior();
    const int b = blockIdx.z, kvh = blockIdx.y / parts, begin = a.qo_indptr[b], ext = a.qo_indptr[b + 1] - begin;
    const int s0 = blockIdx.x * kChunk;
    if (s0 >= ext) return;
    const int n = min(kChunk, ext - s0);
    const int64_t nc = mixed_ld(a), first = begin + s0;
    const __nv_bfloat16* k0 = mixed_rows<__nv_bfloat16>(a) + first * nc + values(a) + static_cast<int64_t>(kvh) * a.padded_dim;
    const int64_t to_q = static_cast<int64_t>(a.kv_heads) * a.padded_dim;
    if (threadIdx.x < kChunk) {
        float kf = 1.f, qf = 1.f;
        if (RULE == kDelta && threadIdx.x < n) {
            kf = a.units[(first + threadIdx.x) * 2 * a.kv_heads + kvh];
            qf = a.units[(first + threadIdx.x) * 2 * a.kv_heads + a.kv_heads + kvh];
        }
        S.kf[threadIdx.x] = kf;
        S.qf[threadIdx.x] = qf;
    }
    // ---- k . k and q . k of this warp's 16 rows ----
    float kk[8][4] = {}, qk[8][4] = {};
    for (int d0 = 0; d0 < a.padded_dim; d0 += 64) {
        if (d0 > 0) __syncthreads();
        for (int i = threadIdx.x; i < kChunk * 8; i += kPrepareThreads) {
            const int t = i >> 3, c = (i & 7) * 8;
            const __nv_bfloat16* row = k0 + (t < n ? t : 0) * nc + d0 + c;
            cp_async16(smem_u32(&S.k[t * ROW + c]), row, t < n);
            cp_async16(smem_u32(&S.q[t * ROW + c]), row + to_q, t < n);
        }
        cp_async_wait_all();
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            uint32_t ak[4], aq[4], b0, b1, b2, b3;
            const int aoff = (warp * 16 + (mi & 1) * 8 + r8) * ROW + ks * 16 + (mi >> 1) * 8;
            ldmatrix_x4(smem_u32(&S.q[aoff]), aq[0], aq[1], aq[2], aq[3]);
            if (RULE == kDelta) ldmatrix_x4(smem_u32(&S.k[aoff]), ak[0], ak[1], ak[2], ak[3]);
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) {
                if (kt > warp) continue;
                ldmatrix_x4(smem_u32(&S.k[(kt * 16 + (mi >> 1) * 8 + r8) * ROW + ks * 16 + (mi & 1) * 8]), b0, b1, b2, b3);
                mma_bf16_16816(qk[2 * kt], aq, b0, b1);
                mma_bf16_16816(qk[2 * kt + 1], aq, b2, b3);
                if (RULE == kDelta) {
                    mma_bf16_16816(kk[2 * kt], ak, b0, b1);
                    mma_bf16_16816(kk[2 * kt + 1], ak, b2, b3);
                }
            }
        }
    }
    // ---- per head: P and, two heads at a time, the inverse ----
    const int group = a.heads / a.kv_heads, part = blockIdx.y % parts;
    const int from = part * kPrepareHeads, to = min(group, from + kPrepareHeads);
    uint4* chunks = static_cast<uint4*>(a.chunks) + chunk_number(begin, b, blockIdx.x) * a.heads * kMatrices * kMatrixVecs;
    for (int h0 = from; h0 < to; h0 += 2) {
        __syncthreads();
        if ((warp & 1) == 0 && h0 + (warp >> 1) < to) {
            const int h = kvh * group + h0 + (warp >> 1);
            const float2* steps = reinterpret_cast<const float2*>(a.steps) + first * a.heads + h;
            const float2 none = no_step<RULE>();
            const float2 x = 2 * lane < n ? steps[static_cast<int64_t>(2 * lane) * a.heads] : none;
            const float2 y = 2 * lane + 1 < n ? steps[static_cast<int64_t>(2 * lane + 1) * a.heads] : none;
            const float2 B = running_sums(make_float2(x.x, y.x));
            if (RULE == kMemory) {   // the exponent of P_ts is weight_s - sum_t: sum holds the maxima here
                const float2 e = make_float2(x.y - B.x, y.y - B.y);
                *reinterpret_cast<float2*>(&S.sum[warp >> 1][2 * lane]) = running_maxima(e);
                *reinterpret_cast<float2*>(&S.weight[warp >> 1][2 * lane]) = e;
            } else {
                *reinterpret_cast<float2*>(&S.sum[warp >> 1][2 * lane]) = B;
                *reinterpret_cast<float2*>(&S.weight[warp >> 1][2 * lane]) = make_float2(x.y, y.y);
            }
        }
        __syncthreads();
#pragma unroll
        for (int hp = 0; hp < 2; ++hp) {
            if (h0 + hp >= to) continue;
            uint4* out = chunks + (static_cast<int64_t>(kvh * group + h0 + hp) * kMatrices) * kMatrixVecs + lane;
            const int t0 = warp * 16 + g;
            const float sum_t[2] = {S.sum[hp][t0], S.sum[hp][t0 + 8]};
            float q_t[2] = {1.f, 1.f}, k_t[2] = {0.f, 0.f}, row_sum[2] = {0.f, 0.f};
            if (RULE == kMemory) q_t[0] = q_t[1] = rsqrtf(static_cast<float>(a.dim));
            if (RULE == kDelta) {
                q_t[0] = S.qf[t0];
                q_t[1] = S.qf[t0 + 8];
                k_t[0] = S.kf[t0] * S.weight[hp][t0];
                k_t[1] = S.kf[t0 + 8] * S.weight[hp][t0 + 8];
            }
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) {
                if (kt > warp) continue;
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int side = 0; side < 2; ++side) {
                    const int s = kt * 16 + side * 8 + 2 * tq;
                    const float2 sum_s = *reinterpret_cast<const float2*>(&S.sum[hp][s]);
                    const float2 f_s = RULE == kDelta ? *reinterpret_cast<const float2*>(&S.kf[s])
                                                      : *reinterpret_cast<const float2*>(&S.weight[hp][s]);
                    float2 am[2];
#pragma unroll
                    for (int half = 0; half < 2; ++half) {   // rows g, g + 8
                        const int t = t0 + half * 8, tile = 2 * kt + side;
                        float rx, ry;
                        if (RULE == kMemory) {
                            rx = s <= t ? ex2(f_s.x - sum_t[half]) : 0.f;
                            ry = s + 1 <= t ? ex2(f_s.y - sum_t[half]) : 0.f;
                            row_sum[half] += qk[tile][2 * half] * (rx * q_t[half]) + qk[tile][2 * half + 1] * (ry * q_t[half]);
                        } else {
                            rx = (s <= t ? ex2(sum_t[half] - sum_s.x) : 0.f) * f_s.x;
                            ry = (s + 1 <= t ? ex2(sum_t[half] - sum_s.y) : 0.f) * f_s.y;
                        }
                        split2(qk[tile][2 * half] * (rx * q_t[half]), qk[tile][2 * half + 1] * (ry * q_t[half]), hi[2 * side + half],
                               lo[2 * side + half]);
                        am[half] = make_float2(s < t ? kk[tile][2 * half] * (rx * k_t[half]) : 0.f,
                                               s + 1 < t ? kk[tile][2 * half + 1] * (ry * k_t[half]) : 0.f);
                    }
                    if (RULE == kDelta) {
                        *reinterpret_cast<float2*>(&S.a[hp][t0 * kARow + s]) = am[0];
                        *reinterpret_cast<float2*>(&S.a[hp][(t0 + 8) * kARow + s]) = am[1];
                    }
                }
                const int tile = warp * (warp + 1) / 2 + kt;
                out[tile * 64] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                out[tile * 64 + 32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
            if (RULE == kMemory) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    float r = row_sum[half];
                    r += __shfl_xor_sync(0xffffffffu, r, 1);
                    r += __shfl_xor_sync(0xffffffffu, r, 2);
                    if (tq == 0 && t0 + half * 8 < n) a.units[(first + t0 + half * 8) * a.heads + kvh * group + h0 + hp] = r;
                }
            }
        }
        if (RULE != kDelta) continue;
        __syncthreads();
        const int hp = warp >> 1;
        if (h0 + hp >= to) continue;   // (both warps of the pair)
        float* m = S.a[hp];
        invert_chunk(m, warp & 1);
        uint4* out = chunks + (static_cast<int64_t>(kvh * group + h0 + hp) * kMatrices + 1) * kMatrixVecs + lane;
        // tiles of the pair's warps: rows 0 and 3, rows 1 and 2
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int mt = (warp & 1) == 0 ? i * 3 : 1 + i;
            for (int kt = 0; kt <= mt; ++kt) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int part = 0; part < 4; ++part) {
                    const float2 v = *reinterpret_cast<const float2*>(m + (mt * 16 + g + (part & 1) * 8) * kARow + kt * 16 +
                                                                      (part >> 1) * 8 + 2 * tq);
                    split2(v.x, v.y, hi[part], lo[part]);
                }
                const int tile = mt * (mt + 1) / 2 + kt;
                out[tile * 64] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                out[tile * 64 + 32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
        }
    }
}

// An 8 x 8 matrix of bf16 pairs, one per lane, transposed across the warp.
__device__ __forceinline__ uint32_t transpose_8x8(uint32_t x) {
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}

constexpr int kWalkThreads = 256;
constexpr int kSlice = 64;            // value columns per CTA, 16 per pair of warps

template <int DK, int RULE>
struct WalkSmem {
    static constexpr int kRow = DK + kPad, kVRow = kSlice + kPad;
    __nv_bfloat16 k[2][kChunk * kRow], q[2][kChunk * kRow], v[2][kChunk * kVRow];   // this chunk's and the next one's
    uint4 m[2][(RULE == kDelta ? 2 : 1) * kMatrixVecs];   // P and inverse
    // what the warps of a pair hand to one another as left operands, per 16 tokens upper and lower parts:
    // beta (V - G K S), U, U as it enters the state
    uint4 hand[RULE == kDelta ? 3 : 1][kSlice / 16][RULE == kDelta ? 4 : 1][2][32];
    // and what a warp's state rows add to the other one's tokens: [pair][warp][token tile][Q S, K S][8 tokens]
    float4 sums[kSlice / 16][2][2][RULE == kDelta ? 2 : 1][2][32];
    float out[2][kChunk];      // G_t times q's factor
    float beta[2][kChunk], read[2][kChunk];   // beta_t; beta_t G_t times k's factor
    float write[2][kChunk];    // exp(B_n - B_t) times k's factor (or times dt)
    float keep[2];             // G_n
    // matrix memory: factors of P V, exp(-m_t), what the chunk's tokens add to n . q; n; one over the denominator
    float own[RULE == kMemory ? 2 : 1][kChunk], floor[RULE == kMemory ? 2 : 1][kChunk], row_sum[RULE == kMemory ? 2 : 1][kChunk];
    float n[RULE == kMemory ? DK : 4], over[RULE == kMemory ? kChunk : 4];
};

// Grid: slices of 64 value columns, heads, requests.  All products are formed transposed, 16 value columns by tokens (or
// by state rows), so that what one leaves in a warp's accumulators is the next one's left operand where it is.  Two
// warps share 16 columns: each keeps half of the state rows and works out the results of half of the tokens (tiles 0
// and 3, tiles 1 and 2).
template <int DK, int RULE>
__global__ void __launch_bounds__(kWalkThreads, 1)
chunk_kernel(const Recurrence a) {
    using Smem = WalkSmem<DK, RULE>;
    constexpr int ROW = Smem::kRow, VROW = Smem::kVRow, kMatrices = RULE == kDelta ? 2 : 1;
    extern __shared__ __align__(16) uint8_t smem_raw[];
    Smem& S = *reinterpret_cast<Smem*>(smem_raw);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, tq = lane & 3, mi = lane >> 3, r8 = lane & 7;
    const int h = blockIdx.y, req = blockIdx.z, v0 = blockIdx.x * kSlice, pair = warp >> 1, half = warp & 1, col0 = pair * 16;
    const int vp = a.padded_value_dim, kvh = h / (a.heads / a.kv_heads);
    const int own[4] = {half, 3 - half, 1 - half, 2 + half};   // this warp's 16-token tiles, then the other one's
    constexpr int kRows = DK / 2;                              // state rows per warp
    pdl_launch_dependents();
    pdl_wait_prior();
    const int begin = a.qo_indptr[req], ext = a.qo_indptr[req + 1] - begin;
    if (ext <= 0) return;
    const int64_t nc = mixed_ld(a);
    const __nv_bfloat16* mixed = mixed_rows<__nv_bfloat16>(a) + begin * nc;
    const int64_t at_k = values(a) + static_cast<int64_t>(kvh) * DK, to_q = static_cast<int64_t>(a.kv_heads) * DK;
    const int64_t at_v = static_cast<int64_t>(h) * vp + v0;

    auto load_chunk = [&](int s0, int buf) {
        const int n = min(kChunk, ext - s0);
        for (int i = threadIdx.x; i < kChunk * (DK / 8); i += kWalkThreads) {
            const int t = i / (DK / 8), c = (i % (DK / 8)) * 8;
            const __nv_bfloat16* row = mixed + static_cast<int64_t>(t < n ? s0 + t : s0) * nc + at_k + c;
            cp_async16(smem_u32(&S.k[buf][t * ROW + c]), row, t < n);
            cp_async16(smem_u32(&S.q[buf][t * ROW + c]), row + to_q, t < n);
        }
        for (int i = threadIdx.x; i < kChunk * (kSlice / 8); i += kWalkThreads) {
            const int t = i / (kSlice / 8), c = (i % (kSlice / 8)) * 8;
            cp_async16(smem_u32(&S.v[buf][t * VROW + c]), mixed + static_cast<int64_t>(t < n ? s0 + t : s0) * nc + at_v + c, t < n);
        }
    };
    // Factors of a chunk's tokens: the first warp fetches them a chunk ahead and works them out behind it.
    float2 st0, st1, un0, un1;
    auto fetch_factors = [&](int s0) {
        const int n = min(kChunk, ext - s0);
        const float2* steps = reinterpret_cast<const float2*>(a.steps) + static_cast<int64_t>(begin + s0) * a.heads + h;
        st0 = st1 = no_step<RULE>();
        un0 = un1 = make_float2(1.f, 1.f);
        auto sum_of = [&](int t) { return make_float2(a.units[static_cast<int64_t>(begin + s0 + t) * a.heads + h], 0.f); };
        auto unit = [&](int t) {
            const float* u = a.units + static_cast<int64_t>(begin + s0 + t) * 2 * a.kv_heads + kvh;
            return make_float2(u[0], u[a.kv_heads]);
        };
        if (2 * lane < n) {
            st0 = steps[static_cast<int64_t>(2 * lane) * a.heads];
            if (RULE == kDelta) un0 = unit(2 * lane);
            if (RULE == kMemory) un0 = sum_of(2 * lane);
        }
        if (2 * lane + 1 < n) {
            st1 = steps[static_cast<int64_t>(2 * lane + 1) * a.heads];
            if (RULE == kDelta) un1 = unit(2 * lane + 1);
            if (RULE == kMemory) un1 = sum_of(2 * lane + 1);
        }
    };
    float top = 0.f;   // the matrix memory's running maximum (first warp)
    auto put_factors = [&](int buf) {
        const float2 B = running_sums(make_float2(st0.x, st1.x));
        const float last = __shfl_sync(0xffffffffu, B.y, 31);
        if constexpr (RULE == kMemory) {
            const float2 e = make_float2(st0.y - B.x, st1.y - B.y), c = running_maxima(e);
            const float c_n = __shfl_sync(0xffffffffu, c.y, 31), qf = rsqrtf(static_cast<float>(a.dim));
            const float r0 = fmaxf(top, c.x), r1 = fmaxf(top, c.y), r = fmaxf(top, c_n);
            auto put = [&](float* to, float x, float y) { *reinterpret_cast<float2*>(to + 2 * lane) = make_float2(x, y); };
            put(S.out[buf], ex2(top - r0) * qf, ex2(top - r1) * qf);
            put(S.own[buf], ex2(c.x - r0), ex2(c.y - r1));
            put(S.floor[buf], ex2(-(B.x + r0)), ex2(-(B.y + r1)));
            put(S.row_sum[buf], un0.x, un1.x);
            put(S.write[buf], ex2(e.x - r), ex2(e.y - r));
            if (lane == 0) S.keep[buf] = ex2(top - r);
            top = last + r;
            return;
        }
        const float g0 = ex2(B.x), g1 = ex2(B.y), w0 = ex2(last - B.x), w1 = ex2(last - B.y);
        *reinterpret_cast<float2*>(&S.out[buf][2 * lane]) = make_float2(g0 * un0.y, g1 * un1.y);
        if (RULE == kDelta) {
            *reinterpret_cast<float2*>(&S.beta[buf][2 * lane]) = make_float2(st0.y, st1.y);
            *reinterpret_cast<float2*>(&S.read[buf][2 * lane]) = make_float2(st0.y * g0 * un0.x, st1.y * g1 * un1.x);
            *reinterpret_cast<float2*>(&S.write[buf][2 * lane]) = make_float2(w0 * un0.x, w1 * un1.x);
        } else {
            *reinterpret_cast<float2*>(&S.write[buf][2 * lane]) = make_float2(w0 * st0.y, w1 * st1.y);
        }
        if (lane == 0) S.keep[buf] = ex2(last);
    };
    const uint4* chunks = static_cast<const uint4*>(a.chunks) + (chunk_number(begin, req, 0) * a.heads + h) * kMatrices * kMatrixVecs;
    const int64_t chunk_vecs = static_cast<int64_t>(a.heads) * kMatrices * kMatrixVecs;
    auto load_matrices = [&](const uint4* m, int buf) {
        for (int i = threadIdx.x; i < kMatrices * kMatrixVecs; i += kWalkThreads) cp_async16(smem_u32(&S.m[buf][i]), m + i, true);
    };
    load_chunk(0, 0);
    load_matrices(chunks, 0);

    // This warp's part of the state, transposed: tile j holds rows 8 j + 2 tq, + 1 of its half, of columns g and g + 8.
    float* state = a.state + ((static_cast<int64_t>(a.table_idx[req]) * a.heads + h) * DK + half * kRows) * vp + v0 + col0 + g;
    float st[kRows / 8][4];
    const bool fresh = a.cached[req] == 0;
#pragma unroll
    for (int j = 0; j < kRows / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[j][e] = fresh ? 0.f : state[static_cast<int64_t>(8 * j + 2 * tq + (e & 1)) * vp + (e >> 1) * 8];
    if constexpr (RULE == kMemory) {
        const float* memory = memory_of(a, a.table_idx[req], h, v0);
        for (int i = threadIdx.x; i < DK; i += kWalkThreads) S.n[i] = fresh ? 0.f : memory[i];
        if (!fresh) top = memory[DK];
    }
    if (warp == 0) {
        fetch_factors(0);
        put_factors(0);
    }
    const float skip = RULE == kStateSpace ? a.skip[h] : 0.f;

    // acc (16 columns by this warp's tokens) += X M^T for a lower triangular M, X as left operands of 16 tokens each
    // (neighbouring products go to different accumulators)
    auto multiply = [&](float (&acc)[2][2][4], const uint32_t (&xh)[4][4], const uint32_t (*xl)[4], const uint4* m) {
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
            uint4 hi[2], lo[2];
#pragma unroll
            for (int i = 0; i < 2; ++i)
                if (kt <= own[i]) {
                    hi[i] = m[(own[i] * (own[i] + 1) / 2 + kt) * 64 + lane];
                    lo[i] = m[(own[i] * (own[i] + 1) / 2 + kt) * 64 + 32 + lane];
                }
#pragma unroll
            for (int part = 0; part < 3; ++part) {
                if (part == 2 && xl == nullptr) continue;
#pragma unroll
                for (int i = 0; i < 2; ++i)
                    if (kt <= own[i]) {
                        const uint4 b = part == 1 ? lo[i] : hi[i];
                        mma_bf16_16816(acc[i][0], part == 2 ? xl[kt] : xh[kt], b.x, b.z);
                        mma_bf16_16816(acc[i][1], part == 2 ? xl[kt] : xh[kt], b.y, b.w);
                    }
            }
        }
    };
    // V^T of 16 tokens: token pairs 2 tq of columns g and g + 8, then eight tokens on
    auto values_of = [&](const __nv_bfloat16* V, int tile, uint32_t (&x)[4]) {
        ldmatrix_x4_trans(smem_u32(&V[(tile * 16 + (mi >> 1) * 8 + r8) * VROW + col0 + (mi & 1) * 8]), x[0], x[1], x[2], x[3]);
    };
    // accumulators of 16 tokens (tile, eight tokens further) as a left operand in two parts, for the pair
    auto hand_over = [&](int which, int tile, const float (&c)[2][4]) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int p = 0; p < 4; ++p) split2(c[p >> 1][(p & 1) * 2], c[p >> 1][(p & 1) * 2 + 1], hi[p], lo[p]);
        S.hand[which][pair][tile][0][lane] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        S.hand[which][pair][tile][1][lane] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    };
    auto take = [&](int which, int tile, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
        const uint4 x = S.hand[which][pair][tile][0][lane], y = S.hand[which][pair][tile][1][lane];
        hi[0] = x.x, hi[1] = x.y, hi[2] = x.z, hi[3] = x.w;
        lo[0] = y.x, lo[1] = y.y, lo[2] = y.z, lo[3] = y.w;
    };
    auto pair_barrier = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(1 + pair) : "memory"); };

    int buf = 0;
    for (int s0 = 0; s0 < ext; s0 += kChunk, buf ^= 1) {
        const int n = min(kChunk, ext - s0);
        const bool more = s0 + kChunk < ext;
        cp_async_wait_all();
        __syncthreads();   // this chunk and its factors are in place; nobody needs the last one's
        if (more) {
            chunks += chunk_vecs;
            load_chunk(s0 + kChunk, buf ^ 1);
            load_matrices(chunks, buf ^ 1);
            if (warp == 0) fetch_factors(s0 + kChunk);
        }
        const __nv_bfloat16 *K = S.k[buf], *Q = S.q[buf], *V = S.v[buf];
        if constexpr (RULE == kMemory) {
            // denominators of the chunk's tokens, four threads each; then n moves on, kParts threads per element
            constexpr int kEach = DK / 4;
            const int t = threadIdx.x >> 2, d0 = (threadIdx.x & 3) * kEach;
            float dot = 0.f;
#pragma unroll
            for (int d = 0; d < kEach; d += 8) {
                const Vec8 x = load8(Q + t * ROW + d0 + d);
#pragma unroll
                for (int j = 0; j < 8; ++j) dot = fmaf(x.v[j], S.n[d0 + d + j], dot);
            }
            dot += __shfl_xor_sync(0xffffffffu, dot, 1);
            dot += __shfl_xor_sync(0xffffffffu, dot, 2);
            if ((threadIdx.x & 3) == 0)
                S.over[t] = 1.f / (fmaxf(fabsf(fmaf(S.out[buf][t], dot, S.own[buf][t] * S.row_sum[buf][t])), S.floor[buf][t]) + kMemoryEps);
            __syncthreads();
            constexpr int kParts = kWalkThreads / DK;
            const int i = threadIdx.x / kParts, part = threadIdx.x % kParts;
            float sum = 0.f;
#pragma unroll 8
            for (int s = part; s < kChunk; s += kParts) sum = fmaf(S.write[buf][s], __bfloat162float(K[s * ROW + i]), sum);
#pragma unroll
            for (int o = 1; o < kParts; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            if (part == 0) S.n[i] = fmaf(S.keep[buf], S.n[i], sum);
        }
        // ---- S^T Q^T and S^T K^T ----
        float o[2][2][4], u[2][2][4];
        {
            float po[4][2][4] = {}, pu[4][2][4] = {};
#pragma unroll
            for (int ks = 0; ks < kRows / 16; ++ks) {
                uint32_t ah[4], al[4];
#pragma unroll
                for (int p = 0; p < 4; ++p)
                    split2(st[2 * ks + (p >> 1)][(p & 1) * 2], st[2 * ks + (p >> 1)][(p & 1) * 2 + 1], ah[p], al[p]);
#pragma unroll
                for (int i0 = 0; i0 < 4; i0 += 2) {
                    uint32_t bq[2][4], bk[2][4];
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const int off = (own[i0 + i] * 16 + (mi >> 1) * 8 + r8) * ROW + half * kRows + ks * 16 + (mi & 1) * 8;
                        ldmatrix_x4(smem_u32(&Q[off]), bq[i][0], bq[i][1], bq[i][2], bq[i][3]);
                        if (RULE == kDelta) ldmatrix_x4(smem_u32(&K[off]), bk[i][0], bk[i][1], bk[i][2], bk[i][3]);
                    }
#pragma unroll
                    for (int part = 0; part < 2; ++part) {
                        const uint32_t(&x)[4] = part == 0 ? ah : al;
#pragma unroll
                        for (int i = 0; i < 2; ++i) {
                            mma_bf16_16816(po[i0 + i][0], x, bq[i][0], bq[i][1]);
                            mma_bf16_16816(po[i0 + i][1], x, bq[i][2], bq[i][3]);
                            if (RULE == kDelta) {
                                mma_bf16_16816(pu[i0 + i][0], x, bk[i][0], bk[i][1]);
                                mma_bf16_16816(pu[i0 + i][1], x, bk[i][2], bk[i][3]);
                            }
                        }
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int side = 0; side < 2; ++side) {
                    const float *x = po[2 + i][side], *y = pu[2 + i][side];
                    S.sums[pair][half][i][0][side][lane] = make_float4(x[0], x[1], x[2], x[3]);
                    if (RULE == kDelta) S.sums[pair][half][i][RULE == kDelta ? 1 : 0][side][lane] = make_float4(y[0], y[1], y[2], y[3]);
                }
            pair_barrier();
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int side = 0; side < 2; ++side) {
                    const float4 x = S.sums[pair][half ^ 1][i][0][side][lane];
                    o[i][side][0] = po[i][side][0] + x.x;
                    o[i][side][1] = po[i][side][1] + x.y;
                    o[i][side][2] = po[i][side][2] + x.z;
                    o[i][side][3] = po[i][side][3] + x.w;
                    if (RULE == kDelta) {
                        const float4 y = S.sums[pair][half ^ 1][i][RULE == kDelta ? 1 : 0][side][lane];
                        u[i][side][0] = pu[i][side][0] + y.x;
                        u[i][side][1] = pu[i][side][1] + y.y;
                        u[i][side][2] = pu[i][side][2] + y.z;
                        u[i][side][3] = pu[i][side][3] + y.w;
                    }
                }
        }
        uint32_t xh[4][4], xl[4][4];
        if (RULE == kDelta) {
            // ---- U = (I + A)^-1 (beta V - beta G K S) ----
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                uint32_t x[4];
                values_of(V, own[i], x);
#pragma unroll
                for (int side = 0; side < 2; ++side) {
                    const int t = own[i] * 16 + side * 8 + 2 * tq;
                    const float2 be = *reinterpret_cast<const float2*>(&S.beta[buf][t]), rd = *reinterpret_cast<const float2*>(&S.read[buf][t]);
                    float* c = u[i][side];
                    c[0] = be.x * bf16_lo(x[2 * side]) - rd.x * c[0];
                    c[1] = be.y * bf16_hi(x[2 * side]) - rd.y * c[1];
                    c[2] = be.x * bf16_lo(x[2 * side + 1]) - rd.x * c[2];
                    c[3] = be.y * bf16_hi(x[2 * side + 1]) - rd.y * c[3];
                }
                hand_over(0, own[i], u[i]);
#pragma unroll
                for (int e = 0; e < 8; ++e) u[i][e >> 2][e & 3] = 0.f;
            }
            pair_barrier();
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) take(0, kt, xh[kt], xl[kt]);
            multiply(u, xh, xl, S.m[buf] + kMatrixVecs);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                hand_over(1, own[i], u[i]);
#pragma unroll
                for (int side = 0; side < 2; ++side) {
                    const float2 w = *reinterpret_cast<const float2*>(&S.write[buf][own[i] * 16 + side * 8 + 2 * tq]);
                    u[i][side][0] *= w.x;
                    u[i][side][1] *= w.y;
                    u[i][side][2] *= w.x;
                    u[i][side][3] *= w.y;
                }
                hand_over(2, own[i], u[i]);
            }
        } else {
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) values_of(V, kt, xh[kt]);
        }
        // ---- O = G Q S + P U (+ skip V) ----
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            uint32_t x[4];
            if (RULE == kStateSpace) values_of(V, own[i], x);
#pragma unroll
            for (int side = 0; side < 2; ++side) {
                const float2 f = *reinterpret_cast<const float2*>(&S.out[buf][own[i] * 16 + side * 8 + 2 * tq]);
                float* c = o[i][side];
                c[0] *= f.x;
                c[1] *= f.y;
                c[2] *= f.x;
                c[3] *= f.y;
                if (RULE == kStateSpace) {
                    c[0] = fmaf(skip, bf16_lo(x[2 * side]), c[0]);
                    c[1] = fmaf(skip, bf16_hi(x[2 * side]), c[1]);
                    c[2] = fmaf(skip, bf16_lo(x[2 * side + 1]), c[2]);
                    c[3] = fmaf(skip, bf16_hi(x[2 * side + 1]), c[3]);
                }
            }
        }
        if (RULE == kDelta) {
            pair_barrier();
#pragma unroll
            for (int kt = 0; kt < 4; ++kt) take(1, kt, xh[kt], xl[kt]);
        }
        if constexpr (RULE == kMemory) {
            float pv[2][2][4] = {};
            multiply(pv, xh, nullptr, S.m[buf]);
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int side = 0; side < 2; ++side) {
                    const int t = own[i] * 16 + side * 8 + 2 * tq;
                    const float2 f = *reinterpret_cast<const float2*>(&S.own[buf][t]), z = *reinterpret_cast<const float2*>(&S.over[t]);
                    float *c = o[i][side], *x = pv[i][side];
                    c[0] = fmaf(f.x, x[0], c[0]) * z.x;
                    c[1] = fmaf(f.y, x[1], c[1]) * z.y;
                    c[2] = fmaf(f.x, x[2], c[2]) * z.x;
                    c[3] = fmaf(f.y, x[3], c[3]) * z.y;
                }
        } else {
            multiply(o, xh, RULE == kDelta ? xl : nullptr, S.m[buf]);
        }
        {
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + static_cast<int64_t>(begin + s0) * a.out_ld + at_v + col0 + 2 * tq;
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int side = 0; side < 2; ++side) {
                    const float* c = o[i][side];
                    const uint32_t left = transpose_8x8(pack_bf16(c[0], c[1])), right = transpose_8x8(pack_bf16(c[2], c[3]));
                    const int t = own[i] * 16 + side * 8 + g;
                    if (t >= n) continue;
                    *reinterpret_cast<uint32_t*>(out + t * a.out_ld) = left;
                    *reinterpret_cast<uint32_t*>(out + t * a.out_ld + 8) = right;
                }
        }
        // ---- the state after the chunk ----
        const float keep = S.keep[buf];
#pragma unroll
        for (int j = 0; j < kRows / 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) st[j][e] *= keep;
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
            if (kt * 16 >= n) continue;
            uint32_t wh[4], wl[4];
            if (RULE == kDelta) {
                take(2, kt, wh, wl);
            } else {
#pragma unroll
                for (int p = 0; p < 4; ++p) {
                    const float2 w = *reinterpret_cast<const float2*>(&S.write[buf][kt * 16 + (p >> 1) * 8 + 2 * tq]);
                    split2(bf16_lo(xh[kt][p]) * w.x, bf16_hi(xh[kt][p]) * w.y, wh[p], wl[p]);
                }
            }
            uint32_t bk[kRows / 16][4];
#pragma unroll
            for (int e = 0; e < kRows / 16; ++e)
                ldmatrix_x4_trans(smem_u32(&K[(kt * 16 + (mi & 1) * 8 + r8) * ROW + half * kRows + e * 16 + (mi >> 1) * 8]), bk[e][0],
                                  bk[e][1], bk[e][2], bk[e][3]);
#pragma unroll
            for (int part = 0; part < 2; ++part)
#pragma unroll
                for (int e = 0; e < kRows / 16; ++e) {
                    const uint32_t(&x)[4] = part == 0 ? wh : wl;
                    mma_bf16_16816(st[2 * e], x, bk[e][0], bk[e][1]);
                    mma_bf16_16816(st[2 * e + 1], x, bk[e][2], bk[e][3]);
                }
        }
        if (more && warp == 0) put_factors(buf ^ 1);
    }
    if constexpr (RULE == kMemory) {
        __syncthreads();
        for (int at = v0; at < v0 + kSlice; at += memory_columns(DK)) {
            float* memory = memory_of(a, a.table_idx[req], h, at);
            for (int i = threadIdx.x; i < DK; i += kWalkThreads) memory[i] = S.n[i];
            if (threadIdx.x == 0) memory[DK] = top;
        }
    }
#pragma unroll
    for (int j = 0; j < kRows / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) state[static_cast<int64_t>(8 * j + 2 * tq + (e & 1)) * vp + (e >> 1) * 8] = st[j][e];
}

bool chunked_supported(const Recurrence& a, int dtype) {
    return dtype == B200_DTYPE_BF16 && !a.plain && (a.padded_dim == 64 || a.padded_dim == 128) && a.padded_value_dim % kSlice == 0;
}

int max_smem(const void* kernel, size_t bytes) {
    B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)));
    return B200_OK;
}

template <typename T>
int launch_mix(const Recurrence& a, cudaStream_t stream) {
    auto kernel = a.conv == nullptr ? mix_kernel<T, 1> : a.taps == 2 ? mix_kernel<T, 2> : a.taps == 3 ? mix_kernel<T, 3> : a.taps == 4 ? mix_kernel<T, 4> : mix_kernel<T, 0>;
    const int v_blocks = div_ceil(a.heads * a.padded_value_dim, kMixThreads * 8);
    const int per_block = kMixThreads / (a.padded_dim / 8);
    // (of the matrix memory's channels nothing is made: the steps alone)
    const int blocks = a.rule == kMemory ? 1 : v_blocks + div_ceil(2 * a.kv_heads, per_block) + 1;
    const dim3 grid(div_ceil(a.max_extend, kMixTokens), blocks, a.batch);
    B200_CHECK_CUDA(launch_kernel(kernel, grid, dim3(kMixThreads), 0, stream, dim3(1, 1, 1), a, v_blocks, per_block));
    return B200_OK;
}

template <int RULE>
int launch_chunked(const Recurrence& a, cudaStream_t stream) {
    auto prepare = prepare_kernel<RULE>;
    int err = max_smem(reinterpret_cast<const void*>(prepare), sizeof(PrepareSmem));
    if (err != B200_OK) return err;
    const int parts = div_ceil(a.heads / a.kv_heads, kPrepareHeads);
    B200_CHECK_CUDA(launch_kernel(prepare, dim3(div_ceil(a.max_extend, kChunk), a.kv_heads * parts, a.batch), dim3(kPrepareThreads),
                                  sizeof(PrepareSmem), stream, dim3(1, 1, 1), a, parts));
    auto kernel = a.padded_dim == 64 ? chunk_kernel<64, RULE> : chunk_kernel<128, RULE>;
    const size_t smem = a.padded_dim == 64 ? sizeof(WalkSmem<64, RULE>) : sizeof(WalkSmem<128, RULE>);
    err = max_smem(reinterpret_cast<const void*>(kernel), smem);
    if (err != B200_OK) return err;
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.padded_value_dim / kSlice, a.heads, a.batch), dim3(kWalkThreads), smem, stream,
                                  dim3(1, 1, 1), a));
    return B200_OK;
}

template <typename T, int RULE>
int launch_steps(const Recurrence& a, int log_cols, int slices, bool finish, cudaStream_t stream) {
    const size_t smem = ((4ull << log_cols) + (RULE == kMemory ? 3ull : 2ull) * a.padded_dim + kStepThreads * 4) * 4;
    const bool few = div_ceil(a.padded_dim, kStepThreads >> log_cols) <= 4;
    auto kernel = a.decode ? (few ? step_kernel<T, RULE, true, 4> : step_kernel<T, RULE, true, kMaxAhead>)
                           : (few ? step_kernel<T, RULE, false, 4> : step_kernel<T, RULE, false, kMaxAhead>);
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.heads, a.batch, slices), dim3(kStepThreads), smem, stream, dim3(1, 1, 1), a,
                                  log_cols, finish));
    return B200_OK;
}

template <typename T>
int run(const Recurrence& a, int dtype, cudaStream_t stream) {
    const bool delta = a.rule == kDelta;
    int err = B200_OK;
    if (!a.decode) err = launch_mix<T>(a, stream);
    if (err != B200_OK) return err;
    bool finished = false;
    if (!a.decode && chunked_supported(a, dtype)) {
        err = delta ? launch_chunked<kDelta>(a, stream)
              : a.rule == kStateSpace ? launch_chunked<kStateSpace>(a, stream)
              : a.rule == kLightning ? launch_chunked<kLightning>(a, stream) : launch_chunked<kMemory>(a, stream);
    } else {
        // groups of four columns per CTA: a thread has room for kMaxAhead rows, and one output column
        const int most = kMaxAhead * kStepThreads / a.padded_dim;
        int log_cols = 0;
        while ((4 << log_cols) < a.padded_value_dim && (2 << log_cols) <= most && (8 << log_cols) <= kStepThreads) ++log_cols;
        const int slices = div_ceil(a.padded_value_dim, 4 << log_cols);
        finished = a.decode && slices == 1 && (delta || (a.rule == kMemory && a.norm_groups == a.heads));
        err = delta ? launch_steps<T, kDelta>(a, log_cols, slices, finished, stream)
              : a.rule == kStateSpace ? launch_steps<T, kStateSpace>(a, log_cols, slices, finished, stream)
              : a.rule == kLightning ? launch_steps<T, kLightning>(a, log_cols, slices, finished, stream)
                                     : launch_steps<T, kMemory>(a, log_cols, slices, finished, stream);
    }
    if (err != B200_OK || finished) return err;
    if (delta || (a.rule == kMemory && a.norm_groups == a.heads)) {
        const int64_t rows = static_cast<int64_t>(a.tokens) * a.heads;
        B200_CHECK_CUDA(launch_kernel(finish_heads_kernel<T>, dim3(static_cast<unsigned>(div_ceil64(rows, kFinishWarps))),
                                      dim3(kFinishWarps * 32), 0, stream, dim3(1, 1, 1), a));
    } else {
        const int per = a.heads * a.value_dim / a.norm_groups;
        auto kernel = per % 8 == 0 && a.value_dim % 8 == 0 ? finish_parts_kernel<T, 8> : finish_parts_kernel<T, 1>;
        B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.tokens, a.norm_groups), dim3(kPartThreads), 0, stream, dim3(1, 1, 1), a));
    }
    return B200_OK;
}

}  // namespace

// A thread of the step kernel holds kMaxAhead state rows of four columns.
bool recurrence_supported(int padded_value_dim, int padded_dim, int taps) {
    return padded_value_dim <= 65535 && padded_dim <= 1024 && taps >= 1 && taps <= kMaxTaps;
}

RecurrenceScratch recurrence_scratch(int rule, int max_tokens, int max_batch, int heads, int kv_heads, int padded_dim,
                                     int padded_value_dim, int dtype) {
    RecurrenceScratch s;
    const int64_t T = max_tokens, esz = dtype == B200_DTYPE_F32 ? 4 : 2;
    s.mixed = T * (static_cast<int64_t>(heads) * padded_value_dim + 2ll * kv_heads * padded_dim) * esz;
    s.steps = T * heads * 8;
    s.units = rule == kDelta ? T * kv_heads * 8 : rule == kMemory ? T * heads * 4 : 0;
    if (rule == kMemory) s.mixed = 0;
    s.chunks = dtype == B200_DTYPE_F32 || padded_dim > 128
                   ? 0
                   : (T / kChunk + max_batch + 1) * heads * (rule == kDelta ? 2 : 1) * kMatrixVecs * 16;
    return s;
}

int64_t recurrence_memory_floats(int padded_dim, int padded_value_dim) {
    return static_cast<int64_t>(memory_copies(padded_dim, padded_value_dim)) * memory_width(padded_dim);
}

int launch_recurrence(const Recurrence& a, int dtype, cudaStream_t stream) {
    if (a.tokens == 0 || a.batch == 0) return B200_OK;
    return dtype == B200_DTYPE_F32 ? run<float>(a, dtype, stream) : run<__nv_bfloat16>(a, dtype, stream);
}

}  // namespace b200

extern "C" {

int b200_recurrence_scratch(int rule, int max_tokens, int max_batch, int heads, int kv_heads, int padded_dim,
                            int padded_value_dim, int dtype, int64_t* bytes) {
    B200_CHECK_ARG(bytes && max_tokens >= 0 && max_batch >= 0 && heads > 0 && kv_heads > 0 && padded_dim > 0 && padded_value_dim > 0,
                   "recurrence_scratch: bad sizes");
    const b200::RecurrenceScratch s =
        b200::recurrence_scratch(rule, max_tokens, max_batch, heads, kv_heads, padded_dim, padded_value_dim, dtype);
    bytes[0] = s.mixed;
    bytes[1] = s.steps;
    bytes[2] = s.units;
    bytes[3] = s.chunks;
    return B200_OK;
}

int64_t b200_recurrence_memory_bytes(int padded_dim, int padded_value_dim) {
    if (padded_dim <= 0 || padded_dim % 64 != 0 || padded_value_dim <= 0 || padded_value_dim % 64 != 0 ||
        !b200::recurrence_supported(padded_value_dim, padded_dim, 1))
        return -1;
    return b200::recurrence_memory_floats(padded_dim, padded_value_dim) * 4;
}

int b200_recurrence(const b200_recurrence_args* p, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(p, "recurrence: NULL argument");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "recurrence: unknown dtype");
    B200_CHECK_ARG(p->rule >= B200_RULE_STATE_SPACE && p->rule <= B200_RULE_MATRIX_MEMORY, "recurrence: unknown rule");
    const bool conv = b200::has_convolution(p->rule), memory = p->rule == B200_RULE_MATRIX_MEMORY;
    B200_CHECK_ARG(conv || (p->kv_heads == p->heads && !p->conv && !p->conv_bias), "recurrence: no convolution with this rule");
    B200_CHECK_ARG(!memory || p->gate_cap > 0.f, "recurrence: bad gate cap");
    B200_CHECK_ARG(p->tokens >= 0 && p->batch >= 0 && p->batch <= 65535 && p->heads > 0 && p->heads <= 65535 && p->kv_heads > 0 &&
                       p->heads % p->kv_heads == 0, "recurrence: bad sizes");
    B200_CHECK_ARG(p->dim > 0 && p->padded_dim >= p->dim && p->padded_dim % 64 == 0 && p->value_dim > 0 &&
                       p->padded_value_dim >= p->value_dim && p->padded_value_dim % 64 == 0 &&
                       b200::recurrence_supported(p->padded_value_dim, p->padded_dim, conv ? p->taps : 1), "recurrence: bad head sizes");
    B200_CHECK_ARG(p->joint_ld % 8 == 0 && p->out_ld % 8 == 0 && p->out_ld >= static_cast<int64_t>(p->heads) * p->padded_value_dim,
                   "recurrence: bad strides");
    B200_CHECK_ARG(p->rule == B200_RULE_DELTA || (p->norm_groups > 0 && p->heads * p->value_dim % p->norm_groups == 0),
                   "recurrence: bad norm groups");
    B200_CHECK_ARG(static_cast<int64_t>(p->tokens) * p->heads < (1ll << 31), "recurrence: too many tokens");
    B200_CHECK_ARG(!p->decode || p->tokens == p->batch, "recurrence: a decode step brings one token per request");
    if (p->tokens == 0 || p->batch == 0) return B200_OK;
    B200_CHECK_ARG(p->out && p->joint && p->table_idx && p->cached && p->state && p->norm &&
                       (!conv || (p->conv_state && p->conv && p->step_bias)) && (memory || p->decay_log) &&
                       (p->rule != B200_RULE_STATE_SPACE || p->skip) && (!memory || (p->step_bias && p->memory)),
                   "recurrence: NULL tensor");
    B200_CHECK_ARG(p->decode || (p->qo_indptr && (p->mixed || memory) && p->steps &&
                                 (p->units || (p->rule != B200_RULE_DELTA && !memory)) && p->chunks && p->max_extend > 0),
                   "recurrence: NULL scratch");
    return b200::launch_recurrence(*p, dtype, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
