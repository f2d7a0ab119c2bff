// Softmax attention of layer stacks: per-head query and key norms, partial rotation, values mixed with those of
// an earlier layer, a sliding window that keeps the first keys or chunks of the sequence, sinks, and gates on the
// output (AttentionWindow).
//
//   * head_prepare_kernel: between the joint projection and the attention.  One warp per (token, head) row of
//     the joint output [q heads | k heads | v heads | gate]: queries are normalised and rotated in place, keys
//     and values go straight into the pools.
//   * heads that mix their weights run in talking_heads.cu.
//   * the attention itself: bf16 heads padded to 128 run on the paged kernels of the grouped-query models
//     (attention_prefill_tc2.cu, attention_decode.cu) with their window; everything else (fp32, wider heads,
//     head counts those do not take) on the plain kernel below, one CTA per (token, query head).
#include "common.cuh"
#include "kernels.h"

namespace b200 {
namespace {

constexpr int kPrepareWarps = 4;

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

// A token's position, inside the tables; one outside is reported by the threads with `report`.
__device__ __forceinline__ int position(const HeadPrepare& a, int64_t t, bool report) {
    const int pos = a.positions[t];
    if (pos >= 0 && pos < a.max_pos) return pos;
    if (report) atomicExch(&a.status[kStatusBadIndex], pos + 1);
    return min(max(pos, 0), a.max_pos - 1);
}

template <typename T>
__global__ void __launch_bounds__(kPrepareWarps * 32)
head_prepare_kernel(const HeadPrepare a) {
    extern __shared__ float s_rows[];   // one row of dp floats per warp
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int rows_per_token = a.heads + 2 * a.kv_heads;
    const int64_t row = static_cast<int64_t>(blockIdx.x) * kPrepareWarps + warp;
    pdl_launch_dependents();
    pdl_wait_prior();
    if (row >= static_cast<int64_t>(a.tokens) * rows_per_token) return;
    const int64_t t = row / rows_per_token;
    const int r = static_cast<int>(row - t * rows_per_token);
    T* joint = static_cast<T*>(a.joint) + t * a.ld;
    int64_t slot = 0;
    if (r >= a.heads) {
        slot = a.out_loc[t];
        if (slot < 0 || slot >= a.num_slots) {
            if (lane == 0) atomicExch(&a.status[kStatusBadIndex], static_cast<int>(slot) + 1);
            return;
        }
    }
    if (r >= a.heads + a.kv_heads) {   // a value row
        const int h = r - a.heads - a.kv_heads;
        const T* src = joint + static_cast<int64_t>(a.heads + a.kv_heads) * a.dp + h * a.vp;
        T* first = static_cast<T*>(a.first_values) + (t * a.kv_heads + h) * a.vp;
        T* dst = static_cast<T*>(a.v_cache) + (slot * a.kv_heads + h) * a.vp;
        const float lambda = a.mix == HeadPrepare::kMix ? *a.lambda : 0.f;
        if (a.value_rotary > 0) {
            const int half = a.value_rotary >> 1, pos = position(a, t, lane == 0);
            const float* c = a.value_cos + static_cast<int64_t>(pos) * half;
            const float* s = a.value_sin + static_cast<int64_t>(pos) * half;
            for (int i = lane; i < half; i += 32) {
                const float x = to_f32(src[i]), y = to_f32(src[i + half]);
                dst[i] = from_f32<T>(x * c[i] - y * s[i]);
                dst[i + half] = from_f32<T>(y * c[i] + x * s[i]);
            }
            for (int i = a.value_rotary + lane; i < a.vp; i += 32) dst[i] = src[i];
            return;
        }
        for (int i = lane * 4; i < a.vp; i += 128) {
            float4 v = load4(src + i);
            if (a.mix == HeadPrepare::kSave) store4(first + i, v);
            if (a.mix == HeadPrepare::kMix) {
                const float4 f = load4(first + i);
                v.x = (1.f - lambda) * v.x + lambda * f.x;
                v.y = (1.f - lambda) * v.y + lambda * f.y;
                v.z = (1.f - lambda) * v.z + lambda * f.z;
                v.w = (1.f - lambda) * v.w + lambda * f.w;
            }
            store4(dst + i, v);
        }
        return;
    }
    const bool is_q = r < a.heads;
    T* src = joint + static_cast<int64_t>(r) * a.dp;
    T* dst = is_q ? src : static_cast<T*>(a.k_cache) + (slot * a.kv_heads + (r - a.heads)) * a.dp;
    const T* weight = static_cast<const T*>(is_q ? a.q_weight : a.k_weight);
    float* buf = s_rows + warp * a.dp;
    float ss = 0.f;
    for (int i = lane * 4; i < a.dp; i += 128) {
        const float4 v = load4(src + i);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        *reinterpret_cast<float4*>(buf + i) = v;
    }
    if (a.unit_norm) {
        const float scale = rsqrtf(warp_sum(ss) / static_cast<float>(a.dim) + a.eps);
        for (int i = lane * 4; i < a.dp; i += 128) {
            const float4 v = *reinterpret_cast<float4*>(buf + i);
            *reinterpret_cast<float4*>(buf + i) = make_float4(v.x * scale, v.y * scale, v.z * scale, v.w * scale);
        }
    } else if (weight != nullptr) {
        const float scale = rsqrtf(warp_sum(ss) / static_cast<float>(a.dim) + a.eps);
        for (int i = lane * 4; i < a.dp; i += 128) {
            const float4 v = *reinterpret_cast<float4*>(buf + i), w = load4(weight + i);
            *reinterpret_cast<float4*>(buf + i) =
                make_float4(v.x * scale * w.x, v.y * scale * w.y, v.z * scale * w.z, v.w * scale * w.w);
        }
    }
    __syncwarp();
    const int pos = position(a, t, lane == 0);
    const int half = a.rotary_dim >> 1;
    const float* c = a.cos_t + static_cast<int64_t>(pos) * half;
    const float* s = a.sin_t + static_cast<int64_t>(pos) * half;
    for (int i = lane * 4; i < a.dp; i += 128) {
        float v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = i + e;
            if (d >= a.rotary_dim)
                v[e] = buf[d];
            else if (d < half)
                v[e] = buf[d] * c[d] - buf[d + half] * s[d];
            else
                v[e] = buf[d] * c[d - half] + buf[d - half] * s[d - half];
        }
        store4(dst + i, make_float4(v[0], v[1], v[2], v[3]));
    }
}

// The same for heads of 128 whose rotation pairs lie whole groups of four elements apart: a lane keeps four elements
// of a row and gets their partners from another lane; one CTA per token, a warp has the loads of kFastRows rows in flight.
constexpr int kFastRows = 4;

template <typename T>
__global__ void __launch_bounds__(kPrepareWarps * 32)
head_prepare_128_kernel(const HeadPrepare a) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, e0 = lane * 4;
    const int rows = a.heads + 2 * a.kv_heads;
    const int64_t t = blockIdx.x;
    pdl_launch_dependents();
    pdl_wait_prior();
    const int half = a.rotary_dim >> 1;
    const bool turns = e0 < a.rotary_dim;
    const int pair = !turns ? lane : e0 < half ? lane + half / 4 : lane - half / 4;
    const int64_t slot = a.out_loc[t];
    const int pos = position(a, t, threadIdx.x == 0);
    const bool slot_ok = slot >= 0 && slot < a.num_slots;
    if (threadIdx.x == 0 && !slot_ok) atomicExch(&a.status[kStatusBadIndex], static_cast<int>(slot) + 1);
    float4 c = make_float4(1.f, 1.f, 1.f, 1.f), s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (turns) {
        const int64_t at = static_cast<int64_t>(pos) * half + (e0 < half ? e0 : e0 - half);
        c = load4(a.cos_t + at);
        s = load4(a.sin_t + at);
        if (e0 < half) s = make_float4(-s.x, -s.y, -s.z, -s.w);
    }
    // the same for values
    const int vhalf = a.value_rotary >> 1;
    const bool vturns = e0 < a.value_rotary;
    const int vpair = !vturns ? lane : e0 < vhalf ? lane + vhalf / 4 : lane - vhalf / 4;
    float4 vc = make_float4(1.f, 1.f, 1.f, 1.f), vs = make_float4(0.f, 0.f, 0.f, 0.f);
    if (vturns) {
        const int64_t at = static_cast<int64_t>(pos) * vhalf + (e0 < vhalf ? e0 : e0 - vhalf);
        vc = load4(a.value_cos + at);
        vs = load4(a.value_sin + at);
        if (e0 < vhalf) vs = make_float4(-vs.x, -vs.y, -vs.z, -vs.w);
    }
    const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
    const float4 wq = a.q_weight != nullptr ? load4(static_cast<const T*>(a.q_weight) + e0) : one;
    const float4 wk = a.k_weight != nullptr ? load4(static_cast<const T*>(a.k_weight) + e0) : one;
    const float lambda = a.mix == HeadPrepare::kMix ? *a.lambda : 0.f;
    T* joint = static_cast<T*>(a.joint) + t * a.ld;
    for (int r0 = warp; r0 < rows; r0 += kPrepareWarps * kFastRows) {
        float4 x[kFastRows];
#pragma unroll
        for (int i = 0; i < kFastRows; ++i) {
            const int r = r0 + i * kPrepareWarps;
            if (r < rows) x[i] = load4(joint + r * 128 + e0);
        }
#pragma unroll
        for (int i = 0; i < kFastRows; ++i) {
            const int r = r0 + i * kPrepareWarps;
            if (r >= rows) break;
            float4 v = x[i];
            const bool is_q = r < a.heads;
            if (r >= a.heads + a.kv_heads) {   // a value row
                const int h = r - a.heads - a.kv_heads;
                T* first = static_cast<T*>(a.first_values) + (t * a.kv_heads + h) * 128 + e0;
                if (a.mix == HeadPrepare::kSave) store4(first, v);
                if (a.mix == HeadPrepare::kMix) {
                    const float4 f = load4(first);
                    v.x = (1.f - lambda) * v.x + lambda * f.x;
                    v.y = (1.f - lambda) * v.y + lambda * f.y;
                    v.z = (1.f - lambda) * v.z + lambda * f.z;
                    v.w = (1.f - lambda) * v.w + lambda * f.w;
                }
                if (a.value_rotary > 0) {   // (the whole warp has this row)
                    float4 o;
                    o.x = __shfl_sync(0xffffffffu, v.x, vpair);
                    o.y = __shfl_sync(0xffffffffu, v.y, vpair);
                    o.z = __shfl_sync(0xffffffffu, v.z, vpair);
                    o.w = __shfl_sync(0xffffffffu, v.w, vpair);
                    v = make_float4(v.x * vc.x + o.x * vs.x, v.y * vc.y + o.y * vs.y, v.z * vc.z + o.z * vs.z, v.w * vc.w + o.w * vs.w);
                }
                if (slot_ok) store4(static_cast<T*>(a.v_cache) + (slot * a.kv_heads + h) * 128 + e0, v);
                continue;
            }
            if (a.unit_norm || (is_q ? a.q_weight : a.k_weight) != nullptr) {
                const float scale =
                    rsqrtf(warp_sum(v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w) / static_cast<float>(a.dim) + a.eps);
                const float4 w = is_q ? wq : wk;
                v = make_float4(v.x * scale * w.x, v.y * scale * w.y, v.z * scale * w.z, v.w * scale * w.w);
            }
            float4 o;
            o.x = __shfl_sync(0xffffffffu, v.x, pair);
            o.y = __shfl_sync(0xffffffffu, v.y, pair);
            o.z = __shfl_sync(0xffffffffu, v.z, pair);
            o.w = __shfl_sync(0xffffffffu, v.w, pair);
            v = make_float4(v.x * c.x + o.x * s.x, v.y * c.y + o.y * s.y, v.z * c.z + o.z * s.z, v.w * c.w + o.w * s.w);
            T* dst = is_q ? joint + r * 128 : static_cast<T*>(a.k_cache) + (slot * a.kv_heads + (r - a.heads)) * 128;
            if (is_q || slot_ok) store4(dst + e0, v);
        }
    }
}

// ---- plain attention: any sizes, fp32 or bf16 ------------------------------------

constexpr int kPlainThreads = 128;
constexpr int kPlainKeys = 128;     // keys per round
constexpr int kPlainMaxVec = 8;     // value elements per thread: heads of up to 1024 values

// ALL: over the values of all key / value heads, 1024 columns per CTA; the averages themselves go to a.mix.scratch.
template <typename T, bool ALL>
__global__ void __launch_bounds__(kPlainThreads)
window_attention_plain_kernel(const WindowAttention a) {
    extern __shared__ float s_q[];      // the query, dp floats
    __shared__ float s_p[kPlainKeys];
    __shared__ int s_slot[kPlainKeys];
    __shared__ float s_red[kPlainThreads / 32];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    pdl_launch_dependents();
    pdl_wait_prior();
    const int64_t t = blockIdx.x;
    const int h = blockIdx.y, g = h / (a.heads / a.kv_heads);
    const T* q = static_cast<const T*>(a.q) + t * a.q_st + static_cast<int64_t>(h) * a.dp;
    for (int i = threadIdx.x; i < a.dp; i += kPlainThreads) s_q[i] = to_f32(q[i]) * a.scale;
    const int32_t* pages = a.page_table + static_cast<int64_t>(a.row_table[t]) * a.pt_stride;
    const int len = a.row_len[t];
    const int oldest = len > 0 ? a.window.oldest(len - 1) : 0;
    const int kept = min(a.window.keep_first, oldest);
    const int count = kept + len - oldest;             // keys it sees: [0, kept) and [oldest, len)
    // this CTA's columns of a slot's row of values
    const int col0 = ALL ? static_cast<int>(blockIdx.z) * kPlainMaxVec * kPlainThreads : 0;
    const int cols = ALL ? min(a.kv_heads * a.vp - col0, kPlainMaxVec * kPlainThreads) : a.vp;
    float acc[kPlainMaxVec];
#pragma unroll
    for (int i = 0; i < kPlainMaxVec; ++i) acc[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    auto block_reduce = [&](float x, bool is_max) {
        x = is_max ? warp_max(x) : warp_sum(x);
        __syncthreads();
        if (lane == 0) s_red[warp] = x;
        __syncthreads();
        float y = s_red[0];
#pragma unroll
        for (int i = 1; i < kPlainThreads / 32; ++i) y = is_max ? fmaxf(y, s_red[i]) : y + s_red[i];
        return y;
    };
    for (int base = 0; base < count; base += kPlainKeys) {
        const int n = min(kPlainKeys, count - base);
        __syncthreads();   // the last round's weights and slots have been used (and the query is in place)
        if (threadIdx.x < n) {
            const int i = base + threadIdx.x;
            int slot = pages[i < kept ? i : oldest + i - kept];
            if (slot < 0 || slot >= a.num_slots) {
                atomicExch(&a.status[kStatusBadIndex], slot + 1);
                slot = 0;
            }
            s_slot[threadIdx.x] = slot;
        }
        __syncthreads();
        for (int j = warp; j < n; j += kPlainThreads / 32) {
            const T* k = static_cast<const T*>(a.k_cache) + (static_cast<int64_t>(s_slot[j]) * a.kv_heads + g) * a.dp;
            float dot = 0.f;
            for (int i = lane * 4; i < a.dp; i += 128) {
                const float4 kv = load4(k + i), qv = *reinterpret_cast<const float4*>(s_q + i);
                dot += kv.x * qv.x + kv.y * qv.y + kv.z * qv.z + kv.w * qv.w;
            }
            dot = warp_sum(dot);
            if (lane == 0) s_p[j] = dot;
        }
        __syncthreads();
        const float score = threadIdx.x < n ? s_p[threadIdx.x] : -INFINITY;
        const float m_new = fmaxf(m, block_reduce(score, true));
        const float p = threadIdx.x < n ? expf(score - m_new) : 0.f;
        s_p[threadIdx.x] = p;
        const float sum = block_reduce(p, false);      // (its barriers publish s_p)
        const float keep = expf(m - m_new);
        l = l * keep + sum;
        m = m_new;
#pragma unroll
        for (int i = 0; i < kPlainMaxVec; ++i) acc[i] *= keep;
        for (int j = 0; j < n; ++j) {
            const T* v = static_cast<const T*>(a.v_cache) + (static_cast<int64_t>(s_slot[j]) * a.kv_heads + (ALL ? 0 : g)) * a.vp + col0;
            const float w = s_p[j];
#pragma unroll
            for (int i = 0; i < kPlainMaxVec; ++i) {
                const int c = threadIdx.x + i * kPlainThreads;
                if (c < cols) acc[i] += w * to_f32(v[c]);
            }
        }
    }
    if (ALL) {
        T* raw = static_cast<T*>(a.mix.scratch) + (t * a.heads + h) * a.kv_heads * a.vp + col0;
        const float over = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
        for (int i = 0; i < kPlainMaxVec; ++i) {
            const int c = threadIdx.x + i * kPlainThreads;
            if (c < cols) raw[c] = from_f32<T>(acc[i] * over);
        }
        return;
    }
    T* out = static_cast<T*>(a.out) + t * a.window.out_st + static_cast<int64_t>(h) * a.vp;
    const T* gate = a.window.gate == nullptr ? nullptr : static_cast<const T*>(a.window.gate) + t * a.window.gate_st;
    if (a.window.sinks != nullptr) l += expf(a.window.sinks[h] - m);
    float inv = l > 0.f ? a.window.out_scale / l : 0.f;
    if (gate != nullptr && a.window.gate_per_head) {
        inv *= 1.f / (1.f + expf(-to_f32(gate[h])));
        gate = nullptr;
    }
    if (gate != nullptr) gate += static_cast<int64_t>(h) * a.vp;
#pragma unroll
    for (int i = 0; i < kPlainMaxVec; ++i) {
        const int c = threadIdx.x + i * kPlainThreads;
        if (c >= a.vp) continue;
        float y = acc[i] * inv;
        if (gate != nullptr) y *= 1.f / (1.f + expf(-to_f32(gate[c])));
        out[c] = from_f32<T>(y);
    }
}

}  // namespace

int launch_head_prepare(const HeadPrepare& a, int dtype, cudaStream_t stream) {
    if (a.tokens == 0) return B200_OK;
    const int64_t rows = static_cast<int64_t>(a.tokens) * (a.heads + 2 * a.kv_heads);
    if (a.dp == 128 && a.vp == 128 && a.rotary_dim % 8 == 0 && a.value_rotary % 8 == 0 && rows >= 4096) {
        auto fast = dtype == B200_DTYPE_F32 ? head_prepare_128_kernel<float> : head_prepare_128_kernel<__nv_bfloat16>;
        B200_CHECK_CUDA(launch_kernel(fast, dim3(a.tokens), dim3(kPrepareWarps * 32), 0, stream, dim3(1, 1, 1), a));
        return B200_OK;
    }
    auto kernel = dtype == B200_DTYPE_F32 ? head_prepare_kernel<float> : head_prepare_kernel<__nv_bfloat16>;
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(static_cast<unsigned>((rows + kPrepareWarps - 1) / kPrepareWarps)),
                                  dim3(kPrepareWarps * 32), static_cast<size_t>(kPrepareWarps) * a.dp * 4, stream,
                                  dim3(1, 1, 1), a));
    return B200_OK;
}

bool window_attention_tc_supported(const WindowAttention& a, int dtype) {
    const int group = a.heads / a.kv_heads;
    if (dtype != B200_DTYPE_BF16 || a.plain || a.dp != 128 || a.vp != 128 || a.scale <= 0.f || group > 16) return false;
    if (a.window.gate_st % 8 != 0 || a.window.out_st % 8 != 0 || !attention_prefill_tc_supported(a.q, a.q_st, a.dp, a.out)) return false;
    if (a.decode) return a.kv_heads <= 8 && 8 % a.kv_heads == 0 && a.batch <= 1024;
    return (group & (group - 1)) == 0;
}

int launch_plain_all_values(const WindowAttention& a, int dtype, cudaStream_t stream) {
    auto kernel = dtype == B200_DTYPE_F32 ? window_attention_plain_kernel<float, true> : window_attention_plain_kernel<__nv_bfloat16, true>;
    const dim3 grid(a.tokens, a.heads, div_ceil(a.kv_heads * a.vp, kPlainMaxVec * kPlainThreads));
    B200_CHECK_CUDA(launch_kernel(kernel, grid, dim3(kPlainThreads), static_cast<size_t>(a.dp) * 4, stream, dim3(1, 1, 1), a));
    return B200_OK;
}

int launch_window_attention(const WindowAttention& a, int dtype, cudaStream_t stream) {
    if (a.tokens == 0) return B200_OK;
    if (a.mix.weights != nullptr) return launch_talking_heads(a, dtype, stream);
    if (window_attention_tc_supported(a, dtype)) {
        if (!a.decode)
            return launch_attention_prefill_tc2(a.out, a.q, a.q_st, a.dp, a.k_cache, a.v_cache, a.num_slots, a.page_table,
                                                a.pt_stride, a.table_idx, a.seq_lens, a.qo_indptr, a.batch, a.max_extend,
                                                a.heads, a.kv_heads, a.page_size, a.scale, a.status, stream, &a.window);
        CUtensorMap tk, tv;
        int err = make_kv_tmap(&tk, a.k_cache, a.num_slots, a.kv_heads, a.page_size);
        if (err != B200_OK) return err;
        err = make_kv_tmap(&tv, a.v_cache, a.num_slots, a.kv_heads, a.page_size);
        if (err != B200_OK) return err;
        return launch_attention_decode(a.out, a.q, a.q_st, a.dp, tk, tv, a.num_slots, a.page_table, a.pt_stride,
                                       a.table_idx, a.seq_lens, a.batch, a.heads, a.kv_heads, a.page_size, a.scale,
                                       a.workspace, a.workspace_bytes, a.status, stream, true, &a.window);
    }
    WindowAttention plain = a;
    if (plain.window.out_st == 0) plain.window.out_st = static_cast<int64_t>(a.heads) * a.vp;
    auto kernel = dtype == B200_DTYPE_F32 ? window_attention_plain_kernel<float, false> : window_attention_plain_kernel<__nv_bfloat16, false>;
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.tokens, a.heads), dim3(kPlainThreads), static_cast<size_t>(a.dp) * 4, stream,
                                  dim3(1, 1, 1), plain));
    return B200_OK;
}

}  // namespace b200

extern "C" {

int b200_head_prepare(const b200_head_prepare_args* p, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(p, "head_prepare: NULL argument");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "head_prepare: unknown dtype");
    B200_CHECK_ARG(p->tokens >= 0 && p->heads > 0 && p->kv_heads >= 0 && p->dim > 0 && p->padded_dim >= p->dim &&
                       p->padded_dim % 64 == 0 && p->padded_value_dim > 0 && p->padded_value_dim % 64 == 0,
                   "head_prepare: bad shape");
    B200_CHECK_ARG(p->rotary_dim >= 0 && p->rotary_dim % 2 == 0 && p->rotary_dim <= p->dim, "head_prepare: bad rotary_dim");
    B200_CHECK_ARG(p->mix >= 0 && p->mix <= 2 && (p->mix == 0 || p->first_values) && (p->mix != 2 || p->lambda),
                   "head_prepare: bad value mixing");
    B200_CHECK_ARG(p->value_rotary >= 0 && p->value_rotary % 2 == 0 && p->value_rotary <= p->padded_value_dim &&
                       (p->value_rotary == 0 || (p->mix == 0 && p->value_cos && p->value_sin)), "head_prepare: bad value rotation");
    if (p->tokens == 0) return B200_OK;
    B200_CHECK_ARG(p->joint && p->positions && p->out_loc && p->k_cache && p->v_cache && p->cos_table && p->sin_table,
                   "head_prepare: NULL tensor");
    b200::HeadPrepare a;
    int err = B200_OK;
    a.status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    a.joint = p->joint;
    a.ld = p->joint_ld;
    a.tokens = p->tokens;
    a.heads = p->heads;
    a.kv_heads = p->kv_heads;
    a.dim = p->dim;
    a.dp = p->padded_dim;
    a.vp = p->padded_value_dim;
    a.q_weight = p->q_norm;
    a.k_weight = p->k_norm;
    a.eps = p->eps;
    a.rotary_dim = p->rotary_dim;
    a.cos_t = p->cos_table;
    a.sin_t = p->sin_table;
    a.max_pos = p->max_pos;
    a.positions = p->positions;
    a.out_loc = p->out_loc;
    a.k_cache = p->k_cache;
    a.v_cache = p->v_cache;
    a.num_slots = p->num_slots;
    a.mix = p->mix;
    a.lambda = p->lambda;
    a.first_values = p->first_values;
    a.unit_norm = p->unit_norm != 0;
    a.value_rotary = p->value_rotary;
    a.value_cos = p->value_cos;
    a.value_sin = p->value_sin;
    return b200::launch_head_prepare(a, dtype, static_cast<cudaStream_t>(stream));
}

int b200_window_attention(const b200_window_attention_args* p, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(p, "window_attention: NULL argument");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "window_attention: unknown dtype");
    B200_CHECK_ARG(p->tokens >= 0 && p->batch >= 0 && p->batch <= 65535 && p->heads > 0 && p->heads <= 65535 &&
                       p->kv_heads > 0 && p->heads % p->kv_heads == 0, "window_attention: bad head counts");
    B200_CHECK_ARG(p->padded_dim > 0 && p->padded_dim % 64 == 0 && p->padded_dim <= 8192 && p->padded_value_dim > 0 &&
                       p->padded_value_dim % 64 == 0 && p->padded_value_dim <= b200::kPlainMaxVec * b200::kPlainThreads,
                   "window_attention: bad head sizes");
    B200_CHECK_ARG(p->page_size >= 1 && (p->page_size & (p->page_size - 1)) == 0, "window_attention: page_size must be a power of two");
    B200_CHECK_ARG(p->window >= 1 && p->keep_first >= 0 && p->chunk >= 0, "window_attention: bad window");
    B200_CHECK_ARG(p->out_stride == 0 || p->out_stride >= static_cast<int64_t>(p->heads) * p->padded_value_dim,
                   "window_attention: bad output stride");
    if (p->tokens == 0) return B200_OK;
    B200_CHECK_ARG(p->out && p->q && p->k_cache && p->v_cache && p->page_table && p->table_idx && p->seq_lens && p->qo_indptr &&
                       p->row_table && p->row_len && p->workspace, "window_attention: NULL tensor");
    b200::WindowAttention a;
    int err = B200_OK;
    a.status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    a.out = p->out;
    a.q = p->q;
    a.q_st = p->q_stride;
    a.k_cache = p->k_cache;
    a.v_cache = p->v_cache;
    a.num_slots = p->num_slots;
    a.page_table = p->page_table;
    a.pt_stride = p->page_table_stride;
    a.table_idx = p->table_idx;
    a.seq_lens = p->seq_lens;
    a.qo_indptr = p->qo_indptr;
    a.row_table = p->row_table;
    a.row_len = p->row_len;
    a.tokens = p->tokens;
    a.batch = p->batch;
    a.max_extend = p->max_extend;
    a.decode = p->decode != 0;
    a.plain = p->plain != 0;
    a.heads = p->heads;
    a.kv_heads = p->kv_heads;
    a.dp = p->padded_dim;
    a.vp = p->padded_value_dim;
    a.page_size = p->page_size;
    a.scale = p->scale;
    a.window.size = p->window;
    a.window.keep_first = p->keep_first;
    a.window.gate = p->gate;
    a.window.gate_st = p->gate_stride;
    a.window.gate_per_head = p->gate_per_head != 0;
    a.window.chunk = p->chunk;
    a.window.sinks = p->sinks;
    a.window.out_scale = p->out_scale == 0.f ? 1.f : p->out_scale;
    a.window.out_st = p->out_stride;
    a.workspace = p->workspace;
    a.workspace_bytes = p->workspace_bytes;
    if (p->head_mix != nullptr) {
        B200_CHECK_ARG(p->mix_scratch && !p->sinks && p->value_rotary >= 0 && p->value_rotary % 2 == 0 &&
                           p->value_rotary <= p->padded_value_dim, "window_attention: bad head mixing");
        B200_CHECK_ARG(p->value_rotary == 0 || (p->value_cos && p->value_sin && p->positions && p->max_pos > 0),
                       "window_attention: NULL rotation");
        a.mix.weights = p->head_mix;
        a.mix.rotary = p->value_rotary;
        a.mix.max_pos = p->max_pos;
        a.mix.cos_t = p->value_cos;
        a.mix.sin_t = p->value_sin;
        a.mix.positions = p->positions;
        a.mix.score_bound = p->score_bound;
        a.mix.scratch = p->mix_scratch;
    }
    return b200::launch_window_attention(a, dtype, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
