// The end of attention whose heads mix their softmax weights.  Mixing weights before they meet the values is the same as
// mixing what they make of the values: with O_gc what the weights of head g make of the values of key / value head c,
//     out_h = sum_g mix[h, g] O_g,c(h)
// so the attention kernels leave O_gc for all pairs, and the kernels that include this file sum them up, turn the result
// back by the token's position, gate it and store it.
#pragma once

#include "common.cuh"
#include "kernels.h"

namespace b200 {

struct MixOutput {
    void* out;
    int64_t out_st;
    const float* weights;      // [heads, heads]
    int heads, kv_heads, vp;
    int rotary, max_pos;
    const float *cos_t, *sin_t;
    const int32_t* positions;
    const void* gate;
    int64_t gate_st;
    bool gate_per_head;
    float out_scale;
    int* status;
    // Element m of a head's values goes with element m + pairs(): the two turn together.
    __host__ __device__ int pairs() const { return (rotary > 0 ? rotary : vp) >> 1; }
};

inline MixOutput mix_output(const WindowAttention& a) {
    MixOutput m;
    m.out = a.out;
    m.out_st = a.window.out_st > 0 ? a.window.out_st : static_cast<int64_t>(a.heads) * a.vp;
    m.weights = a.mix.weights;
    m.heads = a.heads;
    m.kv_heads = a.kv_heads;
    m.vp = a.vp;
    m.rotary = a.mix.rotary;
    m.max_pos = a.mix.max_pos;
    m.cos_t = a.mix.cos_t;
    m.sin_t = a.mix.sin_t;
    m.positions = a.mix.positions;
    m.gate = a.window.gate;
    m.gate_st = a.window.gate_st;
    m.gate_per_head = a.window.gate_per_head;
    m.out_scale = a.window.out_scale;
    m.status = a.status;
    return m;
}

#ifdef __CUDACC__
__device__ __forceinline__ float2 load_pair(const float* p, bool even) {
    return even ? *reinterpret_cast<const float2*>(p) : make_float2(p[0], p[1]);
}
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p, bool even) {
    if (!even) return make_float2(__bfloat162float(p[0]), __bfloat162float(p[1]));
    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(bf16_lo(u), bf16_hi(u));
}
__device__ __forceinline__ void store_pair(float* p, float2 x, bool even) {
    if (even) *reinterpret_cast<float2*>(p) = x;
    else p[0] = x.x, p[1] = x.y;
}
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float2 x, bool even) {
    if (even) *reinterpret_cast<uint32_t*>(p) = pack_bf16(x.x, x.y);
    else p[0] = __float2bfloat16_rn(x.x), p[1] = __float2bfloat16_rn(x.y);
}
__device__ __forceinline__ float exact_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// Elements m, m + 1 (u) and m + pairs, m + pairs + 1 (v) of head h's mixed values for token t.  With an odd number of
// pairs the last m stands alone: the second elements are neither turned nor stored.
template <typename T>
__device__ __forceinline__ void finish_mixed(const MixOutput& a, int64_t t, int h, int m, float2 u, float2 v) {
    const int pairs = a.pairs();
    const bool even = (pairs & 1) == 0, two = m + 1 < pairs;
    if (a.rotary > 0) {
        int pos = a.positions[t];
        if (pos < 0 || pos >= a.max_pos) {
            atomicExch(&a.status[kStatusBadIndex], pos + 1);
            pos = min(max(pos, 0), a.max_pos - 1);
        }
        const int64_t at = static_cast<int64_t>(pos) * pairs + m;
        float2 c = make_float2(a.cos_t[at], 1.f), s = make_float2(a.sin_t[at], 0.f);
        if (two) c.y = a.cos_t[at + 1], s.y = a.sin_t[at + 1];
        const float2 x = u;
        u = make_float2(x.x * c.x + v.x * s.x, x.y * c.y + v.y * s.y);
        v = make_float2(v.x * c.x - x.x * s.x, v.y * c.y - x.y * s.y);
    }
    float2 fu = make_float2(a.out_scale, a.out_scale), fv = fu;
    const T* gate = static_cast<const T*>(a.gate);
    if (gate != nullptr) {
        gate += t * a.gate_st;
        if (a.gate_per_head) {
            const float g = exact_sigmoid(static_cast<float>(gate[h]));
            fu.x *= g, fu.y *= g, fv.x *= g, fv.y *= g;
        } else {
            gate += static_cast<int64_t>(h) * a.vp + m;
            const float2 gu = load_pair(gate, even && two), gv = two ? load_pair(gate + pairs, even) : make_float2(static_cast<float>(gate[pairs]), 0.f);
            fu.x *= exact_sigmoid(gu.x), fu.y *= exact_sigmoid(gu.y);
            fv.x *= exact_sigmoid(gv.x), fv.y *= exact_sigmoid(gv.y);
        }
    }
    u.x *= fu.x, u.y *= fu.y, v.x *= fv.x, v.y *= fv.y;
    T* out = static_cast<T*>(a.out) + t * a.out_st + static_cast<int64_t>(h) * a.vp;
    if (two) {
        store_pair(out + m, u, even);
        store_pair(out + m + pairs, v, even);
    } else {
        out[m] = static_cast<T>(u.x);
        out[m + pairs] = static_cast<T>(v.x);
    }
}

// The padding behind a rotated head is zero.  Called by a whole warp.
template <typename T>
__device__ __forceinline__ void clear_padding(const MixOutput& a, int64_t t, int h) {
    T* out = static_cast<T*>(a.out) + t * a.out_st + static_cast<int64_t>(h) * a.vp;
    for (int i = 2 * a.pairs() + (threadIdx.x & 31); i < a.vp; i += 32) out[i] = static_cast<T>(0.f);
}
#endif

}  // namespace b200
