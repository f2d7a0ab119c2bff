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
// Four neighbouring elements, 8 or 16 bytes at once where `vec`; of the others the first n.
__device__ __forceinline__ float4 load_quad(const float* p, bool vec, int n) {
    if (vec) return *reinterpret_cast<const float4*>(p);
    return make_float4(n > 0 ? p[0] : 0.f, n > 1 ? p[1] : 0.f, n > 2 ? p[2] : 0.f, n > 3 ? p[3] : 0.f);
}
__device__ __forceinline__ float4 load_quad(const __nv_bfloat16* p, bool vec, int n) {
    if (vec) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        return make_float4(bf16_lo(u.x), bf16_hi(u.x), bf16_lo(u.y), bf16_hi(u.y));
    }
    auto at = [&](int i) { return n > i ? __bfloat162float(p[i]) : 0.f; };
    return make_float4(at(0), at(1), at(2), at(3));
}
__device__ __forceinline__ float exact_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// Cosines and sines of what elements m, m + 1 of token t turn back by (1 and 0 without a rotation).
struct Turn {
    float2 c, s;
};
__device__ __forceinline__ Turn turn_of(const MixOutput& a, int64_t t, int m) {
    Turn r = {make_float2(1.f, 1.f), make_float2(0.f, 0.f)};
    if (a.rotary == 0) return r;
    int pos = __ldg(a.positions + t);
    if (pos < 0 || pos >= a.max_pos) {
        atomicExch(&a.status[kStatusBadIndex], pos + 1);
        pos = min(max(pos, 0), a.max_pos - 1);
    }
    const int pairs = a.pairs();
    const int64_t at = static_cast<int64_t>(pos) * pairs + m;
    r.c.x = __ldg(a.cos_t + at), r.s.x = __ldg(a.sin_t + at);
    if (m + 1 < pairs) r.c.y = __ldg(a.cos_t + at + 1), r.s.y = __ldg(a.sin_t + at + 1);
    return r;
}

// Elements m, m + 1 (u) and m + pairs, m + pairs + 1 (v) of head h's mixed values for token t.  With an odd number of
// pairs the last m stands alone: the second elements are not stored.
template <typename T>
__device__ __forceinline__ void finish_mixed(const MixOutput& a, int64_t t, int h, int m, float2 u, float2 v, const Turn& r) {
    const int pairs = a.pairs();
    const bool even = (pairs & 1) == 0, two = m + 1 < pairs;
    const float2 x = u;
    u = make_float2(x.x * r.c.x + v.x * r.s.x, x.y * r.c.y + v.y * r.s.y);
    v = make_float2(v.x * r.c.x - x.x * r.s.x, v.y * r.c.y - x.y * r.s.y);
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

// The padding behind a rotated head is zero.  Called by `lanes` neighbouring threads.
template <typename T>
__device__ __forceinline__ void clear_padding(const MixOutput& a, int64_t t, int h, int lanes) {
    T* out = static_cast<T*>(a.out) + t * a.out_st + static_cast<int64_t>(h) * a.vp;
    for (int i = 2 * a.pairs() + (threadIdx.x & (lanes - 1)); i < a.vp; i += lanes) out[i] = static_cast<T>(0.f);
}
#endif

}  // namespace b200
