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
// Elements m .. m + 3 of a row whose elements up to m + n are there; 8 or 16 bytes at once under VEC (all four are).
template <bool VEC>
__device__ __forceinline__ float4 load_quad(const float* p, int n) {
    if (VEC) return *reinterpret_cast<const float4*>(p);
    auto at = [&](int i) { return n > i ? p[i] : 0.f; };
    return make_float4(at(0), at(1), at(2), at(3));
}
template <bool VEC>
__device__ __forceinline__ float4 load_quad(const __nv_bfloat16* p, int n) {
    if (VEC) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        return make_float4(bf16_lo(u.x), bf16_hi(u.x), bf16_lo(u.y), bf16_hi(u.y));
    }
    auto at = [&](int i) { return n > i ? __bfloat162float(p[i]) : 0.f; };
    return make_float4(at(0), at(1), at(2), at(3));
}
template <bool VEC>
__device__ __forceinline__ void store_quad(float* p, const float4& x, int n) {
    if (VEC) {
        *reinterpret_cast<float4*>(p) = x;
        return;
    }
    const float v[4] = {x.x, x.y, x.z, x.w};
    for (int i = 0; i < 4; ++i)
        if (n > i) p[i] = v[i];
}
template <bool VEC>
__device__ __forceinline__ void store_quad(__nv_bfloat16* p, const float4& x, int n) {
    if (VEC) {
        *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(x.x, x.y), pack_bf16(x.z, x.w));
        return;
    }
    const float v[4] = {x.x, x.y, x.z, x.w};
    for (int i = 0; i < 4; ++i)
        if (n > i) p[i] = __float2bfloat16_rn(v[i]);
}
template <typename T>
__device__ __forceinline__ float open_gate(float x) { return 1.f / (1.f + expf(-x)); }
template <>
__device__ __forceinline__ float open_gate<__nv_bfloat16>(float x) { return sigmoid_f(x); }

// Cosines and sines of what elements m .. m + 3 of token t turn back by (1 and 0 without a rotation).
struct Turn {
    float4 c, s;
};
template <bool VEC>
__device__ __forceinline__ Turn turn_of(const MixOutput& a, int64_t t, int m) {
    Turn r = {make_float4(1.f, 1.f, 1.f, 1.f), make_float4(0.f, 0.f, 0.f, 0.f)};
    if (a.rotary == 0) return r;
    int pos = a.positions[t];
    if (pos < 0 || pos >= a.max_pos) {
        atomicExch(&a.status[kStatusBadIndex], pos + 1);
        pos = min(max(pos, 0), a.max_pos - 1);
    }
    const int64_t at = static_cast<int64_t>(pos) * a.pairs() + m;
    r.c = load_quad<VEC>(a.cos_t + at, a.pairs() - m);
    r.s = load_quad<VEC>(a.sin_t + at, a.pairs() - m);
    return r;
}

// Elements m .. m + 3 (u) and those a.pairs() further (v) of head h's mixed values for token t.  VEC: the number of pairs is
// a multiple of four.
template <typename T, bool VEC>
__device__ __forceinline__ void finish_mixed(const MixOutput& a, int64_t t, int h, int m, const float4& u, const float4& v, const Turn& r) {
    const int pairs = a.pairs(), n = pairs - m;
    float4 x = make_float4(u.x * r.c.x + v.x * r.s.x, u.y * r.c.y + v.y * r.s.y, u.z * r.c.z + v.z * r.s.z, u.w * r.c.w + v.w * r.s.w);
    float4 y = make_float4(v.x * r.c.x - u.x * r.s.x, v.y * r.c.y - u.y * r.s.y, v.z * r.c.z - u.z * r.s.z, v.w * r.c.w - u.w * r.s.w);
    auto scale = [](float4& z, float f) { z.x *= f, z.y *= f, z.z *= f, z.w *= f; };
    float factor = a.out_scale;
    const T* gate = static_cast<const T*>(a.gate);
    if (gate != nullptr) {
        gate += t * a.gate_st;
        if (a.gate_per_head) {
            factor *= open_gate<T>(static_cast<float>(gate[h]));
        } else {
            gate += static_cast<int64_t>(h) * a.vp + m;
            const float4 gx = load_quad<VEC>(gate, n), gy = load_quad<VEC>(gate + pairs, n);
            auto open = [](float4& z, const float4& g) {
                z.x *= open_gate<T>(g.x), z.y *= open_gate<T>(g.y), z.z *= open_gate<T>(g.z), z.w *= open_gate<T>(g.w);
            };
            open(x, gx);
            open(y, gy);
        }
    }
    scale(x, factor);
    scale(y, factor);
    T* out = static_cast<T*>(a.out) + t * a.out_st + static_cast<int64_t>(h) * a.vp + m;
    store_quad<VEC>(out, x, n);
    store_quad<VEC>(out + pairs, y, n);
}

// The padding behind a rotated head is zero.  Called by `lanes` neighbouring threads.
template <typename T>
__device__ __forceinline__ void clear_padding(const MixOutput& a, int64_t t, int h, int lanes) {
    T* out = static_cast<T*>(a.out) + t * a.out_st + static_cast<int64_t>(h) * a.vp;
    for (int i = 2 * a.pairs() + (threadIdx.x & (lanes - 1)); i < a.vp; i += lanes) out[i] = static_cast<T>(0.f);
}
#endif

}  // namespace b200
