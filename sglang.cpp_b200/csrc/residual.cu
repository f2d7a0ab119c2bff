// The fp32 residual stream of a layer stack: one kernel adds what the previous block produced (an
// embedding row, a projection's output, or the weighted outputs of a token's experts), stores the sum and
// writes its RMS norm for the next block - to the token's own row, or straight into the expert-sorted
// rows that the next block's grouped GEMM reads.  One CTA per token, the row in registers.
#include "common.cuh"
#include "kernels.h"

namespace b200 {
namespace {

constexpr int kVec = 8;   // float4 vectors a thread keeps; wider rows are read again from the residual

template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <>
__device__ __forceinline__ float4 load4<float>(const float* p) {
    return *reinterpret_cast<const float4*>(p);
}
template <>
__device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf16_lo(u.x), bf16_hi(u.x), bf16_lo(u.y), bf16_hi(u.y));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

struct Args {
    void* out;
    const int32_t* out_rows;
    float* residual;
    const void* src;
    const int32_t* src_rows;
    const void* weight;
    int64_t src_count;
    int out_top, src_top, init, width, padded;
    float src_scale, weight_offset, out_scale, eps;
    int* status;
};

template <typename T>
__global__ void __launch_bounds__(256)
residual_norm_kernel(const Args a) {
    __shared__ float red[8];
    pdl_launch_dependents();
    const int nvec = a.padded >> 2;
    const T* weight = static_cast<const T*>(a.weight);
    // the norm weights do not come from the kernel before this one
    float4 w[kVec];
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        w[i] = v < nvec ? load4(weight + v * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait_prior();
    const int64_t t = blockIdx.x;
    float* res = a.residual + t * a.padded;
    const T* src = static_cast<const T*>(a.src);
    auto sum_at = [&](int v) {
        float4 s = a.init ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(static_cast<const float*>(res) + v * 4);
        if (src != nullptr) {
            float4 add = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int k = 0; k < a.src_top; ++k) {
                const int64_t row = a.src_rows ? a.src_rows[t * a.src_top + k] : t;
                if (row < 0 || row >= a.src_count) {
                    if (v == 0) atomicExch(&a.status[kStatusBadIndex], static_cast<int>(row) + 1);
                    continue;
                }
                const float4 x = load4(src + row * a.padded + v * 4);
                add.x += x.x;
                add.y += x.y;
                add.z += x.z;
                add.w += x.w;
            }
            s.x += a.src_scale * add.x;
            s.y += a.src_scale * add.y;
            s.z += a.src_scale * add.z;
            s.w += a.src_scale * add.w;
        }
        return s;
    };
    float4 val[kVec];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < nvec) {
            val[i] = sum_at(v);
            if (src != nullptr) store4(res + v * 4, val[i]);
            ss += val[i].x * val[i].x + val[i].y * val[i].y + val[i].z * val[i].z + val[i].w * val[i].w;
        }
    }
    for (int v = threadIdx.x + kVec * blockDim.x; v < nvec; v += blockDim.x) {
        const float4 s = sum_at(v);
        if (src != nullptr) store4(res + v * 4, s);
        ss += s.x * s.x + s.y * s.y + s.z * s.z + s.w * s.w;
    }
    ss = warp_sum(ss);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = warp_sum(lane < static_cast<int>(blockDim.x >> 5) ? red[lane] : 0.f);
    const float scale = rsqrtf(ss / static_cast<float>(a.width) + a.eps) * a.out_scale;
    T* out = static_cast<T*>(a.out);
    if (out == nullptr) return;
    auto emit = [&](int v, float4 s, float4 g) {
        const float o = a.weight_offset;
        const float4 y = make_float4(s.x * scale * (g.x + o), s.y * scale * (g.y + o), s.z * scale * (g.z + o),
                                     s.w * scale * (g.w + o));
        for (int k = 0; k < a.out_top; ++k) {
            const int64_t row = a.out_rows ? a.out_rows[t * a.out_top + k] : t;
            store4(out + row * a.padded + v * 4, y);
        }
    };
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < nvec) emit(v, val[i], w[i]);
    }
    for (int v = threadIdx.x + kVec * blockDim.x; v < nvec; v += blockDim.x)
        emit(v, load4(static_cast<const float*>(res) + v * 4), load4(weight + v * 4));
}

}  // namespace

int launch_residual_norm(const ResidualNorm& r, int dtype, int* status, cudaStream_t stream) {
    if (r.tokens == 0) return B200_OK;
    Args a;
    a.out = r.out;
    a.out_rows = r.out_rows;
    a.residual = r.residual;
    a.src = r.src;
    a.src_rows = r.src_rows;
    a.weight = r.weight;
    a.src_count = r.src_count;
    a.out_top = r.out_rows ? r.out_top : 1;
    a.src_top = r.src_rows ? r.src_top : 1;
    a.init = r.init ? 1 : 0;
    a.width = r.width;
    a.padded = r.padded;
    a.src_scale = r.src_scale;
    a.weight_offset = r.weight_offset;
    a.out_scale = r.out_scale;
    a.eps = r.eps;
    a.status = status;
    int threads = 64;
    while (threads < 256 && threads * 8 < r.padded) threads *= 2;
    auto kernel = dtype == B200_DTYPE_F32 ? residual_norm_kernel<float> : residual_norm_kernel<__nv_bfloat16>;
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(r.tokens), dim3(threads), 0, stream, dim3(1, 1, 1), a));
    return B200_OK;
}

}  // namespace b200

extern "C" {

int b200_residual_norm(void* out, const int32_t* out_rows, int out_top, float* residual, const void* src,
                       const int32_t* src_rows, int src_top, int64_t src_count, float src_scale, int init,
                       const void* weight, float weight_offset, float out_scale, int tokens, int width,
                       int padded, float eps, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0 && width > 0 && padded >= width && padded % 64 == 0, "residual_norm: bad shape");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "residual_norm: unknown dtype");
    B200_CHECK_ARG(out_top >= 1 && src_top >= 1, "residual_norm: bad row counts");
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(out && residual && weight, "residual_norm: NULL tensor");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    b200::ResidualNorm r;
    r.out = out;
    r.out_rows = out_rows;
    r.out_top = out_top;
    r.residual = residual;
    r.src = src;
    r.src_rows = src_rows;
    r.src_top = src_top;
    r.src_count = src_count;
    r.src_scale = src_scale;
    r.init = init != 0;
    r.weight = weight;
    r.weight_offset = weight_offset;
    r.out_scale = out_scale;
    r.tokens = tokens;
    r.width = width;
    r.padded = padded;
    r.eps = eps;
    return b200::launch_residual_norm(r, dtype, status, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
