// The fp32 residual stream of a layer stack: one kernel adds what the previous block produced (an
// embedding row, a projection's output, or the weighted outputs of a token's experts), stores the sum and
// writes its RMS norm for the next block - to the token's own row, or straight into the expert-sorted
// rows that the next block's grouped GEMM reads.  One CTA per token, the row in registers.
#include "common.cuh"
#include "kernels.h"

namespace b200 {
namespace {

// A thread works on pieces of 8 elements; it keeps up to VEC of them, wider rows are read again.
constexpr int kRows = 16;   // row numbers of a token kept in shared memory; wider choices are read from global

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

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
residual_norm_kernel(const Args a) {
    __shared__ float red[8];
    __shared__ int s_src[kRows], s_out[kRows];
    pdl_launch_dependents();
    const int nvec = a.padded >> 3;
    const T* weight = static_cast<const T*>(a.weight);
    // the norm weights do not come from the kernel before this one
    Vec8 w[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < nvec) w[i] = load8(weight + v * 8);
    }
    pdl_wait_prior();
    const int64_t t = blockIdx.x;
    if (a.src_rows != nullptr || a.out_rows != nullptr) {
        if (threadIdx.x < kRows) {
            const int k = threadIdx.x;
            if (a.src_rows != nullptr && k < a.src_top) s_src[k] = a.src_rows[t * a.src_top + k];
            if (a.out_rows != nullptr && k < a.out_top) s_out[k] = a.out_rows[t * a.out_top + k];
        }
        __syncthreads();
    }
    float* res = a.residual + t * a.padded;
    const T* src = static_cast<const T*>(a.src);
    // row k of what is added; a row outside the source adds nothing and is reported
    auto src_row = [&](int k) -> int64_t {
        if (a.src_rows == nullptr) return t;
        const int64_t row = k < kRows ? s_src[k] : a.src_rows[t * a.src_top + k];
        if (row >= 0 && row < a.src_count) return row;
        if (threadIdx.x == 0) atomicExch(&a.status[kStatusBadIndex], static_cast<int>(row) + 1);
        return -1;
    };
    Vec8 val[VEC], add[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int j = 0; j < 8; ++j) val[i].v[j] = add[i].v[j] = 0.f;
        if (v < nvec && !a.init) val[i] = load8(static_cast<const float*>(res) + v * 8);
    }
    if (src != nullptr) {
#pragma unroll 4
        for (int k = 0; k < a.src_top; ++k) {
            const int64_t row = src_row(k);
            if (row < 0) continue;
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                const int v = threadIdx.x + i * blockDim.x;
                if (v < nvec) {
                    const Vec8 x = load8(src + row * a.padded + v * 8);
#pragma unroll
                    for (int j = 0; j < 8; ++j) add[i].v[j] += x.v[j];
                }
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            val[i].v[j] += a.src_scale * add[i].v[j];
            ss += val[i].v[j] * val[i].v[j];
        }
        if (v < nvec && src != nullptr) store8(res + v * 8, val[i]);
    }
    for (int v = threadIdx.x + VEC * blockDim.x; v < nvec; v += blockDim.x) {   // rows wider than the registers
        Vec8 x, y;
#pragma unroll
        for (int j = 0; j < 8; ++j) x.v[j] = y.v[j] = 0.f;
        if (!a.init) x = load8(static_cast<const float*>(res) + v * 8);
        for (int k = 0; src != nullptr && k < a.src_top; ++k) {
            const int64_t row = src_row(k);
            if (row < 0) continue;
            const Vec8 z = load8(src + row * a.padded + v * 8);
#pragma unroll
            for (int j = 0; j < 8; ++j) y.v[j] += z.v[j];
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            x.v[j] += a.src_scale * y.v[j];
            ss += x.v[j] * x.v[j];
        }
        store8(res + v * 8, x);
    }
    ss = warp_sum(ss);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = warp_sum(lane < static_cast<int>(blockDim.x >> 5) ? red[lane] : 0.f);
    const float scale = rsqrtf(ss / static_cast<float>(a.width) + a.eps) * a.out_scale;
    T* out = static_cast<T*>(a.out);
    auto emit = [&](int v, const Vec8& x, const Vec8& g) {
        Vec8 y;
#pragma unroll
        for (int j = 0; j < 8; ++j) y.v[j] = x.v[j] * scale * (g.v[j] + a.weight_offset);
        if (a.out_rows == nullptr) {
            store8(out + t * a.padded + v * 8, y);
            return;
        }
        for (int k = 0; k < a.out_top; ++k) {
            const int64_t row = k < kRows ? s_out[k] : a.out_rows[t * a.out_top + k];
            store8(out + row * a.padded + v * 8, y);
        }
    };
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < nvec) emit(v, val[i], w[i]);
    }
    for (int v = threadIdx.x + VEC * blockDim.x; v < nvec; v += blockDim.x)
        emit(v, load8(static_cast<const float*>(res) + v * 8), load8(weight + v * 8));
}

template <typename T>
auto kernel_for(int pieces) {   // pieces of 8 elements per thread
    return pieces <= 1 ? residual_norm_kernel<T, 1> : pieces <= 2 ? residual_norm_kernel<T, 2> : residual_norm_kernel<T, 4>;
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
    int threads = 32;
    while (threads < 256 && threads * 8 < r.padded) threads *= 2;
    const int pieces = div_ceil(r.padded, threads * 8);
    auto kernel = dtype == B200_DTYPE_F32 ? kernel_for<float>(pieces) : kernel_for<__nv_bfloat16>(pieces);
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
