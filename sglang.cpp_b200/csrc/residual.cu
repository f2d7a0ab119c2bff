// The fp32 residual stream of a layer stack: one kernel adds what the previous block produced (an
// embedding row, a projection's output, or the weighted outputs of a token's experts), stores the sum and
// writes its RMS norm for the next block - to the token's own row, or straight into the expert-sorted
// rows that the next block's grouped GEMM reads.  One CTA per token, the row in registers.
//
// Wirings: the norm on what the next block reads (residual_norm_kernel), or on what the previous block
// returned, before it is added, or both (residual_post_norm_kernel, which also has layer norms).
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

struct PostArgs {
    void* out;
    float* residual;
    const void* src;
    const int32_t* src_rows;
    const float* src_weights;
    const void* src2;
    const void* pair_weight;
    const void* pair_weight2;
    float pair_scale;
    const void* add_weight;
    const void* out_weight;
    int64_t src_count;
    int src_top, init, width, padded;
    float weight_offset, out_scale, eps;
    int32_t* clear;
    int clear_count;
    int* status;
    const void *add_bias, *out_bias, *self;   // KIND kLayer
    float src_scale;                          // (kRms as well)
};
enum { kRms = 0, kPair = 1, kLayer = 2 };

// What is added is a token's row of the source, or the weighted rows src_rows names, plus its row of a second
// source (kPair: both normalised by themselves first, the sum scaled); it is normalised when there is a weight
// for it.  The sum goes to the residual and, rounded (or normalised once more), to `out`.  kLayer: the norms are
// layer norms, and a source row of -1 stands for the token's row of `self`.
template <typename T, int VEC, int KIND>
__global__ void __launch_bounds__(256)
residual_post_norm_kernel(const PostArgs a) {
    constexpr bool PAIR = KIND == kPair, LAYER = KIND == kLayer;
    __shared__ float red[KIND == kRms ? 2 : 4][8];
    __shared__ int s_row[kRows];
    __shared__ float s_weight[kRows];
    pdl_launch_dependents();
    const int nvec = a.padded >> 3;
    const T* add_weight = static_cast<const T*>(a.add_weight);
    const T* out_weight = static_cast<const T*>(a.out_weight);
    // the norm weights do not come from the kernel before this one
    Vec8 w[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < nvec && add_weight != nullptr) w[i] = load8(add_weight + v * 8);
    }
    pdl_wait_prior();
    const int64_t t = blockIdx.x;
    if (blockIdx.x == 0)
        for (int i = threadIdx.x; i < a.clear_count; i += blockDim.x) a.clear[i] = 0;
    if (a.src_rows != nullptr) {
        if (threadIdx.x < kRows && threadIdx.x < a.src_top) {
            s_row[threadIdx.x] = a.src_rows[t * a.src_top + threadIdx.x];
            s_weight[threadIdx.x] = a.src_weights != nullptr ? a.src_weights[t * a.src_top + threadIdx.x] : 1.f;
        }
        __syncthreads();
    }
    float* res = a.residual + t * a.padded;
    const T* src = static_cast<const T*>(a.src);
    const T* src2 = static_cast<const T*>(a.src2);
    float scale_a = 1.f, scale_b = 1.f;   // PAIR: one over the root mean square of either row
    auto addend = [&](int v) {
        Vec8 y;
        if (PAIR) {
            y = load8(src + t * a.padded + v * 8);
            const Vec8 x = load8(src2 + t * a.padded + v * 8);
            const Vec8 ga = load8(static_cast<const T*>(a.pair_weight) + v * 8), gb = load8(static_cast<const T*>(a.pair_weight2) + v * 8);
#pragma unroll
            for (int j = 0; j < 8; ++j) y.v[j] = a.pair_scale * (y.v[j] * scale_a * ga.v[j] + x.v[j] * scale_b * gb.v[j]);
            return y;
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) y.v[j] = 0.f;
        if (a.src_rows == nullptr) {
            y = load8(src + t * a.padded + v * 8);
        } else {
#pragma unroll 4
            for (int k = 0; k < a.src_top; ++k) {
                const int64_t row = k < kRows ? s_row[k] : a.src_rows[t * a.src_top + k];
                const float g = k < kRows ? s_weight[k] : a.src_weights != nullptr ? a.src_weights[t * a.src_top + k] : 1.f;
                if (LAYER && row == -1 && a.self != nullptr) {
                    const Vec8 x = load8(static_cast<const T*>(a.self) + t * a.padded + v * 8);
#pragma unroll
                    for (int j = 0; j < 8; ++j) y.v[j] += g * x.v[j];
                    continue;
                }
                if (row < 0 || row >= a.src_count) {   // adds nothing and is reported
                    if (v == 0) atomicExch(&a.status[kStatusBadIndex], static_cast<int>(row) + 1);
                    continue;
                }
                const Vec8 x = load8(src + row * a.padded + v * 8);
#pragma unroll
                for (int j = 0; j < 8; ++j) y.v[j] += g * x.v[j];
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) y.v[j] *= a.src_scale;
        if (src2 != nullptr) {
            const Vec8 x = load8(src2 + t * a.padded + v * 8);
#pragma unroll
            for (int j = 0; j < 8; ++j) y.v[j] += x.v[j];
        }
        return y;
    };
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    auto block_sum = [&](float x, float* scratch) {
        x = warp_sum(x);
        if (lane == 0) scratch[warp] = x;
        __syncthreads();
        return warp_sum(lane < static_cast<int>(blockDim.x >> 5) ? scratch[lane] : 0.f);
    };
    if (PAIR) {
        float sa = 0.f, sb = 0.f;
        for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
            const Vec8 x = load8(src + t * a.padded + v * 8), y = load8(src2 + t * a.padded + v * 8);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                sa += x.v[j] * x.v[j];
                sb += y.v[j] * y.v[j];
            }
        }
        scale_a = rsqrtf(block_sum(sa, red[PAIR ? 2 : 0]) / static_cast<float>(a.width) + a.eps);
        scale_b = rsqrtf(block_sum(sb, red[PAIR ? 3 : 0]) / static_cast<float>(a.width) + a.eps);
    }
    Vec8 val[VEC], add[VEC];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int j = 0; j < 8; ++j) val[i].v[j] = add[i].v[j] = 0.f;
        if (v < nvec) {
            if (!a.init) val[i] = load8(static_cast<const float*>(res) + v * 8);
            add[i] = addend(v);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += LAYER ? add[i].v[j] : add[i].v[j] * add[i].v[j];
    }
    // layer norms: the sum of a piece's squared deviations (the padding deviates from nothing)
    auto deviation = [&](const Vec8& x, int v, float mean) {
        float d = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j)
            if (v * 8 + j < a.width) d += (x.v[j] - mean) * (x.v[j] - mean);
        return d;
    };
    const T* add_bias = static_cast<const T*>(a.add_bias);
    const T* out_bias = static_cast<const T*>(a.out_bias);
    float mean = 0.f;
    const int wide0 = threadIdx.x + VEC * static_cast<int>(blockDim.x);   // rows wider than the registers
    float scale = 1.f;
    if (add_weight != nullptr) {
        for (int v = wide0; v < nvec; v += blockDim.x) {
            const Vec8 y = addend(v);
#pragma unroll
            for (int j = 0; j < 8; ++j) ss += LAYER ? y.v[j] : y.v[j] * y.v[j];
        }
        ss = block_sum(ss, red[0]);
        if (LAYER) {
            mean = ss / static_cast<float>(a.width);
            ss = 0.f;
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss += deviation(add[i], threadIdx.x + i * blockDim.x, mean);
            for (int v = wide0; v < nvec; v += blockDim.x) ss += deviation(addend(v), v, mean);
            ss = block_sum(ss, red[LAYER ? 2 : 0]);
        }
        scale = rsqrtf(ss / static_cast<float>(a.width) + a.eps);
    }
    float ss2 = 0.f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v >= nvec) continue;
        Vec8 shift;
#pragma unroll
        for (int j = 0; j < 8; ++j) shift.v[j] = 0.f;
        if (LAYER && add_weight != nullptr) shift = load8(add_bias + v * 8);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (LAYER) {
                val[i].v[j] += add_weight != nullptr ? fmaf((add[i].v[j] - mean) * scale, w[i].v[j], shift.v[j]) : add[i].v[j];
                ss2 += val[i].v[j];
            } else {
                val[i].v[j] += add_weight != nullptr ? add[i].v[j] * scale * (w[i].v[j] + a.weight_offset) : add[i].v[j];
                ss2 += val[i].v[j] * val[i].v[j];
            }
        }
        store8(res + v * 8, val[i]);
    }
    for (int v = wide0; v < nvec; v += blockDim.x) {
        const Vec8 y = addend(v);
        Vec8 x, g;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            x.v[j] = 0.f;
            g.v[j] = 1.f - a.weight_offset;
        }
        if (!a.init) x = load8(static_cast<const float*>(res) + v * 8);
        if (add_weight != nullptr) g = load8(add_weight + v * 8);
        if constexpr (LAYER) {
            Vec8 shift;
#pragma unroll
            for (int j = 0; j < 8; ++j) shift.v[j] = 0.f;
            if (add_weight != nullptr) shift = load8(add_bias + v * 8);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                x.v[j] += add_weight != nullptr ? fmaf((y.v[j] - mean) * scale, g.v[j], shift.v[j]) : y.v[j];
                ss2 += x.v[j];
            }
        } else {
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                x.v[j] += y.v[j] * scale * (g.v[j] + a.weight_offset);
                ss2 += x.v[j] * x.v[j];
            }
        }
        store8(res + v * 8, x);
    }
    float out_scale = 1.f;
    if (out_weight != nullptr) {
        ss2 = block_sum(ss2, red[1]);
        if (LAYER) {
            mean = ss2 / static_cast<float>(a.width);
            ss2 = 0.f;
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss2 += deviation(val[i], threadIdx.x + i * blockDim.x, mean);
            for (int v = wide0; v < nvec; v += blockDim.x) ss2 += deviation(load8(static_cast<const float*>(res) + v * 8), v, mean);
            ss2 = block_sum(ss2, red[LAYER ? 3 : 1]);
        }
        out_scale = rsqrtf(ss2 / static_cast<float>(a.width) + a.eps) * (LAYER ? 1.f : a.out_scale);
    }
    T* out = static_cast<T*>(a.out) + t * a.padded;
    auto emit = [&](int v, Vec8 x) {
        if (out_weight != nullptr) {
            const Vec8 g = load8(out_weight + v * 8);
            if (LAYER) {
                const Vec8 shift = load8(out_bias + v * 8);
#pragma unroll
                for (int j = 0; j < 8; ++j) x.v[j] = fmaf((x.v[j] - mean) * out_scale, g.v[j], shift.v[j]);
            } else {
#pragma unroll
                for (int j = 0; j < 8; ++j) x.v[j] *= out_scale * (g.v[j] + a.weight_offset);
            }
        }
        store8(out + v * 8, x);
    };
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < nvec) emit(v, val[i]);
    }
    for (int v = wide0; v < nvec; v += blockDim.x) emit(v, load8(static_cast<const float*>(res) + v * 8));
}

template <typename T, int KIND>
auto post_kernel_for(int pieces) {
    return pieces <= 1 ? residual_post_norm_kernel<T, 1, KIND>
                       : pieces <= 2 ? residual_post_norm_kernel<T, 2, KIND> : residual_post_norm_kernel<T, 4, KIND>;
}
template <typename T>
auto post_kernel_for(const ResidualPostNorm& r, int pieces) {
    return r.layer ? post_kernel_for<T, kLayer>(pieces)
                   : r.pair_weight != nullptr ? post_kernel_for<T, kPair>(pieces) : post_kernel_for<T, kRms>(pieces);
}

}  // namespace

int launch_residual_post_norm(const ResidualPostNorm& r, int dtype, int* status, cudaStream_t stream) {
    if (r.tokens == 0) return B200_OK;
    PostArgs a;
    a.out = r.out;
    a.residual = r.residual;
    a.src = r.src;
    a.src_rows = r.src_rows;
    a.src_weights = r.src_weights;
    a.src2 = r.src2;
    a.pair_weight = r.pair_weight;
    a.pair_weight2 = r.pair_weight2;
    a.pair_scale = r.pair_scale;
    a.add_weight = r.add_weight;
    a.out_weight = r.out_weight;
    a.src_count = r.src_count;
    a.src_top = r.src_rows ? r.src_top : 1;
    a.init = r.init ? 1 : 0;
    a.width = r.width;
    a.padded = r.padded;
    a.weight_offset = r.weight_offset;
    a.out_scale = r.out_scale;
    a.eps = r.eps;
    a.clear = r.clear;
    a.clear_count = r.clear ? r.clear_count : 0;
    a.status = status;
    int threads = 32;
    while (threads < 256 && threads * 8 < r.padded) threads *= 2;
    const int pieces = div_ceil(r.padded, threads * 8);
    a.add_bias = r.add_bias;
    a.out_bias = r.out_bias;
    a.self = r.self;
    a.src_scale = r.init ? r.src_scale : 1.f;
    auto kernel = dtype == B200_DTYPE_F32 ? post_kernel_for<float>(r, pieces) : post_kernel_for<__nv_bfloat16>(r, pieces);
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(r.tokens), dim3(threads), 0, stream, dim3(1, 1, 1), a));
    return B200_OK;
}

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

int b200_residual_post_norm(void* out, float* residual, const void* src, const int32_t* src_rows,
                            const float* src_weights, int src_top, int64_t src_count, const void* src2, int init,
                            const void* add_weight, const void* out_weight, int tokens, int width, int padded,
                            float eps, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0 && width > 0 && padded >= width && padded % 64 == 0, "residual_post_norm: bad shape");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "residual_post_norm: unknown dtype");
    B200_CHECK_ARG(src_top >= 1, "residual_post_norm: bad row count");
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(out && residual && src, "residual_post_norm: NULL tensor");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    b200::ResidualPostNorm r;
    r.out = out;
    r.residual = residual;
    r.src = src;
    r.src_rows = src_rows;
    r.src_weights = src_weights;
    r.src_top = src_top;
    r.src_count = src_count;
    r.src2 = src2;
    r.init = init != 0;
    r.add_weight = add_weight;
    r.out_weight = out_weight;
    r.tokens = tokens;
    r.width = width;
    r.padded = padded;
    r.eps = eps;
    return b200::launch_residual_post_norm(r, dtype, status, static_cast<cudaStream_t>(stream));
}

int b200_residual_layer_norm(void* out, float* residual, const void* src, const int32_t* src_rows,
                             const float* src_weights, int src_top, int64_t src_count, const void* self, float src_scale,
                             int init, const void* add_weight, const void* add_bias, const void* out_weight,
                             const void* out_bias, int tokens, int width, int padded, float eps, int dtype,
                             b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0 && width > 0 && padded >= width && padded % 64 == 0, "residual_layer_norm: bad shape");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "residual_layer_norm: unknown dtype");
    B200_CHECK_ARG(src_top >= 1, "residual_layer_norm: bad row count");
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(out && residual && src && (!add_weight || add_bias) && (!out_weight || out_bias),
                   "residual_layer_norm: NULL tensor");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    b200::ResidualPostNorm r;
    r.layer = true;
    r.out = out;
    r.residual = residual;
    r.src = src;
    r.src_rows = src_rows;
    r.src_weights = src_weights;
    r.src_top = src_top;
    r.src_count = src_count;
    r.self = self;
    r.src_scale = src_scale;
    r.init = init != 0;
    r.add_weight = add_weight;
    r.add_bias = add_bias;
    r.out_weight = out_weight;
    r.out_bias = out_bias;
    r.tokens = tokens;
    r.width = width;
    r.padded = padded;
    r.eps = eps;
    return b200::launch_residual_post_norm(r, dtype, status, static_cast<cudaStream_t>(stream));
}

int b200_residual_pair_norm(void* out, float* residual, const void* src, const void* src2, const void* weight,
                            const void* weight2, float pair_scale, const void* add_weight, const void* out_weight,
                            int tokens, int width, int padded, float eps, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0 && width > 0 && padded >= width && padded % 64 == 0, "residual_pair_norm: bad shape");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "residual_pair_norm: unknown dtype");
    if (tokens == 0) return B200_OK;
    B200_CHECK_ARG(out && residual && src && src2 && weight && weight2, "residual_pair_norm: NULL tensor");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    b200::ResidualPostNorm r;
    r.out = out;
    r.residual = residual;
    r.src = src;
    r.src_count = tokens;
    r.src2 = src2;
    r.pair_weight = weight;
    r.pair_weight2 = weight2;
    r.pair_scale = pair_scale;
    r.add_weight = add_weight;
    r.out_weight = out_weight;
    r.tokens = tokens;
    r.width = width;
    r.padded = padded;
    r.eps = eps;
    return b200::launch_residual_post_norm(r, dtype, status, static_cast<cudaStream_t>(stream));
}

}  // extern "C"
