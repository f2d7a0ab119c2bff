// fp32 GEMM on the CUDA cores for models that run in true fp32: plain, per-head and grouped (expert)
// forms of y = x W^T with the same epilogues as the tensor-core GEMMs.  64 x 64 output tiles, 4 x 4 per
// thread, 16-deep k steps through shared memory.
#include "common.cuh"
#include "kernels.h"

namespace b200 {
namespace {

constexpr int kTile = 64;
constexpr int kStep = 16;

struct F32Params {
    float* y;
    const float* x;
    const float* w;
    int M, n_out, K, w_rows;   // w_rows: rows of W per group
    int64_t x_pitch, y_pitch;
    const int32_t* counts;     // grouped mode
    const int32_t* offsets;
    int per_head;              // z selects a column block of x and y
    const float* bias;         // [n_out] or NULL, before the activation
    float act_limit;
};

__device__ __forceinline__ float gate_f32(int epi, float g) {
    if (epi == B200_EPILOGUE_SWIGLU) return g / (1.0f + expf(-g));
    if (epi == B200_EPILOGUE_GEGLU_ERF) return 0.5f * g * (1.0f + erff(g * 0.70710678118654752f));
    return 0.5f * g * (1.0f + tanhf(0.79788456080286536f * (g + 0.044715f * g * g * g)));
}

template <int EPI>
__global__ void __launch_bounds__(256)
linear_f32_kernel(const F32Params p) {
    constexpr bool GATED = epilogue_is_gated(EPI);
    __shared__ float sx[kStep][kTile + 4];
    __shared__ float sw[GATED ? 2 : 1][kStep][kTile + 4];
    pdl_launch_dependents();
    pdl_wait_prior();
    const int z = blockIdx.z;
    int rows = p.M, row0 = 0;
    if (p.counts) {
        rows = p.counts[z];
        row0 = p.offsets[z];
    }
    const int m0 = blockIdx.y * kTile, n0 = blockIdx.x * kTile;
    if (m0 >= rows) return;
    const float* x = p.x + static_cast<int64_t>(row0) * p.x_pitch + (p.per_head ? static_cast<int64_t>(z) * p.K : 0);
    const float* w = p.w + static_cast<int64_t>(z) * p.w_rows * p.K;
    float* y = p.y + static_cast<int64_t>(row0) * p.y_pitch + (p.per_head ? static_cast<int64_t>(z) * p.n_out : 0);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {}, up[GATED ? 4 : 1][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += kStep) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int idx = threadIdx.x + i * 256;
            const int r = idx >> 4, k = idx & 15;
            sx[k][r] = m0 + r < rows ? x[static_cast<int64_t>(m0 + r) * p.x_pitch + k0 + k] : 0.f;
            const bool in = n0 + r < p.n_out;
            sw[0][k][r] = in ? w[static_cast<int64_t>(n0 + r) * p.K + k0 + k] : 0.f;
            if (GATED) sw[GATED ? 1 : 0][k][r] = in ? w[static_cast<int64_t>(p.n_out + n0 + r) * p.K + k0 + k] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kStep; ++k) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[i] = sx[k][ty * 4 + i];
                b[i] = sw[0][k][tx * 4 + i];
            }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
            if (GATED) {
#pragma unroll
                for (int j = 0; j < 4; ++j) b[j] = sw[GATED ? 1 : 0][k][tx * 4 + j];
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) up[GATED ? i : 0][j] = fmaf(a[i], b[j], up[GATED ? i : 0][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int n = n0 + tx * 4 + j;
            if (n >= p.n_out) continue;
            float v = acc[i][j];
            if (p.bias != nullptr) v += p.bias[n];
            if (EPI == B200_EPILOGUE_CLAMPED_SWIGLU)
                v = clamped_swiglu<true>(v, up[GATED ? i : 0][j], p.act_limit);
            else if (GATED)
                v = gate_f32(EPI, v) * up[GATED ? i : 0][j];
            if (EPI == B200_EPILOGUE_GELU_ERF) v = gate_f32(B200_EPILOGUE_GEGLU_ERF, v);
            if (EPI == B200_EPILOGUE_RELU2) v = fmaxf(v, 0.f) * fmaxf(v, 0.f);
            y[static_cast<int64_t>(m) * p.y_pitch + n] = v;
        }
    }
}

}  // namespace

int launch_linear_f32(float* y, const float* x, const float* w, int max_rows, int N, int K, int groups,
                      const int32_t* counts, const int32_t* offsets, int epilogue, cudaStream_t stream,
                      float act_limit, const float* bias) {
    if (max_rows == 0 || groups == 0) return B200_OK;
    const bool per_head = counts == nullptr && groups > 1;
    F32Params p;
    p.y = y;
    p.x = x;
    p.w = w;
    p.M = max_rows;
    p.n_out = epilogue_is_gated(epilogue) ? N / 2 : N;
    p.K = K;
    p.w_rows = N;
    p.x_pitch = per_head ? static_cast<int64_t>(groups) * K : K;
    p.y_pitch = per_head ? static_cast<int64_t>(groups) * p.n_out : p.n_out;
    p.counts = counts;
    p.offsets = offsets;
    p.per_head = per_head ? 1 : 0;
    p.act_limit = act_limit;
    p.bias = bias;
    void (*kernel)(F32Params) = linear_f32_kernel<B200_EPILOGUE_NONE>;
    if (epilogue == B200_EPILOGUE_SWIGLU) kernel = linear_f32_kernel<B200_EPILOGUE_SWIGLU>;
    if (epilogue == B200_EPILOGUE_GEGLU) kernel = linear_f32_kernel<B200_EPILOGUE_GEGLU>;
    if (epilogue == B200_EPILOGUE_GEGLU_ERF) kernel = linear_f32_kernel<B200_EPILOGUE_GEGLU_ERF>;
    if (epilogue == B200_EPILOGUE_RELU2) kernel = linear_f32_kernel<B200_EPILOGUE_RELU2>;
    if (epilogue == B200_EPILOGUE_GELU_ERF) kernel = linear_f32_kernel<B200_EPILOGUE_GELU_ERF>;
    if (epilogue == B200_EPILOGUE_CLAMPED_SWIGLU) kernel = linear_f32_kernel<B200_EPILOGUE_CLAMPED_SWIGLU>;
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(div_ceil(p.n_out, kTile), div_ceil(max_rows, kTile), groups), dim3(256), 0,
                                  stream, dim3(1, 1, 1), p));
    return B200_OK;
}

}  // namespace b200

extern "C" {

int b200_linear_f32(float* y, const float* x, const float* w, int max_rows, int N, int K, int groups,
                    const int32_t* counts, const int32_t* offsets, int epilogue, b200_stream_t stream) {
    B200_CHECK_ARG(max_rows >= 0 && N > 0 && K > 0 && groups > 0 && groups <= 65535, "linear_f32: bad shape");
    B200_CHECK_ARG(K % 16 == 0, "linear_f32: K must be a multiple of 16");
    B200_CHECK_ARG((counts == nullptr) == (offsets == nullptr), "linear_f32: counts and offsets go together");
    B200_CHECK_ARG(epilogue >= B200_EPILOGUE_NONE && epilogue <= B200_EPILOGUE_RELU2, "linear_f32: unknown epilogue");
    B200_CHECK_ARG(!b200::epilogue_is_gated(epilogue) || N % 2 == 0, "linear_f32: a gated epilogue needs an even N");
    if (max_rows == 0) return B200_OK;
    B200_CHECK_ARG(y && x && w, "linear_f32: NULL tensor");
    B200_CHECK_ARG(max_rows <= 65535 * 64, "linear_f32: too many rows");
    return b200::launch_linear_f32(y, x, w, max_rows, N, K, groups, counts, offsets, epilogue,
                                   static_cast<cudaStream_t>(stream));
}

}  // extern "C"
