// Attention over a shared low-rank latent: the paged latent pool, the plain attention kernel, and the
// gathers that feed the expanded form.
//
// One row of `width` numbers per token is key and value of every head at once.  With the per-head
// up-projections moved to the other side of the products (k_h = U_h c  =>  q_h . k_h = (U_h^T q_h) . c,
// and sum_j p_j (V_h c_j) = V_h sum_j p_j c_j) attention runs in the latent space and reads one latent per
// token whatever the number of heads: that is the form decode steps and short extensions take.  Long
// extensions expand keys and values once per step instead (layer_stack.cu), which costs fewer
// multiplications per query.
#include <math.h>

#include "common.cuh"
#include "kernels.h"

namespace b200 {
namespace {

template <typename T>
__device__ __forceinline__ float as_float(T v);
template <>
__device__ __forceinline__ float as_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ float as_float<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Columns [0, qp) of a token's joint row are its query latent, [qp, qp + rp) its key/value latent; each is
// divided by its own root mean square (over the true widths) and scaled by its own weight, but for the part of
// the key/value latent that turns with the position instead.  One warp per latent: warps 0 and 1 of a pair take
// the two latents of one token, four tokens per CTA, the row in registers (latents of up to kKeep x 256 elements;
// wider ones are read again).
template <typename T, int kKeep>
__global__ void __launch_bounds__(256)
latent_norm_store_kernel(const LatentNorm a) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int64_t t = static_cast<int64_t>(blockIdx.x) * (blockDim.x >> 6) + (warp >> 1);
    if (t >= a.tokens) return;
    const bool kv = (warp & 1) != 0;
    if (kv && a.cache == nullptr) return;
    const T* src = static_cast<const T*>(a.joint) + t * (a.qp + a.rp) + (kv ? a.qp : 0);
    const T* weight = static_cast<const T*>(kv ? a.kv_weight : a.q_weight);
    const int nvec = (kv ? a.rp : a.qp) >> 3;
    const int rope0 = kv && a.rope_dim > 0 ? a.rope_at >> 3 : nvec;   // the first vector that turns
    int64_t slot = 0;
    if (kv) slot = a.out_loc[t];
    int pos = kv && a.rope_dim > 0 ? a.positions[t] : 0;
    if (pos < 0 || pos >= a.max_pos) {
        if (lane == 0) atomicExch(&a.status[kStatusBadIndex], pos + 1);
        pos = min(max(pos, 0), a.max_pos - 1);
    }
    Vec8 x[kKeep];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
        const int v = lane + i * 32;
        if (v < nvec) {
            x[i] = load8(src + v * 8);
#pragma unroll
            for (int j = 0; j < 8; ++j) ss += v < rope0 ? x[i].v[j] * x[i].v[j] : 0.f;
        }
    }
    for (int v = lane + kKeep * 32; v < rope0; v += 32) {
        const Vec8 y = load8(src + v * 8);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += y.v[j] * y.v[j];
    }
    const float r = rsqrtf(warp_sum(ss) / static_cast<float>(kv ? a.kv_rank : a.q_rank) + a.eps);
    T* dst = static_cast<T*>(a.q_latent) + t * a.qp;
    if (kv) {
        if (slot < 0 || slot >= a.num_slots) {
            if (lane == 0) atomicExch(&a.status[kStatusBadIndex], static_cast<int>(slot) + 1);
            return;
        }
        dst = static_cast<T*>(a.cache) + slot * a.rp;
    }
    auto emit = [&](int v, const Vec8& y) {
        Vec8 o;
        if (v < rope0) {
            const Vec8 g = load8(weight + v * 8);
#pragma unroll
            for (int j = 0; j < 8; ++j) o.v[j] = y.v[j] * r * g.v[j];
        } else {
            const int half = a.rope_dim >> 1, pair0 = (v - rope0) * 4;
            const float* ct = a.cos_t + static_cast<int64_t>(pos) * half + pair0;
            const float* st = a.sin_t + static_cast<int64_t>(pos) * half + pair0;
            float c[4] = {0.f, 0.f, 0.f, 0.f}, s[4] = {0.f, 0.f, 0.f, 0.f};
            if (half % 4 == 0) {
                if (pair0 < half) {
                    const float4 c4 = *reinterpret_cast<const float4*>(ct), s4 = *reinterpret_cast<const float4*>(st);
                    c[0] = c4.x, c[1] = c4.y, c[2] = c4.z, c[3] = c4.w;
                    s[0] = s4.x, s[1] = s4.y, s[2] = s4.z, s[3] = s4.w;
                }
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (pair0 + j < half) {
                        c[j] = ct[j];
                        s[j] = st[j];
                    }
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                o.v[2 * j] = y.v[2 * j] * c[j] - y.v[2 * j + 1] * s[j];
                o.v[2 * j + 1] = y.v[2 * j + 1] * c[j] + y.v[2 * j] * s[j];
            }
        }
        store8(dst + v * 8, o);
    };
#pragma unroll
    for (int i = 0; i < kKeep; ++i)
        if (lane + i * 32 < nvec) emit(lane + i * 32, x[i]);
    for (int v = lane + kKeep * 32; v < nvec; v += 32) emit(v, load8(src + v * 8));
}

// One thread per 8 elements of a head's rotated part.
template <typename T>
__global__ void __launch_bounds__(256)
rotate_pairs_kernel(T* __restrict__ x, int64_t count, int vecs, int heads, int ld, int dims, const float* __restrict__ cos_t,
                    const float* __restrict__ sin_t, const int32_t* __restrict__ positions, int max_pos, int* status) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i >= count) return;
    const int64_t row = i / vecs;
    const int v = static_cast<int>(i - row * vecs), half = dims >> 1;
    int pos = positions[row / heads];
    if (pos < 0 || pos >= max_pos) {
        atomicExch(&status[kStatusBadIndex], pos + 1);
        pos = min(max(pos, 0), max_pos - 1);
    }
    T* p = x + row * ld + v * 8;
    Vec8 y = load8(p);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int pair = v * 4 + j;
        if (pair >= half) break;
        const float c = cos_t[static_cast<int64_t>(pos) * half + pair], s = sin_t[static_cast<int64_t>(pos) * half + pair];
        const float a = y.v[2 * j], b = y.v[2 * j + 1];
        y.v[2 * j] = a * c - b * s;
        y.v[2 * j + 1] = b * c + a * s;
    }
    store8(p, y);
}

// One CTA per (query row, head); its warps take every fourth key each with an online softmax whose
// output row is in shared memory, and merge at the end.  Any width, either dtype; not built for speed.
template <typename T>
__global__ void __launch_bounds__(128)
latent_attention_plain_kernel(T* __restrict__ out, const T* __restrict__ q, const T* __restrict__ cache,
                              int64_t num_slots, const int32_t* __restrict__ page_table, int64_t pt_stride,
                              const int32_t* __restrict__ row_table, const int32_t* __restrict__ row_len, int heads,
                              int width, int out_width, float scale, int* status) {
    extern __shared__ float smem[];   // q [width], then o [4][width]
    __shared__ float s_m[4], s_l[4];
    pdl_launch_dependents();
    pdl_wait_prior();
    const int64_t row = blockIdx.x;
    const int h = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* sq = smem;
    float* so = smem + (1 + warp) * width;
    const T* qr = q + (row * heads + h) * width;
    for (int i = threadIdx.x; i < width; i += blockDim.x) sq[i] = as_float(qr[i]);
    for (int i = lane; i < out_width; i += 32) so[i] = 0.f;
    __syncthreads();
    const int32_t* pt = page_table + static_cast<int64_t>(row_table[row]) * pt_stride;
    const int len = row_len[row];
    float m = -INFINITY, l = 0.f;
    for (int j = warp; j < len; j += 4) {
        int64_t slot = pt[j];
        if (slot < 0 || slot >= num_slots) {
            if (lane == 0) atomicExch(&status[kStatusBadIndex], static_cast<int>(slot) + 1);
            slot = 0;
        }
        const T* c = cache + slot * width;
        float s = 0.f;
        for (int i = lane; i < width; i += 32) s = fmaf(sq[i], as_float(c[i]), s);
        s = warp_sum(s) * scale;
        const float m_new = fmaxf(m, s);
        const float alpha = expf(m - m_new), p = expf(s - m_new);
        l = l * alpha + p;
        m = m_new;
        for (int i = lane; i < out_width; i += 32) so[i] = so[i] * alpha + p * as_float(c[i]);
    }
    if (lane == 0) {
        s_m[warp] = m;
        s_l[warp] = l;
    }
    __syncthreads();
    float mx = -INFINITY, tot = 0.f, f[4];
#pragma unroll
    for (int w = 0; w < 4; ++w) mx = fmaxf(mx, s_m[w]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
        f[w] = s_m[w] == -INFINITY ? 0.f : expf(s_m[w] - mx);
        tot += f[w] * s_l[w];
    }
    const float inv = tot > 0.f ? 1.f / tot : 0.f;
    for (int i = threadIdx.x; i < out_width; i += blockDim.x) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) v += f[w] * smem[(1 + w) * width + i];
        put(out + (row * heads + h) * out_width + i, v * inv);
    }
}

__global__ void __launch_bounds__(256)
gather_latents_kernel(uint4* __restrict__ out, const uint4* __restrict__ cache, int64_t num_slots,
                      const int32_t* __restrict__ page_table, int64_t pt_stride,
                      const int32_t* __restrict__ table_idx, const int32_t* __restrict__ seq_lens,
                      const int32_t* __restrict__ base, int vec_per_row, int* status) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int b = blockIdx.y;
    const int at = base[b];
    const int len = seq_lens[b];
    if (at < 0) return;
    const int32_t* pt = page_table + static_cast<int64_t>(table_idx[b]) * pt_stride;
    const int64_t total = static_cast<int64_t>(len) * vec_per_row;
    for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
         i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
        const int64_t pos = i / vec_per_row;
        const int v = static_cast<int>(i - pos * vec_per_row);
        int64_t slot = pt[pos];
        if (slot < 0 || slot >= num_slots) {
            if (v == 0) atomicExch(&status[kStatusBadIndex], static_cast<int>(slot) + 1);
            slot = 0;
        }
        out[(at + pos) * vec_per_row + v] = cache[slot * vec_per_row + v];
    }
}

template <bool SCATTER>
__global__ void __launch_bounds__(128)
move_rows_kernel(uint4* __restrict__ out, const uint4* __restrict__ in, const int32_t* __restrict__ rows,
                 int vec_per_row) {
    pdl_launch_dependents();
    pdl_wait_prior();
    const int64_t i = blockIdx.x, r = rows[i];
    const uint4* src = in + (SCATTER ? i : r) * vec_per_row;
    uint4* dst = out + (SCATTER ? r : i) * vec_per_row;
    for (int v = threadIdx.x; v < vec_per_row; v += blockDim.x) dst[v] = src[v];
}

}  // namespace

int launch_latent_norm_store(const LatentNorm& a, int dtype, cudaStream_t stream) {
    if (a.tokens == 0) return B200_OK;
    // few tokens: a CTA each, for latency; many: four per CTA
    const int threads = a.tokens <= 2 * sm_count() ? 64 : 256;
    const int grid = div_ceil(a.tokens, threads / 64);
    const bool f32 = dtype == B200_DTYPE_F32;
    const int widest = a.qp > a.rp ? a.qp : a.rp;
    auto kernel = widest <= 512    ? (f32 ? latent_norm_store_kernel<float, 2> : latent_norm_store_kernel<__nv_bfloat16, 2>)
                  : widest <= 1024 ? (f32 ? latent_norm_store_kernel<float, 4> : latent_norm_store_kernel<__nv_bfloat16, 4>)
                                   : (f32 ? latent_norm_store_kernel<float, 8> : latent_norm_store_kernel<__nv_bfloat16, 8>);
    B200_CHECK_CUDA(launch_kernel(kernel, dim3(grid), dim3(threads), 0, stream, dim3(1, 1, 1), a));
    return B200_OK;
}

int launch_rotate_pairs(void* x, int tokens, int heads, int ld, int dims, const float* cos_t, const float* sin_t,
                        const int32_t* positions, int max_pos, int dtype, int* status, cudaStream_t stream) {
    if (tokens == 0 || dims == 0) return B200_OK;
    const int vecs = div_ceil(dims, 8);
    const int64_t count = static_cast<int64_t>(tokens) * heads * vecs;
    const dim3 grid(static_cast<unsigned>(div_ceil64(count, 256)));
    auto run = [&](auto* p) -> int {
        using T = typename std::remove_pointer<decltype(p)>::type;
        B200_CHECK_CUDA(launch_kernel(rotate_pairs_kernel<T>, grid, dim3(256), 0, stream, dim3(1, 1, 1), p, count, vecs, heads,
                                      ld, dims, cos_t, sin_t, positions, max_pos, status));
        return B200_OK;
    };
    return dtype == B200_DTYPE_F32 ? run(static_cast<float*>(x)) : run(static_cast<__nv_bfloat16*>(x));
}

int launch_latent_attention_plain(const LatentAttention& a, int dtype, int* status, cudaStream_t stream) {
    if (a.rows == 0) return B200_OK;
    const int smem = 5 * a.width * static_cast<int>(sizeof(float));
    if (smem > 200 * 1024 || a.heads > 65535) {
        set_last_error("latent attention: width %d or %d heads exceed the plain kernel", a.width, a.heads);
        return B200_ERR_UNSUPPORTED;
    }
    auto run = [&](auto* tag) -> int {
        using T = typename std::remove_pointer<decltype(tag)>::type;
        auto kernel = latent_attention_plain_kernel<T>;
        B200_CHECK_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        B200_CHECK_CUDA(launch_kernel(kernel, dim3(a.rows, a.heads), dim3(128), smem, stream, dim3(1, 1, 1),
                                      static_cast<T*>(a.out), static_cast<const T*>(a.q),
                                      static_cast<const T*>(a.cache), a.num_slots, a.page_table, a.pt_stride,
                                      a.row_table, a.row_len, a.heads, a.width, a.out_width > 0 ? a.out_width : a.width, a.scale,
                                      status));
        return B200_OK;
    };
    return dtype == B200_DTYPE_F32 ? run(static_cast<float*>(nullptr)) : run(static_cast<__nv_bfloat16*>(nullptr));
}

int launch_gather_latents(void* out, const void* cache, int64_t num_slots, const int32_t* page_table,
                          int64_t pt_stride, const int32_t* table_idx, const int32_t* seq_lens,
                          const int32_t* base, int batch, int max_len, int rp, int* status, cudaStream_t stream) {
    if (batch == 0 || max_len == 0) return B200_OK;
    const int vec = rp / 8;
    const int64_t blocks = div_ceil64(static_cast<int64_t>(max_len) * vec, 256);
    B200_CHECK_CUDA(launch_kernel(gather_latents_kernel, dim3(static_cast<unsigned>(blocks < 592 ? blocks : 592), batch),
                                  dim3(256), 0, stream, dim3(1, 1, 1), static_cast<uint4*>(out),
                                  static_cast<const uint4*>(cache), num_slots, page_table, pt_stride, table_idx,
                                  seq_lens, base, vec, status));
    return B200_OK;
}

int launch_move_rows(void* out, const void* in, const int32_t* rows, int count, int vec_per_row, bool scatter,
                     cudaStream_t stream) {
    if (count == 0) return B200_OK;
    B200_CHECK_CUDA(launch_kernel(scatter ? move_rows_kernel<true> : move_rows_kernel<false>, dim3(count), dim3(128), 0,
                                  stream, dim3(1, 1, 1), static_cast<uint4*>(out), static_cast<const uint4*>(in), rows,
                                  vec_per_row));
    return B200_OK;
}

}  // namespace b200

extern "C" {

int64_t b200_latent_attention_workspace_bytes(int rows, int heads, int width) {
    if (rows < 0 || heads <= 0 || width <= 0) return -1;
    return b200::latent_attention_workspace_bytes(rows, heads, width);
}

int b200_latent_attention(void* out, const void* q, const void* cache, int64_t num_slots, const int32_t* page_table,
                          int64_t page_table_stride, const int32_t* row_table, const int32_t* row_len, int rows,
                          int heads, int width, int page_size, float scale, int dtype, int plain, void* workspace,
                          int64_t workspace_bytes, b200_stream_t stream) {
    return b200_latent_attention_part(out, q, cache, num_slots, page_table, page_table_stride, row_table, row_len, rows, heads,
                                      width, width, page_size, scale, dtype, plain, workspace, workspace_bytes, stream);
}

int b200_latent_attention_part(void* out, const void* q, const void* cache, int64_t num_slots, const int32_t* page_table,
                               int64_t page_table_stride, const int32_t* row_table, const int32_t* row_len, int rows,
                               int heads, int width, int out_width, int page_size, float scale, int dtype, int plain,
                               void* workspace, int64_t workspace_bytes, b200_stream_t stream) {
    B200_CHECK_ARG(out_width > 0 && out_width <= width && out_width % 128 == 0, "latent_attention: bad output width");
    B200_CHECK_ARG(rows >= 0 && heads > 0 && width > 0 && width % 128 == 0 && num_slots > 0,
                   "latent_attention: bad shape");
    B200_CHECK_ARG(page_size >= 1 && (page_size & (page_size - 1)) == 0, "latent_attention: page_size must be a power of two");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "latent_attention: unknown dtype");
    if (rows == 0) return B200_OK;
    B200_CHECK_ARG(out && q && cache && page_table && row_table && row_len, "latent_attention: NULL tensor");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    b200::LatentAttention a;
    a.out = out;
    a.q = q;
    a.cache = cache;
    a.num_slots = num_slots;
    a.page_table = page_table;
    a.pt_stride = page_table_stride;
    a.row_table = row_table;
    a.row_len = row_len;
    a.rows = rows;
    a.heads = heads;
    a.width = width;
    a.out_width = out_width;
    a.page_size = page_size;
    a.scale = scale;
    a.workspace = workspace;
    a.workspace_bytes = workspace_bytes;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == B200_DTYPE_BF16 && !plain && b200::latent_attention_tc_supported(a)) {
        B200_CHECK_ARG(workspace && workspace_bytes >= b200::latent_attention_workspace_bytes(rows, heads, width),
                       "latent_attention: workspace too small");
        return b200::launch_latent_attention_tc(a, status, s);
    }
    return b200::launch_latent_attention_plain(a, dtype, status, s);
}

int b200_rotate_pairs(void* x, int tokens, int heads, int ld, int dims, const float* cos_table, const float* sin_table,
                      const int32_t* positions, int max_pos, int dtype, b200_stream_t stream) {
    B200_CHECK_ARG(tokens >= 0 && heads > 0 && ld > 0 && ld % 8 == 0 && dims >= 0 && dims % 2 == 0 && dims <= ld && max_pos > 0,
                   "rotate_pairs: bad shape");
    B200_CHECK_ARG(dtype == B200_DTYPE_BF16 || dtype == B200_DTYPE_F32, "rotate_pairs: unknown dtype");
    if (tokens == 0 || dims == 0) return B200_OK;
    B200_CHECK_ARG(x && cos_table && sin_table && positions, "rotate_pairs: NULL tensor");
    int err = B200_OK;
    int* status = b200::device_status_words(&err);
    if (err != B200_OK) return err;
    return b200::launch_rotate_pairs(x, tokens, heads, ld, dims, cos_table, sin_table, positions, max_pos, dtype, status,
                                     static_cast<cudaStream_t>(stream));
}

}  // extern "C"
