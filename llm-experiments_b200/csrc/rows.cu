// Row operations around a 32-bit residual stream: the token rows that start it, RMS norms that read it, and layer norms that
// read it or add a sublayer's normed output to it.
// These kernels may be scheduled ahead of the end of the kernel that writes their inputs, so no pointer to such data is
// const __restrict__: the compiler would take it for data that nothing writes and could load it before the wait.
#include "b2kv_common.cuh"

namespace b2kv {
namespace {

constexpr int kThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kThreads) embed_rows_kernel(const T* table, const int32_t* ids,
                                                              float* out, T* copy, float scale, int dim, int vocab,
                                                              int32_t* dev_status) {
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    int id = ids[blockIdx.x];
    if (id < 0 || id >= vocab) {
        if (threadIdx.x == 0) report_status(dev_status, B2KV_DEV_BAD_TOKEN);
        id = id < 0 ? 0 : vocab - 1;
    }
    const T* src = table + static_cast<int64_t>(id) * dim;
    float* dst = out + static_cast<int64_t>(blockIdx.x) * dim;
    T* cp = copy == nullptr ? nullptr : copy + static_cast<int64_t>(blockIdx.x) * dim;
    for (int i = threadIdx.x; i < dim; i += kThreads) {
        const float v = Elt<T>::to_float(src[i]) * scale;
        dst[i] = v;
        if (cp != nullptr) cp[i] = Elt<T>::from_float(v);
    }
}

__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const uint32_t*>(&lo);
    u.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
}

// One CTA per row; a row of up to 1024 * kKeep elements stays in registers between the two passes.
template <typename T, int kKeep>
__global__ void __launch_bounds__(kThreads) rmsnorm_kernel(const float* x, int64_t ld_x,
                                                           const int32_t* row_index, const float* w,
                                                           float w_offset, T* out, int64_t ld_out, int size,
                                                           float eps, bool vec) {
    __shared__ float part[kThreads / 32];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int64_t row = row_index ? row_index[blockIdx.x] : static_cast<int>(blockIdx.x);
    const float* xr = x + row * ld_x;
    T* yr = out + static_cast<int64_t>(blockIdx.x) * ld_out;
    const int chunks = vec ? size / 4 : 0;
    float4 keep[kKeep];
    float sum = 0.f;
    if (vec) {
#pragma unroll
        for (int c = 0; c < kKeep; ++c) {
            const int i = threadIdx.x + c * kThreads;
            if (i < chunks) {
                keep[c] = reinterpret_cast<const float4*>(xr)[i];
                sum += (keep[c].x * keep[c].x + keep[c].y * keep[c].y) + (keep[c].z * keep[c].z + keep[c].w * keep[c].w);
            }
        }
    } else {
        for (int i = threadIdx.x; i < size; i += kThreads) sum = fmaf(xr[i], xr[i], sum);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sum;
    __syncthreads();
    sum = 0.f;
#pragma unroll
    for (int i = 0; i < kThreads / 32; ++i) sum += part[i];
    const float scale = 1.0f / sqrtf(sum / static_cast<float>(size) + eps);
    if (vec) {
#pragma unroll
        for (int c = 0; c < kKeep; ++c) {
            const int i = threadIdx.x + c * kThreads;
            if (i < chunks) {
                const float4 wv = reinterpret_cast<const float4*>(w)[i];
                float4 v = keep[c];
                v.x *= scale * (wv.x + w_offset), v.y *= scale * (wv.y + w_offset);
                v.z *= scale * (wv.z + w_offset), v.w *= scale * (wv.w + w_offset);
                store4(yr + 4 * i, v);
            }
        }
    } else {
        for (int i = threadIdx.x; i < size; i += kThreads) yr[i] = Elt<T>::from_float(xr[i] * scale * (w[i] + w_offset));
    }
}

template <typename T>
int launch_rmsnorm(const float* x, int64_t ld_x, const int32_t* row_index, const float* w, float w_offset, T* out, int64_t ld_out,
                   int rows, int size, float eps, bool vec, void* stream) {
    // few registers per thread for rows of usual width: more CTAs per SM hide each other's two passes
    auto kernel = size <= 4096 ? rmsnorm_kernel<T, 4> : (size <= 8192 ? rmsnorm_kernel<T, 8> : rmsnorm_kernel<T, 16>);
    OverlapLaunch launch(rows, kThreads, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, kernel, x, ld_x, row_index, w, w_offset, out, ld_out, size, eps, vec));
    return B2KV_OK;
}

// Sum over the CTA, the same in every thread.  `part` may be used again after the next __syncthreads.
__device__ __forceinline__ float block_sum(float v, float* part) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    v = 0.f;
#pragma unroll
    for (int i = 0; i < kThreads / 32; ++i) v += part[i];
    return v;
}

// One CTA per row; a row of up to 1024 * kKeep elements stays in registers between the passes (mean, deviations, result).
template <typename T, int kKeep>
__global__ void __launch_bounds__(kThreads) layernorm_rows_kernel(const float* y, int64_t ld_y, const int32_t* row_index,
                                                                  const float* w, const float* b, float* x, int64_t ld_x,
                                                                  T* out, int64_t ld_out, int size, float eps, bool vec) {
    __shared__ float part[2][kThreads / 32];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int64_t row = row_index ? row_index[blockIdx.x] : static_cast<int>(blockIdx.x);
    const float* yr = y + row * ld_y;
    float* xr = x == nullptr ? nullptr : x + static_cast<int64_t>(blockIdx.x) * ld_x;
    T* outr = out == nullptr ? nullptr : out + static_cast<int64_t>(blockIdx.x) * ld_out;
    const float inv = 1.0f / static_cast<float>(size);
    if (!vec) {
        float sum = 0.f, sq = 0.f;
        for (int i = threadIdx.x; i < size; i += kThreads) sum += yr[i];
        const float mean = block_sum(sum, part[0]) * inv;
        for (int i = threadIdx.x; i < size; i += kThreads) sq = fmaf(yr[i] - mean, yr[i] - mean, sq);
        const float scale = 1.0f / sqrtf(block_sum(sq, part[1]) * inv + eps);
        for (int i = threadIdx.x; i < size; i += kThreads) {
            float v = fmaf((yr[i] - mean) * scale, w[i], b[i]);
            if (xr != nullptr) xr[i] = v = xr[i] + v;
            if (outr != nullptr) outr[i] = Elt<T>::from_float(v);
        }
        return;
    }
    const int chunks = size / 4;
    float4 keep[kKeep], res[kKeep];
    float sum = 0.f, sq = 0.f;
#pragma unroll
    for (int c = 0; c < kKeep; ++c) {
        const int i = threadIdx.x + c * kThreads;
        if (i < chunks) {
            keep[c] = reinterpret_cast<const float4*>(yr)[i];
            if (xr != nullptr) res[c] = reinterpret_cast<const float4*>(xr)[i];
            sum += (keep[c].x + keep[c].y) + (keep[c].z + keep[c].w);
        }
    }
    const float mean = block_sum(sum, part[0]) * inv;
#pragma unroll
    for (int c = 0; c < kKeep; ++c) {
        if (static_cast<int>(threadIdx.x) + c * kThreads < chunks) {
            keep[c].x -= mean, keep[c].y -= mean, keep[c].z -= mean, keep[c].w -= mean;
            sq += (keep[c].x * keep[c].x + keep[c].y * keep[c].y) + (keep[c].z * keep[c].z + keep[c].w * keep[c].w);
        }
    }
    const float scale = 1.0f / sqrtf(block_sum(sq, part[1]) * inv + eps);
#pragma unroll
    for (int c = 0; c < kKeep; ++c) {
        const int i = threadIdx.x + c * kThreads;
        if (i < chunks) {
            const float4 wv = reinterpret_cast<const float4*>(w)[i], bv = reinterpret_cast<const float4*>(b)[i];
            float4 v = keep[c];
            v.x = fmaf(v.x * scale, wv.x, bv.x), v.y = fmaf(v.y * scale, wv.y, bv.y);
            v.z = fmaf(v.z * scale, wv.z, bv.z), v.w = fmaf(v.w * scale, wv.w, bv.w);
            if (xr != nullptr) {
                v.x += res[c].x, v.y += res[c].y, v.z += res[c].z, v.w += res[c].w;
                store4(xr + 4 * i, v);
            }
            if (outr != nullptr) store4(outr + 4 * i, v);
        }
    }
}

template <typename T>
int launch_layernorm_rows(const float* y, int64_t ld_y, const int32_t* row_index, const float* w, const float* b, float* x,
                          int64_t ld_x, T* out, int64_t ld_out, int rows, int size, float eps, bool vec, void* stream) {
    auto kernel = size <= 4096 ? layernorm_rows_kernel<T, 4> : (size <= 8192 ? layernorm_rows_kernel<T, 8> : layernorm_rows_kernel<T, 16>);
    OverlapLaunch launch(rows, kThreads, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, kernel, y, ld_y, row_index, w, b, x, ld_x, out, ld_out, size, eps, vec));
    return B2KV_OK;
}

}  // namespace
}  // namespace b2kv

using namespace b2kv;

extern "C" int b2kv_embed_rows(const void* table, const int32_t* ids, float* out, void* copy, float scale, int rows, int dim,
                               int vocab, int dtype, int32_t* dev_status, void* stream) {
    if (elt_bytes(dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!table || !ids || !out || rows <= 0 || dim <= 0 || vocab <= 0) return B2KV_ERR_BAD_ARG;
    OverlapLaunch launch(rows, kThreads, 0, stream);
    if (dtype == B2KV_DTYPE_F32)
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, embed_rows_kernel<float>, static_cast<const float*>(table), ids, out,
                                         static_cast<float*>(copy), scale, dim, vocab, dev_status));
    else
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, embed_rows_kernel<__nv_bfloat16>, static_cast<const __nv_bfloat16*>(table),
                                         ids, out, static_cast<__nv_bfloat16*>(copy), scale, dim, vocab, dev_status));
    return B2KV_OK;
}

extern "C" int b2kv_layernorm_rows(const float* y, int64_t ld_y, const int32_t* row_index, const float* w, const float* b, float* x,
                                   int64_t ld_x, void* out, int64_t ld_out, int rows, int size, float eps, int dtype,
                                   void* stream) {
    if (elt_bytes(dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!y || !w || !b || (!x && !out) || rows <= 0 || size <= 0 || ld_y < size || (x && ld_x < size) || (out && ld_out < size))
        return B2KV_ERR_BAD_ARG;
    const bool vec = size % 4 == 0 && ld_y % 4 == 0 && size <= 16384 && aligned16(y) && aligned16(w) && aligned16(b) &&
                     (!x || (ld_x % 4 == 0 && aligned16(x))) && (!out || (ld_out % 4 == 0 && aligned16(out)));
    if (dtype == B2KV_DTYPE_F32)
        return launch_layernorm_rows(y, ld_y, row_index, w, b, x, ld_x, static_cast<float*>(out), ld_out, rows, size, eps, vec, stream);
    return launch_layernorm_rows(y, ld_y, row_index, w, b, x, ld_x, static_cast<__nv_bfloat16*>(out), ld_out, rows, size, eps, vec, stream);
}

extern "C" int b2kv_rmsnorm(const float* x, int64_t ld_x, const int32_t* row_index, const float* w, float w_offset, void* out,
                            int64_t ld_out, int rows, int size, float eps, int dtype, void* stream) {
    if (elt_bytes(dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!x || !w || !out || rows <= 0 || size <= 0 || ld_x < size || ld_out < size) return B2KV_ERR_BAD_ARG;
    const bool vec = size % 4 == 0 && ld_x % 4 == 0 && ld_out % 4 == 0 && size <= 16384 && aligned16(x) && aligned16(w) && aligned16(out);
    if (dtype == B2KV_DTYPE_F32) return launch_rmsnorm(x, ld_x, row_index, w, w_offset, static_cast<float*>(out), ld_out, rows, size, eps, vec, stream);
    return launch_rmsnorm(x, ld_x, row_index, w, w_offset, static_cast<__nv_bfloat16*>(out), ld_out, rows, size, eps, vec, stream);
}
