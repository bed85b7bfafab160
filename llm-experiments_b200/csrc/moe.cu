// Mixture of experts around the grouped products of b2kv_linear: expert choice, the sort of the chosen rows by expert, and
// the weighted sum of the experts' outputs onto the 32-bit residual stream.
// These kernels may be scheduled ahead of the end of the kernel that writes their inputs, so no pointer to such data is
// const __restrict__: the compiler would take it for data that nothing writes and could load it before the wait.
#include <math.h>

#include "b2kv_common.cuh"

namespace b2kv {
namespace {

constexpr int kMaxExperts = 1024, kMaxTop = 64;
constexpr int kRouteWarps = 4;

// Largest value over a warp and, among equals, the lowest index.
__device__ __forceinline__ void warp_best(float& v, int& i) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, off);
        const int oi = __shfl_xor_sync(0xffffffffu, i, off);
        if (ov > v || (ov == v && oi < i)) v = ov, i = oi;
    }
}

__global__ void zero_counts_kernel(int32_t* counts, int n) {
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) counts[i] = 0;
}

// A warp per row.  A score that is taken, or whose group is not kept, is replaced by -1 (scores are positive).
__global__ void __launch_bounds__(kRouteWarps * 32)
route_kernel(const float* logits, int64_t ld, int rows, int experts, int groups, int keep, int top,
             int32_t* idx, float* score, int32_t* counts) {
    extern __shared__ float sm_route[];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int row = blockIdx.x * kRouteWarps + warp;
    if (row >= rows) return;
    float* s = sm_route + warp * 2 * experts;  // scores
    float* best = s + experts;                 // largest score of every group (-1: taken)
    const float* z = logits + row * ld;
    float mx = -INFINITY;
    for (int e = lane; e < experts; e += 32) mx = fmaxf(mx, s[e] = z[e]);
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    float sum = 0.f;
    for (int e = lane; e < experts; e += 32) sum += s[e] = expf(s[e] - mx);
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
    for (int e = lane; e < experts; e += 32) s[e] = s[e] / sum;
    __syncwarp();
    if (keep < groups) {
        const int per = experts / groups;
        for (int g = lane; g < groups; g += 32) {
            float b = s[g * per];
            for (int e = 1; e < per; ++e) b = fmaxf(b, s[g * per + e]);
            best[g] = b;
        }
        __syncwarp();
        // what is not among the best is dropped: take the `keep` best away, the rest loses its experts
        for (int k = 0; k < keep; ++k) {
            float v = -2.f;
            int i = 0x7fffffff;
            for (int g = lane; g < groups; g += 32)
                if (best[g] > v) v = best[g], i = g;
            warp_best(v, i);
            if (i >= groups) i = k;  // scores that are not numbers: any group, but one that exists
            if (lane == 0) best[i] = -1.f;
            __syncwarp();
        }
        for (int e = lane; e < experts; e += 32)
            if (best[e / per] >= 0.f) s[e] = -1.f;
        __syncwarp();
    }
    for (int k = 0; k < top; ++k) {
        float v = -2.f;
        int i = 0x7fffffff;
        for (int e = lane; e < experts; e += 32)
            if (s[e] > v) v = s[e], i = e;
        warp_best(v, i);
        if (i >= experts) i = k, v = 0.f;
        if (lane == 0) {
            idx[static_cast<int64_t>(row) * top + k] = i;
            score[static_cast<int64_t>(row) * top + k] = v;
            atomicAdd(&counts[i], 1);
            s[i] = -1.f;
        }
        __syncwarp();
    }
}

// A CTA per choice: its place among the sorted rows, and the copy of its row there (128-bit when aligned).
constexpr int kPlanThreads = 128;

__global__ void __launch_bounds__(kPlanThreads)
moe_plan_kernel(const int32_t* idx, int32_t* counts, int experts, int top, int32_t* offsets,
                int32_t* slot, const uint8_t* h, int64_t pitch_h, uint8_t* sorted,
                int64_t pitch_sorted, int row_bytes, bool vec) {
    __shared__ int place;
    __shared__ int part[kPlanThreads / 32];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int choice = blockIdx.x;
    const int e = idx[choice];
    int before = 0;
    for (int i = threadIdx.x; i < e; i += kPlanThreads) before += counts[i];
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) before += __shfl_xor_sync(0xffffffffu, before, off);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = before;
    __syncthreads();
    if (threadIdx.x == 0) {
        before = 0;
        for (int w = 0; w < kPlanThreads / 32; ++w) before += part[w];
        place = before + atomicAdd(&counts[experts + e], 1);
        slot[choice] = place;
    }
    if (choice == 0) {
        // offsets of all experts, by one CTA (experts are few: a serial prefix per thread range would cost more to set up)
        for (int i = threadIdx.x; i <= experts; i += kPlanThreads) {
            int sum = 0;
            for (int j = 0; j < i; ++j) sum += counts[j];
            offsets[i] = sum;
        }
    }
    __syncthreads();
    const uint8_t* src = h + static_cast<int64_t>(choice / top) * pitch_h;
    uint8_t* dst = sorted + static_cast<int64_t>(place) * pitch_sorted;
    if (vec) {
        for (int i = threadIdx.x; i < row_bytes / 16; i += kPlanThreads)
            reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
    } else {
        for (int i = threadIdx.x; i < row_bytes / 2; i += kPlanThreads)
            reinterpret_cast<uint16_t*>(dst)[i] = reinterpret_cast<const uint16_t*>(src)[i];
    }
}

template <typename T>
__global__ void __launch_bounds__(256) moe_combine_kernel(float* x, int64_t ld_x, const T* y,
                                                          int64_t ld_y, const int32_t* slot,
                                                          const float* score, int top, int dim, bool vec) {
    __shared__ int32_t sl[kMaxTop];
    __shared__ float sc[kMaxTop];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int64_t row = blockIdx.x;
    if (threadIdx.x < top) {
        sl[threadIdx.x] = slot[row * top + threadIdx.x];
        sc[threadIdx.x] = score[row * top + threadIdx.x];
    }
    __syncthreads();
    float* xr = x + row * ld_x;
    if (vec) {
        constexpr int kC = Elt<T>::kPerChunk;
        for (int i = threadIdx.x; i < dim / kC; i += blockDim.x) {
            float acc[kC] = {};
            for (int k = 0; k < top; ++k) {
                float v[kC];
                Elt<T>::widen(reinterpret_cast<const uint4*>(y + sl[k] * ld_y)[i], v);
#pragma unroll
                for (int j = 0; j < kC; ++j) acc[j] = fmaf(sc[k], v[j], acc[j]);
            }
#pragma unroll
            for (int j = 0; j < kC; j += 4) {
                float4* p = reinterpret_cast<float4*>(xr + i * kC + j);
                float4 o = *p;
                o.x += acc[j], o.y += acc[j + 1], o.z += acc[j + 2], o.w += acc[j + 3];
                *p = o;
            }
        }
        return;
    }
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        float acc = 0.f;
        for (int k = 0; k < top; ++k) acc = fmaf(sc[k], Elt<T>::to_float(y[sl[k] * ld_y + i]), acc);
        xr[i] += acc;
    }
}

}  // namespace
}  // namespace b2kv

using namespace b2kv;

extern "C" int b2kv_route(const float* logits, int64_t ld, int rows, int experts, int groups, int keep, int top, int32_t* idx,
                          float* score, int32_t* counts, void* stream) {
    if (!logits || !idx || !score || !counts || rows <= 0 || experts <= 0 || ld < experts || groups <= 0 || keep <= 0 ||
        keep > groups || experts % groups != 0 || top <= 0 || top > keep * (experts / groups))
        return B2KV_ERR_BAD_ARG;
    if (experts > kMaxExperts || top > kMaxTop) return B2KV_ERR_UNSUPPORTED;
    OverlapLaunch zero(1, 256, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&zero.cfg, zero_counts_kernel, counts, 2 * experts));
    OverlapLaunch launch((rows + kRouteWarps - 1) / kRouteWarps, kRouteWarps * 32,
                         static_cast<size_t>(kRouteWarps) * 2 * experts * sizeof(float), stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, route_kernel, logits, ld, rows, experts, groups, keep, top, idx, score, counts));
    return B2KV_OK;
}

extern "C" int b2kv_moe_plan(const int32_t* idx, int32_t* counts, int rows, int experts, int top, int32_t* offsets,
                             int32_t* slot, const void* h, int64_t ld_h, void* sorted, int64_t ld_sorted, int dim, int dtype,
                             void* stream) {
    const int es = elt_bytes(dtype);
    if (es == 0) return B2KV_ERR_UNSUPPORTED;
    if (!idx || !counts || !offsets || !slot || !h || !sorted || rows <= 0 || experts <= 0 || top <= 0 || dim <= 0 || ld_h < dim ||
        ld_sorted < dim)
        return B2KV_ERR_BAD_ARG;
    if (static_cast<long long>(rows) * top > 0x7fffffffLL) return B2KV_ERR_UNSUPPORTED;
    const bool vec = (dim * es) % 16 == 0 && (ld_h * es) % 16 == 0 && (ld_sorted * es) % 16 == 0 && aligned16(h) && aligned16(sorted);
    OverlapLaunch launch(rows * top, kPlanThreads, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, moe_plan_kernel, idx, counts, experts, top, offsets, slot,
                                     static_cast<const uint8_t*>(h), ld_h * es, static_cast<uint8_t*>(sorted), ld_sorted * es,
                                     dim * es, vec));
    return B2KV_OK;
}

extern "C" int b2kv_moe_combine(float* x, int64_t ld_x, const void* y, int64_t ld_y, const int32_t* slot, const float* score,
                                int rows, int top, int dim, int dtype, void* stream) {
    const int es = elt_bytes(dtype);
    if (es == 0) return B2KV_ERR_UNSUPPORTED;
    if (!x || !y || !slot || !score || rows <= 0 || top <= 0 || dim <= 0 || ld_x < dim || ld_y < dim) return B2KV_ERR_BAD_ARG;
    if (top > kMaxTop) return B2KV_ERR_UNSUPPORTED;
    const bool vec = (dim * es) % 16 == 0 && (ld_y * es) % 16 == 0 && ld_x % 4 == 0 && dim % 4 == 0 && aligned16(x) && aligned16(y);
    OverlapLaunch launch(rows, 256, 0, stream);
    if (dtype == B2KV_DTYPE_F32)
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, moe_combine_kernel<float>, x, ld_x, static_cast<const float*>(y), ld_y, slot,
                                         score, top, dim, vec));
    else
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, moe_combine_kernel<__nv_bfloat16>, x, ld_x,
                                         static_cast<const __nv_bfloat16*>(y), ld_y, slot, score, top, dim, vec));
    return B2KV_OK;
}
