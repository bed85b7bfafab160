// Grouped-query attention, the parts on CUDA cores: norms and temperature of the queries with the cache append, and attention
// of single query rows for every shape and both storage types.
// These kernels may be scheduled ahead of the end of the kernel that writes their inputs, so no pointer to such data is
// const __restrict__: the compiler would take it for data that nothing writes and could load it before the wait.
#include "gqa.cuh"

#include <math.h>

namespace b2kv {
namespace {

constexpr int kAppendThreads = 256;

__device__ __forceinline__ void narrow_store(float* p, const float (&f)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
__device__ __forceinline__ void narrow_store(__nv_bfloat16* p, const float (&f)[8]) {
    __nv_bfloat162 h[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(f[2 * e], f[2 * e + 1]);
    *reinterpret_cast<uint4*>(p) = *reinterpret_cast<uint4*>(h);
}

// This thread's share of a row of n elements: 16-byte pieces when kVec (n a whole number of them), the first kKeep of which
// stay in registers.
template <typename T, bool kVec, int kKeep>
struct Row {
    static constexpr int kC = Elt<T>::kPerChunk;
    uint4 keep[kKeep];
    __device__ __forceinline__ uint4 piece(const T* src, int j) const {
        return reinterpret_cast<const uint4*>(src)[threadIdx.x + j * kAppendThreads];
    }
    __device__ __forceinline__ void load(const T* src, int n) {
        if (!kVec) return;
#pragma unroll
        for (int j = 0; j < kKeep; ++j)
            if (static_cast<int>(threadIdx.x) + j * kAppendThreads < n / kC) keep[j] = piece(src, j);
    }
    // fn(piece, index of its first element)
    template <typename F>
    __device__ __forceinline__ void each(const T* src, int n, F&& fn) const {
#pragma unroll
        for (int j = 0; j < kKeep; ++j)
            if (static_cast<int>(threadIdx.x) + j * kAppendThreads < n / kC) fn(keep[j], (threadIdx.x + j * kAppendThreads) * kC);
        for (int j = kKeep; static_cast<int>(threadIdx.x) + j * kAppendThreads < n / kC; ++j)
            fn(piece(src, j), (threadIdx.x + j * kAppendThreads) * kC);
    }
    __device__ __forceinline__ float squares(const T* src, int n) const {
        float sum = 0.f;
        if (kVec) {
            each(src, n, [&](const uint4& p, int) {
                float f[kC];
                Elt<T>::widen(p, f);
#pragma unroll
                for (int e = 0; e < kC; ++e) sum = fmaf(f[e], f[e], sum);
            });
        } else {
            for (int i = threadIdx.x; i < n; i += kAppendThreads) sum = fmaf(Elt<T>::to_float(src[i]), Elt<T>::to_float(src[i]), sum);
        }
        return sum;
    }
    // dst = src * factor * w (w NULL: src * factor); dst may be src.
    __device__ __forceinline__ void scaled(T* dst, const T* src, const float* w, float factor, int n) const {
        if (kVec) {
            each(src, n, [&](const uint4& p, int at) {
                float f[kC];
                Elt<T>::widen(p, f);
                if (w != nullptr) {
#pragma unroll
                    for (int e = 0; e < kC; e += 4) {
                        const float4 wv = *reinterpret_cast<const float4*>(w + at + e);
                        f[e] *= factor * wv.x, f[e + 1] *= factor * wv.y, f[e + 2] *= factor * wv.z, f[e + 3] *= factor * wv.w;
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < kC; ++e) f[e] *= factor;
                }
                narrow_store(dst + at, f);
            });
        } else {
            for (int i = threadIdx.x; i < n; i += kAppendThreads)
                dst[i] = Elt<T>::from_float(Elt<T>::to_float(src[i]) * (w != nullptr ? factor * w[i] : factor));
        }
    }
};

struct AppendArgs {
    const float *q_norm, *k_norm;
    const int32_t *row_slot, *row_pos;
    int32_t* dev_status;
    int64_t ld_y;
    int H, G, dim, vdim, n_slots, T_max, temp_every;
    float eps, temp_coef;
};

template <typename T, bool kVec>
__global__ void __launch_bounds__(kAppendThreads) gqa_append_kernel(T* y, T* k_cache, T* v_cache, const AppendArgs a) {
    __shared__ float part[2][kAppendThreads / 32];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    int slot, pos;
    if (!row_place(a.row_slot, a.row_pos, blockIdx.x, a.n_slots, a.T_max, slot, pos)) {
        if (threadIdx.x == 0) report_status(a.dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const int nq = a.H * a.dim, nk = a.G * a.dim, nv = a.G * a.vdim;
    T* q = y + static_cast<int64_t>(blockIdx.x) * a.ld_y;
    const T *k = q + nq, *v = k + nk;
    const bool own = k_cache != nullptr;
    // the first pieces of q, k and v stay in registers between the two passes, all loads on their way together
    Row<T, kVec, 2> rq;
    Row<T, kVec, 1> rk, rv;
    rq.load(q, nq);
    if (own) rk.load(k, nk), rv.load(v, nv);
    float sq = a.q_norm != nullptr ? rq.squares(q, nq) : 0.f;
    float sk = own && a.k_norm != nullptr ? rk.squares(k, nk) : 0.f;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, off);
        sk += __shfl_xor_sync(0xffffffffu, sk, off);
    }
    if ((threadIdx.x & 31) == 0) part[0][threadIdx.x >> 5] = sq, part[1][threadIdx.x >> 5] = sk;
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < kAppendThreads / 32; ++i) sq += part[0][i], sk += part[1][i];
    float fq = a.q_norm != nullptr ? 1.0f / sqrtf(sq / static_cast<float>(nq) + a.eps) : 1.f;
    if (a.temp_every > 0) fq *= 1.0f + a.temp_coef * logf(static_cast<float>((pos + 1) / a.temp_every) + 1.0f);
    if (a.q_norm != nullptr || a.temp_every > 0) rq.scaled(q, q, a.q_norm, fq, nq);
    if (!own) return;
    const int64_t place = static_cast<int64_t>(slot) * a.T_max + pos;
    const float fk = a.k_norm != nullptr ? 1.0f / sqrtf(sk / static_cast<float>(nk) + a.eps) : 1.f;
    rk.scaled(k_cache + place * nk, k, a.k_norm, fk, nk);
    rv.scaled(v_cache + place * nv, v, nullptr, 1.f, nv);
}

// One CTA per (head, query row); its warps take the visible tokens in turn, each with an online softmax of its own, and are
// merged at the end.  A lane holds kPer elements of the query and of the output.
constexpr int kWarps = 4;

template <typename T, int kPer>
__global__ void __launch_bounds__(kWarps * 32) gqa_decode_kernel(const GqaDecodeArgs a) {
    extern __shared__ float sm_acc[];  // [kWarps][vdim]
    __shared__ float sm_m[kWarps], sm_l[kWarps];
    const int h = blockIdx.x, i = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int slot, pos;
    if (!row_place(a.row_slot, a.row_pos, i, a.n_slots, a.T_max, slot, pos)) {
        if (threadIdx.x == 0) report_status(a.dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const int g = h / (a.H / a.G);
    const T* qr = static_cast<const T*>(a.q) + i * a.ld_q + h * a.dim;
    const T* keys = static_cast<const T*>(a.k_cache) + (static_cast<int64_t>(slot) * a.T_max * a.G + g) * a.dim;
    const T* values = static_cast<const T*>(a.v_cache) + (static_cast<int64_t>(slot) * a.T_max * a.G + g) * a.vdim;
    const float slope = a.slopes != nullptr ? a.slopes[h] : 0.f;
    float q[kPer], acc[kPer];
#pragma unroll
    for (int c = 0; c < kPer; ++c) {
        const int d = c * 32 + lane;
        q[c] = d < a.dim ? Elt<T>::to_float(qr[d]) : 0.f;
        acc[c] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    for (int t = warp; t <= pos; t += kWarps) {
        const T* key = keys + static_cast<int64_t>(t) * a.G * a.dim;
        const T* value = values + static_cast<int64_t>(t) * a.G * a.vdim;
        float v[kPer], s = 0.f;
#pragma unroll
        for (int c = 0; c < kPer; ++c) {
            const int d = c * 32 + lane;
            v[c] = d < a.vdim ? Elt<T>::to_float(value[d]) : 0.f;
            s = fmaf(q[c], d < a.dim ? Elt<T>::to_float(key[d]) : 0.f, s);
        }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
        s = s * a.scale - slope * static_cast<float>(pos - t);
        const float mn = fmaxf(m, s), f = expf(m - mn), p = expf(s - mn);
        l = l * f + p;
        m = mn;
#pragma unroll
        for (int c = 0; c < kPer; ++c) acc[c] = fmaf(acc[c], f, p * v[c]);
    }
#pragma unroll
    for (int c = 0; c < kPer; ++c)
        if (c * 32 + lane < a.vdim) sm_acc[warp * a.vdim + c * 32 + lane] = acc[c];
    if (lane == 0) sm_m[warp] = m, sm_l[warp] = l;
    __syncthreads();
    float mx = sm_m[0];
#pragma unroll
    for (int w = 1; w < kWarps; ++w) mx = fmaxf(mx, sm_m[w]);
    float f[kWarps], sum = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
        f[w] = expf(sm_m[w] - mx);
        sum += f[w] * sm_l[w];
    }
    T* out = static_cast<T*>(a.out) + i * a.ld_out + h * a.vdim;
    for (int d = threadIdx.x; d < a.vdim; d += kWarps * 32) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) o = fmaf(f[w], sm_acc[w * a.vdim + d], o);
        out[d] = Elt<T>::from_float(o / sum);
    }
}

template <typename T>
int launch_simt(const GqaDecodeArgs& a, void* stream) {
    const int widest = a.dim > a.vdim ? a.dim : a.vdim;
    if (widest > 512 || a.rows > 65535) return B2KV_ERR_UNSUPPORTED;
    const dim3 grid(a.H, a.rows);
    const size_t smem = static_cast<size_t>(kWarps) * a.vdim * sizeof(float);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (widest <= 64)
        gqa_decode_kernel<T, 2><<<grid, kWarps * 32, smem, s>>>(a);
    else if (widest <= 128)
        gqa_decode_kernel<T, 4><<<grid, kWarps * 32, smem, s>>>(a);
    else
        gqa_decode_kernel<T, 16><<<grid, kWarps * 32, smem, s>>>(a);
    B2KV_CUDA_TRY(cudaGetLastError());
    return B2KV_OK;
}

template <typename T>
int launch_append(T* y, T* k, T* v, const AppendArgs& a, int rows, void* stream) {
    constexpr int per = 16 / static_cast<int>(sizeof(T));
    const bool vec = aligned16(y) && aligned16(a.q_norm) && aligned16(a.k_norm) && aligned16(k) && aligned16(v) && a.ld_y % per == 0 && (a.H * a.dim) % per == 0 &&
                     (a.G * a.dim) % per == 0 && (a.G * a.vdim) % per == 0;
    OverlapLaunch launch(rows, kAppendThreads, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, vec ? gqa_append_kernel<T, true> : gqa_append_kernel<T, false>, y, k, v, a));
    return B2KV_OK;
}

}  // namespace
}  // namespace b2kv

using namespace b2kv;

extern "C" int b2kv_gqa_append(void* y, int64_t ld_y, int H, int G, int dim, int vdim, const float* q_norm, const float* k_norm,
                               float eps, float temp_coef, int temp_every, void* k_cache, void* v_cache,
                               const int32_t* row_slot, const int32_t* row_pos, int n_slots, int T_max, int rows, int dtype,
                               int32_t* dev_status, void* stream) {
    if (elt_bytes(dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!y || !row_pos || H <= 0 || G <= 0 || H % G != 0 || dim <= 0 || vdim <= 0 || rows <= 0 || n_slots <= 0 || T_max <= 0)
        return B2KV_ERR_BAD_ARG;
    if ((k_cache == nullptr) != (v_cache == nullptr)) return B2KV_ERR_BAD_ARG;
    const int64_t cols = static_cast<int64_t>(H) * dim + (k_cache ? static_cast<int64_t>(G) * (dim + vdim) : 0);
    if (ld_y < cols) return B2KV_ERR_BAD_ARG;
    const AppendArgs a{q_norm, k_norm, row_slot, row_pos, dev_status, ld_y, H, G, dim, vdim, n_slots, T_max, temp_every, eps, temp_coef};
    if (dtype == B2KV_DTYPE_F32)
        return launch_append(static_cast<float*>(y), static_cast<float*>(k_cache), static_cast<float*>(v_cache), a, rows, stream);
    return launch_append(static_cast<__nv_bfloat16*>(y), static_cast<__nv_bfloat16*>(k_cache), static_cast<__nv_bfloat16*>(v_cache),
                         a, rows, stream);
}

extern "C" size_t b2kv_gqa_decode_workspace_bytes(int rows, int H, int G, int vdim, int span, int dtype) {
    if (dtype != B2KV_DTYPE_BF16 || rows <= 0 || H <= 0 || G <= 0 || H % G != 0 || vdim <= 0 || span <= 0) return 0;
    return gqa_decode_tc_workspace(rows, H, G, vdim, span);
}

extern "C" int b2kv_gqa_decode(const void* q, int64_t ld_q, const void* k_cache, const void* v_cache, void* out, int64_t ld_out,
                               const float* slopes, const int32_t* row_slot, const int32_t* row_pos, int n_slots, int T_max,
                               int rows, int H, int G, int dim, int vdim, int span, float scale, int dtype, int path,
                               void* workspace, size_t workspace_bytes, int32_t* dev_status, void* stream) {
    if (elt_bytes(dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!q || !k_cache || !v_cache || !out || !row_pos) return B2KV_ERR_BAD_ARG;
    if (n_slots <= 0 || T_max <= 0 || rows <= 0 || H <= 0 || G <= 0 || H % G != 0 || dim <= 0 || vdim <= 0 || span <= 0 ||
        path < 0 || path > 2 || ld_q < static_cast<int64_t>(H) * dim || ld_out < static_cast<int64_t>(H) * vdim)
        return B2KV_ERR_BAD_ARG;
    const GqaDecodeArgs a{q, k_cache, v_cache, out, slopes, row_slot, row_pos, dev_status, ld_q, ld_out,
                          n_slots, T_max, rows, H, G, dim, vdim, span, scale};
    if (path == 2 && dtype != B2KV_DTYPE_BF16) return B2KV_ERR_UNSUPPORTED;
    if (dtype == B2KV_DTYPE_BF16 && path != 1) {
        const int rc = gqa_decode_tc(a, workspace, workspace_bytes, stream);
        if (rc != B2KV_ERR_UNSUPPORTED || path == 2) return rc;
    }
    return dtype == B2KV_DTYPE_F32 ? launch_simt<float>(a, stream) : launch_simt<__nv_bfloat16>(a, stream);
}
