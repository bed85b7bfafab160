// Gated linear attention, token after token on CUDA cores: a decode step, short portions, and every shape and storage type.
// One CTA per (head, segment).  A thread owns fixed elements of the head's state - a few neighbouring value columns in every
// RY-th key row - and streams them through registers once per token: for a single token that is the state read and written
// once, which is all the memory traffic there is.  The head's norm and gate are applied before the output is stored.
// No pointer to data of the kernel before is const __restrict__: this kernel may be scheduled ahead of that one's end.
#include "gla.cuh"

#include <algorithm>

namespace b2kv {
namespace gla {
namespace {

constexpr int kThreads = 256;
constexpr int kBatch = 8;  // state rows in flight per thread

template <int kVec>
struct Piece;
template <>
struct Piece<1> {
    float f[1];
    __device__ __forceinline__ void load(const float* p) { f[0] = *p; }
    __device__ __forceinline__ void store(float* p) const { *p = f[0]; }
};
template <>
struct Piece<4> {
    float f[4];
    __device__ __forceinline__ void load(const float* p) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        f[0] = v.x, f[1] = v.y, f[2] = v.z, f[3] = v.w;
    }
    __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]); }
};

template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads, 3) gla_step_kernel(const b2kv_gla_args a, int cx_count, int32_t* dev_status) {
    extern __shared__ float sm[];
    __shared__ float red[kThreads / 32];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int h = blockIdx.x;
    b2kv_row_segment sg;
    if (!segment_place(a, blockIdx.y, sg)) {
        if (threadIdx.x == 0) report_status(dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const int ry_count = kThreads / cx_count;
    const int cx = threadIdx.x % cx_count, ry = threadIdx.x / cx_count;
    float* const s_alpha = sm;
    float* const s_k = s_alpha + a.dim;
    float* const s_q = s_k + a.dim;
    float* const part = s_q + a.dim;  // [ry_count][vdim]
    float* const state = a.state + (static_cast<int64_t>(sg.slot) * a.H + h) * a.dim * a.vdim;
    bool fresh = a.row_pos[sg.row0] == 0;
    for (int i = 0; i < sg.n; ++i) {
        const int64_t row = sg.row0 + i;
        const T* y = static_cast<const T*>(a.y) + row * a.ld_y;
        const float* alpha = a.alpha + row * a.ld_alpha + static_cast<int64_t>(h) * a.dim;
        for (int d = threadIdx.x; d < a.dim; d += kThreads) {
            s_alpha[d] = alpha[d];
            s_k[d] = Elt<T>::to_float(y[a.k_col + h * a.dim + d]);
            s_q[d] = Elt<T>::to_float(y[a.q_col + h * a.dim + d]) * a.q_scale;
        }
        __syncthreads();
        for (int c = cx * kVec; c < a.vdim; c += cx_count * kVec) {
            float v[kVec], o[kVec];
#pragma unroll
            for (int e = 0; e < kVec; ++e) {
                v[e] = Elt<T>::to_float(y[a.v_col + h * a.vdim + c + e]);
                o[e] = 0.f;
            }
            for (int d0 = ry; d0 < a.dim; d0 += ry_count * kBatch) {
                Piece<kVec> s[kBatch];
#pragma unroll
                for (int u = 0; u < kBatch; ++u) {
                    const int d = d0 + u * ry_count;
                    if (!fresh && d < a.dim) {
                        s[u].load(state + static_cast<int64_t>(d) * a.vdim + c);
                    } else {
#pragma unroll
                        for (int e = 0; e < kVec; ++e) s[u].f[e] = 0.f;
                    }
                }
#pragma unroll
                for (int u = 0; u < kBatch; ++u) {
                    const int d = d0 + u * ry_count;
                    if (d >= a.dim) break;
                    const float al = s_alpha[d], k = s_k[d], q = s_q[d];
#pragma unroll
                    for (int e = 0; e < kVec; ++e) {
                        s[u].f[e] = fmaf(s[u].f[e], al, k * v[e]);
                        o[e] = fmaf(q, s[u].f[e], o[e]);
                    }
                    s[u].store(state + static_cast<int64_t>(d) * a.vdim + c);
                }
            }
#pragma unroll
            for (int e = 0; e < kVec; ++e) part[ry * a.vdim + c + e] = o[e];
        }
        fresh = false;
        __syncthreads();
        float sum = 0.f;
        for (int c = threadIdx.x; c < a.vdim; c += kThreads) {
            float o = part[c];
            for (int r = 1; r < ry_count; ++r) o += part[r * a.vdim + c];
            part[c] = o;
            sum = fmaf(o, o, sum);
        }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = sum;
        __syncthreads();
        sum = 0.f;
#pragma unroll
        for (int w = 0; w < kThreads / 32; ++w) sum += red[w];
        const float scale = 1.0f / sqrtf(sum / static_cast<float>(a.vdim) + a.eps);
        T* out = static_cast<T*>(a.out) + row * a.ld_out + static_cast<int64_t>(h) * a.vdim;
        for (int c = threadIdx.x; c < a.vdim; c += kThreads) {
            const float g = Elt<T>::to_float(y[a.g_col + h * a.vdim + c]);
            out[c] = Elt<T>::from_float(part[c] * scale * a.norm[c] * (sizeof(T) == 4 ? silu(g) : silu_fast(g)));
        }
        // (the next token's first barrier comes before anything of shared memory but alpha, k, q is written again, and those were
        // read before the last two)
    }
}

template <typename T>
int launch_step(const b2kv_gla_args& a, int32_t* dev_status, void* stream) {
    if (a.n_segments > 65535) return B2KV_ERR_UNSUPPORTED;
    const bool vec = a.vdim % 4 == 0 && aligned16(a.state);
    const int cols = vec ? a.vdim / 4 : a.vdim;
    int cx = 1;
    while (cx < cols && cx < kThreads) cx *= 2;
    const size_t smem = (3 * static_cast<size_t>(a.dim) + static_cast<size_t>(kThreads / cx) * a.vdim) * sizeof(float);
    if (smem > 48 * 1024) return B2KV_ERR_UNSUPPORTED;
    OverlapLaunch launch(dim3(a.H, a.n_segments), kThreads, smem, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, vec ? gla_step_kernel<T, 4> : gla_step_kernel<T, 1>, a, cx, dev_status));
    return B2KV_OK;
}

}  // namespace
}  // namespace gla
}  // namespace b2kv

using namespace b2kv;

static bool takes_chunks(int path, int dtype, int max_n) { return path == 2 || (path == 0 && dtype == B2KV_DTYPE_BF16 && max_n > 16); }

extern "C" size_t b2kv_gla_workspace_bytes(int H, int dim, int vdim, int n_segments, int max_n, int dtype, int path) {
    if (H <= 0 || dim <= 0 || vdim <= 0 || n_segments <= 0 || max_n <= 0 || !takes_chunks(path, dtype, max_n)) return 0;
    return gla_chunked_workspace(H, dim, vdim, n_segments, max_n, dtype);
}

extern "C" int b2kv_gla(const b2kv_gla_args* args, int32_t* dev_status, void* stream) {
    if (args == nullptr) return B2KV_ERR_BAD_ARG;
    const b2kv_gla_args& a = *args;
    if (elt_bytes(a.dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!a.y || !a.alpha || !a.norm || !a.state || !a.out || !a.row_pos || a.path < 0 || a.path > 2) return B2KV_ERR_BAD_ARG;
    if (a.H <= 0 || a.dim <= 0 || a.vdim <= 0 || a.n_segments <= 0 || a.max_n <= 0 || a.rows <= 0 || a.n_slots <= 0) return B2KV_ERR_BAD_ARG;
    if (!a.segments && (a.n_segments > a.rows || a.n_segments > a.n_slots)) return B2KV_ERR_BAD_ARG;
    const int64_t keys = static_cast<int64_t>(a.H) * a.dim, values = static_cast<int64_t>(a.H) * a.vdim;
    if (a.q_col < 0 || a.k_col < 0 || a.v_col < 0 || a.g_col < 0 || a.ld_y < a.q_col + keys || a.ld_y < a.k_col + keys ||
        a.ld_y < a.v_col + values || a.ld_y < a.g_col + values || a.ld_alpha < keys || a.ld_out < values)
        return B2KV_ERR_BAD_ARG;
    if (takes_chunks(a.path, a.dtype, a.max_n)) {
        const int rc = gla_chunked(a, dev_status, stream);
        if (rc != B2KV_ERR_UNSUPPORTED || a.path == 2) return rc;
    }
    return a.dtype == B2KV_DTYPE_F32 ? gla::launch_step<float>(a, dev_status, stream)
                                     : gla::launch_step<__nv_bfloat16>(a, dev_status, stream);
}
