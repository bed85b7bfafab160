// Latent attention, the parts on CUDA cores: rotation of the queries and the cache append (norm of the latent row,
// rotation of the shared key part), and attention of single query rows in the latent space for every shape and both
// storage types.
// These kernels may be scheduled ahead of the end of the kernel that writes their inputs, so no pointer to such data is
// const __restrict__: the compiler would take it for data that nothing writes and could load it before the wait.
#include "latent.cuh"

#include <math.h>

namespace b2kv {
namespace {

constexpr int kAppendThreads = 256;
constexpr int kMaxRot = 512;

// Floats narrowed to one 16-byte piece of the storage type.
__device__ __forceinline__ uint4 narrow(const float (&f)[4]) {
    return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
}
__device__ __forceinline__ uint4 narrow(const float (&f)[8]) {
    uint32_t w[4];
#pragma unroll
    for (int e = 0; e < 4; ++e)
        w[e] = static_cast<uint32_t>(__bfloat16_as_ushort(__float2bfloat16_rn(f[2 * e]))) |
               static_cast<uint32_t>(__bfloat16_as_ushort(__float2bfloat16_rn(f[2 * e + 1]))) << 16;
    return make_uint4(w[0], w[1], w[2], w[3]);
}

// kPerChunk pairs of elements turned in place: (u, v) -> (u cos - v sin, v cos + u sin).
template <typename T>
__device__ __forceinline__ void rotate_pieces(uint4* pu, uint4* pv, const float* cs, const float* sn) {
    constexpr int kC = Elt<T>::kPerChunk;
    float u[kC], v[kC], a[kC], b[kC];
    Elt<T>::widen(*pu, u);
    Elt<T>::widen(*pv, v);
#pragma unroll
    for (int e = 0; e < kC; ++e) {
        a[e] = u[e] * cs[e] - v[e] * sn[e];
        b[e] = v[e] * cs[e] + u[e] * sn[e];
    }
    *pu = narrow(a);
    *pv = narrow(b);
}

// vec: every head's rotated part, row and half of the rotated elements is made of whole 16-byte pieces.
template <typename T>
__global__ void __launch_bounds__(kAppendThreads)
latent_append_kernel(T* y, int64_t ld_y, int H, int dim, int rot, int rot_dims, const float* inv_freq,
                     int down_col, int kv_rank, const float* w_norm, float eps, T* key_cache,
                     T* latent_cache, const int32_t* row_slot, const int32_t* row_pos,
                     int n_slots, int T_max, int32_t* dev_status, bool vec) {
    __shared__ float cs[kMaxRot / 2], sn[kMaxRot / 2], part[kAppendThreads / 32];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    int slot, pos;
    if (!row_place(row_slot, row_pos, blockIdx.x, n_slots, T_max, slot, pos)) {
        if (threadIdx.x == 0) report_status(dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const int half = rot_dims / 2;
    for (int j = threadIdx.x; j < half; j += kAppendThreads) sincosf(static_cast<float>(pos) * inv_freq[j], &sn[j], &cs[j]);
    T* row = y + static_cast<int64_t>(blockIdx.x) * ld_y;
    float sum = 0.f;
    if (latent_cache != nullptr) {
        for (int i = threadIdx.x; i < kv_rank; i += kAppendThreads) {
            const float v = Elt<T>::to_float(row[down_col + i]);
            sum = fmaf(v, v, sum);
        }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
        if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = sum;
    }
    __syncthreads();
    constexpr int kC = Elt<T>::kPerChunk;
    if (vec) {  // 16-byte pieces: kC pairs at a time
        const int pieces = half / kC;
        for (int i = threadIdx.x; i < H * pieces; i += kAppendThreads) {
            const int h = i / pieces, j = i % pieces;
            uint4* q = reinterpret_cast<uint4*>(row + h * (dim + rot) + dim);
            rotate_pieces<T>(q + j, q + j + pieces, cs + j * kC, sn + j * kC);
        }
    } else {
        for (int i = threadIdx.x; i < H * half; i += kAppendThreads) {
            const int h = i / half, j = i % half;
            T* q = row + h * (dim + rot) + dim;
            const float u = Elt<T>::to_float(q[j]), v = Elt<T>::to_float(q[j + half]);
            q[j] = Elt<T>::from_float(u * cs[j] - v * sn[j]);
            q[j + half] = Elt<T>::from_float(v * cs[j] + u * sn[j]);
        }
    }
    if (latent_cache == nullptr) return;
    sum = 0.f;
#pragma unroll
    for (int i = 0; i < kAppendThreads / 32; ++i) sum += part[i];
    const float scale = 1.0f / sqrtf(sum / static_cast<float>(kv_rank) + eps);
    const int64_t place = static_cast<int64_t>(slot) * T_max + pos;
    T* latent = latent_cache + place * kv_rank;
    for (int i = threadIdx.x; i < kv_rank; i += kAppendThreads)
        latent[i] = Elt<T>::from_float(Elt<T>::to_float(row[down_col + i]) * scale * w_norm[i]);
    T* key = key_cache + place * rot;
    const T* kr = row + down_col + kv_rank;
    for (int j = threadIdx.x; j < half; j += kAppendThreads) {
        const float u = Elt<T>::to_float(kr[j]), v = Elt<T>::to_float(kr[j + half]);
        key[j] = Elt<T>::from_float(u * cs[j] - v * sn[j]);
        key[j + half] = Elt<T>::from_float(v * cs[j] + u * sn[j]);
    }
    for (int j = rot_dims + threadIdx.x; j < rot; j += kAppendThreads) key[j] = kr[j];
}

// One CTA per (head, query row); its warps take the visible tokens in turn, each with an online softmax of its own, and
// are merged at the end.  A lane holds kPer elements of the latent space.
constexpr int kWarps = 4;

template <typename T, int kPer>
__global__ void __launch_bounds__(kWarps * 32) latent_decode_kernel(const LatentDecodeArgs a) {
    extern __shared__ float sm_acc[];  // [kWarps][kv_rank]
    __shared__ float sm_m[kWarps], sm_l[kWarps];
    const int h = blockIdx.x, i = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int slot, pos;
    if (!row_place(a.row_slot, a.row_pos, i, a.n_slots, a.T_max, slot, pos)) {
        if (threadIdx.x == 0) report_status(a.dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const T* ql = static_cast<const T*>(a.q_latent) + (static_cast<int64_t>(i) * a.H + h) * a.kv_rank;
    const T* qr = static_cast<const T*>(a.q) + i * a.ld_q + h * (a.dim + a.rot) + a.dim;
    float q[kPer], acc[kPer];
#pragma unroll
    for (int c = 0; c < kPer; ++c) {
        const int d = c * 32 + lane;
        q[c] = d < a.kv_rank ? Elt<T>::to_float(ql[d]) : 0.f;
        acc[c] = 0.f;
    }
    float m = -INFINITY, l = 0.f;
    const int t0 = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    for (int t = t0 + warp; t <= pos; t += kWarps) {
        const int64_t place = static_cast<int64_t>(slot) * a.T_max + t;
        const T* lat = static_cast<const T*>(a.latent_cache) + place * a.kv_rank;
        const T* key = static_cast<const T*>(a.key_cache) + place * a.rot;
        float v[kPer], s = 0.f;
#pragma unroll
        for (int c = 0; c < kPer; ++c) {
            const int d = c * 32 + lane;
            v[c] = d < a.kv_rank ? Elt<T>::to_float(lat[d]) : 0.f;
            s = fmaf(q[c], v[c], s);
        }
        for (int d = lane; d < a.rot; d += 32) s = fmaf(Elt<T>::to_float(qr[d]), Elt<T>::to_float(key[d]), s);
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
        s *= a.scale;
        const float mn = fmaxf(m, s), f = expf(m - mn), p = expf(s - mn);
        l = l * f + p;
        m = mn;
#pragma unroll
        for (int c = 0; c < kPer; ++c) acc[c] = fmaf(acc[c], f, p * v[c]);
    }
#pragma unroll
    for (int c = 0; c < kPer; ++c)
        if (c * 32 + lane < a.kv_rank) sm_acc[warp * a.kv_rank + c * 32 + lane] = acc[c];
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
    T* out = static_cast<T*>(a.out) + (static_cast<int64_t>(i) * a.H + h) * a.kv_rank;
    for (int d = threadIdx.x; d < a.kv_rank; d += kWarps * 32) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) o = fmaf(f[w], sm_acc[w * a.kv_rank + d], o);
        out[d] = Elt<T>::from_float(o / sum);
    }
}

template <typename T>
int launch_simt(const LatentDecodeArgs& a, void* stream) {
    if (a.kv_rank > 1024 || a.rows > 65535) return B2KV_ERR_UNSUPPORTED;
    const dim3 grid(a.H, a.rows);
    const size_t smem = static_cast<size_t>(kWarps) * a.kv_rank * sizeof(float);
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (a.kv_rank <= 128)
        latent_decode_kernel<T, 4><<<grid, kWarps * 32, smem, s>>>(a);
    else if (a.kv_rank <= 512)
        latent_decode_kernel<T, 16><<<grid, kWarps * 32, smem, s>>>(a);
    else
        latent_decode_kernel<T, 32><<<grid, kWarps * 32, smem, s>>>(a);
    B2KV_CUDA_TRY(cudaGetLastError());
    return B2KV_OK;
}

}  // namespace
}  // namespace b2kv

using namespace b2kv;

extern "C" int b2kv_latent_append(void* y, int64_t ld_y, int H, int dim, int rot, int rot_dims, const float* inv_freq,
                                  int down_col, int kv_rank, const float* w_norm, float eps, void* key_cache,
                                  void* latent_cache, const int32_t* row_slot, const int32_t* row_pos, int n_slots, int T_max,
                                  int rows, int dtype, int32_t* dev_status, void* stream) {
    if (elt_bytes(dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!y || !inv_freq || !row_pos || H <= 0 || dim <= 0 || rot <= 0 || rot_dims <= 0 || rows <= 0 || n_slots <= 0 || T_max <= 0)
        return B2KV_ERR_BAD_ARG;
    if (rot_dims > rot || rot_dims % 2 != 0 || ld_y < static_cast<int64_t>(H) * (dim + rot)) return B2KV_ERR_BAD_ARG;
    if (rot_dims > kMaxRot) return B2KV_ERR_UNSUPPORTED;
    if ((key_cache == nullptr) != (latent_cache == nullptr)) return B2KV_ERR_BAD_ARG;
    if (latent_cache && (!w_norm || kv_rank <= 0 || down_col < 0 || ld_y < down_col + kv_rank + rot)) return B2KV_ERR_BAD_ARG;
    const int per = 16 / elt_bytes(dtype);
    const bool vec = aligned16(y) && ld_y % per == 0 && dim % per == 0 && rot % per == 0 && (rot_dims / 2) % per == 0;
    OverlapLaunch launch(rows, kAppendThreads, 0, stream);
    if (dtype == B2KV_DTYPE_F32)
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, latent_append_kernel<float>, static_cast<float*>(y), ld_y, H, dim, rot,
                                         rot_dims, inv_freq, down_col, kv_rank, w_norm, eps, static_cast<float*>(key_cache),
                                         static_cast<float*>(latent_cache), row_slot, row_pos, n_slots, T_max, dev_status, vec));
    else
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, latent_append_kernel<__nv_bfloat16>, static_cast<__nv_bfloat16*>(y), ld_y,
                                         H, dim, rot, rot_dims, inv_freq, down_col, kv_rank, w_norm, eps,
                                         static_cast<__nv_bfloat16*>(key_cache), static_cast<__nv_bfloat16*>(latent_cache),
                                         row_slot, row_pos, n_slots, T_max, dev_status, vec));
    return B2KV_OK;
}

extern "C" size_t b2kv_latent_decode_workspace_bytes(int rows, int H, int kv_rank, int span, int dtype) {
    if (dtype != B2KV_DTYPE_BF16 || rows <= 0 || H <= 0 || kv_rank <= 0 || span <= 0) return 0;
    return latent_decode_tc_workspace(rows, H, kv_rank, span);
}

extern "C" int b2kv_latent_decode(const void* q_latent, const void* q, int64_t ld_q, int dim, const void* key_cache,
                                  const void* latent_cache, void* out, const int32_t* row_slot, const int32_t* row_pos,
                                  int n_slots, int T_max, int rows, int H, int kv_rank, int rot, int window, int span,
                                  float scale, int dtype, int path, void* workspace, size_t workspace_bytes,
                                  int32_t* dev_status, void* stream) {
    if (elt_bytes(dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!q_latent || !q || !key_cache || !latent_cache || !out || !row_pos) return B2KV_ERR_BAD_ARG;
    if (n_slots <= 0 || T_max <= 0 || rows <= 0 || H <= 0 || kv_rank <= 0 || rot <= 0 || dim <= 0 || span <= 0 || path < 0 ||
        path > 2 || ld_q < static_cast<int64_t>(H) * (dim + rot))
        return B2KV_ERR_BAD_ARG;
    const LatentDecodeArgs a{q_latent, q, key_cache, latent_cache, out, row_slot, row_pos, dev_status, ld_q, dim,
                             n_slots, T_max, rows, H, kv_rank, rot, window, span, scale};
    if (path == 2 && dtype != B2KV_DTYPE_BF16) return B2KV_ERR_UNSUPPORTED;
    if (dtype == B2KV_DTYPE_BF16 && path != 1) {
        const int rc = latent_decode_tc(a, workspace, workspace_bytes, stream);
        if (rc != B2KV_ERR_UNSUPPORTED || path == 2) return rc;
    }
    return dtype == B2KV_DTYPE_F32 ? launch_simt<float>(a, stream) : launch_simt<__nv_bfloat16>(a, stream);
}
