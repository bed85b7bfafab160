// b2kv_linear: argument checks, the choice of the kernel, and the CUDA-core kernel for fp32 and for shapes that the
// tensor-core kernels do not take, and the one for few input features (64 x 64 output tiles, 16 input features per step, 4 x 4 outputs per thread, fp32
// accumulation).
#include "linear.cuh"

namespace b2kv {
namespace lin {

constexpr int kTile = 64, kStep = 16, kThreads = 256;

// Exact exponential for the fp32 path; the bf16 paths round the result to 8 bits anyway.
template <typename T>
__device__ __forceinline__ float glu_value(int kind, float g, float u, float limit) {
    if (sizeof(T) == 2) return glu(kind, g, u, limit);
    if (kind == B2KV_SEG_GLU_SILU) return g / (1.0f + expf(-g)) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}

template <typename T>
__global__ void __launch_bounds__(kThreads) linear_simt_kernel(const b2kv_linear_args a) {
    __shared__ float xs[kStep][kTile + 4];
    __shared__ float ws[kStep][kTile + 4];
    const int g = blockIdx.z;
    int first = 0, n_rows = a.rows;
    const T* x = static_cast<const T*>(a.x);
    if (a.group_rows != nullptr) {
        first = a.group_rows[g];
        n_rows = a.group_rows[g + 1] - first;
        x += static_cast<int64_t>(first) * a.ld_x;
    } else {
        x += static_cast<int64_t>(g) * a.group_x;
    }
    const int row0 = blockIdx.y * kTile, col0 = blockIdx.x * kTile;
    if (row0 >= n_rows) return;
    const T* w = static_cast<const T*>(a.w) + static_cast<int64_t>(g) * a.group_w;
    const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.K; k0 += kStep) {
        for (int i = threadIdx.x; i < kTile * kStep; i += kThreads) {
            const int r = i / kStep, k = i % kStep;
            xs[k][r] = (row0 + r < n_rows && k0 + k < a.K)
                           ? Elt<T>::to_float(x[static_cast<int64_t>(row0 + r) * a.ld_x + k0 + k]) : 0.f;
            const int wk = i / kTile, c = i % kTile;
            ws[wk][c] = (k0 + wk < a.K && col0 + c < a.N)
                            ? Elt<T>::to_float(w[static_cast<int64_t>(k0 + wk) * a.ld_w + col0 + c]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kStep; ++k) {
            float xv[4], wv[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) xv[i] = xs[k][ty * 4 + i], wv[i] = ws[k][tx * 4 + i];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = row0 + ty * 4 + i;
        if (r >= n_rows) break;
        const int64_t out_row = first + r;
#pragma unroll
        for (int j = 0; j < 4; j += 2) {  // pairs of columns: boundaries of segments are even
            const int c = col0 + tx * 4 + j;
            if (c >= a.N) break;
            const int s = segment_of(a, c);
            const b2kv_segment& sg = a.seg[s];
            const int local = c - segment_first(a, s);
            const int64_t base = out_row * sg.ld + static_cast<int64_t>(g) * (a.group_rows ? 0 : sg.group);
            if (a.bias != nullptr) {
                acc[i][j] += a.bias[c];
                if (c + 1 < a.N) acc[i][j + 1] += a.bias[c + 1];
            }
            if (is_pair(sg.kind)) {
                static_cast<T*>(sg.out)[base + local / 2] =
                    Elt<T>::from_float(glu_value<T>(sg.kind, acc[i][j], acc[i][j + 1], a.limit));
                continue;
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                if (c + e >= a.N) break;
                float v = sizeof(T) == 4 && sg.kind == B2KV_SEG_DECAY ? decay_exact(acc[i][j + e], a.limit)
                                                                      : single(sg.kind, acc[i][j + e], a.limit);
                if (is_f32(sg.kind)) {
                    if (a.residual != nullptr && sg.kind == B2KV_SEG_F32) v += a.residual[out_row * a.ld_residual + local + e];
                    static_cast<float*>(sg.out)[base + local + e] = v;
                } else {
                    static_cast<T*>(sg.out)[base + local + e] = Elt<T>::from_float(v);
                }
            }
        }
    }
}

static int launch_simt(const b2kv_linear_args& a, void* stream) {
    const int max_rows = a.group_rows ? a.max_group_rows : a.rows;
    const dim3 grid((a.N + kTile - 1) / kTile, (max_rows + kTile - 1) / kTile, a.groups);
    if (grid.y > 65535u || grid.z > 65535u) return B2KV_ERR_UNSUPPORTED;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (a.dtype == B2KV_DTYPE_F32)
        linear_simt_kernel<float><<<grid, kThreads, 0, s>>>(a);
    else
        linear_simt_kernel<__nv_bfloat16><<<grid, kThreads, 0, s>>>(a);
    B2KV_CUDA_TRY(cudaGetLastError());
    return B2KV_OK;
}

// Products with few input features (a low-rank bottleneck): what they cost is the outputs, so there is nothing for the tensor
// cores to win.  A thread keeps two columns of w in registers and goes through a tile of rows, whose few elements lie in shared
// memory; neighbouring threads store neighbouring columns.
constexpr int kThinK = 32, kThinThreads = 128, kThinRows = 64;

template <int kK>
__global__ void __launch_bounds__(kThinThreads) linear_thin_kernel(const __grid_constant__ b2kv_linear_args a, int row_tile) {
    __shared__ float4 xs[kThinRows][kK / 4];
    const int c = (blockIdx.x * kThinThreads + threadIdx.x) * 2;
    const bool live = c < a.N;
    const __nv_bfloat16* const w = static_cast<const __nv_bfloat16*>(a.w);
    float2 wr[kK], bias = make_float2(0.f, 0.f);
#pragma unroll
    for (int k = 0; k < kK; ++k) {
        wr[k] = make_float2(0.f, 0.f);
        if (live && k < a.K) wr[k] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(w + k * a.ld_w + c));
    }
    if (live && a.bias != nullptr) bias = make_float2(a.bias[c], a.bias[c + 1]);
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int row0 = blockIdx.y * row_tile, n = min(row_tile, a.rows - row0);
    const __nv_bfloat16* const x = static_cast<const __nv_bfloat16*>(a.x) + row0 * a.ld_x;
    for (int i = threadIdx.x; i < n * kK; i += kThinThreads) {
        const int r = i / kK, k = i % kK;
        reinterpret_cast<float*>(xs[r])[k] = k < a.K ? __bfloat162float(x[r * a.ld_x + k]) : 0.f;
    }
    __syncthreads();
    if (!live) return;
    const b2kv_segment& sg = a.seg[0];
    for (int r = 0; r < n; ++r) {
        float2 v = bias;
#pragma unroll
        for (int k = 0; k < kK; k += 4) {
            const float4 xv = xs[r][k / 4];
            v = __ffma2_rn(make_float2(xv.x, xv.x), wr[k], v);
            v = __ffma2_rn(make_float2(xv.y, xv.y), wr[k + 1], v);
            v = __ffma2_rn(make_float2(xv.z, xv.z), wr[k + 2], v);
            v = __ffma2_rn(make_float2(xv.w, xv.w), wr[k + 3], v);
        }
        v.x = single(sg.kind, v.x, a.limit);
        v.y = single(sg.kind, v.y, a.limit);
        const int64_t row = row0 + r;
        if (is_f32(sg.kind)) {
            if (a.residual != nullptr && sg.kind == B2KV_SEG_F32) {
                const float2 add = *reinterpret_cast<const float2*>(a.residual + row * a.ld_residual + c);
                v.x += add.x, v.y += add.y;
            }
            *reinterpret_cast<float2*>(static_cast<float*>(sg.out) + row * sg.ld + c) = v;
        } else {
            *reinterpret_cast<__nv_bfloat162*>(static_cast<__nv_bfloat16*>(sg.out) + row * sg.ld + c) = __floats2bfloat162_rn(v.x, v.y);
        }
    }
}

static int launch_thin(const b2kv_linear_args& a, void* stream) {
    const b2kv_segment& sg = a.seg[0];
    if (a.dtype != B2KV_DTYPE_BF16 || a.K > kThinK || a.N % 2 || a.groups > 1 || a.group_rows || a.n_seg > 1 || is_pair(sg.kind))
        return B2KV_ERR_UNSUPPORTED;
    if (!aligned16(a.w) || !aligned16(sg.out) || a.ld_w % 2 || sg.ld % 2 || (a.residual && (!aligned16(a.residual) || a.ld_residual % 2)))
        return B2KV_ERR_UNSUPPORTED;
    // few rows: enough CTAs to be quick; many: the columns of w are loaded once per tile of rows
    const int row_tile = a.rows > 1024 ? kThinRows : 8;
    const dim3 grid((a.N / 2 + kThinThreads - 1) / kThinThreads, (a.rows + row_tile - 1) / row_tile);
    if (grid.y > 65535u) return B2KV_ERR_UNSUPPORTED;
    OverlapLaunch launch(grid, kThinThreads, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, a.K <= 16 ? linear_thin_kernel<16> : linear_thin_kernel<32>, a, row_tile));
    return B2KV_OK;
}

// A per-head product of many rows: the weight-streaming kernel on 128 rows at a time (the heads' matrices are small and
// stay in L2).
static int rows_in_slices(const b2kv_linear_args& all, int32_t* dev_status, void* stream) {
    const int es = elt_bytes(all.dtype);
    for (int r0 = 0; r0 < all.rows; r0 += 128) {
        b2kv_linear_args a = all;
        a.rows = all.rows - r0 < 128 ? all.rows - r0 : 128;
        a.x = static_cast<const char*>(all.x) + r0 * all.ld_x * es;
        if (all.residual) a.residual = all.residual + r0 * all.ld_residual;
        for (int s = 0; s < a.n_seg; ++s)
            a.seg[s].out = static_cast<char*>(all.seg[s].out) + r0 * all.seg[s].ld * (is_f32(all.seg[s].kind) ? 4 : es);
        const int rc = linear_rows_tc(a, dev_status, stream);
        if (rc != B2KV_OK) return rc;
    }
    return B2KV_OK;
}

}  // namespace lin
}  // namespace b2kv

using namespace b2kv;

extern "C" int b2kv_linear(const b2kv_linear_args* args, int32_t* dev_status, void* stream) {
    if (args == nullptr) return B2KV_ERR_BAD_ARG;
    const b2kv_linear_args& a = *args;
    if (elt_bytes(a.dtype) == 0) return B2KV_ERR_UNSUPPORTED;
    if (!a.x || !a.w || a.rows <= 0 || a.K <= 0 || a.N <= 0 || a.groups <= 0 || a.path < 0 || a.path > 4) return B2KV_ERR_BAD_ARG;
    if (a.n_seg < 1 || a.n_seg > B2KV_MAX_SEGMENTS || a.seg[a.n_seg - 1].end != a.N) return B2KV_ERR_BAD_ARG;
    if (a.bias && a.groups > 1) return B2KV_ERR_BAD_ARG;
    if (a.group_rows && (a.max_group_rows <= 0 || a.max_group_rows > a.rows)) return B2KV_ERR_BAD_ARG;
    int first = 0;
    for (int s = 0; s < a.n_seg; ++s) {
        const b2kv_segment& sg = a.seg[s];
        if (!sg.out || (sg.kind >= B2KV_SEG_SOFTCAP && !(a.limit > 0.f)) || sg.end <= first || sg.kind < B2KV_SEG_STORE || sg.kind > B2KV_SEG_DECAY) return B2KV_ERR_BAD_ARG;
        // pairs of columns never straddle a boundary (the last segment may end on an odd column if it has no pairs)
        if ((sg.end & 1) && (s + 1 < a.n_seg || lin::is_pair(sg.kind))) return B2KV_ERR_BAD_ARG;
        first = sg.end;
    }
    if (a.path == 2) return linear_rows_tc(a, dev_status, stream);
    if (a.path == 3) return linear_tiled_tc(a, dev_status, stream);
    if (a.path == 4) return lin::launch_thin(a, stream);
    if (a.path == 0 && a.dtype == B2KV_DTYPE_BF16) {
        int rc = lin::launch_thin(a, stream);
        if (rc != B2KV_ERR_UNSUPPORTED) return rc;
        if ((a.group_rows ? a.max_group_rows : a.rows) <= 128) {
            rc = linear_rows_tc(a, dev_status, stream);
        } else if (a.groups > 1 && a.group_rows == nullptr) {
            rc = lin::rows_in_slices(a, dev_status, stream);
        } else {
            rc = linear_tiled_tc(a, dev_status, stream);
        }
        if (rc != B2KV_ERR_UNSUPPORTED) return rc;
    }
    return lin::launch_simt(a, stream);
}
