// Grouped, segmented linear layers (b2kv_linear): what the three kernels behind the entry point share.
#pragma once

#include "b2kv_common.cuh"

namespace b2kv {
namespace lin {

// x * sigmoid(1.702 x) of the clamped gate times the clamped up part plus one; silu(gate) * up.
__device__ __forceinline__ float glu(int kind, float g, float u, float limit) {
    if (kind == B2KV_SEG_GLU_SILU) return g / (1.0f + __expf(-g)) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + __expf(-1.702f * g)) * (u + 1.0f);
}

// Kinds whose columns are (gate, up) pairs; kinds whose output is fp32.
__host__ __device__ constexpr bool is_pair(int kind) { return kind == B2KV_SEG_GLU_SILU || kind == B2KV_SEG_GLU_CLAMP; }
__host__ __device__ constexpr bool is_f32(int kind) { return kind == B2KV_SEG_F32 || kind >= B2KV_SEG_SOFTCAP; }

// sigmoid(z)^(1 / tau) through ln(sigmoid(z)) = min(z, 0) - ln(1 + u), u = exp(-|z|), which cancels on neither side.  Without
// branches or calls: ln(1 + u) = 2 atanh(s), s = u / (2 + u) <= 1/3, as a series whose first dropped term is below 2^-26 of it.
__device__ __forceinline__ float decay(float z, float inv_tau) {
    const float u = __expf(-fabsf(z)), s = __fdividef(u, 2.0f + u), s2 = s * s;
    float p = 1.0f / 15.0f;
    p = fmaf(p, s2, 1.0f / 13.0f);
    p = fmaf(p, s2, 1.0f / 11.0f);
    p = fmaf(p, s2, 1.0f / 9.0f);
    p = fmaf(p, s2, 1.0f / 7.0f);
    p = fmaf(p, s2, 1.0f / 5.0f);
    p = fmaf(p, s2, 1.0f / 3.0f);
    p = fmaf(p, s2, 1.0f);
    return __expf((fminf(z, 0.f) - 2.0f * s * p) * inv_tau);
}
__device__ __forceinline__ float decay_exact(float z, float tau) { return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) / tau); }

// What happens to a single column before it is stored.
__device__ __forceinline__ float single(int kind, float v, float limit) {
    if (kind == B2KV_SEG_RELU2) {
        v = fmaxf(v, 0.f);
        return v * v;
    }
    if (kind == B2KV_SEG_DECAY) return decay(v, 1.0f / limit);
    return kind == B2KV_SEG_SOFTCAP ? limit * tanhf(v / limit) : v;
}

// Index of the segment that holds column c (segments are in column order).
__device__ __forceinline__ int segment_of(const b2kv_linear_args& a, int c) {
    int s = 0;
    while (s + 1 < a.n_seg && c >= a.seg[s].end) ++s;
    return s;
}

__device__ __forceinline__ int segment_first(const b2kv_linear_args& a, int s) { return s == 0 ? 0 : a.seg[s - 1].end; }

}  // namespace lin

// bf16 kernels on the tensor cores; B2KV_ERR_UNSUPPORTED when the shape is not one they take.
int linear_rows_tc(const b2kv_linear_args& a, int32_t* dev_status, void* stream);   // linear_rows.cu
int linear_tiled_tc(const b2kv_linear_args& a, int32_t* dev_status, void* stream);  // gemm.cu

}  // namespace b2kv
