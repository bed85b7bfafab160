// Gated linear attention: what the token-by-token and the chunked kernel share.
#pragma once

#include <math.h>

#include "b2kv_common.cuh"

namespace b2kv {

// Tensor-core kernel for segments of a prompt (bf16); B2KV_ERR_UNSUPPORTED when the shape is not one it takes.
int gla_chunked(const b2kv_gla_args& a, int32_t* dev_status, void* stream);
size_t gla_chunked_workspace(int H, int dim, int vdim, int n_segments, int max_n, int dtype);  // 0: no such form

namespace gla {

__device__ __forceinline__ float silu(float g) { return g / (1.0f + expf(-g)); }

__device__ __forceinline__ float silu_fast(float g) { return __fdividef(g, 1.0f + __expf(-g)); }

// Segment of a CTA, and whether it lies inside the buffers.
__device__ __forceinline__ bool segment_place(const b2kv_gla_args& a, int i, b2kv_row_segment& sg) {
    if (a.segments == nullptr) {
        sg.row0 = i, sg.n = 1, sg.slot = i;
    } else {
        sg = a.segments[i];
    }
    return sg.row0 >= 0 && sg.n > 0 && sg.n <= a.max_n && sg.row0 + sg.n <= a.rows && sg.slot >= 0 && sg.slot < a.n_slots;
}

}  // namespace gla
}  // namespace b2kv
