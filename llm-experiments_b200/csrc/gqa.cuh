// Grouped-query attention on caches of keys and values: arguments shared by the CUDA-core and the tensor-core kernel for
// single query rows.
#pragma once

#include "latent.cuh"

namespace b2kv {

struct GqaDecodeArgs {
    const void* q;  // head h of row i at q + i * ld_q + h * dim
    const void* k_cache;
    const void* v_cache;
    void* out;  // head h of row i at out + i * ld_out + h * vdim
    const float* slopes;
    const int32_t* row_slot;
    const int32_t* row_pos;
    int32_t* dev_status;
    int64_t ld_q, ld_out;
    int n_slots, T_max, rows, H, G, dim, vdim, span;
    float scale;
};

// Tensor-core kernel (bf16); B2KV_ERR_UNSUPPORTED when the shape is not one it takes.
int gqa_decode_tc(const GqaDecodeArgs& a, void* workspace, size_t workspace_bytes, void* stream);
size_t gqa_decode_tc_workspace(int rows, int H, int G, int vdim, int span);

}  // namespace b2kv
