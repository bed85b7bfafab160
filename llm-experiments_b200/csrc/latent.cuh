// Latent attention: arguments shared by the CUDA-core and the tensor-core kernel for single query rows.
#pragma once

#include "b2kv_common.cuh"

namespace b2kv {

struct LatentDecodeArgs {
    const void* q_latent;  // [rows, H, kv_rank]
    const void* q;         // rotated query rows: head h at column h * (dim + rot), its rotated part from + dim on
    const void* key_cache;
    const void* latent_cache;
    void* out;  // [rows, H, kv_rank]
    const int32_t* row_slot;
    const int32_t* row_pos;
    int32_t* dev_status;
    int64_t ld_q;
    int dim, n_slots, T_max, rows, H, kv_rank, rot, window, span;
    float scale;
};

// Tensor-core kernel (bf16); B2KV_ERR_UNSUPPORTED when the shape is not one it takes.
int latent_decode_tc(const LatentDecodeArgs& a, void* workspace, size_t workspace_bytes, void* stream);
size_t latent_decode_tc_workspace(int rows, int H, int kv_rank, int span);

// Sequence of query row i, and whether its position lies inside that sequence's cache.
__device__ __forceinline__ bool row_place(const int32_t* row_slot, const int32_t* row_pos, int i, int n_slots, int T_max,
                                          int& slot, int& pos) {
    slot = row_slot ? row_slot[i] : i;
    pos = row_pos[i];
    return slot >= 0 && slot < n_slots && pos >= 0 && pos < T_max;
}

}  // namespace b2kv
