#include "linear.cuh"
#include "latent.cuh"
namespace b2kv {
int linear_rows_tc(const b2kv_linear_args& a, int32_t* dev_status, void* stream) { return B2KV_ERR_UNSUPPORTED; }
int linear_tiled_tc(const b2kv_linear_args& a, int32_t* dev_status, void* stream) { return B2KV_ERR_UNSUPPORTED; }
int latent_decode_tc(const LatentDecodeArgs& a, void* workspace, size_t workspace_bytes, void* stream){ return B2KV_ERR_UNSUPPORTED; }
size_t latent_decode_tc_workspace(int rows, int H, int kv_rank, int span){return 0;}
}
