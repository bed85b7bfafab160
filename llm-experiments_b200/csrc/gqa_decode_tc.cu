#include "gqa.cuh"
namespace b2kv {
int gqa_decode_tc(const GqaDecodeArgs&, void*, size_t, void*) { return B2KV_ERR_UNSUPPORTED; }
size_t gqa_decode_tc_workspace(int, int, int, int, int) { return 0; }
}
