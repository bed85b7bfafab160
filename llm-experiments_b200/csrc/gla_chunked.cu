#include "gla.cuh"
namespace b2kv { int gla_chunked(const b2kv_gla_args&, int32_t*, void*) { return B2KV_ERR_UNSUPPORTED; } }
