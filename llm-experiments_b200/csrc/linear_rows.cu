// b2kv_linear for few rows (a decode step) on the tensor cores: the weights are streamed once.
//
// The scheme is that of qkv_append.cu: the product is computed transposed, D[feature, row] = W^T x^T, so that the 128
// rows of an MMA are output features and its columns the few rows of x; one CTA per 128 output features; warp 4 streams W
// (an MN-major operand as it lies in memory) and x (K-major) with TMA through a ring, warp 5 issues tcgen05.mma into one
// accumulator, warps 0-3 are the epilogue (thread = output feature = TMEM lane); a product with few tiles has its input
// features cut into ranges, one per CTA of a cluster, whose partial sums meet in distributed shared memory.  What is
// different here:
//
//   * groups: the tensor maps have a third dimension, so a CTA can take the columns of x and the matrix of one head (exact
//     extents: what lies past a head's features reads as zero), or, with device-side row offsets, the rows and the matrix
//     of one expert.  An expert without rows costs a launched CTA that leaves at once; rows past an expert's last one are
//     columns of D that nobody stores;
//   * the output columns are cut into segments with places and forms of their own.  Gated pairs sit in neighbouring TMEM
//     lanes: the even lane finishes the even rows and the odd lane the odd ones after one shuffle per pair of rows;
//   * fp32 outputs, with an fp32 residual added before the store;
//   * input features and output columns need not fill whole tiles.
#include <algorithm>

#include "linear.cuh"
#include "tc_ptx.cuh"
#include "tma_map.cuh"

namespace b2kv {
namespace linrows {

using namespace tc;

constexpr int kFeat = 128;   // output features per CTA (MMA M)
constexpr int kKTile = 128;  // input features per stage
constexpr int kMaxStages = 6;
constexpr int kRingBytes = 200 * 1024;
constexpr int kRingBytesTwo = 100 * 1024;  // two CTAs per SM, when there are several waves of them
constexpr int kSmemBytes = 224 * 1024;
constexpr int kWBytes = kKTile * kFeat * 2;
constexpr int kWHalf = kWBytes / 2;
constexpr int kMaxRows = 128;
constexpr int kThreads = 192;

struct Shared {
    alignas(8) uint64_t full[kMaxStages], empty[kMaxStages];
    uint64_t done;
    uint32_t tmem_base;
    int got[8];
};

struct Params {
    b2kv_linear_args a;
    int32_t* dev_status;
    int tiles_n, Bn, box_rows, stages, splits, split_shift;
};

__device__ __forceinline__ uint32_t cluster_rank() {
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ void peer_store_u32(uint32_t local, uint32_t rank, uint32_t v) {
    uint32_t addr;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(addr) : "r"(local), "r"(rank));
    asm volatile("st.shared::cluster.u32 [%0], %1;" ::"r"(addr), "r"(v) : "memory");
}

// fp32 accumulate, bf16 operands, A MN-major, B K-major, M = 128, N = n
__host__ __device__ constexpr uint32_t idesc_of(int n) { return instr_desc(1, 0, n); }

// Where one thread's output feature goes.
struct Place {
    void* out;
    const float* residual;
    int64_t ld, ld_residual, col;  // col: element inside the output row
    int kind;
    float bias;
    bool live;
};

// Stores kN values of this thread's feature, for rows row[0 .. kN - 1] (-1: none).
template <int kN>
__device__ __forceinline__ void emit(const Place& pl, float (&v)[kN], const int64_t (&row)[kN], float limit) {
#pragma unroll
    for (int j = 0; j < kN; ++j) v[j] += pl.bias;
    if (lin::is_pair(pl.kind)) {
        // (kind is the same for the whole warp: segments start on multiples of 32 columns)
        const bool odd = threadIdx.x & 1;
        __nv_bfloat16* out = static_cast<__nv_bfloat16*>(pl.out) + pl.col;
#pragma unroll
        for (int j = 0; j < kN; j += 2) {
            const float other = __shfl_xor_sync(0xffffffffu, odd ? v[j] : v[j + 1], 1);
            const float g = odd ? other : v[j], u = odd ? v[j + 1] : other;
            const int64_t r = odd ? row[j + 1] : row[j];
            const float z = lin::glu(pl.kind, g, u, limit);
            if (r >= 0 && pl.live) out[r * pl.ld] = __float2bfloat16_rn(z);
        }
        return;
    }
    if (!pl.live) return;
    if (pl.kind >= B2KV_SEG_RELU2) {
#pragma unroll
        for (int j = 0; j < kN; ++j) v[j] = lin::single(pl.kind, v[j], limit);
    }
    if (lin::is_f32(pl.kind)) {
        float* out = static_cast<float*>(pl.out) + pl.col;
        float add[kN];
#pragma unroll
        for (int j = 0; j < kN; ++j)
            add[j] = (pl.residual != nullptr && row[j] >= 0) ? pl.residual[row[j] * pl.ld_residual + pl.col] : 0.f;
#pragma unroll
        for (int j = 0; j < kN; ++j)
            if (row[j] >= 0) out[row[j] * pl.ld] = v[j] + add[j];
    } else {
        __nv_bfloat16* out = static_cast<__nv_bfloat16*>(pl.out) + pl.col;
#pragma unroll
        for (int j = 0; j < kN; ++j)
            if (row[j] >= 0) out[row[j] * pl.ld] = __float2bfloat16_rn(v[j]);
    }
}

__global__ void __launch_bounds__(kThreads)
linear_rows_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x,
                   const __grid_constant__ Params p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ Shared sm;
    uint8_t* const w_ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = p.splits > 1 ? static_cast<int>(cluster_rank()) : 0;
    const int tile = blockIdx.x / p.splits;
    const int g = tile / p.tiles_n;
    const int c0 = (tile % p.tiles_n) * kFeat;
    const int n_k_all = (p.a.K + kKTile - 1) / kKTile;
    const int k_first = static_cast<int>(static_cast<long long>(n_k_all) * split / p.splits);
    const int n_k = static_cast<int>(static_cast<long long>(n_k_all) * (split + 1) / p.splits) - k_first;
    const bool by_rows = p.a.group_rows != nullptr;

    grid_launch_dependents();
    int row0 = 0, n_rows = p.a.rows;
    if (by_rows) {
        // the row offsets come from the kernel before this one
        if (threadIdx.x == 0) grid_dependency_wait();
        __syncthreads();
        row0 = p.a.group_rows[g];
        n_rows = min(p.a.group_rows[g + 1] - row0, p.Bn);
        if (n_rows <= 0) return;  // all CTAs of a cluster share the group
    }
    const int Bn = by_rows ? (n_rows + 15) / 16 * 16 : p.Bn;
    const uint32_t x_span = static_cast<uint32_t>(Bn) * 128u;  // Bn rows of one 64-feature span
    const uint32_t x_span_max = static_cast<uint32_t>(p.Bn) * 128u;
    uint8_t* const x_ring = w_ring + p.stages * kWBytes;
    const int n_st = p.stages;
    float* const recv = reinterpret_cast<float*>(x_ring + p.stages * 2 * x_span_max);
    const int rows_per_cta = p.Bn >> p.split_shift;
    const uint32_t stage_bytes = kWBytes + 2 * x_span;

    if (threadIdx.x == 0) {
        for (int s = 0; s < kMaxStages; ++s) {
            mbar_init(&sm.full[s], 1);
            mbar_init(&sm.empty[s], 1);
        }
        mbar_init(&sm.done, 1);
        for (int s = 0; s < 8; ++s) sm.got[s] = 0;
        fence_mbar_init();
    }
    __syncthreads();
    // first cluster barrier: once a CTA has waited for it, all its peers are running with their flags cleared
    if (p.splits > 1 && warp != 4) cluster_arrive();
    if (warp == 5) {
        tmem_alloc(&sm.tmem_base, kMaxRows);
        tmem_relinquish();
        tc_fence_before();
    }

    bool done = true;  // this thread's accumulator lane is complete
    if (warp == 4) {
        auto load_w = [&](int st, int k0) {
            tma_load_3d(w_ring + st * kWBytes, &tm_w, &sm.full[st], c0, k0, g);
            tma_load_3d(w_ring + st * kWBytes + kWHalf, &tm_w, &sm.full[st], c0 + 64, k0, g);
        };
        auto load_x = [&](int st, int k0) {
            uint8_t* dst = x_ring + st * 2 * x_span_max;
            for (int r = 0; r < Bn; r += p.box_rows) {
                tma_load_3d(dst + r * 128, &tm_x, &sm.full[st], k0, by_rows ? 0 : g, row0 + r);
                tma_load_3d(dst + x_span + r * 128, &tm_x, &sm.full[st], k0 + 64, by_rows ? 0 : g, row0 + r);
            }
        };
        const int ahead = n_k < n_st ? n_k : n_st;
        if (lane == 0) {
            for (int i = 0; i < ahead; ++i) {
                mbar_arrive_expect_tx(&sm.full[i], stage_bytes);
                load_w(i, (k_first + i) * kKTile);
            }
            grid_dependency_wait();
            for (int i = 0; i < ahead; ++i) load_x(i, (k_first + i) * kKTile);
        }
        __syncwarp();
        if (p.splits > 1) cluster_arrive();
        if (lane == 0) {
            for (int i = ahead; i < n_k; ++i) {
                const int st = i % n_st;
                if (!mbar_wait(&sm.empty[st], ((i / n_st) & 1) ^ 1)) break;
                mbar_arrive_expect_tx(&sm.full[st], stage_bytes);
                load_w(st, (k_first + i) * kKTile);
                load_x(st, (k_first + i) * kKTile);
            }
        }
        __syncwarp();
        if (p.splits > 1) cluster_wait();
    } else if (warp == 5) {
        if (lane == 0) {
            tc_fence_after();
            const uint32_t tmem = *reinterpret_cast<volatile uint32_t*>(&sm.tmem_base);
            const uint32_t idesc = idesc_of(Bn);
            bool ok = true;
            for (int i = 0; i < n_k && ok; ++i) {
                const int st = i % n_st;
                ok = mbar_wait(&sm.full[st], (i / n_st) & 1);
                if (!ok) break;
                tc_fence_after();
                const uint64_t da = smem_desc(smem_u32(w_ring + st * kWBytes), kWHalf, 1024);
                const uint64_t db = smem_desc(smem_u32(x_ring + st * 2 * x_span_max), 16, 1024);
#pragma unroll
                for (int kk = 0; kk < kKTile / 16; ++kk) {
                    const uint32_t b_off = (kk >> 2) * x_span + (kk & 3) * 32;
                    mma_ss(tmem, da + static_cast<uint64_t>((kk * 2048) >> 4), db + static_cast<uint64_t>(b_off >> 4), idesc,
                           (i | kk) ? 1u : 0u);
                }
                mma_commit(&sm.empty[st]);
            }
            if (ok) mma_commit(&sm.done);
        }
        __syncwarp();
        if (p.splits > 1) cluster_wait();
    } else {
        // ------------------------------ epilogue: thread = output feature ------------------------------
        const int m = threadIdx.x;
        // outputs may be read by the kernels before this one and the residual is written by them
        if (threadIdx.x == 0) grid_dependency_wait();
        named_barrier_sync<kFeat>(1);
        if (p.splits > 1) cluster_wait();
        if (mbar_wait(&sm.done, 0)) {
            tc_fence_after();
            const uint32_t t_lane = sm.tmem_base + (static_cast<uint32_t>(warp * 32) << 16);
            if (p.splits > 1) {
                // row b's partial goes to CTA b mod splits, slab `split`, row b / splits
                const uint32_t mine = smem_u32(recv) + static_cast<uint32_t>((split * rows_per_cta) * kFeat + m) * 4u;
                for (int nb = 0; nb < Bn; nb += 16) {
                    uint32_t v[16];
                    tmem_ld16(t_lane + nb, v);
                    tmem_wait_ld();
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        const int b = nb + j;
                        peer_store_u32(mine + static_cast<uint32_t>((b >> p.split_shift) * kFeat) * 4u,
                                       static_cast<uint32_t>(b & (p.splits - 1)), v[j]);
                    }
                }
                if (m < p.splits) peer_store_u32(smem_u32(&sm.got[split]), static_cast<uint32_t>(m), 1u);
            }
        } else {
            report_status(p.dev_status, B2KV_DEV_WAIT_TIMEOUT);
            done = false;
        }
    }

    if (p.splits > 1) {
        // second cluster barrier: the partials of this CTA's rows have arrived, or a CTA gave up and raised no flag
        __syncwarp();
        cluster_arrive();
        cluster_wait();
    }
    if (warp < 4) {
        const int m = threadIdx.x, c = c0 + m;
        Place pl;
        const int s = lin::segment_of(p.a, min(c, p.a.N - 1));
        const b2kv_segment& sg = p.a.seg[s];
        const int local = c - lin::segment_first(p.a, s);
        pl.kind = sg.kind;
        pl.out = sg.out;
        pl.ld = sg.ld;
        pl.ld_residual = p.a.ld_residual;
        pl.col = (lin::is_pair(sg.kind) ? local / 2 : local) + (by_rows ? 0 : static_cast<int64_t>(g) * sg.group);
        pl.residual = sg.kind == B2KV_SEG_F32 ? p.a.residual : nullptr;
        pl.live = c < p.a.N;
        pl.bias = pl.live && p.a.bias != nullptr ? p.a.bias[c] : 0.f;
        if (p.splits > 1) {
            bool all = true;
            for (int sp = 0; sp < p.splits; ++sp) all = all && *reinterpret_cast<volatile int*>(&sm.got[sp]) == 1;
            if (all) {
                for (int r0 = 0; r0 < rows_per_cta; r0 += 8) {
                    float acc[8];
                    int64_t row[8];
#pragma unroll
                    for (int u = 0; u < 8; ++u) {
                        const int b = ((r0 + u) << p.split_shift) + split;
                        row[u] = (r0 + u < rows_per_cta && b < n_rows) ? row0 + b : -1;
                        acc[u] = 0.f;
                    }
                    for (int sp = 0; sp < p.splits; ++sp) {
#pragma unroll
                        for (int u = 0; u < 8; ++u)
                            if (row[u] >= 0) acc[u] += recv[(sp * rows_per_cta + r0 + u) * kFeat + m];
                    }
                    emit<8>(pl, acc, row, p.a.limit);
                }
            }
        } else if (__all_sync(0xffffffffu, done)) {
            const uint32_t t_lane = sm.tmem_base + (static_cast<uint32_t>(warp * 32) << 16);
            for (int nb = 0; nb < Bn; nb += 16) {
                uint32_t v[16];
                __syncwarp();  // the lanes' stores above differ
                tmem_ld16(t_lane + nb, v);
                tmem_wait_ld();
                float f[16];
                int64_t row[16];
#pragma unroll
                for (int j = 0; j < 16; ++j) {
                    f[j] = __uint_as_float(v[j]);
                    row[j] = nb + j < n_rows ? row0 + nb + j : -1;
                }
                emit<16>(pl, f, row, p.a.limit);
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        tc_fence_after();
        tmem_dealloc(sm.tmem_base, kMaxRows);
    }
}

// 3-D map of bf16 elements with 64-element boxes along the contiguous dimension, 128-byte swizzle.
static bool make_map_3d(CUtensorMap* map, const void* base, const cuuint64_t (&dims)[3], int64_t stride1, int64_t stride2,
                        int box1, int box2) {
    EncodeTiledFn fn = tensor_map_encoder();
    if (fn == nullptr) return false;
    const cuuint64_t strides[2] = {static_cast<cuuint64_t>(stride1) * 2, static_cast<cuuint64_t>(stride2) * 2};
    const cuuint32_t box[3] = {64, static_cast<cuuint32_t>(box1), static_cast<cuuint32_t>(box2)};
    const cuuint32_t estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace linrows

int linear_rows_tc(const b2kv_linear_args& a, int32_t* dev_status, void* stream) {
    using namespace linrows;
    if (a.dtype != B2KV_DTYPE_BF16) return B2KV_ERR_UNSUPPORTED;
    const int max_rows = a.group_rows ? a.max_group_rows : a.rows;
    if (max_rows > kMaxRows) return B2KV_ERR_UNSUPPORTED;
    if (!aligned16(a.x) || !aligned16(a.w) || a.ld_x % 8 || a.ld_w % 8 || a.group_x % 8 || a.group_w % 8 || a.ld_x <= 0 || a.ld_w <= 0)
        return B2KV_ERR_UNSUPPORTED;
    if (a.groups > 1 && (a.group_w <= 0 || (!a.group_rows && a.group_x <= 0))) return B2KV_ERR_UNSUPPORTED;
    for (int s = 0; s + 1 < a.n_seg; ++s)
        if (a.seg[s].end % 32 != 0) return B2KV_ERR_UNSUPPORTED;
    Params p{};
    p.a = a;
    p.dev_status = dev_status;
    p.tiles_n = (a.N + kFeat - 1) / kFeat;
    p.Bn = (max_rows + 15) / 16 * 16;
    p.box_rows = a.group_rows ? 16 : p.Bn;
    CUtensorMap tw, tx;
    const cuuint64_t wd[3] = {static_cast<cuuint64_t>(a.N), static_cast<cuuint64_t>(a.K), static_cast<cuuint64_t>(a.groups)};
    const cuuint64_t xd[3] = {static_cast<cuuint64_t>(a.K), static_cast<cuuint64_t>(a.group_rows ? 1 : a.groups),
                              static_cast<cuuint64_t>(a.rows)};
    if (!make_map_3d(&tw, a.w, wd, a.ld_w, a.groups > 1 ? a.group_w : a.ld_w * a.K, kKTile, 1) ||
        !make_map_3d(&tx, a.x, xd, a.group_rows || a.groups == 1 ? a.ld_x : a.group_x, a.ld_x, 1, p.box_rows))
        return B2KV_ERR_UNSUPPORTED;
    const long long tiles = static_cast<long long>(p.tiles_n) * a.groups;
    if (tiles > 0x0fffffff) return B2KV_ERR_UNSUPPORTED;
    const int n_k = (a.K + kKTile - 1) / kKTile;
    p.splits = 1;
    if (tune_get("matmul_splits") > 0) {
        while (p.splits * 2 <= std::min(std::min(tune_get("matmul_splits"), 8), n_k)) p.splits *= 2;
    } else {
        // (clusters of eight find few places: they pay only where there are few of them)
        while (p.splits < 8 && tiles * p.splits * 2 <= (p.splits == 4 ? 64 : 148) && n_k / (p.splits * 2) >= 2) p.splits *= 2;
    }
    while ((1 << p.split_shift) < p.splits) ++p.split_shift;
    const int recv_bytes = p.splits > 1 ? p.Bn * kFeat * 4 : 0;
    const int stage_bytes = kWBytes + 2 * p.Bn * 128;
    const bool waves = tiles * p.splits > device_sm_count();
    const int ring = waves ? kRingBytesTwo : kRingBytes;
    p.stages = std::max(2, std::min(std::min(kMaxStages, std::max(n_k, 1)), std::min(ring, kSmemBytes - recv_bytes) / stage_bytes));
    const size_t smem = static_cast<size_t>(p.stages) * stage_bytes + recv_bytes + 1024;
    static int configured[64] = {0};
    int dev = 0;
    B2KV_CUDA_TRY(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64) return B2KV_ERR_UNSUPPORTED;
    if (configured[dev] < static_cast<int>(smem)) {
        B2KV_CUDA_TRY(cudaFuncSetAttribute(linear_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        configured[dev] = static_cast<int>(smem);
    }
    OverlapLaunch launch(static_cast<unsigned>(tiles * p.splits), kThreads, smem, stream, p.splits);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, linear_rows_kernel, tw, tx, p));
    return B2KV_OK;
}

}  // namespace b2kv
