// Attention of single query rows over cached latent rows on the Blackwell tensor cores (bf16).
//
// All heads of a row read the same latent rows, so the cache is streamed once per row (and group of heads) and the work is
// matrix-shaped: H heads against every key.  Both products are computed transposed, so that the 128 rows of an MMA are the
// plentiful dimension and its columns the few heads (as in the weight-streaming kernels):
//
//   S^T[key, head]     = latent[key, :] q_latent[head, :] + key part[key, :] q_rot[head, :]      A K-major
//   O^T[element, head] += latent[:, element]^T P[key, head]                                       the same tile, A MN-major
//
//   * one CTA per (row, group of up to 64 heads, share of the row's window).  A tile is 64 keys, so that two and a half tiles
//     of 512 + 64 elements fit shared memory: pairs of 64-element chunks of the latent rows, copied with TMA (128-byte swizzle)
//     into a ring of pairs, and a chunk of the rotated key part in a ring of two.  An MMA has 128 rows all the same: the upper
//     64 rows of S^T are made from whatever lies behind a chunk in shared memory, and nobody looks at them (64-row tiles of
//     128-row MMAs waste tensor time that is not the limit; 128-key tiles left no room for the next tile's copies, and every
//     tile then paid a full memory latency);
//   * warp 4 copies, warp 5 issues tcgen05.mma from one thread, in the order S(j + 1), O(j), so that the next tile's scores are
//     made under this tile's softmax.  Warps 0-1 are the softmax: thread = key = TMEM lane, one column per head.  Column maxima
//     take one integer warp reduction per head and an exchange through shared memory; sums stay in registers per key until the
//     end; P goes to shared memory as the K-major operand of the second product; O stays in tensor memory and is rescaled (by
//     warps 0-3) only when a head's maximum has grown by more than 2^8;
//   * the shares of one row (few rows, long windows) leave fp32 partial results that a small kernel merges.
//
// No MMA is predicated; sizes that do not fill a chunk read as zero.  Every wait is bounded.
#include <math.h>

#include <algorithm>

#include "latent.cuh"
#include "tc_ptx.cuh"
#include "tma_map.cuh"

namespace b2kv {
namespace latdec {

using namespace tc;

constexpr int kTile = 64;                // keys per tile
constexpr int kChunkBytes = kTile * 128;  // 64 rows x 64 bf16
constexpr int kPairBytes = 2 * kChunkBytes;
constexpr int kMaxPairs = 12;
constexpr int kMaxHeads = 64;
constexpr int kThreads = 192;
constexpr int kSmemLimit = 226 * 1024;
constexpr float kRescaleThreshold = 8.0f;
constexpr float kNothingSeen = -1e30f;

struct Shared {
    alignas(8) uint64_t q_full;
    uint64_t pair_full[kMaxPairs], pair_empty[kMaxPairs];
    uint64_t rot_full[2], rot_empty[2];
    uint64_t s_full[2], p_ready[2], o_done;
    uint32_t tmem_base;
    volatile int abort_flag;
    int need;
    int warp_max[2][kMaxHeads];
    float m[kMaxHeads], factor[kMaxHeads], sum[2][kMaxHeads];
};

struct Params {
    const int32_t* row_slot;
    const int32_t* row_pos;
    __nv_bfloat16* out;  // [rows, H, kv_rank]
    float* partial;      // [rows, splits, H, kv_rank + 2] when splits > 1
    int32_t* dev_status;
    int n_slots, T_max, H, kv_rank, window, splits, head_groups;
    int tile_pairs;  // pairs per tile: ceil(kv_rank / 128)
    int ring_pairs;  // pairs of the ring
    int tmem_cols;
    float prescale;  // scale * log2(e)
};

// Order-preserving map of floats to signed integers (for the integer warp reduction) and back.
__device__ __forceinline__ int ordered(float f) {
    const int b = __float_as_int(f);
    return b ^ ((b >> 31) & 0x7fffffff);
}
__device__ __forceinline__ float unordered(int o) { return __int_as_float(o ^ ((o >> 31) & 0x7fffffff)); }

template <int kHn>
__global__ void __launch_bounds__(kThreads)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_ql, const __grid_constant__ CUtensorMap tm_qr,
                        const __grid_constant__ CUtensorMap tm_lat, const __grid_constant__ CUtensorMap tm_key, const Params p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ Shared sm;
    uint8_t* const ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* const rot_tile = ring + p.ring_pairs * kPairBytes;
    uint8_t* const q_tile = rot_tile + 2 * kChunkBytes;  // 2 * tile_pairs latent chunks, then the rotated one; kHn rows each
    constexpr int kQChunk = kHn * 128;
    uint8_t* const p_tile = q_tile + (2 * p.tile_pairs + 1) * kQChunk;  // two tiles of [kHn][64 keys]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = blockIdx.x % p.splits;
    const int h0 = blockIdx.x / p.splits % p.head_groups * kHn;
    const int i = blockIdx.x / (p.splits * p.head_groups);

    grid_launch_dependents();
    if (threadIdx.x == 0) {
        mbar_init(&sm.q_full, 1);
        for (int s = 0; s < kMaxPairs; ++s) {
            mbar_init(&sm.pair_full[s], 1);
            mbar_init(&sm.pair_empty[s], 1);
        }
        for (int s = 0; s < 2; ++s) {
            mbar_init(&sm.rot_full[s], 1);
            mbar_init(&sm.rot_empty[s], 1);
            mbar_init(&sm.s_full[s], 1);
            mbar_init(&sm.p_ready[s], 128);
        }
        mbar_init(&sm.o_done, 1);
        sm.abort_flag = 0;
        sm.need = 0;
        fence_mbar_init();
        grid_dependency_wait();  // queries, cache rows and positions come from the kernels before this one
    }
    if (warp == 5) {
        tmem_alloc(&sm.tmem_base, p.tmem_cols);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sm.tmem_base;

    // this CTA's tiles: [first, first + n_tiles) of the row's window, which starts at token t0
    int slot, pos;
    const bool valid = row_place(p.row_slot, p.row_pos, i, p.n_slots, p.T_max, slot, pos);
    const int t0 = valid && p.window > 0 ? max(0, pos - p.window + 1) : 0;
    const int all_tiles = valid ? (pos - t0) / kTile + 1 : 0;
    const int share = (all_tiles + p.splits - 1) / p.splits;
    const int first = split * share;
    const int n_tiles = max(0, min(share, all_tiles - first));
    if (!valid && threadIdx.x == 0) report_status(p.dev_status, B2KV_DEV_BAD_POSITION);
    const uint32_t o_base = tmem + 2 * kHn;  // S of even and odd tiles in columns [0, 2 kHn), O of pair g behind them

    if (warp == 4) {
        // ------------------------------ TMA producer ------------------------------
        if (lane == 0 && n_tiles > 0) {
            bool ok = true;
            mbar_arrive_expect_tx(&sm.q_full, (2 * p.tile_pairs + 1) * kQChunk);
            for (int c = 0; c < 2 * p.tile_pairs; ++c) tma_load_3d(q_tile + c * kQChunk, &tm_ql, &sm.q_full, c * 64, h0, i);
            tma_load_3d(q_tile + 2 * p.tile_pairs * kQChunk, &tm_qr, &sm.q_full, 0, h0, i);
            int slot_i = 0;
            uint32_t phase = 1;  // parity of the "empty" phase to wait for: the ring starts empty
            for (int j = 0; j < n_tiles && ok; ++j) {
                const int row = slot * p.T_max + t0 + (first + j) * kTile;
                ok = mbar_wait(&sm.rot_empty[j & 1], ((j >> 1) & 1) ^ 1);
                if (!ok) break;
                mbar_arrive_expect_tx(&sm.rot_full[j & 1], kChunkBytes);
                tma_load_3d(rot_tile + (j & 1) * kChunkBytes, &tm_key, &sm.rot_full[j & 1], 0, 0, row);
                for (int g = 0; g < p.tile_pairs; ++g) {
                    ok = mbar_wait(&sm.pair_empty[slot_i], phase);
                    if (!ok) break;
                    mbar_arrive_expect_tx(&sm.pair_full[slot_i], kPairBytes);
                    tma_load_3d(ring + slot_i * kPairBytes, &tm_lat, &sm.pair_full[slot_i], g * 128, 0, row);
                    tma_load_3d(ring + slot_i * kPairBytes + kChunkBytes, &tm_lat, &sm.pair_full[slot_i], g * 128 + 64, 0, row);
                    if (++slot_i == p.ring_pairs) slot_i = 0, phase ^= 1;
                }
            }
            if (!ok) sm.abort_flag = 1;
        }
        __syncwarp();
    } else if (warp == 5) {
        // ------------------------------ MMA issuer ------------------------------
        if (lane == 0 && n_tiles > 0) {
            constexpr uint32_t idesc_s = instr_desc(0, 0, kHn), idesc_o = instr_desc(1, 0, kHn);
            const uint64_t d_lat_k = smem_desc(smem_u32(ring), 16, 1024);            // latent rows, K-major (keys are M)
            const uint64_t d_lat_mn = smem_desc(smem_u32(ring), kChunkBytes, 1024);  // the same bytes, MN-major (elements are M)
            const uint64_t d_rot = smem_desc(smem_u32(rot_tile), 16, 1024);
            const uint64_t d_q = smem_desc(smem_u32(q_tile), 16, 1024), d_p = smem_desc(smem_u32(p_tile), 16, 1024);
            constexpr uint32_t kPair16 = kPairBytes >> 4, kChunk16 = kChunkBytes >> 4, kQ16 = kQChunk >> 4;
            const uint64_t d_qr = d_q + static_cast<uint64_t>(2 * p.tile_pairs) * kQ16;
            int slot_i = 0, done_i = 0;  // ring places of the next pair to multiply with the queries / with P
            uint32_t phase = 0;
            bool ok = mbar_wait(&sm.q_full, 0);
            // scores of tile j
            auto issue_s = [&](int j) {
                if (!mbar_wait(&sm.rot_full[j & 1], (j >> 1) & 1)) return false;
                tc_fence_after();
                const uint32_t s_tmem = tmem + (j & 1) * kHn;
                const uint64_t ar = d_rot + static_cast<uint64_t>(j & 1) * kChunk16;
#pragma unroll
                for (int kk = 0; kk < 4; ++kk)
                    mma_ss(s_tmem, ar + static_cast<uint64_t>(2 * kk), d_qr + static_cast<uint64_t>(2 * kk), idesc_s, kk ? 1u : 0u);
                mma_commit(&sm.rot_empty[j & 1]);
                for (int g = 0; g < p.tile_pairs; ++g) {
                    if (!mbar_wait(&sm.pair_full[slot_i], phase)) return false;
                    tc_fence_after();
                    const uint64_t a = d_lat_k + static_cast<uint64_t>(slot_i) * kPair16;
                    const uint64_t b = d_q + static_cast<uint64_t>(2 * g) * kQ16;
#pragma unroll
                    for (int kk = 0; kk < 8; ++kk)
                        mma_ss(s_tmem, a + static_cast<uint64_t>((kk >> 2) * kChunk16 + (kk & 3) * 2),
                               b + static_cast<uint64_t>((kk >> 2) * kQ16 + (kk & 3) * 2), idesc_s, 1u);
                    if (++slot_i == p.ring_pairs) slot_i = 0, phase ^= 1;
                }
                mma_commit(&sm.s_full[j & 1]);
                return true;
            };
            ok = ok && issue_s(0);
            for (int j = 0; j < n_tiles && ok; ++j) {
                // P(j - 1) has been waited for, so S(j - 1) has been read and its columns are free
                if (j + 1 < n_tiles) ok = issue_s(j + 1);
                ok = ok && mbar_wait(&sm.p_ready[j & 1], (j >> 1) & 1);
                if (!ok) break;
                tc_fence_after();
                const uint64_t b = d_p + static_cast<uint64_t>(j & 1) * kQ16;
                for (int g = 0; g < p.tile_pairs; ++g) {
                    const uint64_t a = d_lat_mn + static_cast<uint64_t>(done_i) * kPair16;
                    const uint32_t o = o_base + g * kHn;
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk)  // 16 keys: 2048 bytes of the tile, 32 bytes of P
                        mma_ss(o, a + static_cast<uint64_t>((kk * 2048) >> 4), b + static_cast<uint64_t>(2 * kk), idesc_o,
                               (j | kk) ? 1u : 0u);
                    mma_commit(&sm.pair_empty[done_i]);
                    if (++done_i == p.ring_pairs) done_i = 0;
                }
                mma_commit(&sm.o_done);
            }
            if (!ok) sm.abort_flag = 1;
        }
        __syncwarp();
    } else {
        // ------------------------------ softmax: thread = key of the tile ------------------------------
        const int key = threadIdx.x;
        const uint32_t lane_base = static_cast<uint32_t>(warp * 32) << 16;
        const float c = p.prescale;
        float l[kHn];
#pragma unroll
        for (int h = 0; h < kHn; ++h) l[h] = 0.f;
        bool ok = true;
        for (int j = 0; j < n_tiles; ++j) {
            ok = __all_sync(0xffffffffu, mbar_wait(&sm.s_full[j & 1], (j >> 1) & 1));
            if (!ok) break;
            tc_fence_after();
            uint32_t r[kHn];
            if (warp < kTile / 32) {
                const bool seen = t0 + (first + j) * kTile + key <= pos;
#pragma unroll
                for (int cc = 0; cc < kHn / 16; ++cc)
                    tmem_ld16(tmem + lane_base + (j & 1) * kHn + cc * 16, *reinterpret_cast<uint32_t(*)[16]>(&r[cc * 16]));
                tmem_wait_ld();
#pragma unroll
                for (int h = 0; h < kHn; ++h) {
                    r[h] = seen ? r[h] : 0xff800000u;
                    const int mx = __reduce_max_sync(0xffffffffu, ordered(__uint_as_float(r[h])));
                    if (lane == (h & 31)) sm.warp_max[warp][h] = mx;
                }
            }
            named_barrier_sync<128>(1);
            if (threadIdx.x < kHn) {
                const int h = threadIdx.x;
                const float mx = unordered(max(sm.warp_max[0][h], sm.warp_max[1][h])) * c;
                float m = j == 0 ? fmaxf(mx, kNothingSeen) : sm.m[h], f = 1.f;
                if (mx > m + kRescaleThreshold) {
                    f = ex2(m - mx);
                    m = mx;
                    sm.need = j + 1;
                }
                sm.m[h] = m;
                sm.factor[h] = f;
            }
            named_barrier_sync<128>(1);
            const bool need = *reinterpret_cast<volatile int*>(&sm.need) == j + 1;
            // P of the tile before last has been read: its product was issued before this tile's scores
            if (warp < kTile / 32) {
                uint8_t* const p_row = p_tile + (j & 1) * kQChunk + (key & 7) * 2;
#pragma unroll
                for (int h = 0; h < kHn; ++h) {
                    const float w = ex2(fmaf(__uint_as_float(r[h]), c, -sm.m[h]));
                    l[h] = l[h] * sm.factor[h] + w;
                    *reinterpret_cast<__nv_bfloat16*>(p_row + h * 128 + (((key >> 3) ^ (h & 7)) << 4)) = __float2bfloat16_rn(w);
                }
            }
            if (need && j > 0) {  // (uniform) bring O down to the new reference maxima, once the product before has gone into it
                ok = __all_sync(0xffffffffu, mbar_wait(&sm.o_done, (j - 1) & 1));
                if (!ok) break;
                tc_fence_after();
#pragma unroll 1
                for (int g = 0; g < p.tile_pairs; ++g) {
#pragma unroll
                    for (int cc = 0; cc < kHn / 16; ++cc) {
                        uint32_t o[16];
                        __syncwarp();
                        tmem_ld16(o_base + lane_base + g * kHn + cc * 16, o);
                        tmem_wait_ld();
#pragma unroll
                        for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * sm.factor[cc * 16 + e]);
                        tmem_st16(o_base + lane_base + g * kHn + cc * 16, o);
                    }
                }
                tmem_wait_st();
            }
            fence_proxy_async_smem();  // P was written with ordinary stores and is read by the tensor core
            tc_fence_before();
            mbar_arrive(&sm.p_ready[j & 1]);
        }
        // (a parity wait cannot tell a phase from the one two before: the last scores waited for cover all products but two)
        if (n_tiles > 1 && ok) ok = __all_sync(0xffffffffu, mbar_wait(&sm.o_done, (n_tiles - 2) & 1));
        if (n_tiles > 0 && ok) ok = __all_sync(0xffffffffu, mbar_wait(&sm.o_done, (n_tiles - 1) & 1));
        if (ok) {
            tc_fence_after();
            // sums over the keys: inside the warps, then over the warps
#pragma unroll
            for (int h = 0; h < kHn; ++h) {
#pragma unroll
                for (int off = 16; off > 0; off >>= 1) l[h] += __shfl_xor_sync(0xffffffffu, l[h], off);
                if (lane == (h & 31) && warp < kTile / 32) sm.sum[warp][h] = l[h];
            }
            named_barrier_sync<128>(1);
            const int heads = min(kHn, p.H - h0);
            const int64_t stride = p.kv_rank + 2;
            float* part = p.splits > 1 ? p.partial + ((static_cast<int64_t>(i) * p.splits + split) * p.H + h0) * stride : nullptr;
            if (part != nullptr && threadIdx.x < heads) {
                const int h = threadIdx.x;
                part[h * stride + p.kv_rank] = n_tiles > 0 ? sm.m[h] : kNothingSeen;
                part[h * stride + p.kv_rank + 1] = sm.sum[0][h] + sm.sum[1][h];
            }
            if (n_tiles > 0) {
                __nv_bfloat16* out = p.out + (static_cast<int64_t>(i) * p.H + h0) * p.kv_rank;
#pragma unroll 1
                for (int g = 0; g < p.tile_pairs; ++g) {
                    const int e = g * 128 + threadIdx.x;  // element of the latent space = TMEM lane
#pragma unroll
                    for (int cc = 0; cc < kHn / 16; ++cc) {
                        uint32_t o[16];
                        __syncwarp();
                        tmem_ld16(o_base + lane_base + g * kHn + cc * 16, o);
                        tmem_wait_ld();
#pragma unroll
                        for (int u = 0; u < 16; ++u) {
                            const int h = cc * 16 + u;
                            if (h >= heads || e >= p.kv_rank) continue;
                            const float v = __uint_as_float(o[u]);
                            if (part != nullptr)
                                part[h * stride + e] = v;
                            else
                                out[static_cast<int64_t>(h) * p.kv_rank + e] =
                                    __float2bfloat16_rn(v / (sm.sum[0][h] + sm.sum[1][h]));
                        }
                    }
                }
            }
        } else {
            sm.abort_flag = 1;
        }
    }

    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        tc_fence_after();
        tmem_dealloc(tmem, p.tmem_cols);
    }
    if (threadIdx.x == 0 && sm.abort_flag) report_status(p.dev_status, B2KV_DEV_WAIT_TIMEOUT);
}

// One CTA per (head, row): the shares' partial results, each relative to its own reference maximum.
constexpr int kMaxSplits = 64;
__global__ void __launch_bounds__(128) latent_merge_kernel(const float* partial, __nv_bfloat16* out, int H, int kv_rank, int splits) {
    __shared__ float w[kMaxSplits];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int h = blockIdx.x, i = blockIdx.y;
    const int64_t stride = kv_rank + 2;
    const float* part = partial + (static_cast<int64_t>(i) * splits * H + h) * stride;
    if (threadIdx.x < 32) {
        float mx = kNothingSeen;
        for (int s = threadIdx.x; s < splits; s += 32) mx = fmaxf(mx, part[s * H * stride + kv_rank]);
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        float sum = 0.f;
        for (int s = threadIdx.x; s < splits; s += 32) {
            const float f = ex2(part[s * H * stride + kv_rank] - mx);
            w[s] = f;
            sum += f * part[s * H * stride + kv_rank + 1];
        }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
        for (int s = threadIdx.x; s < splits; s += 32)
            w[s] = part[s * H * stride + kv_rank + 1] > 0.f ? w[s] / sum : -1.f;  // a share without keys wrote no elements
    }
    __syncthreads();
    for (int e = threadIdx.x; e < kv_rank; e += 128) {
        float v = 0.f;
        for (int s = 0; s < splits; ++s)
            if (w[s] >= 0.f) v = fmaf(w[s], part[s * H * stride + e], v);
        out[(static_cast<int64_t>(i) * H + h) * kv_rank + e] = __float2bfloat16_rn(v);
    }
}

// (element, head or 1, row) view with 64-element boxes of box_heads x box_rows, 128-byte swizzle.
static bool make_map(CUtensorMap* map, const void* base, int width, int heads, int64_t rows, int64_t head_stride, int64_t pitch,
                     int box_heads, int box_rows) {
    EncodeTiledFn fn = tensor_map_encoder();
    if (fn == nullptr) return false;
    const cuuint64_t dims[3] = {static_cast<cuuint64_t>(width), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(rows)};
    const cuuint64_t strides[2] = {static_cast<cuuint64_t>(head_stride) * 2, static_cast<cuuint64_t>(pitch) * 2};
    const cuuint32_t box[3] = {64, static_cast<cuuint32_t>(box_heads), static_cast<cuuint32_t>(box_rows)};
    const cuuint32_t estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

static int head_columns(int H) { return H <= 16 ? 16 : (H <= 32 ? 32 : 64); }

// Shares per row: about one CTA per SM, each with at least four tiles where the window has them.
static int choose_splits(int rows, int H, int span) {
    const int groups = (H + kMaxHeads - 1) / kMaxHeads;
    const int tiles = (span + kTile - 1) / kTile;
    const int fill = std::max(1, device_sm_count() / std::max(1, rows * groups));
    return std::max(1, std::min(std::min(fill, kMaxSplits), (tiles + 3) / 4));
}

template <int kHn>
static int launch(const CUtensorMap (&m)[4], const Params& p, unsigned grid, size_t smem, void* stream) {
    static int configured[64] = {0};
    int dev = 0;
    B2KV_CUDA_TRY(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64) return B2KV_ERR_UNSUPPORTED;
    if (configured[dev] < static_cast<int>(smem)) {
        B2KV_CUDA_TRY(cudaFuncSetAttribute(latent_decode_tc_kernel<kHn>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        configured[dev] = static_cast<int>(smem);
    }
    OverlapLaunch cfg(grid, kThreads, smem, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&cfg.cfg, latent_decode_tc_kernel<kHn>, m[0], m[1], m[2], m[3], p));
    return B2KV_OK;
}

}  // namespace latdec

size_t latent_decode_tc_workspace(int rows, int H, int kv_rank, int span) {
    const int splits = latdec::choose_splits(rows, H, span);
    return splits > 1 ? static_cast<size_t>(rows) * splits * H * (kv_rank + 2) * sizeof(float) : 0;
}

int latent_decode_tc(const LatentDecodeArgs& a, void* workspace, size_t workspace_bytes, void* stream) {
    using namespace latdec;
    if (a.kv_rank % 8 != 0 || a.kv_rank > 512 || a.rot % 8 != 0 || a.rot > 64 || a.dim % 8 != 0 || a.ld_q % 8 != 0 || !(a.scale > 0.f))
        return B2KV_ERR_UNSUPPORTED;
    if (!aligned16(a.q_latent) || !aligned16(a.q) || !aligned16(a.key_cache) || !aligned16(a.latent_cache)) return B2KV_ERR_UNSUPPORTED;
    if (static_cast<int64_t>(a.n_slots) * a.T_max > 0x7fffffffLL - 256) return B2KV_ERR_UNSUPPORTED;
    const int tile_pairs = (a.kv_rank + 127) / 128;
    auto fixed_bytes = [&](int hn) {
        return 2 * kChunkBytes + (2 * tile_pairs + 1) * hn * 128 + 2 * hn * 128 + 1024 + static_cast<int>(sizeof(Shared));
    };
    int Hn = head_columns(a.H);
    // 64 heads beside a wide latent do not fit one SM: two groups of 32 then read the same rows, the second out of L2
    while (Hn > 16 && (kSmemLimit - fixed_bytes(Hn)) / kPairBytes < 2 * tile_pairs) Hn /= 2;
    Params p{};
    p.row_slot = a.row_slot;
    p.row_pos = a.row_pos;
    p.out = static_cast<__nv_bfloat16*>(a.out);
    p.partial = static_cast<float*>(workspace);
    p.dev_status = a.dev_status;
    p.n_slots = a.n_slots;
    p.T_max = a.T_max;
    p.H = a.H;
    p.kv_rank = a.kv_rank;
    p.window = a.window;
    p.prescale = a.scale * 1.4426950408889634f;
    p.head_groups = (a.H + Hn - 1) / Hn;
    p.splits = choose_splits(a.rows, a.H, a.span);
    if (p.splits > 1 && (workspace == nullptr || workspace_bytes < latent_decode_tc_workspace(a.rows, a.H, a.kv_rank, a.span)))
        return B2KV_ERR_WORKSPACE;
    p.tile_pairs = tile_pairs;
    p.tmem_cols = 32;
    while (p.tmem_cols < (p.tile_pairs + 2) * Hn) p.tmem_cols *= 2;
    const int fixed = fixed_bytes(Hn);
    p.ring_pairs = std::min(std::min(kMaxPairs, 3 * p.tile_pairs), (kSmemLimit - fixed) / kPairBytes);
    if (p.ring_pairs < 2 * p.tile_pairs) return B2KV_ERR_UNSUPPORTED;
    const size_t smem = static_cast<size_t>(p.ring_pairs) * kPairBytes + fixed - sizeof(Shared);
    const int64_t cache_rows = static_cast<int64_t>(a.n_slots) * a.T_max;
    CUtensorMap m[4];
    if (!make_map(&m[0], a.q_latent, a.kv_rank, a.H, a.rows, a.kv_rank, static_cast<int64_t>(a.H) * a.kv_rank, Hn, 1) ||
        !make_map(&m[1], static_cast<const __nv_bfloat16*>(a.q) + a.dim, a.rot, a.H, a.rows, a.dim + a.rot, a.ld_q, Hn, 1) ||
        !make_map(&m[2], a.latent_cache, a.kv_rank, 1, cache_rows, a.kv_rank, a.kv_rank, 1, kTile) ||
        !make_map(&m[3], a.key_cache, a.rot, 1, cache_rows, a.rot, a.rot, 1, kTile))
        return B2KV_ERR_UNSUPPORTED;
    const long long grid = static_cast<long long>(a.rows) * p.head_groups * p.splits;
    if (grid > 0x7fffffffLL) return B2KV_ERR_UNSUPPORTED;
    const int rc = Hn == 16 ? launch<16>(m, p, static_cast<unsigned>(grid), smem, stream)
                            : (Hn == 32 ? launch<32>(m, p, static_cast<unsigned>(grid), smem, stream)
                                        : launch<64>(m, p, static_cast<unsigned>(grid), smem, stream));
    if (rc != B2KV_OK || p.splits == 1) return rc;
    OverlapLaunch cfg(dim3(a.H, a.rows), 128, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&cfg.cfg, latent_merge_kernel, static_cast<const float*>(p.partial), p.out, a.H, a.kv_rank, p.splits));
    return B2KV_OK;
}

}  // namespace b2kv
