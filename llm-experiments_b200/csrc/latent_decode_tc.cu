// Attention of single query rows over cached latent rows on the Blackwell tensor cores (bf16).
//
// All heads of a row read the same latent rows, so the cache is streamed once per row (and group of heads) and the work is
// matrix-shaped: H heads against every key.  Both products are computed transposed, so that the 128 rows of an MMA are the
// plentiful dimension and its columns the few heads (as in the weight-streaming kernels):
//
//   S^T[key, head]     = latent[key, :] q_latent[head, :] + key part[key, :] q_rot[head, :]      A K-major
//   O^T[element, head] += latent[:, element]^T P[key, head]                                       the same tile, A MN-major
//
//   * one CTA per (row, group of up to 32 heads, share of the row's window).  A tile is 64 keys: pairs of 64-element chunks of
//     the latent rows and one chunk of the rotated key part, copied with TMA (128-byte swizzle) into a ring of whole tiles (two
//     at 512 + 64 elements).  An MMA has 128 rows all the same: the upper 64 rows of S^T are made from whatever lies behind a
//     chunk in shared memory, and nobody looks at them;
//   * even and odd tiles are two streams of their own, each with four softmax warps, a score buffer, reference maxima and an
//     output accumulator in tensor memory, so that one tile's softmax runs under the other's copies and products; the two
//     results are put together at the end.  Warp 8 copies; one thread of warp 9 issues whatever can go next: a product whose P
//     is ready, or the scores of a tile that has arrived;
//   * softmax: thread = key = TMEM lane, one column per head (the upper two warps of a stream only help rescaling).  Weights are
//     taken against the reference maxima in force, which move only when a score has outgrown its reference by more than 2^8:
//     one vote per tile, column maxima and rescaling only then.  Sums stay in registers per key until the end; P goes to shared
//     memory as the K-major operand of the second product;
//   * the shares of one row (few rows, long windows) leave fp32 partial results that a small kernel merges.
//
// No MMA is predicated; sizes that do not fill a chunk read as zero.  Every wait is bounded; a warp whose wait ran out still
// meets its partners at their barrier, tells them there, and all leave together.
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
constexpr int kMaxStages = 8;
constexpr int kMaxHeads = 32;
constexpr int kStream = 128;  // threads of one stream's softmax warps
constexpr int kThreads = 2 * kStream + 64;
constexpr int kSmemLimit = 226 * 1024;
constexpr float kRescaleThreshold = 8.0f;
constexpr float kNothingSeen = -1e30f;

struct Shared {
    alignas(8) uint64_t q_full;
    uint64_t full[kMaxStages], empty[kMaxStages];
    uint64_t s_full[2], p_ready[2], o_done;
    uint32_t tmem_base;
    volatile int abort_flag;
    volatile int fail[2];
    int warp_max[2][2][kMaxHeads];  // [stream][warp][head]
    float m[2][kMaxHeads], factor[2][kMaxHeads], delta[2][kMaxHeads], sum[2][2][kMaxHeads];
};

struct Params {
    const int32_t* row_slot;
    const int32_t* row_pos;
    __nv_bfloat16* out;  // [rows, H, kv_rank]
    float* partial;      // [rows, splits, H, kv_rank + 2] when splits > 1
    int32_t* dev_status;
    int n_slots, T_max, H, kv_rank, window, splits, head_groups;
    int tile_pairs;  // pairs per tile: ceil(kv_rank / 128)
    int stages;      // tiles of the ring
    int tmem_cols;
    float prescale;  // scale * log2(e)
};

// Barrier `id` of kN threads that tells every one of them whether any came with v.
template <int kN>
__device__ __forceinline__ bool barrier_any(int id, bool v) {
    uint32_t any;
    asm volatile(
        "{\n"
        ".reg .pred p, q;\n"
        "setp.ne.u32 p, %3, 0;\n"
        "barrier.cta.red.or.pred q, %1, %2, p;\n"
        "selp.u32 %0, 1, 0, q;\n"
        "}\n"
        : "=r"(any)
        : "r"(id), "n"(kN), "r"(static_cast<uint32_t>(v))
        : "memory");
    return any != 0;
}

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
    const int stage_bytes = p.tile_pairs * kPairBytes + kChunkBytes;  // the latent pairs, then the rotated chunk
    uint8_t* const q_tile = ring + p.stages * stage_bytes;            // 2 * tile_pairs latent chunks, then the rotated one; kHn rows each
    constexpr int kQChunk = kHn * 128;
    uint8_t* const p_tile = q_tile + (2 * p.tile_pairs + 1) * kQChunk;  // per stream [kHn][64 keys]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int split = blockIdx.x % p.splits;
    const int h0 = blockIdx.x / p.splits % p.head_groups * kHn;
    const int i = blockIdx.x / (p.splits * p.head_groups);

    grid_launch_dependents();
    if (threadIdx.x == 0) {
        mbar_init(&sm.q_full, 1);
        for (int s = 0; s < kMaxStages; ++s) {
            mbar_init(&sm.full[s], 1);
            mbar_init(&sm.empty[s], 1);
        }
        for (int s = 0; s < 2; ++s) {
            mbar_init(&sm.s_full[s], 1);
            mbar_init(&sm.p_ready[s], kStream / 32);  // one arrival per warp
            sm.fail[s] = 0;
        }
        mbar_init(&sm.o_done, 1);
        sm.abort_flag = 0;
        fence_mbar_init();
        grid_dependency_wait();  // queries, cache rows and positions come from the kernels before this one
    }
    if (warp == 9) {
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
    const uint32_t o_base = tmem + 2 * kHn;  // the streams' scores in columns [0, 2 kHn), then O of stream 0, O of stream 1

    if (warp == 8) {
        // ------------------------------ TMA producer ------------------------------
        if (lane == 0 && n_tiles > 0) {
            bool ok = true;
            mbar_arrive_expect_tx(&sm.q_full, (2 * p.tile_pairs + 1) * kQChunk);
            for (int c = 0; c < 2 * p.tile_pairs; ++c) tma_load_3d(q_tile + c * kQChunk, &tm_ql, &sm.q_full, c * 64, h0, i);
            tma_load_3d(q_tile + 2 * p.tile_pairs * kQChunk, &tm_qr, &sm.q_full, 0, h0, i);
            int st = 0;
            uint32_t phase = 1;  // parity of the "empty" phase to wait for: the ring starts empty
            for (int j = 0; j < n_tiles; ++j) {
                const int row = slot * p.T_max + t0 + (first + j) * kTile;
                ok = mbar_wait(&sm.empty[st], phase);
                if (!ok) break;
                mbar_arrive_expect_tx(&sm.full[st], stage_bytes);
                uint8_t* dst = ring + st * stage_bytes;
                for (int c = 0; c < 2 * p.tile_pairs; ++c)
                    tma_load_3d(dst + c * kChunkBytes, &tm_lat, &sm.full[st], c * 64, 0, row);
                tma_load_3d(dst + 2 * p.tile_pairs * kChunkBytes, &tm_key, &sm.full[st], 0, 0, row);
                if (++st == p.stages) st = 0, phase ^= 1;
            }
            if (!ok) sm.abort_flag = 1;
        }
        __syncwarp();
    } else if (warp == 9) {
        // ------------------------------ MMA issuer ------------------------------
        if (lane == 0 && n_tiles > 0) {
            constexpr uint32_t idesc_s = instr_desc(0, 0, kHn), idesc_o = instr_desc(1, 0, kHn);
            const uint64_t d_lat_k = smem_desc(smem_u32(ring), 16, 1024);            // latent rows, K-major (keys are M)
            const uint64_t d_lat_mn = smem_desc(smem_u32(ring), kChunkBytes, 1024);  // the same bytes, MN-major (elements are M)
            const uint64_t d_q = smem_desc(smem_u32(q_tile), 16, 1024), d_p = smem_desc(smem_u32(p_tile), 16, 1024);
            constexpr uint32_t kPair16 = kPairBytes >> 4, kChunk16 = kChunkBytes >> 4, kQ16 = kQChunk >> 4;
            const uint32_t stage16 = static_cast<uint32_t>(stage_bytes) >> 4, rot16 = static_cast<uint32_t>(2 * p.tile_pairs) * kChunk16;
            const uint64_t d_qr = d_q + static_cast<uint64_t>(2 * p.tile_pairs) * kQ16;
            auto issue_s = [&](int j, int st) {
                const uint32_t s_tmem = tmem + (j & 1) * kHn;
                const uint64_t a = d_lat_k + static_cast<uint64_t>(st * stage16), ar = a + static_cast<uint64_t>(rot16);
#pragma unroll
                for (int kk = 0; kk < 4; ++kk)
                    mma_ss(s_tmem, ar + static_cast<uint64_t>(2 * kk), d_qr + static_cast<uint64_t>(2 * kk), idesc_s, kk ? 1u : 0u);
                for (int g = 0; g < p.tile_pairs; ++g) {
                    const uint64_t ag = a + static_cast<uint64_t>(g * kPair16), bg = d_q + static_cast<uint64_t>(2 * g * kQ16);
#pragma unroll
                    for (int kk = 0; kk < 8; ++kk)
                        mma_ss(s_tmem, ag + static_cast<uint64_t>((kk >> 2) * kChunk16 + (kk & 3) * 2),
                               bg + static_cast<uint64_t>((kk >> 2) * kQ16 + (kk & 3) * 2), idesc_s, 1u);
                }
                mma_commit(&sm.s_full[j & 1]);
            };
            auto issue_o = [&](int j, int st) {
                const uint64_t a = d_lat_mn + static_cast<uint64_t>(st * stage16), b = d_p + static_cast<uint64_t>((j & 1) * kQ16);
                const uint32_t o = o_base + (j & 1) * p.tile_pairs * kHn;
                const uint32_t more = j > 1 ? 1u : 0u;  // the stream's first tile starts its accumulator
                for (int g = 0; g < p.tile_pairs; ++g) {
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk)  // 16 keys: 2048 bytes of the tile, 32 bytes of P
                        mma_ss(o + g * kHn, a + static_cast<uint64_t>(g * kPair16 + ((kk * 2048) >> 4)),
                               b + static_cast<uint64_t>(2 * kk), idesc_o, kk ? 1u : more);
                }
                mma_commit(&sm.empty[st]);
            };
            bool ok = mbar_wait(&sm.q_full, 0);
            int js = 0, jo = 0, st_s = 0, st_o = 0;  // next tile to score, next product; their ring places
            uint32_t ph_s = 0;
            uint32_t idle = 0;
            unsigned long long since = 0;
            while (ok && jo < n_tiles) {
                if (jo < js && mbar_test(&sm.p_ready[jo & 1], (jo >> 1) & 1)) {
                    tc_fence_after();
                    issue_o(jo, st_o);
                    if (++st_o == p.stages) st_o = 0;
                    ++jo;
                    idle = 0;
                } else if (js < n_tiles && js < jo + 2 && mbar_test(&sm.full[st_s], ph_s)) {
                    // (P(js - 2) has been waited for, so that stream's scores have been read)
                    tc_fence_after();
                    issue_s(js, st_s);
                    if (++st_s == p.stages) st_s = 0, ph_s ^= 1;
                    ++js;
                    idle = 0;
                } else if ((++idle & 1023u) == 0) {
                    if (idle == 1024u) since = globaltimer_ns();
                    else ok = globaltimer_ns() - since < kWaitLimitNs;
                }
            }
            if (ok) mma_commit(&sm.o_done);
            else sm.abort_flag = 1;
        }
        __syncwarp();
    } else {
        // ------------------------------ softmax: thread = key of the tile ------------------------------
        const int x_id = warp >> 2, w_id = warp & 3;  // stream, warp of the stream
        const int key = threadIdx.x & (kStream - 1);
        const uint32_t lane_base = static_cast<uint32_t>(w_id * 32) << 16;
        const bool scores = w_id < kTile / 32;
        const float c = p.prescale;
        const int n_x = (n_tiles + 1 - x_id) / 2;  // tiles of this stream
        float* const m = sm.m[x_id];
        float l[kHn];
#pragma unroll
        for (int h = 0; h < kHn; ++h) l[h] = 0.f;
        if (key < kHn) m[key] = 0.f;
        named_barrier_sync<kStream>(1 + x_id);
        bool ok = true;
        for (int k = 0; k < n_x; ++k) {
            const bool arrived = __all_sync(0xffffffffu, mbar_wait(&sm.s_full[x_id], k & 1));
            if (!arrived && lane == 0) sm.fail[x_id] = 1;
            tc_fence_after();
            float x[kHn];
            float mx = -INFINITY;
            if (scores) {
                const bool seen = t0 + (first + 2 * k + x_id) * kTile + key <= pos;
                uint32_t r[kHn];
#pragma unroll
                for (int cc = 0; cc < kHn / 16; ++cc)
                    tmem_ld16(tmem + lane_base + x_id * kHn + cc * 16, *reinterpret_cast<uint32_t(*)[16]>(&r[cc * 16]));
                tmem_wait_ld();
#pragma unroll
                for (int h = 0; h < kHn; ++h) {
                    x[h] = seen ? fmaf(__uint_as_float(r[h]), c, -m[h]) : -INFINITY;
                    mx = fmaxf(mx, x[h]);
                }
            }
            // the first tile has no reference yet
            const bool need = barrier_any<kStream>(1 + x_id, k == 0 || mx > kRescaleThreshold);
            if (sm.fail[x_id]) {  // set before the barrier, so all of the stream see it
                ok = false;
                break;
            }
            if (need) {
                if (scores) {
#pragma unroll
                    for (int h = 0; h < kHn; ++h) {
                        const int hm = __reduce_max_sync(0xffffffffu, ordered(x[h]));
                        if (lane == h) sm.warp_max[x_id][w_id][h] = hm;
                    }
                }
                named_barrier_sync<kStream>(1 + x_id);
                if (key < kHn) {
                    const float grown = unordered(max(sm.warp_max[x_id][0][key], sm.warp_max[x_id][1][key]));
                    const bool moves = k == 0 || grown > kRescaleThreshold;
                    sm.factor[x_id][key] = moves && k > 0 ? ex2(-grown) : 1.f;
                    sm.delta[x_id][key] = moves ? grown : 0.f;
                    if (moves) m[key] += grown;
                }
                named_barrier_sync<kStream>(1 + x_id);
                if (scores) {
#pragma unroll
                    for (int h = 0; h < kHn; ++h) {
                        x[h] -= sm.delta[x_id][h];
                        l[h] *= sm.factor[x_id][h];
                    }
                }
                if (k > 0) {
                    // the stream's products so far are complete: they were issued ahead of this tile's scores
                    const uint32_t o_mine = o_base + lane_base + x_id * p.tile_pairs * kHn;
#pragma unroll 1
                    for (int g = 0; g < p.tile_pairs; ++g) {
#pragma unroll
                        for (int cc = 0; cc < kHn / 16; ++cc) {
                            uint32_t o[16];
                            __syncwarp();
                            tmem_ld16(o_mine + g * kHn + cc * 16, o);
                            tmem_wait_ld();
#pragma unroll
                            for (int e = 0; e < 16; ++e)
                                o[e] = __float_as_uint(__uint_as_float(o[e]) * sm.factor[x_id][cc * 16 + e]);
                            tmem_st16(o_mine + g * kHn + cc * 16, o);
                        }
                    }
                    tmem_wait_st();
                }
            }
            if (scores) {
                uint8_t* const p_row = p_tile + x_id * kQChunk + (key & 7) * 2;
#pragma unroll
                for (int h = 0; h < kHn; ++h) {
                    const float w = ex2(x[h]);
                    l[h] += w;
                    *reinterpret_cast<__nv_bfloat16*>(p_row + h * 128 + (((key >> 3) ^ (h & 7)) << 4)) = __float2bfloat16_rn(w);
                }
            }
            fence_proxy_async_smem();  // P was written with ordinary stores and is read by the tensor core
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sm.p_ready[x_id]);
        }
        if (ok && n_tiles > 0) ok = __all_sync(0xffffffffu, mbar_wait(&sm.o_done, 0));
        if (!ok && lane == 0) sm.fail[x_id] = 1;
        tc_fence_after();
        // sums over the keys: inside the warps, then over the warps and the streams
#pragma unroll
        for (int h = 0; h < kHn; ++h) {
#pragma unroll
            for (int off = 16; off > 0; off >>= 1) l[h] += __shfl_xor_sync(0xffffffffu, l[h], off);
            if (lane == h && scores) sm.sum[x_id][w_id][h] = l[h];
        }
        named_barrier_sync<2 * kStream>(3);
        if (sm.fail[0] == 0 && sm.fail[1] == 0) {
            const bool both = n_tiles > 1;  // otherwise the second stream has no accumulator
            if (x_id == 0 && key < kHn) {   // weights of the streams, against the larger of their references
                const float m0 = sm.m[0][key], m1 = both ? sm.m[1][key] : m0, top = fmaxf(m0, m1);
                sm.factor[0][key] = ex2(m0 - top);
                sm.factor[1][key] = both ? ex2(m1 - top) : 0.f;
                sm.delta[0][key] = n_tiles > 0 ? top : kNothingSeen;
                sm.delta[1][key] = sm.factor[0][key] * (sm.sum[0][0][key] + sm.sum[0][1][key]) +
                                   (both ? sm.factor[1][key] * (sm.sum[1][0][key] + sm.sum[1][1][key]) : 0.f);
            }
            named_barrier_sync<2 * kStream>(3);
            const int heads = min(kHn, p.H - h0);
            const int64_t stride = p.kv_rank + 2;
            float* part = p.splits > 1 ? p.partial + ((static_cast<int64_t>(i) * p.splits + split) * p.H + h0) * stride : nullptr;
            if (part != nullptr && x_id == 0 && key < heads) {
                part[key * stride + p.kv_rank] = sm.delta[0][key];
                part[key * stride + p.kv_rank + 1] = sm.delta[1][key];
            }
            if (n_tiles > 0) {
                __nv_bfloat16* out = p.out + (static_cast<int64_t>(i) * p.H + h0) * p.kv_rank;
                const uint32_t o_0 = o_base + lane_base, o_1 = o_0 + p.tile_pairs * kHn;
#pragma unroll 1
                for (int g = x_id; g < p.tile_pairs; g += 2) {
                    const int e = g * 128 + key;  // element of the latent space = TMEM lane
#pragma unroll 1
                    for (int cc = 0; cc < kHn / 16; ++cc) {
                        uint32_t o[16], o2[16];
                        __syncwarp();
                        tmem_ld16(o_0 + g * kHn + cc * 16, o);
                        tmem_ld16(o_1 + g * kHn + cc * 16, o2);  // (read in any case, used only if there is a second stream)
                        tmem_wait_ld();
#pragma unroll
                        for (int u = 0; u < 16; ++u) {
                            const int h = cc * 16 + u;
                            if (h >= heads || e >= p.kv_rank) continue;
                            float v = __uint_as_float(o[u]) * sm.factor[0][h];
                            if (both) v = fmaf(__uint_as_float(o2[u]), sm.factor[1][h], v);
                            if (part != nullptr)
                                part[h * stride + e] = v;
                            else
                                out[static_cast<int64_t>(h) * p.kv_rank + e] = __float2bfloat16_rn(v / sm.delta[1][h]);
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
    if (warp == 9) {
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

static int head_columns(int H) { return H <= 16 ? 16 : 32; }

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
    const int Hn = head_columns(a.H);  // further heads are further CTAs, which find the rows in L2
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
    while (p.tmem_cols < (2 * p.tile_pairs + 2) * Hn) p.tmem_cols *= 2;
    const int fixed = (2 * p.tile_pairs + 1) * Hn * 128 + 2 * Hn * 128 + 1024;
    const int stage_bytes = p.tile_pairs * kPairBytes + kChunkBytes;
    p.stages = std::min(kMaxStages, (kSmemLimit - fixed - static_cast<int>(sizeof(Shared))) / stage_bytes);
    if (p.stages < 2) return B2KV_ERR_UNSUPPORTED;
    const size_t smem = static_cast<size_t>(p.stages) * stage_bytes + fixed;
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
                            : launch<32>(m, p, static_cast<unsigned>(grid), smem, stream);
    if (rc != B2KV_OK || p.splits == 1) return rc;
    OverlapLaunch cfg(dim3(a.H, a.rows), 128, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&cfg.cfg, latent_merge_kernel, static_cast<const float*>(p.partial), p.out, a.H, a.kv_rank, p.splits));
    return B2KV_OK;
}

}  // namespace b2kv
