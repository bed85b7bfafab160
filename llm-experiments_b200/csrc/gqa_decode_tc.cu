// Grouped-query attention of single query rows over cached keys and values on the Blackwell tensor cores (bf16).
//
// The query heads of one key / value head read the same rows, so the cache is streamed once per group and the work is
// matrix-shaped.  Both products are computed transposed, so that the 128 rows of an MMA are the plentiful dimension and its
// columns the few heads (the scheme of latent_decode_tc.cu, with keys and values of their own):
//
//   S^T[key, head]      = K[key, :] q[head, :]              A K-major
//   O^T[element, head] += V[:, element]^T P[key, head]      A MN-major
//
//   * one CTA per (row, key / value head, group of up to 32 query heads, share of the row's tokens).  A tile is 128 keys: one or
//     two 64-element chunks of V, then of K, copied with TMA (128-byte swizzle) into a ring of whole tiles (three at
//     128 + 128 elements).  The second product always has 128 rows: for values of a single chunk the upper 64 are made from
//     the K chunk behind it, and nobody looks at them;
//   * even and odd tiles are two streams of their own, each with four softmax warps, a score buffer, reference maxima and an
//     output accumulator in tensor memory, so that one tile's softmax runs under the other's copies and products; the two
//     results are put together at the end.  Warp 8 copies; one thread of warp 9 issues whatever can go next;
//   * softmax: thread = key = TMEM lane, one column per head.  The distance bias is taken off in fp32 before anything else.
//     Weights are taken against the reference maxima in force, which move only when a score has outgrown its reference by more
//     than 2^8: one vote per tile, column maxima and rescaling only then.  Sums stay in registers per key until the end; P
//     goes to shared memory as the K-major operand of the second product;
//   * shares have a fixed number of tiles, so that rows of unequal length load the SMs evenly; a row of a single share writes
//     its output, the shares of longer ones leave fp32 partial results that a small kernel merges.
//
// No MMA is predicated; sizes that do not fill a chunk read as zero.  Every wait is bounded; a warp whose wait ran out still
// meets its partners at their barrier, tells them there, and all leave together.
#include <math.h>

#include <algorithm>

#include "gqa.cuh"
#include "tc_ptx.cuh"
#include "tma_map.cuh"

namespace b2kv {
namespace gqadec {

using namespace tc;

constexpr int kTile = 128;                // keys per tile
constexpr int kChunkBytes = kTile * 128;  // 128 rows x 64 bf16
constexpr int kMaxStages = 6;
constexpr int kMaxHeads = 32;
constexpr int kStream = 128;  // threads of one stream's softmax warps
constexpr int kWarps = kStream / 32;
constexpr int kThreads = 2 * kStream + 64;
constexpr int kSmemLimit = 226 * 1024;
constexpr float kRescaleThreshold = 8.0f;
constexpr float kNothingSeen = -1e30f;
constexpr float kLog2e = 1.4426950408889634f;

struct Shared {
    alignas(8) uint64_t q_full;
    uint64_t full[kMaxStages], empty[kMaxStages];
    uint64_t s_full[2], p_ready[2], o_done;
    uint32_t tmem_base;
    volatile int abort_flag;
    volatile int fail[2];
    int warp_max[2][kWarps][kMaxHeads];  // [stream][warp][head]
    float m[2][kMaxHeads], factor[2][kMaxHeads], delta[2][kMaxHeads], sum[2][kWarps][kMaxHeads], slope[kMaxHeads];
};

struct Params {
    const int32_t* row_slot;
    const int32_t* row_pos;
    const float* slopes;
    __nv_bfloat16* out;
    float* partial;  // [rows, splits, H, vdim + 2] when splits > 1
    int32_t* dev_status;
    int64_t ld_out;
    int n_slots, T_max, H, G, vdim, splits, share, head_groups;
    int v_chunks;  // 64-element chunks per value
    int stages;    // tiles of the ring
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

template <int kHn, int kKc>
__global__ void __launch_bounds__(kThreads)
gqa_decode_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                     const __grid_constant__ CUtensorMap tm_v, const Params p) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ Shared sm;
    constexpr int kTmemCols = 4 * kHn;  // scores and accumulators of the two streams
    constexpr int kQChunk = kHn * 128;
    uint8_t* const ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int v_bytes = p.v_chunks * kChunkBytes, stage_bytes = v_bytes + kKc * kChunkBytes;
    uint8_t* const q_tile = ring + p.stages * stage_bytes;  // kKc chunks of kHn rows
    uint8_t* const p_tile = q_tile + kKc * kQChunk;         // per stream two chunks: [kHn][64 keys]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int per_kv = p.H / p.G;
    int rest = blockIdx.x;
    const int g0 = rest % p.G;  // key / value head: neighbours read neighbouring columns of the same rows
    rest /= p.G;
    const int hg = rest % p.head_groups * kHn;  // first query head inside the group
    rest /= p.head_groups;
    const int split = rest % p.splits, i = rest / p.splits;
    const int h0 = g0 * per_kv + hg, heads = min(kHn, per_kv - hg);

    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();  // queries, cache rows and positions come from the kernels before this one
    __syncthreads();
    // this CTA's tiles: [first, first + n_tiles)
    int slot, pos;
    if (!row_place(p.row_slot, p.row_pos, i, p.n_slots, p.T_max, slot, pos)) {
        if (threadIdx.x == 0) report_status(p.dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const int all_tiles = pos / kTile + 1;
    const int first = split * p.share;
    const int n_tiles = min(p.splits > 1 ? p.share : all_tiles, all_tiles - first);
    if (n_tiles <= 0) return;  // a share behind the row's end

    if (threadIdx.x == 0) {
        mbar_init(&sm.q_full, 1);
        for (int s = 0; s < kMaxStages; ++s) {
            mbar_init(&sm.full[s], 1);
            mbar_init(&sm.empty[s], 1);
        }
        for (int s = 0; s < 2; ++s) {
            mbar_init(&sm.s_full[s], 1);
            mbar_init(&sm.p_ready[s], kWarps);  // one arrival per warp
            sm.fail[s] = 0;
        }
        mbar_init(&sm.o_done, 1);
        sm.abort_flag = 0;
        fence_mbar_init();
    }
    if (threadIdx.x < kHn) sm.slope[threadIdx.x] = p.slopes != nullptr && static_cast<int>(threadIdx.x) < heads ? p.slopes[h0 + threadIdx.x] * kLog2e : 0.f;
    if (warp == 9) {
        tmem_alloc(&sm.tmem_base, kTmemCols);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sm.tmem_base;
    const uint32_t o_base = tmem + 2 * kHn;  // the streams' scores in columns [0, 2 kHn), then O of stream 0, O of stream 1

    if (warp == 8) {
        // ------------------------------ TMA producer ------------------------------
        if (lane == 0) {
            bool ok = true;
            mbar_arrive_expect_tx(&sm.q_full, kKc * kQChunk);
#pragma unroll
            for (int c = 0; c < kKc; ++c) tma_load_3d(q_tile + c * kQChunk, &tm_q, &sm.q_full, c * 64, h0, i);
            int st = 0;
            uint32_t phase = 1;  // parity of the "empty" phase to wait for: the ring starts empty
            for (int j = 0; j < n_tiles; ++j) {
                const int row = slot * p.T_max + (first + j) * kTile;
                ok = mbar_wait(&sm.empty[st], phase);
                if (!ok) break;
                mbar_arrive_expect_tx(&sm.full[st], stage_bytes);
                uint8_t* dst = ring + st * stage_bytes;
#pragma unroll
                for (int c = 0; c < kKc; ++c) tma_load_3d(dst + v_bytes + c * kChunkBytes, &tm_k, &sm.full[st], c * 64, g0, row);
                for (int c = 0; c < p.v_chunks; ++c) tma_load_3d(dst + c * kChunkBytes, &tm_v, &sm.full[st], c * 64, g0, row);
                if (++st == p.stages) st = 0, phase ^= 1;
            }
            if (!ok) sm.abort_flag = 1;
        }
        __syncwarp();
    } else if (warp == 9) {
        // ------------------------------ MMA issuer ------------------------------
        if (lane == 0) {
            constexpr uint32_t idesc_s = instr_desc(0, 0, kHn), idesc_o = instr_desc(1, 0, kHn);
            const uint64_t d_k = smem_desc(smem_u32(ring) + v_bytes, 16, 1024);    // keys are M, K-major
            const uint64_t d_v = smem_desc(smem_u32(ring), kChunkBytes, 1024);     // elements are M, MN-major
            const uint64_t d_q = smem_desc(smem_u32(q_tile), 16, 1024), d_p = smem_desc(smem_u32(p_tile), 16, 1024);
            constexpr uint32_t kChunk16 = kChunkBytes >> 4, kQ16 = kQChunk >> 4;
            const uint32_t stage16 = static_cast<uint32_t>(stage_bytes) >> 4;
            auto issue_s = [&](int j, int st) {
                const uint64_t a = d_k + static_cast<uint64_t>(st * stage16);
#pragma unroll
                for (int kk = 0; kk < 4 * kKc; ++kk)
                    mma_ss(tmem + (j & 1) * kHn, a + static_cast<uint64_t>((kk >> 2) * kChunk16 + (kk & 3) * 2),
                           d_q + static_cast<uint64_t>((kk >> 2) * kQ16 + (kk & 3) * 2), idesc_s, kk ? 1u : 0u);
                mma_commit(&sm.s_full[j & 1]);
            };
            auto issue_o = [&](int j, int st) {
                const uint64_t a = d_v + static_cast<uint64_t>(st * stage16), b = d_p + static_cast<uint64_t>((j & 1) * 2 * kQ16);
                const uint32_t more = j > 1 ? 1u : 0u;  // the stream's first tile starts its accumulator
#pragma unroll
                for (int kk = 0; kk < 8; ++kk)  // 16 keys: 2048 bytes of the tile, 32 bytes of P
                    mma_ss(o_base + (j & 1) * kHn, a + static_cast<uint64_t>((kk * 2048) >> 4),
                           b + static_cast<uint64_t>((kk >> 2) * kQ16 + (kk & 3) * 2), idesc_o, kk ? 1u : more);
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
            const int behind = pos - ((first + 2 * k + x_id) * kTile + key);
            const float dist = static_cast<float>(behind);
            {
                uint32_t r[kHn];
#pragma unroll
                for (int cc = 0; cc < kHn / 16; ++cc)
                    tmem_ld16(tmem + lane_base + x_id * kHn + cc * 16, *reinterpret_cast<uint32_t(*)[16]>(&r[cc * 16]));
                tmem_wait_ld();
#pragma unroll
                for (int h = 0; h < kHn; ++h) {
                    x[h] = behind >= 0 ? fmaf(__uint_as_float(r[h]), c, -fmaf(sm.slope[h], dist, m[h])) : -INFINITY;
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
#pragma unroll
                for (int h = 0; h < kHn; ++h) {
                    const int hm = __reduce_max_sync(0xffffffffu, ordered(x[h]));
                    if (lane == h) sm.warp_max[x_id][w_id][h] = hm;
                }
                named_barrier_sync<kStream>(1 + x_id);
                if (key < kHn) {
                    const int(&wm)[kWarps][kMaxHeads] = sm.warp_max[x_id];
                    const float grown = unordered(max(max(wm[0][key], wm[1][key]), max(wm[2][key], wm[3][key])));
                    const bool moves = k == 0 || grown > kRescaleThreshold;
                    sm.factor[x_id][key] = moves && k > 0 ? ex2(-grown) : 1.f;
                    sm.delta[x_id][key] = moves ? grown : 0.f;
                    if (moves) m[key] += grown;
                }
                named_barrier_sync<kStream>(1 + x_id);
#pragma unroll
                for (int h = 0; h < kHn; ++h) {
                    x[h] -= sm.delta[x_id][h];
                    l[h] *= sm.factor[x_id][h];
                }
                if (k > 0) {
                    // the stream's products so far are complete: they were issued ahead of this tile's scores
                    const uint32_t o_mine = o_base + lane_base + x_id * kHn;
#pragma unroll
                    for (int cc = 0; cc < kHn / 16; ++cc) {
                        uint32_t o[16];
                        __syncwarp();
                        tmem_ld16(o_mine + cc * 16, o);
                        tmem_wait_ld();
#pragma unroll
                        for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * sm.factor[x_id][cc * 16 + e]);
                        tmem_st16(o_mine + cc * 16, o);
                    }
                    tmem_wait_st();
                }
            }
            uint8_t* const p_row = p_tile + (2 * x_id + (key >> 6)) * kQChunk + (key & 7) * 2;
#pragma unroll
            for (int h = 0; h < kHn; ++h) {
                const float w = ex2(x[h]);
                l[h] += w;
                *reinterpret_cast<__nv_bfloat16*>(p_row + h * 128 + ((((key & 63) >> 3) ^ (h & 7)) << 4)) = __float2bfloat16_rn(w);
            }
            fence_proxy_async_smem();  // P was written with ordinary stores and is read by the tensor core
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&sm.p_ready[x_id]);
        }
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&sm.o_done, 0));
        if (!ok && lane == 0) sm.fail[x_id] = 1;
        tc_fence_after();
        // sums over the keys: inside the warps, then over the warps and the streams
#pragma unroll
        for (int h = 0; h < kHn; ++h) {
#pragma unroll
            for (int off = 16; off > 0; off >>= 1) l[h] += __shfl_xor_sync(0xffffffffu, l[h], off);
            if (lane == h) sm.sum[x_id][w_id][h] = l[h];
        }
        named_barrier_sync<2 * kStream>(3);
        if (sm.fail[0] == 0 && sm.fail[1] == 0) {
            const bool both = n_tiles > 1;  // otherwise the second stream has no accumulator
            if (x_id == 0 && key < kHn) {   // weights of the streams, against the larger of their references
                const float m0 = sm.m[0][key], m1 = both ? sm.m[1][key] : m0, top = fmaxf(m0, m1);
                float s0 = 0.f, s1 = 0.f;
#pragma unroll
                for (int w = 0; w < kWarps; ++w) s0 += sm.sum[0][w][key], s1 += sm.sum[1][w][key];
                sm.factor[0][key] = ex2(m0 - top);
                sm.factor[1][key] = both ? ex2(m1 - top) : 0.f;
                sm.delta[0][key] = top;
                sm.delta[1][key] = sm.factor[0][key] * s0 + (both ? sm.factor[1][key] * s1 : 0.f);
            }
            named_barrier_sync<2 * kStream>(3);
            const int64_t stride = p.vdim + 2;
            // a row of a single share writes its output, others leave a partial result
            float* part = all_tiles > n_tiles ? p.partial + ((static_cast<int64_t>(i) * p.splits + split) * p.H + h0) * stride : nullptr;
            if (part != nullptr && x_id == 0 && key < heads) {
                part[key * stride + p.vdim] = sm.delta[0][key];
                part[key * stride + p.vdim + 1] = sm.delta[1][key];
            }
            __nv_bfloat16* out = p.out + static_cast<int64_t>(i) * p.ld_out + static_cast<int64_t>(h0) * p.vdim;
            const uint32_t o_0 = o_base + lane_base, o_1 = o_0 + kHn;
            // element = TMEM lane; the streams' warps take the columns in turn
#pragma unroll 1
            for (int cc = x_id; cc < kHn / 8; cc += 2) {
                uint32_t o[8], o2[8];
                __syncwarp();
                tmem_ld8(o_0 + cc * 8, o);
                tmem_ld8(o_1 + cc * 8, o2);  // (read in any case, used only if there is a second stream)
                tmem_wait_ld();
#pragma unroll
                for (int u = 0; u < 8; ++u) {
                    const int h = cc * 8 + u;
                    if (h >= heads || key >= p.vdim) continue;
                    float v = __uint_as_float(o[u]) * sm.factor[0][h];
                    if (both) v = fmaf(__uint_as_float(o2[u]), sm.factor[1][h], v);
                    if (part != nullptr)
                        part[h * stride + key] = v;
                    else
                        out[static_cast<int64_t>(h) * p.vdim + key] = __float2bfloat16_rn(v / sm.delta[1][h]);
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
        tmem_dealloc(tmem, kTmemCols);
    }
    if (threadIdx.x == 0 && sm.abort_flag) report_status(p.dev_status, B2KV_DEV_WAIT_TIMEOUT);
}

// One CTA per (head, row): the shares' partial results, each relative to its own reference maximum.
constexpr int kMaxSplits = 256;
__global__ void __launch_bounds__(128) gqa_merge_kernel(const Params p) {
    __shared__ float w[kMaxSplits];
    grid_launch_dependents();
    if (threadIdx.x == 0) grid_dependency_wait();
    __syncthreads();
    const int h = blockIdx.x, i = blockIdx.y;
    int slot, pos;
    if (!row_place(p.row_slot, p.row_pos, i, p.n_slots, p.T_max, slot, pos)) return;
    const int splits = min(p.splits, (pos / kTile + p.share) / p.share);  // shares with tiles
    if (splits <= 1) return;                                // the row's only share has written the output
    const int64_t stride = p.vdim + 2;
    const float* part = p.partial + (static_cast<int64_t>(i) * p.splits * p.H + h) * stride;
    if (threadIdx.x < 32) {
        float mx = kNothingSeen;
        for (int s = threadIdx.x; s < splits; s += 32) mx = fmaxf(mx, part[s * p.H * stride + p.vdim]);
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        float sum = 0.f;
        for (int s = threadIdx.x; s < splits; s += 32) {
            const float f = ex2(part[s * p.H * stride + p.vdim] - mx);
            w[s] = f;
            sum += f * part[s * p.H * stride + p.vdim + 1];
        }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
        for (int s = threadIdx.x; s < splits; s += 32) w[s] /= sum;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < p.vdim; e += 128) {
        float v = 0.f;
        for (int s = 0; s < splits; ++s) v = fmaf(w[s], part[s * p.H * stride + e], v);
        p.out[static_cast<int64_t>(i) * p.ld_out + static_cast<int64_t>(h) * p.vdim + e] = __float2bfloat16_rn(v);
    }
}

// (element, head, row) view with 64-element boxes of box_heads x box_rows, 128-byte swizzle.
static bool make_map(CUtensorMap* map, const void* base, int width, int heads, int64_t rows, int64_t pitch, int box_heads,
                     int box_rows) {
    EncodeTiledFn fn = tensor_map_encoder();
    if (fn == nullptr) return false;
    const cuuint64_t dims[3] = {static_cast<cuuint64_t>(width), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(rows)};
    const cuuint64_t strides[2] = {static_cast<cuuint64_t>(width) * 2, static_cast<cuuint64_t>(pitch) * 2};
    const cuuint32_t box[3] = {64, static_cast<cuuint32_t>(box_heads), static_cast<cuuint32_t>(box_rows)};
    const cuuint32_t estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// Tiles per share: enough shares for every SM where the rows are few, and shares long enough to pay for their start.
static int choose_share(int rows, int H, int G, int span) {
    const int tiles = (span + kTile - 1) / kTile;
    int share = tune_get("gqa_decode_share");
    if (share <= 0) {
        const int groups = (H / G + kMaxHeads - 1) / kMaxHeads;
        const long long all = static_cast<long long>(rows) * G * groups * tiles;
        share = static_cast<int>(std::min<long long>(16, std::max<long long>(2, all / (4LL * device_sm_count()))));
    }
    return std::max(share, (tiles + kMaxSplits - 1) / kMaxSplits);
}

template <int kHn, int kKc>
static int launch(const CUtensorMap (&m)[3], const Params& p, unsigned grid, size_t smem, void* stream) {
    static int configured[64] = {0};
    int dev = 0;
    B2KV_CUDA_TRY(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64) return B2KV_ERR_UNSUPPORTED;
    auto kernel = gqa_decode_tc_kernel<kHn, kKc>;
    if (configured[dev] < static_cast<int>(smem)) {
        B2KV_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        configured[dev] = static_cast<int>(smem);
    }
    OverlapLaunch cfg(grid, kThreads, smem, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&cfg.cfg, kernel, m[0], m[1], m[2], p));
    return B2KV_OK;
}

}  // namespace gqadec

size_t gqa_decode_tc_workspace(int rows, int H, int G, int vdim, int span) {
    const int share = gqadec::choose_share(rows, H, G, span);
    const int splits = ((span + gqadec::kTile - 1) / gqadec::kTile + share - 1) / share;
    return splits > 1 ? static_cast<size_t>(rows) * splits * H * (vdim + 2) * sizeof(float) : 0;
}

int gqa_decode_tc(const GqaDecodeArgs& a, void* workspace, size_t workspace_bytes, void* stream) {
    using namespace gqadec;
    if (a.dim % 8 != 0 || a.dim > 128 || a.vdim % 8 != 0 || a.vdim > 128 || a.ld_q % 8 != 0 || !(a.scale > 0.f)) return B2KV_ERR_UNSUPPORTED;
    if (!aligned16(a.q) || !aligned16(a.k_cache) || !aligned16(a.v_cache)) return B2KV_ERR_UNSUPPORTED;
    const int64_t cache_rows = static_cast<int64_t>(a.n_slots) * a.T_max;
    if (cache_rows > 0x7fffffffLL - 256 || a.rows > 65535) return B2KV_ERR_UNSUPPORTED;
    const int per_kv = a.H / a.G, Hn = per_kv <= 16 ? 16 : 32;  // further heads are further CTAs, which find the rows in L2
    Params p{};
    p.row_slot = a.row_slot;
    p.row_pos = a.row_pos;
    p.slopes = a.slopes;
    p.out = static_cast<__nv_bfloat16*>(a.out);
    p.partial = static_cast<float*>(workspace);
    p.dev_status = a.dev_status;
    p.ld_out = a.ld_out;
    p.n_slots = a.n_slots;
    p.T_max = a.T_max;
    p.H = a.H;
    p.G = a.G;
    p.vdim = a.vdim;
    p.prescale = a.scale * kLog2e;
    p.head_groups = (per_kv + Hn - 1) / Hn;
    p.share = choose_share(a.rows, a.H, a.G, a.span);
    p.splits = ((std::min(a.span, a.T_max) + kTile - 1) / kTile + p.share - 1) / p.share;
    if (p.splits > 1 && (workspace == nullptr || workspace_bytes < gqa_decode_tc_workspace(a.rows, a.H, a.G, a.vdim, a.span)))
        return B2KV_ERR_WORKSPACE;
    p.v_chunks = (a.vdim + 63) / 64;
    const int k_chunks = (a.dim + 63) / 64;
    const int fixed = (k_chunks + 4) * Hn * 128 + 1024;
    const int stage_bytes = (k_chunks + p.v_chunks) * kChunkBytes;
    p.stages = std::min(kMaxStages, (kSmemLimit - fixed - static_cast<int>(sizeof(Shared))) / stage_bytes);
    const size_t smem = static_cast<size_t>(p.stages) * stage_bytes + fixed;
    CUtensorMap m[3];
    if (!make_map(&m[0], a.q, a.dim, a.H, a.rows, a.ld_q, Hn, 1) ||
        !make_map(&m[1], a.k_cache, a.dim, a.G, cache_rows, static_cast<int64_t>(a.G) * a.dim, 1, kTile) ||
        !make_map(&m[2], a.v_cache, a.vdim, a.G, cache_rows, static_cast<int64_t>(a.G) * a.vdim, 1, kTile))
        return B2KV_ERR_UNSUPPORTED;
    const long long grid = static_cast<long long>(a.rows) * a.G * p.head_groups * p.splits;
    if (grid > 0x7fffffffLL) return B2KV_ERR_UNSUPPORTED;
    const unsigned n = static_cast<unsigned>(grid);
    const int rc = Hn == 16 ? (k_chunks == 1 ? launch<16, 1>(m, p, n, smem, stream) : launch<16, 2>(m, p, n, smem, stream))
                            : (k_chunks == 1 ? launch<32, 1>(m, p, n, smem, stream) : launch<32, 2>(m, p, n, smem, stream));
    if (rc != B2KV_OK || p.splits == 1) return rc;
    OverlapLaunch cfg(dim3(a.H, a.rows), 128, 0, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&cfg.cfg, gqa_merge_kernel, p));
    return B2KV_OK;
}

}  // namespace b2kv
