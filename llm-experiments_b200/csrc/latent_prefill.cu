// Attention of prompt portions on the Blackwell tensor cores (bf16): over keys and values expanded from cached latent rows, and over
// cached keys and values of grouped heads.
//
// The scheme is that of prefill_tc.cu: one CTA per head and 256 query rows (two 128-row tiles A and B that share every 128-key
// tile), warp 8 copies with TMA, warp 9 issues tcgen05.mma (S = Q K^T from shared memory, O += P V with P read from tensor
// memory) in the order PV_A, QK_A', PV_B, QK_B', warps 0-7 are the softmax (thread = query row = TMEM lane, running maximum in
// the log2 domain, O rescaled only when the maximum has grown by more than 2^8).  What is different here:
//
//   * a query / key row is the concatenation of `dim` unrotated elements of its own head and `rot` rotated ones, which for
//     the keys are one row shared by all heads, read from the cache itself.  Tensor maps with exact extents per head cut both
//     parts into 64-element chunks whose tails read as zero, so nothing is assembled in memory;
//   * values may be narrower or wider than keys;
//   * a sliding window: tiles outside a row tile's window are not visited, and elements are masked by position.  A row can
//     meet tiles without any visible key before its first one; its P is zero there.  That case takes no branch of its own:
//     the rows of a warp differ in it, and the tensor-memory instructions around it have to be met by whole warps;
//   * portions: query row i of a segment sits at key row `own + i` of that segment, so a portion attends to what earlier
//     portions left in the cache.  One launch takes any number of segments (sequences), described by a device table;
//   * with 192-element keys and 128-element values the two query tiles leave room for eight 16 KB chunks: K tiles take a single
//     chunk (a ring of two) and a pair, V tiles a pair, the pairs form one ring of three that K(0) V(0) K(1) V(1) ... pass
//     through.  K(j + 1) and V(j + 1) are then on their way while K(j) and V(j) are in use.
//
// Grouped heads (no rotated part) read the caches in place: key row t of a segment is a cache row, head h takes the columns of
// key / value head h / (H / G).  A distance bias, slope_h * (query position - key position), is taken off the scores in fp32
// without work per score: the part that depends on the key's place in its tile, 0 ... 127, is one more k-step of the score product
// (key rows hold their place, query rows slope / scale in three bf16 pieces, so the products are exact), the rest is a
// constant of the row and the tile.
//
// TMEM columns: S_A 0-127, S_B 128-255, O_A 256-383, O_B 384-511.  Every wait is bounded.
#include <math.h>

#include <algorithm>
#include <type_traits>

#include "tc_ptx.cuh"
#include "tma_map.cuh"

namespace b2kv {
namespace latpre {

using namespace tc;

constexpr int kTileM = 128, kBlockN = 128;
constexpr int kChunkBytes = 128 * 128;  // 128 rows x 64 bf16
constexpr int kThreads = 320;
constexpr int kTmemCols = 512;
constexpr int kColS = 0, kColO = 256;
constexpr float kRescaleThreshold = 8.0f;
constexpr float kNothingSeen = -1e30f;  // reference maximum of a row that has met no visible key yet (finite: P = 2^(-inf) = 0)

struct Params {
    __nv_bfloat16* out;  // row i of the step at out + i * ld_out, head h at column h * vdim
    const b2kv_prompt_segment* seg;
    int32_t* dev_status;
    const float* slopes;  // fp32 [H], with kBias
    int64_t ld_out;
    int n_seg, n_blocks, H, group, dim, rot, vdim, window;
    float prescale;  // scale * log2(e)
    int rows, kv_rows, cache_rows;
    int per_kv;  // query heads per key / value head
};

// kNope chunks per key, with kRot one more for the rotated part; kV chunks per value.
template <int kNope, bool kRot, int kV, bool kBias>
struct Storage {
    static constexpr int kK = kNope + (kRot ? 1 : 0);
    static constexpr bool kSharedRing = kK == 3 && kV == 2;
    static constexpr int kChunks = kSharedRing ? 8 : 2 * (kK + kV);
    alignas(1024) uint8_t q[2][kK][kChunkBytes];
    alignas(1024) uint8_t kv[kChunks][kChunkBytes];
    uint8_t ext[kBias ? kChunkBytes : 16];  // the bias's k-step: elements 0-15 of the key rows, 16-31 of the query rows
    alignas(8) uint64_t q_full;
    uint64_t k_full[2], k_empty[2], v_full[2], v_empty[2];
    uint64_t s_full[2], p_ready[2], o_done[2];
    uint32_t tmem_base;
    volatile int abort_flag;

    // Chunk of K tile j (the first kNope are neighbours) / first chunk of V tile j (j counts from the CTA's first tile).
    __device__ static __forceinline__ int k_chunk(int j, int c) {
        if (kSharedRing) return c == 2 ? 6 + (j & 1) : (2 * j) % 3 * 2 + c;
        return (j & 1) * kK + c;
    }
    __device__ static __forceinline__ int v_chunk(int j) {
        if (kSharedRing) return (2 * j + 1) % 3 * 2;
        return 2 * kK + (j & 1) * kV;
    }
};

template <int kNope, bool kRot, int kV, bool kBias>
__global__ void __launch_bounds__(kThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tm_qn, const __grid_constant__ CUtensorMap tm_qr,
                      const __grid_constant__ CUtensorMap tm_kn, const __grid_constant__ CUtensorMap tm_kr,
                      const __grid_constant__ CUtensorMap tm_v, const Params p) {
    extern __shared__ uint8_t smem_raw[];
    using Smem = Storage<kNope, kRot, kV, kBias>;
    constexpr int kK = Smem::kK;
    Smem& sm = *reinterpret_cast<Smem*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    // groups of heads whose keys and values stay in L2 together; inside a group the last row blocks first
    const int per_group = p.group * p.n_blocks;
    const int gi = static_cast<int>(blockIdx.x) / per_group;
    const int heads_here = min(p.group, p.H - gi * p.group);
    const int within = static_cast<int>(blockIdx.x) - gi * per_group;
    const int block = p.n_blocks - 1 - within / heads_here;
    const int h = gi * p.group + within % heads_here;
    const int h_kv = kRot ? h : h / p.per_kv;
    int si = 0;
    while (si + 1 < p.n_seg && p.seg[si + 1].first_block <= block) ++si;
    const b2kv_prompt_segment sg = p.seg[si];
    if (sg.row0 < 0 || sg.n <= 0 || sg.row0 + sg.n > p.rows || sg.kv_row0 < 0 || sg.own < 0 ||
        sg.kv_row0 + sg.own + sg.n > p.kv_rows || sg.cache_row0 < 0 || sg.cache_row0 + sg.own + sg.n > p.cache_rows ||
        block < sg.first_block || (block - sg.first_block) * 2 * kTileM >= sg.n) {
        if (threadIdx.x == 0) report_status(p.dev_status, B2KV_DEV_BAD_POSITION);  // a table that does not fit the buffers
        return;
    }
    const int q0 = (block - sg.first_block) * 2 * kTileM;  // first query row, inside the segment
    // key tiles of the two row tiles, [first, last]; B is absent past the segment's end
    const bool has_b = q0 + kTileM < sg.n;
    auto first_tile = [&](int r) { return p.window > 0 ? max(0, sg.own + r - p.window + 1) / kBlockN : 0; };
    auto last_tile = [&](int r) { return (sg.own + min(r + kTileM, sg.n) - 1) / kBlockN; };
    const int a0 = first_tile(q0), a1 = last_tile(q0);
    const int b0 = has_b ? first_tile(q0 + kTileM) : a1 + 1, b1 = has_b ? last_tile(q0 + kTileM) : a1;
    const int n_tiles = max(a1, b1) - a0 + 1;
    // relative to the CTA's first tile
    const int end_a = a1 - a0 + 1, beg_b = has_b ? b0 - a0 : n_tiles, end_b = has_b ? b1 - a0 + 1 : n_tiles;

    if (threadIdx.x == 0) {
        mbar_init(&sm.q_full, 1);
        for (int s = 0; s < 2; ++s) {
            mbar_init(&sm.k_full[s], 1);
            mbar_init(&sm.k_empty[s], 1);
            mbar_init(&sm.v_full[s], 1);
            mbar_init(&sm.v_empty[s], 1);
            mbar_init(&sm.s_full[s], 1);
            mbar_init(&sm.p_ready[s], 128);
            mbar_init(&sm.o_done[s], 1);
        }
        sm.abort_flag = 0;
        fence_mbar_init();
    }
    if (warp == 9) {
        tmem_alloc(&sm.tmem_base, kTmemCols);
        tmem_relinquish();
    }
    if (kBias && threadIdx.x < kBlockN) {
        const float whole = p.slopes[h] * 1.4426950408889634f / p.prescale;  // slope / scale
        const float hi = __bfloat162float(__float2bfloat16_rn(whole));
        const float mid = __bfloat162float(__float2bfloat16_rn(whole - hi));
        const float place = static_cast<float>(threadIdx.x);
        uint4 piece[4] = {};
        piece[0].x = pack_bf16(place, place);
        piece[0].y = pack_bf16(place, 0.f);
        piece[2].x = pack_bf16(hi, mid);
        piece[2].y = pack_bf16(whole - hi - mid, 0.f);
#pragma unroll
        for (int c = 0; c < 4; ++c)
            *reinterpret_cast<uint4*>(sm.ext + threadIdx.x * 128 + ((c ^ (threadIdx.x & 7)) << 4)) = piece[c];
        fence_proxy_async_smem();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = sm.tmem_base;

    if (warp == 8) {
        // ------------------------------ TMA producer ------------------------------
        if (lane == 0) {
            mbar_arrive_expect_tx(&sm.q_full, (has_b ? 2 : 1) * kK * kChunkBytes);
            for (int x = 0; x < (has_b ? 2 : 1); ++x) {
                const int row = sg.row0 + q0 + x * kTileM;
#pragma unroll
                for (int c = 0; c < kNope; ++c) tma_load_3d(sm.q[x][c], &tm_qn, &sm.q_full, c * 64, h, row);
                if (kRot) tma_load_3d(sm.q[x][kK - 1], &tm_qr, &sm.q_full, 0, h, row);
            }
            bool ok = true;
            for (int j = 0; j < n_tiles; ++j) {
                const int st = j & 1;
                const uint32_t par = ((j >> 1) & 1) ^ 1;
                const int key = (a0 + j) * kBlockN;
                ok = mbar_wait(&sm.k_empty[st], par);
                if (Smem::kSharedRing && ok) ok = mbar_wait(&sm.v_empty[st], par);  // V(j - 2) leaves its pair to K(j)
                if (!ok) break;
                mbar_arrive_expect_tx(&sm.k_full[st], kK * kChunkBytes);
#pragma unroll
                for (int c = 0; c < kNope; ++c)
                    tma_load_3d(sm.kv[Smem::k_chunk(j, c)], &tm_kn, &sm.k_full[st], c * 64, h_kv, sg.kv_row0 + key);
                if (kRot) tma_load_3d(sm.kv[Smem::k_chunk(j, kNope)], &tm_kr, &sm.k_full[st], 0, 0, sg.cache_row0 + key);
                ok = mbar_wait(&sm.v_empty[st], par);
                // K(j - 1) leaves its pair to V(j)
                if (Smem::kSharedRing && ok && j > 0) ok = mbar_wait(&sm.k_empty[st ^ 1], ((j - 1) >> 1) & 1);
                if (!ok) break;
                mbar_arrive_expect_tx(&sm.v_full[st], kV * kChunkBytes);
#pragma unroll
                for (int c = 0; c < kV; ++c)
                    tma_load_3d(sm.kv[Smem::v_chunk(j) + c], &tm_v, &sm.v_full[st], c * 64, h_kv, sg.kv_row0 + key);
            }
            if (!ok) sm.abort_flag = 1;
        }
        __syncwarp();
    } else if (warp == 9) {
        // ------------------------------ MMA issuer ------------------------------
        if (lane == 0) {
            // Everything an MMA needs beside the tile's place is a compile-time constant: chunks are multiplied whole (what
            // lies past a head's elements is zero in both operands), and the places are chosen by selects.
            constexpr uint32_t idesc_qk = instr_desc(0, 0, kBlockN);
            constexpr uint32_t idesc_pv = instr_desc(0, 1, kV * 64);
            const uint64_t dq0 = smem_desc(smem_u32(sm.q[0][0]), 16, 1024), dq1 = smem_desc(smem_u32(sm.q[1][0]), 16, 1024);
            const uint64_t dk = smem_desc(smem_u32(sm.kv[0]), 16, 1024);
            const uint64_t dv = smem_desc(smem_u32(sm.kv[0]), kChunkBytes, 1024);
            const uint64_t d_ext = smem_desc(smem_u32(sm.ext), 16, 1024);
            constexpr uint32_t kChunk16 = kChunkBytes >> 4;
            auto issue_qk = [&](int x, int j) {
                const uint64_t a = x ? dq1 : dq0;
                const uint64_t b = dk + static_cast<uint64_t>(Smem::k_chunk(j, 0)) * kChunk16;
                const uint64_t b_last = dk + static_cast<uint64_t>(Smem::k_chunk(j, kNope)) * kChunk16;
                const uint32_t s_tmem = tmem + kColS + x * 128;
#pragma unroll
                for (int c = 0; c < kK; ++c) {
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk)
                        mma_ss(s_tmem, a + static_cast<uint64_t>(c * kChunk16 + 2 * kk),
                               kRot && c == kNope ? b_last + static_cast<uint64_t>(2 * kk) : b + static_cast<uint64_t>(c * kChunk16 + 2 * kk),
                               idesc_qk, (c | kk) ? 1u : 0u);
                }
                if (kBias) mma_ss(s_tmem, d_ext + static_cast<uint64_t>(2), d_ext, idesc_qk, 1u);
                mma_commit(&sm.s_full[x]);
            };
            auto issue_pv = [&](int x, int j, bool first) {
                const uint64_t b = dv + static_cast<uint64_t>(Smem::v_chunk(j)) * kChunk16;
                const uint32_t p_tmem = tmem + kColS + x * 128, o_tmem = tmem + kColO + x * 128;
#pragma unroll
                for (int kk = 0; kk < 8; ++kk)
                    mma_ts(o_tmem, p_tmem + kk * 8, b + static_cast<uint64_t>((kk * 2048) >> 4), idesc_pv,
                           (kk || !first) ? 1u : 0u);
                mma_commit(&sm.o_done[x]);
            };
            bool ok = mbar_wait(&sm.q_full, 0) && mbar_wait(&sm.k_full[0], 0);
            if (ok) {
                tc_fence_after();
                issue_qk(0, 0);
                if (beg_b == 0) issue_qk(1, 0);
                mma_commit(&sm.k_empty[0]);
            }
            for (int j = 0; j < n_tiles && ok; ++j) {
                const int st = j & 1, st1 = st ^ 1;
                const uint32_t par = (j >> 1) & 1, par1 = ((j + 1) >> 1) & 1;
                const bool in_a = j < end_a, in_b = j >= beg_b && j < end_b;
                const bool next_a = j + 1 < end_a, next_b = j + 1 >= beg_b && j + 1 < end_b;
                if (in_a) {
                    ok = mbar_wait(&sm.p_ready[0], j & 1) && mbar_wait(&sm.v_full[st], par);
                    if (!ok) break;
                    tc_fence_after();
                    issue_pv(0, j, j == 0);
                }
                if (next_a) {
                    ok = mbar_wait(&sm.k_full[st1], par1);
                    if (!ok) break;
                    tc_fence_after();
                    issue_qk(0, j + 1);
                }
                if (in_b) {
                    ok = mbar_wait(&sm.p_ready[1], (j - beg_b) & 1) && (in_a || mbar_wait(&sm.v_full[st], par));
                    if (!ok) break;
                    tc_fence_after();
                    issue_pv(1, j, j == beg_b);
                }
                mma_commit(&sm.v_empty[st]);
                if (next_b) {
                    ok = next_a || mbar_wait(&sm.k_full[st1], par1);
                    if (!ok) break;
                    tc_fence_after();
                    issue_qk(1, j + 1);
                }
                if (j + 1 < n_tiles) mma_commit(&sm.k_empty[st1]);
            }
            if (!ok) sm.abort_flag = 1;
        }
        __syncwarp();
    } else {
        // ------------------------------ softmax: thread = query row ------------------------------
        const int x = warp >> 2;
        const int row = threadIdx.x & 127;
        const int beg = x ? beg_b : 0, end = x ? end_b : end_a;
        const int n_x = x && !has_b ? 0 : end - beg;
        const uint32_t lane_base = static_cast<uint32_t>((warp & 3) * 32) << 16;
        const uint32_t s_tmem = tmem + lane_base + kColS + x * 128;
        const uint32_t o_tmem = tmem + lane_base + kColO + x * 128;
        const float c = p.prescale;
        const float slope = kBias ? p.slopes[h] * 1.4426950408889634f : 0.f;
        const int own = sg.own + q0 + x * kTileM;  // key row of the tile's first query
        float m_used = -INFINITY, m_run = -INFINITY, l = 0.f;
        bool ok = true;
        for (int i = 0; i < n_x && ok; ++i) {
            const int key0 = (a0 + beg + i) * kBlockN;
            ok = __all_sync(0xffffffffu, mbar_wait(&sm.s_full[x], i & 1));
            if (!ok) break;
            tc_fence_after();
            uint32_t r[128];
            tmem_ld128(s_tmem, r);
            tmem_wait_ld();
            // columns this row sees: [lo, hi]; a tile that every row of the row tile sees whole needs no mask
            const int hi = own + row - key0;
            const int lo = p.window > 0 ? hi - p.window + 1 : -1;
            const float2 c2 = make_float2(c, c);
            const float shift = kBias ? -slope * static_cast<float>(hi) : 0.f;  // what the row and the tile take off
            if (key0 + kBlockN - 1 > own || (p.window > 0 && own + kTileM - 1 - p.window + 1 > key0)) {
#pragma unroll
                for (int e = 0; e < 128; ++e)
                    if (e > hi || e < lo) r[e] = 0xff800000u;
            }
            float mxs[8];
#pragma unroll
            for (int a = 0; a < 8; ++a) mxs[a] = __uint_as_float(r[a]);
#pragma unroll
            for (int e = 8; e < 128; ++e) mxs[e & 7] = fmaxf(mxs[e & 7], __uint_as_float(r[e]));
            const float mx = fmaxf(fmaxf(fmaxf(mxs[0], mxs[1]), fmaxf(mxs[2], mxs[3])),
                                   fmaxf(fmaxf(mxs[4], mxs[5]), fmaxf(mxs[6], mxs[7])));
            m_run = fmaxf(m_run, kBias ? fmaf(mx, c, shift) : mx * c);
            float factor = 1.f;
            bool need = false;
            if (i == 0) {
                m_used = fmaxf(m_run, kNothingSeen);
            } else if (m_run > m_used + kRescaleThreshold) {  // also from kNothingSeen: O and l are zero and stay so
                factor = ex2(m_used - m_run);
                m_used = m_run;
                need = true;
            }
            const float neg_m = shift - m_used;
            __syncwarp();  // the tensor-memory instructions below need the whole warp together
            float sums[8];
#pragma unroll
            for (int a = 0; a < 8; ++a) sums[a] = 0.f;
            const float2 neg_m2 = make_float2(neg_m, neg_m);
#pragma unroll
            for (int cc = 0; cc < 4; ++cc) {
                uint32_t pk[16];
#pragma unroll
                for (int e = 0; e < 16; ++e) {
                    const float2 s2 = make_float2(__uint_as_float(r[cc * 32 + 2 * e]), __uint_as_float(r[cc * 32 + 2 * e + 1]));
                    const float2 z = __ffma2_rn(s2, c2, neg_m2);
                    const float p0 = ex2(z.x), p1 = ex2(z.y);
                    sums[(2 * e) & 7] += p0;
                    sums[(2 * e + 1) & 7] += p1;
                    pk[e] = pack_bf16(p0, p1);
                }
                tmem_st16(s_tmem + cc * 16, pk);
            }
            const float sum0 = (sums[0] + sums[1]) + (sums[2] + sums[3]);
            const float sum1 = (sums[4] + sums[5]) + (sums[6] + sums[7]);
            l = l * factor + (sum0 + sum1);
            // rare: bring O down to the new reference maximum (needs PV of the previous tile finished)
            if (__any_sync(0xffffffffu, need)) {
                ok = __all_sync(0xffffffffu, mbar_wait(&sm.o_done[x], (i - 1) & 1));
                if (ok) {
                    tc_fence_after();
#pragma unroll 1
                    for (int cc = 0; cc < (p.vdim + 31) / 32; ++cc) {
                        uint32_t o[32];
                        tmem_ld32(o_tmem + cc * 32, o);
                        tmem_wait_ld();
#pragma unroll
                        for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * factor);
                        tmem_st32(o_tmem + cc * 32, o);
                    }
                }
            }
            tmem_wait_st();
            tc_fence_before();
            mbar_arrive(&sm.p_ready[x]);
        }
        if (ok && n_x > 0) ok = __all_sync(0xffffffffu, mbar_wait(&sm.o_done[x], (n_x - 1) & 1));
        if (ok && n_x > 0) {
            tc_fence_after();
            const int qrow = q0 + x * kTileM + row;
            const bool live = qrow < sg.n;
            const float inv = 1.f / l;
            __nv_bfloat16* out = p.out + static_cast<int64_t>(sg.row0 + qrow) * p.ld_out + static_cast<int64_t>(h) * p.vdim;
#pragma unroll 1
            for (int cc = 0; cc < (p.vdim + 31) / 32; ++cc) {
                uint32_t o[32];
                __syncwarp();
                tmem_ld32(o_tmem + cc * 32, o);
                tmem_wait_ld();
                if (live) {
#pragma unroll
                    for (int v4 = 0; v4 < 4; ++v4) {
                        if (cc * 32 + v4 * 8 >= p.vdim) break;
                        uint4 w;
                        w.x = pack_bf16(__uint_as_float(o[v4 * 8 + 0]) * inv, __uint_as_float(o[v4 * 8 + 1]) * inv);
                        w.y = pack_bf16(__uint_as_float(o[v4 * 8 + 2]) * inv, __uint_as_float(o[v4 * 8 + 3]) * inv);
                        w.z = pack_bf16(__uint_as_float(o[v4 * 8 + 4]) * inv, __uint_as_float(o[v4 * 8 + 5]) * inv);
                        w.w = pack_bf16(__uint_as_float(o[v4 * 8 + 6]) * inv, __uint_as_float(o[v4 * 8 + 7]) * inv);
                        *reinterpret_cast<uint4*>(out + cc * 32 + v4 * 8) = w;
                    }
                }
            }
        } else if (!ok) {
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

// (element, head, row) view of a matrix: 64 elements of one head in 128 rows per box.
static bool make_map(CUtensorMap* map, const void* base, int width, int heads, int64_t rows, int64_t head_stride, int64_t pitch) {
    EncodeTiledFn fn = tensor_map_encoder();
    if (fn == nullptr) return false;
    const cuuint64_t dims[3] = {static_cast<cuuint64_t>(width), static_cast<cuuint64_t>(heads), static_cast<cuuint64_t>(rows)};
    const cuuint64_t strides[2] = {static_cast<cuuint64_t>(head_stride) * 2, static_cast<cuuint64_t>(pitch) * 2};
    const cuuint32_t box[3] = {64, 1, 128};
    const cuuint32_t estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
              CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int kNope, bool kRot, int kV, bool kBias>
static int launch(const CUtensorMap (&m)[5], const Params& p, long long ctas, void* stream) {
    constexpr size_t smem = sizeof(Storage<kNope, kRot, kV, kBias>) + 1024;
    static_assert(smem <= 227 * 1024, "the tiles must fit one SM's shared memory");
    auto kernel = latent_prefill_kernel<kNope, kRot, kV, kBias>;
    static bool configured[64] = {false};
    int dev = 0;
    B2KV_CUDA_TRY(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64) return B2KV_ERR_UNSUPPORTED;
    if (!configured[dev]) {
        B2KV_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        configured[dev] = true;
    }
    kernel<<<static_cast<unsigned>(ctas), kThreads, smem, static_cast<cudaStream_t>(stream)>>>(m[0], m[1], m[2], m[3], m[4], p);
    B2KV_CUDA_TRY(cudaGetLastError());
    return B2KV_OK;
}

}  // namespace latpre
}  // namespace b2kv

using namespace b2kv;

extern "C" int b2kv_latent_prefill_supported(int dim, int rot, int vdim, int kv_rank, int dtype) {
    return dtype == B2KV_DTYPE_BF16 && dim > 0 && dim <= 128 && dim % 8 == 0 && rot > 0 && rot <= 64 && rot % 8 == 0 && vdim > 0 &&
           vdim <= 128 && vdim % 8 == 0 && kv_rank > 0 && kv_rank % 8 == 0;
}

extern "C" int b2kv_latent_prefill(const void* q, int64_t ld_q, const void* keys, const void* values, int64_t ld_kv,
                                   const void* key_cache, int64_t cache_rows, void* out, int64_t ld_out,
                                   const b2kv_prompt_segment* segments, int n_segments, int n_blocks, int rows, int kv_rows, int H,
                                   int dim, int rot, int vdim, int window, float scale, int dtype, int32_t* dev_status,
                                   void* stream) {
    using namespace latpre;
    if (!q || !keys || !values || !key_cache || !out || !segments || n_segments <= 0 || n_blocks <= 0 || rows <= 0 || kv_rows <= 0 ||
        cache_rows <= 0 || H <= 0)
        return B2KV_ERR_BAD_ARG;
    if (!b2kv_latent_prefill_supported(dim, rot, vdim, 8, dtype) || !(scale > 0.f)) return B2KV_ERR_UNSUPPORTED;
    if (ld_q < static_cast<int64_t>(H) * (dim + rot) || ld_out < static_cast<int64_t>(H) * vdim) return B2KV_ERR_BAD_ARG;
    if (!aligned16(q) || !aligned16(keys) || !aligned16(values) || !aligned16(key_cache) || !aligned16(out) || ld_q % 8 || ld_kv % 8 ||
        ld_out % 8)
        return B2KV_ERR_ALIGN;
    CUtensorMap m[5];
    if (!make_map(&m[0], q, dim, H, rows, dim + rot, ld_q) ||
        !make_map(&m[1], static_cast<const __nv_bfloat16*>(q) + dim, rot, H, rows, dim + rot, ld_q) ||
        !make_map(&m[2], keys, dim, H, kv_rows, dim, ld_kv) || !make_map(&m[3], key_cache, rot, 1, cache_rows, rot, rot) ||
        !make_map(&m[4], values, vdim, H, kv_rows, vdim, ld_kv))
        return B2KV_ERR_UNSUPPORTED;
    Params p{static_cast<__nv_bfloat16*>(out), segments, dev_status, nullptr, ld_out, n_segments, n_blocks, H, 0, dim, rot, vdim,
             window, scale * 1.4426950408889634f, rows, kv_rows, static_cast<int>(cache_rows), 1};
    // heads whose keys and values together take about 32 MB, a quarter of L2, run next to each other
    const long long head_bytes = 2LL * kv_rows * (dim + vdim);
    p.group = static_cast<int>(std::min<long long>(H, std::max<long long>(1, (32LL << 20) / head_bytes)));
    const long long ctas = static_cast<long long>(n_blocks) * H;
    if (ctas > 0x7fffffffLL) return B2KV_ERR_UNSUPPORTED;
    if (dim <= 64) return vdim <= 64 ? launch<1, true, 1, false>(m, p, ctas, stream) : launch<1, true, 2, false>(m, p, ctas, stream);
    return vdim <= 64 ? launch<2, true, 1, false>(m, p, ctas, stream) : launch<2, true, 2, false>(m, p, ctas, stream);
}

extern "C" int b2kv_gqa_prefill_supported(int dim, int vdim, int dtype) {
    return dtype == B2KV_DTYPE_BF16 && dim > 0 && dim <= 128 && dim % 8 == 0 && vdim > 0 && vdim <= 128 && vdim % 8 == 0;
}

extern "C" int b2kv_gqa_prefill(const void* q, int64_t ld_q, const void* k_cache, const void* v_cache, int64_t cache_rows, void* out,
                                int64_t ld_out, const float* slopes, const b2kv_prompt_segment* segments, int n_segments,
                                int n_blocks, int rows, int H, int G, int dim, int vdim, float scale, int dtype,
                                int32_t* dev_status, void* stream) {
    using namespace latpre;
    if (!q || !k_cache || !v_cache || !out || !segments || n_segments <= 0 || n_blocks <= 0 || rows <= 0 || cache_rows <= 0 ||
        cache_rows > 0x7fffff00LL || H <= 0 || G <= 0 || H % G != 0)
        return B2KV_ERR_BAD_ARG;
    if (!b2kv_gqa_prefill_supported(dim, vdim, dtype) || !(scale > 0.f)) return B2KV_ERR_UNSUPPORTED;
    if (ld_q < static_cast<int64_t>(H) * dim || ld_out < static_cast<int64_t>(H) * vdim) return B2KV_ERR_BAD_ARG;
    if (!aligned16(q) || !aligned16(k_cache) || !aligned16(v_cache) || !aligned16(out) || ld_q % 8 || ld_out % 8) return B2KV_ERR_ALIGN;
    CUtensorMap m[5];
    if (!make_map(&m[0], q, dim, H, rows, dim, ld_q) ||
        !make_map(&m[2], k_cache, dim, G, cache_rows, dim, static_cast<int64_t>(G) * dim) ||
        !make_map(&m[4], v_cache, vdim, G, cache_rows, vdim, static_cast<int64_t>(G) * vdim))
        return B2KV_ERR_UNSUPPORTED;
    m[1] = m[0], m[3] = m[2];  // (no rotated parts: not used)
    const int per_kv = H / G;
    Params p{static_cast<__nv_bfloat16*>(out), segments, dev_status, slopes, ld_out, n_segments, n_blocks, H, 0, dim, 0, vdim,
             0, scale * 1.4426950408889634f, rows, static_cast<int>(cache_rows), static_cast<int>(cache_rows), per_kv};
    // heads whose keys and values of the step's own tokens take about 32 MB run next to each other
    const long long head_bytes = 2LL * rows * (dim + vdim);
    p.group = static_cast<int>(std::min<long long>(H, std::max<long long>(1, (32LL << 20) / head_bytes) * per_kv));
    const long long ctas = static_cast<long long>(n_blocks) * H;
    if (ctas > 0x7fffffffLL) return B2KV_ERR_UNSUPPORTED;
    auto go = [&](auto bias) {
        constexpr bool kBias = decltype(bias)::value;
        if (dim <= 64) return vdim <= 64 ? launch<1, false, 1, kBias>(m, p, ctas, stream) : launch<1, false, 2, kBias>(m, p, ctas, stream);
        return vdim <= 64 ? launch<2, false, 1, kBias>(m, p, ctas, stream) : launch<2, false, 2, kBias>(m, p, ctas, stream);
    };
    return slopes != nullptr ? go(std::true_type{}) : go(std::false_type{});
}
