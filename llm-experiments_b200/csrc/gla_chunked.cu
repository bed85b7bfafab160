// Gated linear attention over prompt portions, sixteen tokens at a time (bf16 rows, fp32 state).
//
// With P_t the product of the decays up to token t of a chunk and R_s the product behind token s (both per key channel, both at
// most one, so nothing can overflow however strong the decay), a chunk with incoming state S is
//
//   o_t  = S^T (q_t P_t) + sum_{s <= t} A_ts v_s,   A_ts = sum_d q_td k_sd prod_{s < r <= t} alpha_rd
//   S   <- diag(P_last) S + sum_s (k_s R_s) v_s^T
//
// One CTA per (head, segment) walks the chunks in order:
//   * four warps prepare a chunk (thread = key channel): q P and k R, and A, whose products of decays are carried along
//     exactly instead of being taken apart into factors that could overflow.  They run one chunk ahead, with the next chunk's rows
//     already on their way (TMA);
//   * every other warp owns 16 value columns of the state, transposed, as accumulators of mma.m16n8k16: the state never
//     leaves registers between the first and the last chunk.  As an A operand of the first product the accumulators need no
//     shuffle.  A step of the recurrence is sixteen tokens deep, one k-step of this instruction; larger tiles would have to
//     bring the state through tensor memory, decay it there and write it back as operands sixteen tokens at a time, a chain of
//     copies and waits several times as long as these products.
//   * fp32 operands (q P, k R, A and the state) are split into two bf16 halves, x = hi + lo, and lo * lo is dropped; v is
//     exact.  Accumulation, decay and state are fp32.
//   * o goes through shared memory so that the warps can take whole rows for the head's norm and the gate.
// Producer and consumer warps meet at hardware barriers whose arrivals are fixed by the number of chunks, which all warps know.
#include <algorithm>

#include "gla.cuh"

#include "tc_ptx.cuh"
#include "tma_map.cuh"

namespace b2kv {
namespace gla {
namespace {

constexpr int kChunk = 16;
constexpr int kPrep = 128;    // threads that prepare
constexpr int kSlab = 16;      // value columns per state warp
constexpr int kMaxWarps = 16;  // state warps
constexpr int kBox = 32;       // value columns per copy of v: two warps' slabs
constexpr int kPairs = kChunk * (kChunk + 1) / 2;  // entries of A on and below the diagonal
constexpr int kRing = 3;      // chunks of rows in shared memory
enum { kBarFull = 1, kBarEmpty = 3, kBarPrep = 5, kBarState = 6 };  // the first two: one for even and one for odd chunks

__device__ __forceinline__ void bar_sync(int id, int n) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(n) : "memory"); }
__device__ __forceinline__ void bar_arrive(int id, int n) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(n) : "memory"); }

__device__ __forceinline__ void tma_load_2d(void* dst, const CUtensorMap* map, uint64_t* bar, int x, int y) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
        ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(smem_u32(bar)), "r"(x), "r"(y)
        : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two fp32 numbers as bf16 pairs: the leading halves and what they leave.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = tc::pack_bf16(x, y);
    lo = tc::pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
}
// Entries of A in a fixed order, column after column from the diagonal down, as compile-time constants.
template <int kP>
struct Entry {
    static constexpr int column(int p) {
        int c = 0;
        for (; p >= kChunk - c; ++c) p -= kChunk - c;
        return c;
    }
    static constexpr int p = kP, c = column(kP), t = kP - (c * kChunk - c * (c - 1) / 2) + c;
};
template <int kP, typename F>
__device__ __forceinline__ void each_entry(F&& fn) {
    if constexpr (kP < kPairs) {
        fn(Entry<kP>{});
        each_entry<kP + 1>(fn);
    }
}
// Lane i gets the sum over the warp of everybody's v[i].
__device__ __forceinline__ float sum_by_lane(float (&v)[32], int lane) {
#pragma unroll
    for (int h = 16; h > 0; h >>= 1) {
        const bool up = lane & h;
#pragma unroll
        for (int i = 0; i < h; ++i) {
            const float mine = up ? v[i + h] : v[i], theirs = up ? v[i] : v[i + h];
            v[i] = mine + __shfl_xor_sync(0xffffffffu, theirs, h);
        }
    }
    return v[0];
}
__device__ __forceinline__ void split1(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}

// Shared memory for kD16 * 16 key channels; the arrays that depend on the value width come behind it.
template <int kD16>
struct Smem {
    static constexpr int kD = kD16 * 16;
    static constexpr int kLd = kD + 8;  // bf16 rows an odd number of 16-byte pieces apart: no bank conflicts in ldmatrix
    static constexpr int kLa = 24;
    struct Buffer {
        __nv_bfloat16 q_hi[kChunk][kLd], q_lo[kChunk][kLd], k_hi[kChunk][kLd], k_lo[kChunk][kLd];
        __nv_bfloat16 a_hi[kChunk][kLa], a_lo[kChunk][kLa];
        float decay[kD];
    };
    alignas(16) Buffer buf[2];
    float part[2][4][kPairs];
    alignas(16) float norm[kSlab * kMaxWarps];
    alignas(8) uint64_t full[kRing];
};

// One chunk's rows as TMA brings them, in bytes from the chunk's place in the ring: v in boxes of 32 columns (64-byte swizzle),
// gate, q and k rows side by side, decays.
struct RowPlan {
    int boxes, gate, q, k, alpha, bytes, stride;
    __host__ __device__ RowPlan(int dim, int vdim) {
        auto up = [](int n) { return (n + 127) / 128 * 128; };
        boxes = (vdim + kBox - 1) / kBox;
        gate = boxes * kChunk * kBox * 2;
        q = gate + up(kChunk * vdim * 2);
        k = q + up(kChunk * dim * 2);
        alpha = k + up(kChunk * dim * 2);
        stride = (alpha + up(kChunk * dim * 4) + 1023) / 1024 * 1024;
        bytes = kChunk * (boxes * kBox * 2 + vdim * 2 + 2 * dim * 2 + dim * 4);
    }
};

template <int kD16>
__global__ void __launch_bounds__(kPrep + 32 * kMaxWarps, 1) gla_chunk_kernel(
    const __grid_constant__ CUtensorMap tm_key, const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_gate,
    const __grid_constant__ CUtensorMap tm_alpha, const __grid_constant__ b2kv_gla_args a, int n_warps, int lanes_per_token,
    int32_t* dev_status) {
    extern __shared__ uint8_t smem_raw[];
    using S = Smem<kD16>;
    constexpr int kD = S::kD;
    const RowPlan plan(a.dim, a.vdim);
    const int ldo = kSlab * n_warps + 4;  // row pitch of o
    // (an offset, not a rounded pointer: the compiler has to see that all of this is shared memory)
    uint8_t* const ring = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    S& sm = *reinterpret_cast<S*>(ring + kRing * plan.stride);
    float* const s_o = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(&sm) + sizeof(S));  // [2][kChunk][ldo]
    const int n_threads = kPrep + 32 * n_warps;
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31;

    grid_launch_dependents();
    if (tid == 0) grid_dependency_wait();
    __syncthreads();
    b2kv_row_segment sg;
    if (!segment_place(a, blockIdx.y, sg)) {
        if (tid == 0) report_status(dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const int chunks = (sg.n + kChunk - 1) / kChunk;
    for (int i = tid; i < a.vdim; i += n_threads) sm.norm[i] = a.norm[i];
    if (tid == 0) {
        for (int i = 0; i < kRing; ++i) mbar_init(&sm.full[i], 1);
        fence_mbar_init();
    }
    __syncthreads();
    bool ok = true;  // a wait that ran out is reported at the end; the barriers' arrivals stay as they are

    if (tid < kPrep) {
        // ------------------------------ preparation ------------------------------
        auto request = [&](int ci) {
            const int slot = ci % kRing, row = sg.row0 + ci * kChunk;
            uint8_t* const dst = ring + slot * plan.stride;
            uint64_t* const bar = &sm.full[slot];
            mbar_arrive_expect_tx(bar, plan.bytes);
            tma_load_2d(dst + plan.alpha, &tm_alpha, bar, h * a.dim, row);
            tma_load_2d(dst + plan.q, &tm_key, bar, a.q_col + h * a.dim, row);
            tma_load_2d(dst + plan.k, &tm_key, bar, a.k_col + h * a.dim, row);
            for (int w = 0; w < plan.boxes; ++w)
                tma_load_2d(dst + w * kChunk * kBox * 2, &tm_v, bar, a.v_col + h * a.vdim + w * kBox, row);
            tma_load_2d(dst + plan.gate, &tm_gate, bar, a.g_col + h * a.vdim, row);
        };
        if (tid == 0) request(0);
        const int warp = tid >> 5;
        // A's entries in the order of the products below: column after column from the diagonal down
        auto entry = [](int p, int& t, int& c) {
            for (c = 0; p >= kChunk - c; ++c) p -= kChunk - c;
            t = c + p;
        };
        int t0, c0, t1, c1;
        entry(tid, t0, c0);
        entry(min(kPrep + tid, kPairs - 1), t1, c1);
        for (int i = tid; i < 2 * kChunk * S::kLa; i += kPrep) {  // what is above the diagonal stays zero
            (&sm.buf[i / (kChunk * S::kLa)].a_hi[0][0])[i % (kChunk * S::kLa)] = __nv_bfloat16(0.f);
            (&sm.buf[i / (kChunk * S::kLa)].a_lo[0][0])[i % (kChunk * S::kLa)] = __nv_bfloat16(0.f);
        }
        for (int ci = 0; ci < chunks; ++ci) {
            typename S::Buffer& b = sm.buf[ci & 1];
            const uint8_t* const rows = ring + ci % kRing * plan.stride;
            if (ci >= 2) bar_sync(kBarEmpty + (ci & 1), n_threads);
            if (tid == 0 && ci + 1 < chunks) request(ci + 1);  // in the place of chunk ci - 2
            ok = ok && mbar_wait(&sm.full[ci % kRing], (ci / kRing) & 1);
            if (tid < kD) {  // thread = key channel
                const int n = tid < a.dim ? min(kChunk, sg.n - ci * kChunk) : 0;  // tokens; what lies behind them is not theirs
                const float* const ra = reinterpret_cast<const float*>(rows + plan.alpha) + tid;
                const __nv_bfloat16* const rq = reinterpret_cast<const __nv_bfloat16*>(rows + plan.q) + tid;
                const __nv_bfloat16* const rk = reinterpret_cast<const __nv_bfloat16*>(rows + plan.k) + tid;
                // (loads in front of stores: the compiler cannot tell that they never meet)
                float al[kChunk], q[kChunk], k[kChunk], prod = 1.f;
#pragma unroll
                for (int t = 0; t < kChunk; ++t) {
                    al[t] = t < n ? ra[t * a.dim] : 1.f;
                    q[t] = t < n ? __bfloat162float(rq[t * a.dim]) * a.q_scale : 0.f;
                    k[t] = t < n ? __bfloat162float(rk[t * a.dim]) : 0.f;
                }
#pragma unroll
                for (int t = 0; t < kChunk; ++t) {
                    prod *= al[t];
                    split1(q[t] * prod, b.q_hi[t][tid], b.q_lo[t][tid]);
                }
                b.decay[tid] = prod;
                prod = 1.f;
#pragma unroll
                for (int t = kChunk - 1; t >= 0; --t) {
                    split1(k[t] * prod, b.k_hi[t][tid], b.k_lo[t][tid]);
                    prod *= al[t];
                }
                // This channel's part of every entry of A; 32 entries at a time are summed over the warp's channels, after
                // which lane i holds entry i.
                float v[32], w = 0.f;
                each_entry<0>([&](auto entry) {
                    constexpr int p = entry.p, t = entry.t, c = entry.c;
                    w = t == c ? k[c] : w * al[t];
                    v[p % 32] = q[t] * w;
                    if constexpr (p % 32 == 31) sm.part[ci & 1][warp][p - 31 + lane] = sum_by_lane(v, lane);
                });
#pragma unroll
                for (int i = kPairs % 32; i < 32; ++i) v[i] = 0.f;
                const float last = sum_by_lane(v, lane);
                if (lane < kPairs % 32) sm.part[ci & 1][warp][kPairs / 32 * 32 + lane] = last;
            }
            bar_sync(kBarPrep, kPrep);
            auto total = [&](int p) {
                float v = sm.part[ci & 1][0][p];
#pragma unroll
                for (int w = 1; w < kD / 32; ++w) v += sm.part[ci & 1][w][p];
                return v;
            };
            split1(total(tid), b.a_hi[t0][c0], b.a_lo[t0][c0]);
            if (tid < kPairs - kPrep) split1(total(kPrep + tid), b.a_hi[t1][c1], b.a_lo[t1][c1]);
            bar_arrive(kBarFull + (ci & 1), n_threads);
        }
        if (!ok) report_status(dev_status, B2KV_DEV_WAIT_TIMEOUT);
        return;
    }

    // ------------------------------ state: 16 value columns per warp ------------------------------
    const int w = (tid - kPrep) >> 5;
    const int row = lane >> 2, col = (lane & 3) * 2;  // place of this thread's first accumulator in a tile
    float* const state = a.state + (static_cast<int64_t>(sg.slot) * a.H + h) * a.dim * a.vdim;
    const bool fresh = a.row_pos[sg.row0] == 0;
    float c[2 * kD16][4];  // [tile of 8 key channels]
    auto each_state = [&](auto&& fn) {
#pragma unroll
        for (int j = 0; j < 2 * kD16; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int v = w * kSlab + row + (e >> 1) * 8, d = j * 8 + col + (e & 1);
                fn(c[j][e], static_cast<int64_t>(d) * a.vdim + v, v < a.vdim && d < a.dim);
            }
    };
    each_state([&](float& x, int64_t at, bool live) { x = live && !fresh ? state[at] : 0.f; });

    const int mat = lane >> 3, r8 = lane & 7;
    // ldmatrix row addresses: [token][channel] tiles as they lie (tokens 0-7 | 8-15 outermost), and transposed
    const int plain_t = r8 + 8 * (mat >> 1), plain_c = 8 * (mat & 1);
    const int trans_t = r8 + 8 * (mat & 1), trans_c = 8 * (mat >> 1);
    const float inv_vdim = 1.0f / static_cast<float>(a.vdim);
    const int group = lane / lanes_per_token, sub = lane % lanes_per_token, groups = 32 / lanes_per_token;
    for (int ci = 0; ci < chunks; ++ci) {
        typename S::Buffer& b = sm.buf[ci & 1];
        const uint8_t* const rows = ring + ci % kRing * plan.stride;
        bar_sync(kBarFull + (ci & 1), n_threads);
        ok = ok && mbar_wait(&sm.full[ci % kRing], (ci / kRing) & 1);  // (complete: the other warps have waited for it)
        // this warp's half of a box of v: rows of 64 bytes, 16-byte pieces exchanged by row
        const uint32_t v_addr = smem_u32(rows + (w >> 1) * kChunk * kBox * 2 + plain_t * 64) +
                                (((2 * (w & 1) + (plain_c >> 3)) ^ ((plain_t >> 1) & 3)) << 4);
        // (operands share registers: with 64 of the state there are few to spare)
        uint32_t f[4], x[4];
        float o[2][4];
        ldsm4t(f, v_addr);
        ldsm4(x, smem_u32(&b.a_hi[plain_t][plain_c]));
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
            mma16816(o[n], f, x[2 * n], x[2 * n + 1]);
        }
        ldsm4(x, smem_u32(&b.a_lo[plain_t][plain_c]));
#pragma unroll
        for (int n = 0; n < 2; ++n) mma16816(o[n], f, x[2 * n], x[2 * n + 1]);
#pragma unroll
        for (int kk = 0; kk < kD16; ++kk) {
            uint32_t s_hi[4], s_lo[4];
            ldsm4(x, smem_u32(&b.q_hi[plain_t][kk * 16 + plain_c]));
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float(&t)[4] = c[2 * kk + (e >> 1)];
                split2(t[2 * (e & 1)], t[2 * (e & 1) + 1], s_hi[e], s_lo[e]);
            }
#pragma unroll
            for (int n = 0; n < 2; ++n) mma16816(o[n], s_hi, x[2 * n], x[2 * n + 1]);
#pragma unroll
            for (int n = 0; n < 2; ++n) mma16816(o[n], s_lo, x[2 * n], x[2 * n + 1]);
            ldsm4(x, smem_u32(&b.q_lo[plain_t][kk * 16 + plain_c]));
#pragma unroll
            for (int n = 0; n < 2; ++n) mma16816(o[n], s_hi, x[2 * n], x[2 * n + 1]);
        }
        float* const so = s_o + (ci & 1) * kChunk * ldo;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) so[(n * 8 + col + (e & 1)) * ldo + w * kSlab + row + (e >> 1) * 8] = o[n][e];
        ldsm4t(f, v_addr);
#pragma unroll
        for (int kk = 0; kk < kD16; ++kk) {
            ldsm4t(x, smem_u32(&b.k_hi[trans_t][kk * 16 + trans_c]));
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float2 d = *reinterpret_cast<const float2*>(&b.decay[(2 * kk + u) * 8 + col]);
                float(&t)[4] = c[2 * kk + u];
                t[0] *= d.x, t[1] *= d.y, t[2] *= d.x, t[3] *= d.y;
                mma16816(t, f, x[2 * u], x[2 * u + 1]);
            }
            ldsm4t(x, smem_u32(&b.k_lo[trans_t][kk * 16 + trans_c]));
#pragma unroll
            for (int u = 0; u < 2; ++u) mma16816(c[2 * kk + u], f, x[2 * u], x[2 * u + 1]);
        }
        bar_sync(kBarState, 32 * n_warps);
        // whole rows of o: lanes_per_token lanes with eight values each
        for (int t0 = w * groups; t0 < kChunk; t0 += n_warps * groups) {
            const int t = t0 + group;
            const bool mine = sub * 8 < a.vdim && t < kChunk && ci * kChunk + t < sg.n;
            const float* const src = so + t * ldo + sub * 8;
            float sum = 0.f;
            if (mine) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const float4 x = *reinterpret_cast<const float4*>(src + half * 4);
                    sum = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, fmaf(x.w, x.w, sum))));
                }
            }
            for (int off = lanes_per_token / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
            if (mine) {
                const float scale = rsqrtf(fmaf(sum, inv_vdim, a.eps));
                const uint8_t* const gate = rows + plan.gate + (t * a.vdim + sub * 8) * 2;
                __nv_bfloat16* const dst = static_cast<__nv_bfloat16*>(a.out) + (static_cast<int64_t>(sg.row0) + ci * kChunk + t) * a.ld_out +
                                           static_cast<int64_t>(h) * a.vdim + sub * 8;
#pragma unroll 1
                for (int half = 0; half < 2; ++half) {  // (four values at a time, for the registers' sake)
                    const float4 x = *reinterpret_cast<const float4*>(src + half * 4);
                    const float4 n = *reinterpret_cast<const float4*>(&sm.norm[sub * 8 + half * 4]);
                    const uint2 g = *reinterpret_cast<const uint2*>(gate + half * 8);
                    uint2 out;
                    out.x = tc::pack_bf16(x.x * scale * n.x * silu_fast(__uint_as_float(g.x << 16)),
                                          x.y * scale * n.y * silu_fast(__uint_as_float(g.x & 0xffff0000u)));
                    out.y = tc::pack_bf16(x.z * scale * n.z * silu_fast(__uint_as_float(g.y << 16)),
                                          x.w * scale * n.w * silu_fast(__uint_as_float(g.y & 0xffff0000u)));
                    *reinterpret_cast<uint2*>(dst + half * 4) = out;
                }
            }
        }
        if (ci + 2 < chunks) bar_arrive(kBarEmpty + (ci & 1), n_threads);
    }
    each_state([&](float& x, int64_t at, bool live) {
        if (live) state[at] = x;
    });
    if (!ok) report_status(dev_status, B2KV_DEV_WAIT_TIMEOUT);
}

// Row-major matrix, boxes of kChunk rows.
bool make_map(CUtensorMap* map, CUtensorMapDataType type, int es, const void* base, int64_t rows, int64_t cols, int64_t pitch, int box,
              CUtensorMapSwizzle swizzle) {
    EncodeTiledFn fn = tensor_map_encoder();
    if (fn == nullptr) return false;
    const cuuint64_t dims[2] = {static_cast<cuuint64_t>(cols), static_cast<cuuint64_t>(rows)};
    const cuuint64_t strides[1] = {static_cast<cuuint64_t>(pitch) * es};
    const cuuint32_t boxes[2] = {static_cast<cuuint32_t>(box), kChunk};
    const cuuint32_t estr[2] = {1, 1};
    return fn(map, type, 2, const_cast<void*>(base), dims, strides, boxes, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, swizzle,
              CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int kD16>
int launch_chunked(const b2kv_gla_args& a, int n_warps, int32_t* dev_status, void* stream) {
    const RowPlan plan(a.dim, a.vdim);
    const size_t smem = 1024 + kRing * plan.stride + sizeof(Smem<kD16>) + 2 * kChunk * (kSlab * n_warps + 4) * sizeof(float);
    CUtensorMap tk, tv, tg, ta;
    const int64_t keys = static_cast<int64_t>(a.H) * a.dim, values = static_cast<int64_t>(a.H) * a.vdim;
    const int64_t cols = std::max(std::max(a.q_col, a.k_col) + keys, std::max(a.v_col, a.g_col) + values);
    const auto bf16 = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
    if (!make_map(&tk, bf16, 2, a.y, a.rows, cols, a.ld_y, a.dim, CU_TENSOR_MAP_SWIZZLE_NONE) ||
        !make_map(&tv, bf16, 2, a.y, a.rows, cols, a.ld_y, kBox, CU_TENSOR_MAP_SWIZZLE_64B) ||
        !make_map(&tg, bf16, 2, a.y, a.rows, cols, a.ld_y, a.vdim, CU_TENSOR_MAP_SWIZZLE_NONE) ||
        !make_map(&ta, CU_TENSOR_MAP_DATA_TYPE_FLOAT32, 4, a.alpha, a.rows, keys, a.ld_alpha, a.dim, CU_TENSOR_MAP_SWIZZLE_NONE))
        return B2KV_ERR_UNSUPPORTED;
    static int configured[64] = {0};
    int dev = 0;
    B2KV_CUDA_TRY(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64) return B2KV_ERR_UNSUPPORTED;
    auto kernel = gla_chunk_kernel<kD16>;
    if (configured[dev] < static_cast<int>(smem)) {
        B2KV_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        configured[dev] = static_cast<int>(smem);
    }
    int lanes = 4;  // lanes per row of o, eight values each: a power of two
    while (lanes * 8 < a.vdim) lanes *= 2;
    OverlapLaunch launch(dim3(a.H, a.n_segments), kPrep + 32 * n_warps, smem, stream);
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, kernel, tk, tv, tg, ta, a, n_warps, lanes, dev_status));
    return B2KV_OK;
}

}  // namespace
}  // namespace gla

int gla_chunked(const b2kv_gla_args& a, int32_t* dev_status, void* stream) {
    using namespace gla;
    if (a.dtype != B2KV_DTYPE_BF16 || a.dim % 8 != 0 || a.dim > 128 || a.vdim % 8 != 0 || a.vdim > kSlab * kMaxWarps || a.n_segments > 65535)
        return B2KV_ERR_UNSUPPORTED;
    // 16-byte pieces of v, gate and output rows
    if (!aligned16(a.y) || !aligned16(a.out) || a.ld_y % 8 || a.ld_out % 8 || a.v_col % 8 || a.g_col % 8 || a.q_col % 8 || a.k_col % 8)
        return B2KV_ERR_UNSUPPORTED;
    if (!aligned16(a.alpha) || a.ld_alpha % 4) return B2KV_ERR_UNSUPPORTED;
    const int n_warps = (a.vdim + kSlab - 1) / kSlab;
    if (a.dim <= 32) return launch_chunked<2>(a, n_warps, dev_status, stream);
    if (a.dim <= 64) return launch_chunked<4>(a, n_warps, dev_status, stream);
    return launch_chunked<8>(a, n_warps, dev_status, stream);
}

}  // namespace b2kv
