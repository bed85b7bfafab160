// Gated linear attention over prompt portions, sixteen tokens at a time (bf16 rows, fp32 state).
//
// With P_t the product of the decays up to token t of a chunk and R_s the product behind token s (both per key channel, both at
// most one, so nothing can overflow however strong the decay), a chunk with incoming state S is
//
//   o_t  = S^T (q_t P_t) + sum_{s <= t} A_ts v_s,   A_ts = sum_d q_td k_sd prod_{s < r <= t} alpha_rd
//   S   <- diag(P_last) S + sum_s (k_s R_s) v_s^T
//
// Two kernels.  What does not depend on the state is made for many chunks at once (gla_prepare_kernel): one CTA per chunk and
// head, thread = two key channels; A's products of decays are carried along exactly instead of being taken apart into factors that
// could overflow, and its entries are summed over the channels 32 at a time.  The result is a record per chunk and head that is
// byte for byte what the second kernel wants in shared memory.  Records are made a slice of the segments at a time, small enough
// to stay in L2.
//
// gla_state_kernel has one CTA per (head, segment) and walks the chunks in order:
//   * every warp owns 16 value columns of the state, transposed, as accumulators of mma.m16n8k16: the state never
//     leaves registers between the first and the last chunk.  As an A operand of the first product the accumulators need no
//     shuffle.  A step of the recurrence is sixteen tokens deep, one k-step of this instruction; larger tiles would have to
//     bring the state through tensor memory, decay it there and write it back as operands sixteen tokens at a time, a chain of
//     copies and waits several times as long as these products.
//   * fp32 operands (q P, k R, A and the state) are split into two bf16 halves, x = hi + lo, and lo * lo is dropped; v is
//     exact.  Accumulation, decay and state are fp32.
//   * o goes through shared memory so that the warps can take whole rows for the head's norm and the gate.
//   * copies run ahead through a ring: records with one bulk copy each, rows of v and gate with TMA.  A thread of the first warp
//     asks for them when everybody has left the chunk before (a warp of its own would take registers from all others).
// Every wait is bounded; a thread whose wait ran out goes on without waiting (so that nobody is left at a barrier) and reports.
#include <algorithm>

#include "gla.cuh"
#include "tc_ptx.cuh"
#include "tma_map.cuh"

namespace b2kv {
namespace gla {
namespace {

constexpr int kChunk = 16;
constexpr int kPairs = kChunk * (kChunk + 1) / 2;  // entries of A on and below the diagonal
constexpr int kSlab = 16;                          // value columns per state warp
constexpr int kMaxWarps = 16;                      // state warps
constexpr int kBox = 32;                           // value columns per copy of v: two warps' slabs
constexpr int kMaxRing = 6;
constexpr int kSmemLimit = 220 * 1024;
constexpr size_t kSliceBytes = 64u << 20;  // records of a slice, at most (but at least kMinSlice chunks per segment)
constexpr int kMinSlice = 8;

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
__device__ __forceinline__ void split1(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(x);
    lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}

// What a chunk brings to a head beside v, for kD16 * 16 key channels.
template <int kD16>
struct alignas(128) Record {
    static constexpr int kD = kD16 * 16;
    static constexpr int kLd = kD + 8;  // bf16 rows an odd number of 16-byte pieces apart: no bank conflicts in ldmatrix
    static constexpr int kLa = 24;
    __nv_bfloat16 q_hi[kChunk][kLd], q_lo[kChunk][kLd], k_hi[kChunk][kLd], k_lo[kChunk][kLd];  // q P, k R
    __nv_bfloat16 a_hi[kChunk][kLa], a_lo[kChunk][kLa];
    float decay[kD];  // P_last
};

// Chunks [first, first + count) of every segment; record (segment, head, chunk) at ((segment * H + head) * count + chunk - first).
struct Slice {
    int first, count;
};

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

template <int kD16>
__global__ void __launch_bounds__(kD16 <= 4 ? 32 : 8 * kD16) gla_prepare_kernel(const __grid_constant__ b2kv_gla_args a, const Slice slice,
                                                                               int32_t* dev_status) {
    using R = Record<kD16>;
    constexpr int kD = R::kD, kThreads = kD16 <= 4 ? 32 : 8 * kD16, kWarps = kThreads / 32;
    __shared__ R out;
    __shared__ float part[kWarps][kPairs];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, d = 2 * tid;
    grid_launch_dependents();
    if (tid == 0) grid_dependency_wait();
    __syncthreads();
    b2kv_row_segment sg;
    if (!segment_place(a, blockIdx.z, sg)) {
        if (tid == 0) report_status(dev_status, B2KV_DEV_BAD_POSITION);
        return;
    }
    const int first = (slice.first + static_cast<int>(blockIdx.x)) * kChunk;
    if (sg.n <= first) return;
    const int n = d < a.dim ? min(kChunk, sg.n - first) : 0;  // tokens of this chunk (none in channels that are padding)
    const int64_t row = sg.row0 + first;
    const float* const ra = a.alpha + row * a.ld_alpha + h * a.dim + d;
    const __nv_bfloat16* const y = static_cast<const __nv_bfloat16*>(a.y) + row * a.ld_y + h * a.dim + d;
    float2 al[kChunk], q[kChunk], k[kChunk], prod = make_float2(1.f, 1.f);
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
        al[t] = t < n ? *reinterpret_cast<const float2*>(ra + t * a.ld_alpha) : make_float2(1.f, 1.f);
        const uint32_t qb = t < n ? *reinterpret_cast<const uint32_t*>(y + t * a.ld_y + a.q_col) : 0u;
        const uint32_t kb = t < n ? *reinterpret_cast<const uint32_t*>(y + t * a.ld_y + a.k_col) : 0u;
        q[t] = make_float2(__uint_as_float(qb << 16) * a.q_scale, __uint_as_float(qb & 0xffff0000u) * a.q_scale);
        k[t] = make_float2(__uint_as_float(kb << 16), __uint_as_float(kb & 0xffff0000u));
    }
    if (d < kD) {
        auto store = [&](__nv_bfloat16* hi_at, __nv_bfloat16* lo_at, float2 v) {
            uint32_t hi, lo;
            split2(v.x, v.y, hi, lo);
            *reinterpret_cast<uint32_t*>(hi_at) = hi;
            *reinterpret_cast<uint32_t*>(lo_at) = lo;
        };
#pragma unroll
        for (int t = 0; t < kChunk; ++t) {
            prod = __fmul2_rn(prod, al[t]);
            store(&out.q_hi[t][d], &out.q_lo[t][d], __fmul2_rn(q[t], prod));
        }
        *reinterpret_cast<float2*>(&out.decay[d]) = prod;
        prod = make_float2(1.f, 1.f);
#pragma unroll
        for (int t = kChunk - 1; t >= 0; --t) {
            store(&out.k_hi[t][d], &out.k_lo[t][d], __fmul2_rn(k[t], prod));
            prod = __fmul2_rn(prod, al[t]);
        }
    }
    // these channels' part of every entry of A; 32 entries at a time are summed over the warp's channels
    float v[32];
    float2 w = make_float2(0.f, 0.f);
    each_entry<0>([&](auto entry) {
        constexpr int p = entry.p, t = entry.t, c = entry.c;
        w = t == c ? k[c] : __fmul2_rn(w, al[t]);
        const float2 z = __fmul2_rn(q[t], w);
        v[p % 32] = z.x + z.y;
        if constexpr (p % 32 == 31) part[warp][p - 31 + lane] = sum_by_lane(v, lane);
    });
#pragma unroll
    for (int i = kPairs % 32; i < 32; ++i) v[i] = 0.f;
    const float last = sum_by_lane(v, lane);
    if (lane < kPairs % 32) part[warp][kPairs / 32 * 32 + lane] = last;
    __syncthreads();
    for (int e = tid; e < kChunk * kChunk; e += kThreads) {
        const int t = e / kChunk, c = e % kChunk;
        float sum = 0.f;
        if (c <= t) {
            const int p = c * kChunk - c * (c - 1) / 2 + t - c;
#pragma unroll
            for (int i = 0; i < kWarps; ++i) sum += part[i][p];
        }
        split1(sum, out.a_hi[t][c], out.a_lo[t][c]);
    }
    __syncthreads();
    uint4* const dst = reinterpret_cast<uint4*>(reinterpret_cast<R*>(a.workspace) +
                                                (static_cast<int64_t>(blockIdx.z) * a.H + h) * slice.count + blockIdx.x);
    for (int i = tid; i < static_cast<int>(sizeof(R) / 16); i += kThreads) dst[i] = reinterpret_cast<const uint4*>(&out)[i];
}

// One place of the ring: the record, then v in boxes of 32 columns (64-byte swizzle), then the gate's rows.
struct RowPlan {
    int boxes, v, gate, stride, bytes;
    __host__ __device__ RowPlan(int record, int vdim) {
        boxes = (vdim + kBox - 1) / kBox;
        v = (record + 1023) / 1024 * 1024;
        gate = v + boxes * kChunk * kBox * 2;
        stride = (gate + kChunk * vdim * 2 + 1023) / 1024 * 1024;
        bytes = record + kChunk * (boxes * kBox + vdim) * 2;
    }
};

struct Shared {
    alignas(16) float norm[kSlab * kMaxWarps];
    alignas(8) uint64_t full[kMaxRing];
    uint64_t o_ready[2];  // o of an even / odd chunk is in shared memory: one arrival per warp
};

template <int kD16>
__global__ void __launch_bounds__(32 * kMaxWarps, 1) gla_state_kernel(
    const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_gate, const __grid_constant__ b2kv_gla_args a,
    const Slice slice, int n_warps, int n_ring, int lanes_per_token, int32_t* dev_status) {
    extern __shared__ uint8_t smem_raw[];
    __shared__ Shared sm;
    using R = Record<kD16>;
    const RowPlan plan(sizeof(R), a.vdim);
    const int ldo = kSlab * n_warps + 4;  // row pitch of o
    // (an offset, not a rounded pointer: the compiler has to see that all of this is shared memory)
    uint8_t* const ring = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
    float* const s_o = reinterpret_cast<float*>(ring + n_ring * plan.stride);  // [2][kChunk][ldo]
    const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;

    grid_launch_dependents();
    if (tid == 0) grid_dependency_wait();
    __syncthreads();
    b2kv_row_segment sg;
    if (!segment_place(a, blockIdx.y, sg)) return;  // (reported by the other kernel)
    const int chunks = min((sg.n + kChunk - 1) / kChunk - slice.first, slice.count);
    if (chunks <= 0) return;
    for (int i = tid; i < a.vdim; i += blockDim.x) sm.norm[i] = a.norm[i];
    if (tid == 0) {
        for (int i = 0; i < kMaxRing; ++i) mbar_init(&sm.full[i], 1);
        for (int i = 0; i < 2; ++i) mbar_init(&sm.o_ready[i], n_warps);
        fence_mbar_init();
    }
    __syncthreads();
    bool ok = true;
    const int row0 = sg.row0 + slice.first * kChunk, rows_left = sg.n - slice.first * kChunk;

    const R* const records = reinterpret_cast<const R*>(a.workspace) + (static_cast<int64_t>(blockIdx.y) * a.H + h) * slice.count;
    auto request = [&](int ci, int slot) {
        uint8_t* const dst = ring + slot * plan.stride;
        uint64_t* const bar = &sm.full[slot];
        mbar_arrive_expect_tx(bar, plan.bytes);
        bulk_g2s(dst, records + ci, sizeof(R), bar);
        for (int b = 0; b < plan.boxes; ++b)
            tma_load_2d(dst + plan.v + b * kChunk * kBox * 2, &tm_v, bar, a.v_col + h * a.vdim + b * kBox, row0 + ci * kChunk);
        tma_load_2d(dst + plan.gate, &tm_gate, bar, a.g_col + h * a.vdim, row0 + ci * kChunk);
    };
    if (tid == 0)
        for (int i = 0; i < min(n_ring, chunks); ++i) request(i, i);

    // ------------------------------ state: 16 value columns per warp ------------------------------
    const int row = lane >> 2, col = (lane & 3) * 2;  // place of this thread's first accumulator in a tile
    float* const state = a.state + (static_cast<int64_t>(sg.slot) * a.H + h) * a.dim * a.vdim;
    const bool fresh = slice.first == 0 && a.row_pos[sg.row0] == 0;
    float c[2 * kD16][4];  // [tile of 8 key channels]
    auto each_state = [&](auto&& fn) {
#pragma unroll
        for (int j = 0; j < 2 * kD16; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int v = warp * kSlab + row + (e >> 1) * 8, d = j * 8 + col + (e & 1);
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
    int slot = 0;
    uint32_t phase = 0;
    for (int ci = 0; ci < chunks; ++ci) {
        const uint8_t* const place = ring + slot * plan.stride;
        const R& b = *reinterpret_cast<const R*>(place);
        ok = ok && mbar_wait(&sm.full[slot], phase);
        // this warp's half of a box of v: rows of 64 bytes, 16-byte pieces exchanged by row
        const uint32_t v_addr = smem_u32(place + plan.v + (warp >> 1) * kChunk * kBox * 2 + plain_t * 64) +
                                (((2 * (warp & 1) + (plain_c >> 3)) ^ ((plain_t >> 1) & 3)) << 4);
        const uint32_t q_addr = smem_u32(&b.q_hi[plain_t][plain_c]), k_addr = smem_u32(&b.k_hi[trans_t][trans_c]);
        constexpr uint32_t kLo = sizeof(b.q_hi);  // from a matrix of leading halves to that of what they leave
        uint32_t vf[4], x[2][4], z[2][4];
        float o[2][4];
        ldsm4t(vf, v_addr);
        {
            ldsm4(x[1], smem_u32(&b.a_hi[plain_t][plain_c]));
            ldsm4(z[1], smem_u32(&b.a_lo[plain_t][plain_c]));
            ldsm4(x[0], q_addr);
            ldsm4(z[0], q_addr + kLo);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
                mma16816(o[n], vf, x[1][2 * n], x[1][2 * n + 1]);
            }
#pragma unroll
            for (int n = 0; n < 2; ++n) mma16816(o[n], vf, z[1][2 * n], z[1][2 * n + 1]);
        }
#pragma unroll
        for (int kk = 0; kk < kD16; ++kk) {
            if (kk + 1 < kD16) {  // the next step's operands are on their way during this one's products
                ldsm4(x[(kk + 1) & 1], q_addr + (kk + 1) * 32);
                ldsm4(z[(kk + 1) & 1], q_addr + kLo + (kk + 1) * 32);
            }
            uint32_t s_hi[4], s_lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float(&t)[4] = c[2 * kk + (e >> 1)];
                split2(t[2 * (e & 1)], t[2 * (e & 1) + 1], s_hi[e], s_lo[e]);
            }
            const uint32_t(&hi)[4] = x[kk & 1], (&lo)[4] = z[kk & 1];
#pragma unroll
            for (int n = 0; n < 2; ++n) mma16816(o[n], s_hi, hi[2 * n], hi[2 * n + 1]);
#pragma unroll
            for (int n = 0; n < 2; ++n) mma16816(o[n], s_hi, lo[2 * n], lo[2 * n + 1]);
#pragma unroll
            for (int n = 0; n < 2; ++n) mma16816(o[n], s_lo, hi[2 * n], hi[2 * n + 1]);
        }
        ldsm4t(x[0], k_addr);
        ldsm4t(z[0], k_addr + kLo);
        float* const so = s_o + (ci & 1) * kChunk * ldo;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) so[(n * 8 + col + (e & 1)) * ldo + warp * kSlab + row + (e >> 1) * 8] = o[n][e];
        __syncwarp();
        if (lane == 0) mbar_arrive(&sm.o_ready[ci & 1]);
#pragma unroll
        for (int kk = 0; kk < kD16; ++kk) {
            if (kk + 1 < kD16) {
                ldsm4t(x[(kk + 1) & 1], k_addr + (kk + 1) * 32);
                ldsm4t(z[(kk + 1) & 1], k_addr + kLo + (kk + 1) * 32);
            }
            const uint32_t(&hi)[4] = x[kk & 1], (&lo)[4] = z[kk & 1];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float2 d = *reinterpret_cast<const float2*>(&b.decay[(2 * kk + u) * 8 + col]);
                float(&t)[4] = c[2 * kk + u];
                t[0] *= d.x, t[1] *= d.y, t[2] *= d.x, t[3] *= d.y;
                mma16816(t, vf, hi[2 * u], hi[2 * u + 1]);
            }
#pragma unroll
            for (int u = 0; u < 2; ++u) mma16816(c[2 * kk + u], vf, lo[2 * u], lo[2 * u + 1]);
        }
        // All warps have stored their part of o, so they have left the chunk before: its place in the ring is free, and so is the
        // other buffer of o.  Nobody waits for the others' updates here: the warps drift apart and keep the tensor pipe busy.
        ok = ok && mbar_wait(&sm.o_ready[ci & 1], (ci >> 1) & 1);
        __syncwarp();
        if (tid == 0 && ci > 0 && ci - 1 + n_ring < chunks) request(ci - 1 + n_ring, slot == 0 ? n_ring - 1 : slot - 1);
        // whole rows of o: lanes_per_token lanes with eight values each
        for (int t0 = warp * groups; t0 < kChunk; t0 += n_warps * groups) {
            const int t = t0 + group;
            const bool mine = sub * 8 < a.vdim && t < kChunk && ci * kChunk + t < rows_left;
            const float* const src = so + t * ldo + sub * 8;
            float sum = 0.f;
            if (mine) {
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const float4 f = *reinterpret_cast<const float4*>(src + half * 4);
                    sum = fmaf(f.x, f.x, fmaf(f.y, f.y, fmaf(f.z, f.z, fmaf(f.w, f.w, sum))));
                }
            }
            for (int off = lanes_per_token / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
            if (mine) {
                const float scale = rsqrtf(fmaf(sum, inv_vdim, a.eps));
                const uint8_t* const gate = place + plan.gate + (t * a.vdim + sub * 8) * 2;
                __nv_bfloat16* const dst = static_cast<__nv_bfloat16*>(a.out) + (static_cast<int64_t>(row0) + ci * kChunk + t) * a.ld_out +
                                           static_cast<int64_t>(h) * a.vdim + sub * 8;
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const float4 f = *reinterpret_cast<const float4*>(src + half * 4);
                    const float4 n = *reinterpret_cast<const float4*>(&sm.norm[sub * 8 + half * 4]);
                    const uint2 g = *reinterpret_cast<const uint2*>(gate + half * 8);
                    uint2 out;
                    out.x = tc::pack_bf16(f.x * scale * n.x * silu_fast(__uint_as_float(g.x << 16)),
                                          f.y * scale * n.y * silu_fast(__uint_as_float(g.x & 0xffff0000u)));
                    out.y = tc::pack_bf16(f.z * scale * n.z * silu_fast(__uint_as_float(g.y << 16)),
                                          f.w * scale * n.w * silu_fast(__uint_as_float(g.y & 0xffff0000u)));
                    *reinterpret_cast<uint2*>(dst + half * 4) = out;
                }
            }
        }
        if (++slot == n_ring) slot = 0, phase ^= 1;
    }
    each_state([&](float& x, int64_t at, bool live) {
        if (live) state[at] = x;
    });
    if (!ok) {
        // (whoever asked for copies sees to it that they have landed before this memory is given up)
        if (tid == 0)
            for (int i = max(0, chunks - n_ring); i < chunks; ++i) mbar_wait(&sm.full[i % n_ring], (i / n_ring) & 1);
        report_status(dev_status, B2KV_DEV_WAIT_TIMEOUT);
    }
}

// Row-major bf16 matrix, boxes of kChunk rows.
bool make_map(CUtensorMap* map, const void* base, int64_t rows, int64_t cols, int64_t pitch, int box, CUtensorMapSwizzle swizzle) {
    EncodeTiledFn fn = tensor_map_encoder();
    if (fn == nullptr) return false;
    const cuuint64_t dims[2] = {static_cast<cuuint64_t>(cols), static_cast<cuuint64_t>(rows)};
    const cuuint64_t strides[1] = {static_cast<cuuint64_t>(pitch) * 2};
    const cuuint32_t boxes[2] = {static_cast<cuuint32_t>(box), kChunk};
    const cuuint32_t estr[2] = {1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, boxes, estr,
              CU_TENSOR_MAP_INTERLEAVE_NONE, swizzle, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

int record_bytes(int dim) {
    return static_cast<int>(dim <= 32 ? sizeof(Record<2>) : (dim <= 64 ? sizeof(Record<4>) : sizeof(Record<8>)));
}

int slice_chunks(int H, int dim, int n_segments, int max_n) {
    const int chunks = (max_n + kChunk - 1) / kChunk;
    const size_t per_chunk = static_cast<size_t>(record_bytes(dim)) * H * n_segments;
    const int fit = static_cast<int>(std::min<size_t>(kSliceBytes / per_chunk, 1u << 20));
    return std::min(chunks, std::max(kMinSlice, fit));
}

template <int kD16>
int launch_chunked(const b2kv_gla_args& a, int32_t* dev_status, void* stream) {
    const int n_warps = (a.vdim + kSlab - 1) / kSlab;
    const RowPlan plan(sizeof(Record<kD16>), a.vdim);
    const int fixed = 1024 + 2 * kChunk * (kSlab * n_warps + 4) * static_cast<int>(sizeof(float));
    const int n_ring = std::min(kMaxRing, (kSmemLimit - fixed) / plan.stride);
    const size_t smem = fixed + static_cast<size_t>(n_ring) * plan.stride;
    CUtensorMap tv, tg;
    const int64_t cols = std::max(a.v_col, a.g_col) + static_cast<int64_t>(a.H) * a.vdim;
    if (!make_map(&tv, a.y, a.rows, cols, a.ld_y, kBox, CU_TENSOR_MAP_SWIZZLE_64B) ||
        !make_map(&tg, a.y, a.rows, cols, a.ld_y, a.vdim, CU_TENSOR_MAP_SWIZZLE_NONE))
        return B2KV_ERR_UNSUPPORTED;
    static int configured[64] = {0};
    int dev = 0;
    B2KV_CUDA_TRY(cudaGetDevice(&dev));
    if (dev < 0 || dev >= 64) return B2KV_ERR_UNSUPPORTED;
    auto kernel = gla_state_kernel<kD16>;
    if (configured[dev] < static_cast<int>(smem)) {
        B2KV_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
        configured[dev] = static_cast<int>(smem);
    }
    int lanes = 2;  // lanes per row of o, eight values each: a power of two
    while (lanes * 8 < a.vdim) lanes *= 2;
    const int chunks = (a.max_n + kChunk - 1) / kChunk;
    Slice slice{0, slice_chunks(a.H, a.dim, a.n_segments, a.max_n)};
    for (; slice.first < chunks; slice.first += slice.count) {
        const unsigned here = static_cast<unsigned>(std::min(slice.count, chunks - slice.first));
        OverlapLaunch prep(dim3(here, a.H, a.n_segments), kD16 <= 4 ? 32 : 8 * kD16, 0, stream);
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&prep.cfg, gla_prepare_kernel<kD16>, a, slice, dev_status));
        OverlapLaunch walk(dim3(a.H, a.n_segments), 32 * n_warps, smem, stream);
        B2KV_CUDA_TRY(cudaLaunchKernelEx(&walk.cfg, kernel, tv, tg, a, slice, n_warps, n_ring, lanes, dev_status));
    }
    return B2KV_OK;
}

bool chunked_sizes(int dim, int vdim, int dtype) {
    return dtype == B2KV_DTYPE_BF16 && dim > 0 && dim % 8 == 0 && dim <= 128 && vdim > 0 && vdim % 8 == 0 && vdim <= kSlab * kMaxWarps;
}

}  // namespace
}  // namespace gla

size_t gla_chunked_workspace(int H, int dim, int vdim, int n_segments, int max_n, int dtype) {
    if (!gla::chunked_sizes(dim, vdim, dtype)) return 0;
    return static_cast<size_t>(gla::slice_chunks(H, dim, n_segments, max_n)) * gla::record_bytes(dim) * H * n_segments;
}

int gla_chunked(const b2kv_gla_args& a, int32_t* dev_status, void* stream) {
    using namespace gla;
    if (!chunked_sizes(a.dim, a.vdim, a.dtype) || a.n_segments > 65535 || a.H > 65535) return B2KV_ERR_UNSUPPORTED;
    // 16-byte pieces of v, gate and output rows
    if (!aligned16(a.y) || !aligned16(a.out) || a.ld_y % 8 || a.ld_out % 8 || a.v_col % 8 || a.g_col % 8) return B2KV_ERR_UNSUPPORTED;
    if (!aligned16(a.alpha) || a.ld_alpha % 2 || a.q_col % 2 || a.k_col % 2) return B2KV_ERR_UNSUPPORTED;  // pairs of channels
    if (!a.workspace || (reinterpret_cast<uintptr_t>(a.workspace) & 127) ||
        a.workspace_bytes < gla_chunked_workspace(a.H, a.dim, a.vdim, a.n_segments, a.max_n, a.dtype))
        return B2KV_ERR_WORKSPACE;
    if (a.dim <= 32) return launch_chunked<2>(a, dev_status, stream);
    if (a.dim <= 64) return launch_chunked<4>(a, dev_status, stream);
    return launch_chunked<8>(a, dev_status, stream);
}

}  // namespace b2kv
