// Gated linear attention over prompt portions, sixteen tokens at a time (bf16 rows, fp32 state).
//
// With P_t the product of the decays up to token t of a chunk and R_s the product behind token s (both per key channel, both at
// most one, so nothing can overflow however strong the decay), a chunk with incoming state S is
//
//   o_t  = S^T (q_t P_t) + sum_{s <= t} A_ts v_s,   A_ts = sum_d q_td k_sd prod_{s < r <= t} alpha_rd
//   S   <- diag(P_last) S + sum_s (k_s R_s) v_s^T
//
// One CTA per (head, segment) walks the chunks in order:
//   * four warps prepare a chunk: decays, q P and k R (thread = key channel), and A, whose products of decays are carried along
//     exactly instead of being taken apart into factors that could overflow (thread = token s and a range of channels).  They run
//     one chunk ahead, with the next chunk's rows already on their way;
//   * every other warp owns 32 value columns of the state, transposed, as accumulators of mma.m16n8k16: the state never
//     leaves registers between the first and the last chunk.  As an A operand of the first product the accumulators need no
//     shuffle.  A step of the recurrence is sixteen tokens deep, one k-step of this instruction; larger tiles would have to
//     bring the state through tensor memory, decay it there and write it back as operands sixteen tokens at a time, a chain of
//     copies and waits several times as long as these products.
//   * fp32 operands (q P, k R, A and the state) are split into two bf16 halves, x = hi + lo, and lo * lo is dropped; v is
//     exact.  Accumulation, decay and state are fp32.
//   * o goes through shared memory so that the warps can take whole rows for the head's norm and the gate.
// Producer and consumer warps meet at hardware barriers whose arrivals are fixed by the number of chunks, which all warps know.
#include "gla.cuh"

#include "tc_ptx.cuh"

namespace b2kv {
namespace gla {
namespace {

constexpr int kChunk = 16;
constexpr int kPrep = 128;    // threads that prepare
constexpr int kSlab = 32;     // value columns per state warp
constexpr int kMaxWarps = 8;  // state warps
constexpr int kRing = 3;      // chunks of v and gate rows in shared memory
enum { kBarFull = 1, kBarEmpty = 3, kBarPrep = 5, kBarState = 6 };

__device__ __forceinline__ void bar_sync(int id, int n) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(n) : "memory"); }
__device__ __forceinline__ void bar_arrive(int id, int n) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(n) : "memory"); }

// 16 bytes global -> shared, or 16 zero bytes.
__device__ __forceinline__ void copy16(void* dst, const void* src, bool live) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
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

// Shared memory for kD16 * 16 key channels; the arrays that depend on the value width come behind it.
template <int kD16>
struct Smem {
    static constexpr int kD = kD16 * 16;
    static constexpr int kLd = kD + 8;  // bf16 rows an odd number of 16-byte pieces apart: no bank conflicts in ldmatrix
    static constexpr int kLf = kD + 4;
    static constexpr int kLa = 24;
    struct Buffer {
        __nv_bfloat16 q_hi[kChunk][kLd], q_lo[kChunk][kLd], k_hi[kChunk][kLd], k_lo[kChunk][kLd];
        __nv_bfloat16 a_hi[kChunk][kLa], a_lo[kChunk][kLa];
        float decay[kD];
    };
    alignas(16) Buffer buf[2];
    alignas(16) float q[kChunk][kLf], k[kChunk][kLf], alpha[kChunk][kLf];
    float part[4][kChunk * kChunk];
};

template <int kD16>
__global__ void __launch_bounds__(kPrep + 32 * kMaxWarps, 1) gla_chunk_kernel(const b2kv_gla_args a, int n_warps, int lanes_per_token,
                                                                             int32_t* dev_status) {
    extern __shared__ uint8_t smem_raw[];
    using S = Smem<kD16>;
    constexpr int kD = S::kD;
    S& sm = *reinterpret_cast<S*>(smem_raw);
    const int ldv = kSlab * n_warps + 8, ldo = kSlab * n_warps + 4;  // row pitches of v and gate (bf16), of o (fp32)
    __nv_bfloat16* const s_v = reinterpret_cast<__nv_bfloat16*>(smem_raw + sizeof(S));  // [kRing][kChunk][ldv]
    __nv_bfloat16* const s_g = s_v + kRing * kChunk * ldv;
    float* const s_o = reinterpret_cast<float*>(s_g + kRing * kChunk * ldv);  // [2][kChunk][ldo]
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

    if (tid < kPrep) {
        // ------------------------------ preparation ------------------------------
        const __nv_bfloat16* const y = static_cast<const __nv_bfloat16*>(a.y) + static_cast<int64_t>(sg.row0) * a.ld_y;
        const __nv_bfloat16* const yq = y + a.q_col + h * a.dim;
        const __nv_bfloat16* const yk = y + a.k_col + h * a.dim;
        const float* const z = a.z + static_cast<int64_t>(sg.row0) * a.ld_z + static_cast<int64_t>(h) * a.dim;
        const float inv_tau = 1.0f / a.tau;
        const bool live_d = tid < a.dim;  // thread = key channel
        const int pieces = kSlab * n_warps / 8;
        auto request = [&](int ci) {  // v and gate rows of a chunk
            for (int p = tid; p < 2 * kChunk * pieces; p += kPrep) {
                const bool gate = p >= kChunk * pieces;
                const int t = (gate ? p - kChunk * pieces : p) / pieces, c = p % pieces * 8;
                const bool live = ci * kChunk + t < sg.n && c < a.vdim;
                const __nv_bfloat16* src = y + (gate ? a.g_col : a.v_col) + h * a.vdim;
                if (live) src += static_cast<int64_t>(ci * kChunk + t) * a.ld_y + c;
                copy16((gate ? s_g : s_v) + (ci % kRing * kChunk + t) * ldv + c, src, live);
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        float nz[kChunk];
        __nv_bfloat16 nq[kChunk], nk[kChunk];
        auto fetch = [&](int ci) {  // this channel's numbers of a chunk
#pragma unroll
            for (int t = 0; t < kChunk; ++t) {
                const bool live = live_d && ci * kChunk + t < sg.n;
                const int64_t row = ci * kChunk + t;
                nz[t] = live ? z[row * a.ld_z + tid] : 0.f;
                nq[t] = live ? yq[row * a.ld_y + tid] : __nv_bfloat16(0.f);
                nk[t] = live ? yk[row * a.ld_y + tid] : __nv_bfloat16(0.f);
            }
        };
        request(0);
        fetch(0);
        const int s = lane & 15, warp = tid >> 5;
        const int d0 = warp * (kD / 4) + (lane >> 4) * (kD / 8);  // channels of this thread's part of A's column s
        for (int ci = 0; ci < chunks; ++ci) {
            typename S::Buffer& b = sm.buf[ci & 1];
            if (ci >= 2) bar_sync(kBarEmpty + (ci & 1), n_threads);
            if (ci + 1 < chunks) request(ci + 1);
            if (tid < kD) {
                float al[kChunk], prod = 1.f;
#pragma unroll
                for (int t = 0; t < kChunk; ++t) {
                    const bool live = live_d && ci * kChunk + t < sg.n;
                    al[t] = live ? expf(log_sigmoid(nz[t]) * inv_tau) : 1.f;
                    prod *= al[t];
                    const float q = __bfloat162float(nq[t]) * a.q_scale;
                    sm.q[t][tid] = q;
                    sm.k[t][tid] = __bfloat162float(nk[t]);
                    sm.alpha[t][tid] = al[t];
                    split1(q * prod, b.q_hi[t][tid], b.q_lo[t][tid]);
                }
                b.decay[tid] = prod;
                prod = 1.f;
#pragma unroll
                for (int t = kChunk - 1; t >= 0; --t) {
                    split1(__bfloat162float(nk[t]) * prod, b.k_hi[t][tid], b.k_lo[t][tid]);
                    prod *= al[t];
                }
            }
            if (ci + 1 < chunks) fetch(ci + 1);
            bar_sync(kBarPrep, kPrep);
            float acc[kChunk];
#pragma unroll
            for (int t = 0; t < kChunk; ++t) acc[t] = 0.f;
            for (int d = d0; d < d0 + kD / 8; d += 4) {
                float4 w = *reinterpret_cast<const float4*>(&sm.k[s][d]);
#pragma unroll
                for (int t = 0; t < kChunk; ++t) {
                    const float4 q = *reinterpret_cast<const float4*>(&sm.q[t][d]);
                    const float4 f = *reinterpret_cast<const float4*>(&sm.alpha[t][d]);
                    if (t > s) w.x *= f.x, w.y *= f.y, w.z *= f.z, w.w *= f.w;
                    acc[t] = fmaf(q.x, w.x, fmaf(q.y, w.y, fmaf(q.z, w.z, fmaf(q.w, w.w, acc[t]))));
                }
            }
#pragma unroll
            for (int t = 0; t < kChunk; ++t) {
                acc[t] += __shfl_xor_sync(0xffffffffu, acc[t], 16);
                if (lane < 16) sm.part[warp][t * kChunk + s] = acc[t];
            }
            bar_sync(kBarPrep, kPrep);
            for (int e = tid; e < kChunk * kChunk; e += kPrep) {
                const int t = e / kChunk, c = e % kChunk;
                const float v = c <= t ? (sm.part[0][e] + sm.part[1][e]) + (sm.part[2][e] + sm.part[3][e]) : 0.f;
                split1(v, b.a_hi[t][c], b.a_lo[t][c]);
            }
            if (ci + 1 < chunks)
                asm volatile("cp.async.wait_group 1;" ::: "memory");
            else
                asm volatile("cp.async.wait_group 0;" ::: "memory");
            bar_arrive(kBarFull + (ci & 1), n_threads);
        }
        return;
    }

    // ------------------------------ state: 32 value columns per warp ------------------------------
    const int w = (tid - kPrep) >> 5;
    const int row = lane >> 2, col = (lane & 3) * 2;  // place of this thread's first accumulator in a tile
    float* const state = a.state + (static_cast<int64_t>(sg.slot) * a.H + h) * a.dim * a.vdim;
    const bool fresh = a.row_pos[sg.row0] == 0;
    float c[2][2 * kD16][4];  // [slab of 16 value columns][tile of 8 key channels]
    auto each_state = [&](auto&& fn) {
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int j = 0; j < 2 * kD16; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int v = w * kSlab + m * 16 + row + (e >> 1) * 8, d = j * 8 + col + (e & 1);
                    fn(c[m][j][e], static_cast<int64_t>(d) * a.vdim + v, v < a.vdim && d < a.dim);
                }
    };
    each_state([&](float& x, int64_t at, bool live) { x = live && !fresh ? state[at] : 0.f; });

    const int mat = lane >> 3, r8 = lane & 7;
    // ldmatrix row addresses: [token][channel] tiles as they lie (tokens 0-7 | 8-15 outermost), and transposed
    const int plain_t = r8 + 8 * (mat >> 1), plain_c = 8 * (mat & 1);
    const int trans_t = r8 + 8 * (mat & 1), trans_c = 8 * (mat >> 1);
    const int group = lane / lanes_per_token, sub = lane % lanes_per_token, groups = 32 / lanes_per_token;
    for (int ci = 0; ci < chunks; ++ci) {
        typename S::Buffer& b = sm.buf[ci & 1];
        const int slot = ci % kRing;
        bar_sync(kBarFull + (ci & 1), n_threads);
        const uint32_t v_addr = smem_u32(s_v + (slot * kChunk + plain_t) * ldv + w * kSlab + plain_c);
        float o[2][2][4];
        {
            uint32_t vf[2][4], hi[4], lo[4];
            ldsm4t(vf[0], v_addr);
            ldsm4t(vf[1], v_addr + 32);
            ldsm4(hi, smem_u32(&b.a_hi[plain_t][plain_c]));
            ldsm4(lo, smem_u32(&b.a_lo[plain_t][plain_c]));
#pragma unroll
            for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;
                    mma16816(o[m][n], vf[m], hi[2 * n], hi[2 * n + 1]);
                    mma16816(o[m][n], vf[m], lo[2 * n], lo[2 * n + 1]);
                }
        }
#pragma unroll
        for (int kk = 0; kk < kD16; ++kk) {
            uint32_t hi[4], lo[4];
            ldsm4(hi, smem_u32(&b.q_hi[plain_t][kk * 16 + plain_c]));
            ldsm4(lo, smem_u32(&b.q_lo[plain_t][kk * 16 + plain_c]));
#pragma unroll
            for (int m = 0; m < 2; ++m) {
                uint32_t s_hi[4], s_lo[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float(&t)[4] = c[m][2 * kk + (e >> 1)];
                    split2(t[2 * (e & 1)], t[2 * (e & 1) + 1], s_hi[e], s_lo[e]);
                }
#pragma unroll
                for (int n = 0; n < 2; ++n) mma16816(o[m][n], s_hi, hi[2 * n], hi[2 * n + 1]);
#pragma unroll
                for (int n = 0; n < 2; ++n) mma16816(o[m][n], s_hi, lo[2 * n], lo[2 * n + 1]);
#pragma unroll
                for (int n = 0; n < 2; ++n) mma16816(o[m][n], s_lo, hi[2 * n], hi[2 * n + 1]);
            }
        }
        float* const so = s_o + (ci & 1) * kChunk * ldo;
#pragma unroll
        for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    so[(n * 8 + col + (e & 1)) * ldo + w * kSlab + m * 16 + row + (e >> 1) * 8] = o[m][n][e];
        uint32_t vf[2][4];  // (loaded again: no registers to keep it in)
        ldsm4t(vf[0], v_addr);
        ldsm4t(vf[1], v_addr + 32);
#pragma unroll
        for (int kk = 0; kk < kD16; ++kk) {
            uint32_t hi[4], lo[4];
            ldsm4t(hi, smem_u32(&b.k_hi[trans_t][kk * 16 + trans_c]));
            ldsm4t(lo, smem_u32(&b.k_lo[trans_t][kk * 16 + trans_c]));
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float2 f = *reinterpret_cast<const float2*>(&b.decay[(2 * kk + u) * 8 + col]);
#pragma unroll
                for (int m = 0; m < 2; ++m) {
                    float(&t)[4] = c[m][2 * kk + u];
                    t[0] *= f.x, t[1] *= f.y, t[2] *= f.x, t[3] *= f.y;
                    mma16816(t, vf[m], hi[2 * u], hi[2 * u + 1]);
                    mma16816(t, vf[m], lo[2 * u], lo[2 * u + 1]);
                }
            }
        }
        bar_sync(kBarState, 32 * n_warps);
        // whole rows of o: lanes_per_token lanes with eight values each
        for (int t0 = w * groups; t0 < kChunk; t0 += n_warps * groups) {
            const int t = t0 + group;
            const bool mine = sub * 8 < a.vdim && t < kChunk && ci * kChunk + t < sg.n;
            float f[8], g[8], sum = 0.f;
            if (mine) {
                const float* src = so + t * ldo + sub * 8;
                const float4 x0 = *reinterpret_cast<const float4*>(src), x1 = *reinterpret_cast<const float4*>(src + 4);
                f[0] = x0.x, f[1] = x0.y, f[2] = x0.z, f[3] = x0.w, f[4] = x1.x, f[5] = x1.y, f[6] = x1.z, f[7] = x1.w;
                Elt<__nv_bfloat16>::widen(*reinterpret_cast<const uint4*>(s_g + (slot * kChunk + t) * ldv + sub * 8), g);
#pragma unroll
                for (int e = 0; e < 8; ++e) sum = fmaf(f[e], f[e], sum);
            }
            for (int off = lanes_per_token / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
            if (mine) {
                const float scale = 1.0f / sqrtf(sum / static_cast<float>(a.vdim) + a.eps);
#pragma unroll
                for (int e = 0; e < 8; ++e) f[e] *= scale * a.norm[sub * 8 + e] * silu(g[e]);
                uint4 out;
                out.x = tc::pack_bf16(f[0], f[1]), out.y = tc::pack_bf16(f[2], f[3]);
                out.z = tc::pack_bf16(f[4], f[5]), out.w = tc::pack_bf16(f[6], f[7]);
                __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + (static_cast<int64_t>(sg.row0) + ci * kChunk + t) * a.ld_out +
                                     static_cast<int64_t>(h) * a.vdim + sub * 8;
                *reinterpret_cast<uint4*>(dst) = out;
            }
        }
        if (ci + 2 < chunks) bar_arrive(kBarEmpty + (ci & 1), n_threads);
    }
    each_state([&](float& x, int64_t at, bool live) {
        if (live) state[at] = x;
    });
}

template <int kD16>
int launch_chunked(const b2kv_gla_args& a, int n_warps, int32_t* dev_status, void* stream) {
    const size_t smem = sizeof(Smem<kD16>) + 2 * kRing * kChunk * (kSlab * n_warps + 8) * sizeof(__nv_bfloat16) +
                        2 * kChunk * (kSlab * n_warps + 4) * sizeof(float);
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
    B2KV_CUDA_TRY(cudaLaunchKernelEx(&launch.cfg, kernel, a, n_warps, lanes, dev_status));
    return B2KV_OK;
}

}  // namespace
}  // namespace gla

int gla_chunked(const b2kv_gla_args& a, int32_t* dev_status, void* stream) {
    using namespace gla;
    if (a.dtype != B2KV_DTYPE_BF16 || a.dim % 8 != 0 || a.dim > 128 || a.vdim % 8 != 0 || a.vdim > kSlab * kMaxWarps || a.n_segments > 65535)
        return B2KV_ERR_UNSUPPORTED;
    // 16-byte pieces of v, gate and output rows
    if (!aligned16(a.y) || !aligned16(a.out) || a.ld_y % 8 || a.ld_out % 8 || a.v_col % 8 || a.g_col % 8) return B2KV_ERR_UNSUPPORTED;
    const int n_warps = (a.vdim + kSlab - 1) / kSlab;
    if (a.dim <= 32) return launch_chunked<2>(a, n_warps, dev_status, stream);
    if (a.dim <= 64) return launch_chunked<4>(a, n_warps, dev_status, stream);
    return launch_chunked<8>(a, n_warps, dev_status, stream);
}

}  // namespace b2kv
