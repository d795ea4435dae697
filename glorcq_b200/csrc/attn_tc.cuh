// Causal attention of a prompt (or a portion of one) on tcgen05: keys of up to two parts, the second of which all heads
// share, grouped query heads, values position by position or transposed.
#pragma once

#include "tma.cuh"

namespace glq {

// 2^x by the special-function unit alone (2 ulp; -inf -> 0; results below the normal range flush to zero)
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// Shared-memory operand whose rows of 128 bytes run along the other dimension (MN-major, 128-byte swizzle): 8 rows to an
// atom of 1024 bytes, atoms of the next 64 columns 8192 bytes on
__device__ __forceinline__ uint64_t at_desc_mn(uint32_t saddr) {
    return (uint64_t)((saddr & 0x3FFFFu) >> 4) | ((uint64_t)(8192 >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) |
           ((uint64_t)2 << 61);
}
inline size_t at_smem(size_t chunks, int dv) { return chunks * (2 * 16384 + 2 * 8192) + 2 * (size_t)dv * 128 + 1024; }

// One CTA takes 256 queries of a head, as two groups of 128 that alternate between the tensor core and the soft-max.
// Per key block of 64: S = Q K^T (operands in shared memory by TMA) into tensor memory; a thread owns a query row, turns
// its 64 scores into weights and writes them back to tensor memory as two bf16 parts; O += P V takes them from there,
// the values from shared memory: rows of a value dimension over positions (VMN false), or positions as they are cached (VMN),
// the transposed operand then being the tensor core's business.  The running maximum a row works with is replaced (and O rescaled) only when
// a score exceeds it by more than 8 in the base-2 exponent: weights stay below 2^8 and the final division makes the
// result the same.
// Tensor memory (512 columns): S 2 x 64, P 2 x (32 + 32), O 2 x 128.
constexpr int kAtThreads = 320;      // warps 0-3, 4-7: soft-max of the two groups, 8: TMA, 9: MMA
struct AtParams {
    const float* gate;               // (rows, ldg), one per head, or NULL
    void* out;                       // (rows, H * V)
    long long ldg;
    int B, T, H, V, S;               // S: positions with keys, the last T of them the queries'
    int krows, rrows;                // rows of a sequence in the keys' (and VMN: values') map, in the second key part's
    int group;                       // query heads to a key head
    float scale;
};
struct AtMaps {
    CUtensorMap qn, qr, kn, kr, vt;
};
struct AtGeom {
    int cd, nc;                      // 64-column chunks of the unrotated part, of both parts
    int steps_last_d, steps_last_r;  // 16-column steps in the last chunk of either part
};

__device__ __forceinline__ void at_st16(uint32_t taddr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};" ::"r"(taddr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
        "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
        : "memory");
}

template <int DV, bool VMN>
__global__ void __launch_bounds__(kAtThreads, 1) causal_attn_tc_kernel(const __grid_constant__ AtMaps maps, const AtParams p,
                                                                         const AtGeom geo) {
    extern __shared__ unsigned char at_raw[];
    __shared__ __align__(8) unsigned long long bars[15];
    __shared__ uint32_t s_tmem;
    __shared__ int s_dead;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int nc = geo.nc;
    const uint32_t sq = (smem_u32(at_raw) + 1023u) & ~1023u;
    const uint32_t sk = sq + (uint32_t)nc * 2 * 16384, sv = sk + (uint32_t)nc * 2 * 8192;
    const uint32_t q_full = smem_u32(bars), k_full = q_full + 8, k_empty = k_full + 16, v_full = k_empty + 16, v_empty = v_full + 16,
                   s_full = v_empty + 16, p_full = s_full + 16, pv_done = p_full + 16;
    volatile int* dead = &s_dead;
    // work order: the query blocks with the most keys first, over all heads and sequences
    const int n_hb = p.H * p.B;
    const int qb = (int)(gridDim.x / n_hb) - 1 - (int)(blockIdx.x / n_hb);
    const int h = (int)(blockIdx.x % n_hb) % p.H, b = (int)(blockIdx.x % n_hb) / p.H;
    const int start = p.S - p.T, q0 = qb * 256, kh = h / p.group, v0 = (int)blockIdx.y * DV;
    int nblk[2];
#pragma unroll
    for (int g = 0; g < 2; ++g) nblk[g] = q0 + 128 * g < p.T ? (start + min(p.T, q0 + 128 * (g + 1)) - 1) / 64 + 1 : 0;
    const int nmax = max(nblk[0], nblk[1]);
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int i = 0; i < 2; ++i) {
            mbar_init(k_full + 8 * i, 1);
            mbar_init(k_empty + 8 * i, 1);
            mbar_init(v_full + 8 * i, 1);
            mbar_init(v_empty + 8 * i, 1);
            mbar_init(s_full + 8 * i, 1);
            mbar_init(p_full + 8 * i, 4);
            mbar_init(pv_done + 8 * i, 1);
        }
        s_dead = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 9) tc_alloc(smem_u32(&s_tmem), 512);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    pdl_wait();
    pdl_release();

    if (warp == 8) {
        if (lane == 0) {
            mbar_expect_tx(q_full, (uint32_t)nc * 2 * 16384);
            for (int g = 0; g < 2; ++g)
                for (int c = 0; c < nc; ++c) {
                    const uint32_t dst = sq + (uint32_t)(g * nc + c) * 16384;
                    const int row = b * p.T + q0 + 128 * g;      // rows past the sequence are read and not used
                    if (c < geo.cd) tma_load_3d(dst, &maps.qn, 64 * c, h, row, q_full);
                    else tma_load_3d(dst, &maps.qr, 64 * (c - geo.cd), h, row, q_full);
                }
            int jk = 0, jv = 0;
            for (int j = 0; j < nmax; ++j) {
                const int s = j & 1;
                const uint32_t ph = ((uint32_t)(j >> 1) & 1u) ^ 1u;
                if (!tc_wait(k_empty + 8 * s, ph, dead, 120)) break;
                mbar_expect_tx(k_full + 8 * s, (uint32_t)nc * 8192);
                for (int c = 0; c < nc; ++c) {
                    const uint32_t dst = sk + (uint32_t)(s * nc + c) * 8192;
                    if (c < geo.cd) tma_load_3d(dst, &maps.kn, 64 * c, kh, b * p.krows + 64 * j, k_full + 8 * s);
                    else tma_load_2d(dst, &maps.kr, 64 * (c - geo.cd), b * p.rrows + 64 * j, k_full + 8 * s);
                }
                ++jk;
                if (!tc_wait(v_empty + 8 * s, ph, dead, 121)) break;
                mbar_expect_tx(v_full + 8 * s, DV * 128);
                if constexpr (VMN) {
#pragma unroll
                    for (int c = 0; c < DV / 64; ++c)
                        tma_load_3d(sv + (uint32_t)s * DV * 128 + c * 8192, &maps.vt, v0 + 64 * c, kh, b * p.krows + 64 * j, v_full + 8 * s);
                } else {
                    tma_load_2d(sv + (uint32_t)s * DV * 128, &maps.vt, 64 * j, (b * p.H + h) * p.V, v_full + 8 * s);
                }
                ++jv;
            }
            if (*dead) {   // copies in flight must land before the CTA leaves (bounded)
                const unsigned long long t0 = global_ns();
                auto drain = [&](uint32_t bar, uint32_t parity) {
                    while (!mbar_test_wait(bar, parity) && global_ns() - t0 < 4000000ull) __nanosleep(64);
                };
                drain(q_full, 0);
                for (int j = max(0, jk - 2); j < jk; ++j) drain(k_full + 8 * (j & 1), (uint32_t)(j >> 1) & 1u);
                for (int j = max(0, jv - 2); j < jv; ++j) drain(v_full + 8 * (j & 1), (uint32_t)(j >> 1) & 1u);
            }
        }
        __syncwarp();
    } else if (warp == 9) {
        if (lane == 0) {
            auto scores = [&](int g, int j) {
                uint32_t acc = 0;
                for (int c = 0; c < nc; ++c) {
                    const int steps = c == geo.cd - 1 ? geo.steps_last_d : (c == nc - 1 ? geo.steps_last_r : 4);
                    const uint32_t a = sq + (uint32_t)(g * nc + c) * 16384, kb = sk + (uint32_t)((j & 1) * nc + c) * 8192;
                    for (int kk = 0; kk < steps; ++kk) {
                        tc_mma_f16(tmem + (uint32_t)g * 64, tc_smem_desc(a + 32u * kk), tc_smem_desc(kb + 32u * kk), dt_idesc(64), acc);
                        acc = 1;
                    }
                }
                tc_commit(s_full + 8 * g);
            };
            // a stage is handed back only where a later block waits for it: no commit is pending when the CTA ends
            bool ok = tc_wait(q_full, 0, dead, 122) && tc_wait(k_full, 0, dead, 123);
            tc_fence_after();
            if (ok) {
                for (int g = 0; g < 2; ++g)
                    if (nblk[g] > 0) scores(g, 0);
                if (2 < nmax) tc_commit(k_empty);
            }
            for (int j = 0; j < nmax && ok; ++j) {
                if (j + 1 < nmax) ok = tc_wait(k_full + 8 * ((j + 1) & 1), (uint32_t)((j + 1) >> 1) & 1u, dead, 124);
                ok = ok && tc_wait(v_full + 8 * (j & 1), (uint32_t)(j >> 1) & 1u, dead, 125);
                for (int g = 0; g < 2 && ok; ++g) {
                    if (j >= nblk[g]) continue;
                    ok = tc_wait(p_full + 8 * g, (uint32_t)j & 1u, dead, 126);
                    if (!ok) break;
                    tc_fence_after();
                    if (j + 1 < nblk[g]) scores(g, j + 1);      // the group's scores of block j have been read
                    const uint32_t vb = sv + (uint32_t)(j & 1) * DV * 128;
#pragma unroll
                    for (int part = 0; part < 2; ++part)
#pragma unroll
                        for (int kk = 0; kk < 4; ++kk)
                            tc_mma_f16_ts(tmem + 256u + 128u * g, tmem + 128u + 64u * g + 32u * part + 8u * kk,
                                          VMN ? at_desc_mn(vb + 2048u * kk) : tc_smem_desc(vb + 32u * kk),
                                          dt_idesc(DV) | (VMN ? 1u << 16 : 0u), (j | part | kk) != 0);
                    tc_commit(pv_done + 8 * g);
                }
                if (!ok) break;
                if (j + 2 < nmax) tc_commit(v_empty + 8 * (j & 1));
                if (j + 3 < nmax) tc_commit(k_empty + 8 * ((j + 1) & 1));
            }
        }
        __syncwarp();
    } else {
        const int g = warp >> 2, n = nblk[g];
        const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
        const uint32_t ts = tmem + 64u * g + lanes, tp = tmem + 128u + 64u * g + lanes, to = tmem + 256u + 128u * g + lanes;
        const int wrow = q0 + 128 * g + (warp & 3) * 32, row = wrow + lane;      // query of the warp's first lane, of this lane
        const float sc = p.scale * 1.4426950408889634f;
        float m = 0.f, l = 0.f;
        bool ok = true;
        for (int j = 0; j < n; ++j) {
            ok = tc_wait_warp(s_full + 8 * g, (uint32_t)j & 1u, dead, 127);
            if (!ok) break;
            tc_fence_after();
            float s[64];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                uint32_t v[16];
                tc_ld16(ts + 16u * c, v);
                tc_ld_wait();
#pragma unroll
                for (int i = 0; i < 16; ++i) s[16 * c + i] = __uint_as_float(v[i]) * sc;
            }
            if (64 * j + 63 > start + wrow) {        // some key of the block lies after some query of the warp
                const int seen = start + row - 64 * j;
#pragma unroll
                for (int i = 0; i < 64; ++i)
                    if (i > seen) s[i] = -INFINITY;
            }
            float mx = s[0];
#pragma unroll
            for (int i = 1; i < 64; ++i) mx = fmaxf(mx, s[i]);
            bool waited = j == 0;
            if (j == 0) {
                m = mx == -INFINITY ? 0.f : mx;
            } else if (__any_sync(0xffffffffu, mx > m + 8.f)) {
                ok = tc_wait_warp(pv_done + 8 * g, (uint32_t)(j - 1) & 1u, dead, 128);
                if (!ok) break;
                waited = true;
                tc_fence_after();
                const float mn = fmaxf(m, mx), f = ex2(m - mn);
                m = mn;
                l *= f;
#pragma unroll
                for (int c = 0; c < DV / 16; ++c) {
                    uint32_t v[16];
                    tc_ld16(to + 16u * c, v);
                    tc_ld_wait();
#pragma unroll
                    for (int i = 0; i < 16; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * f);
                    at_st16(to + 16u * c, v);
                }
                tc_st_wait();
            }
            uint32_t hi[32], lo[32];
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                const float a = ex2(s[2 * i] - m), c = ex2(s[2 * i + 1] - m);
                sum += a + c;
                split_bf2(a, c, hi[i], lo[i]);
            }
            l += sum;
            if (!waited) {                           // the weights of the last block have been used
                ok = tc_wait_warp(pv_done + 8 * g, (uint32_t)(j - 1) & 1u, dead, 129);
                if (!ok) break;
                tc_fence_after();
            }
            at_st16(tp, hi);
            at_st16(tp + 16u, hi + 16);
            at_st16(tp + 32u, lo);
            at_st16(tp + 48u, lo + 16);
            tc_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(p_full + 8 * g);
        }
        if (n > 0 && ok) ok = tc_wait_warp(pv_done + 8 * g, (uint32_t)(n - 1) & 1u, dead, 130);
        if (n > 0 && ok) {
            tc_fence_after();
            const size_t orow = (size_t)b * p.T + row;
            const float inv = row < p.T ? (p.gate ? sigmoid_f(p.gate[orow * p.ldg + h]) : 1.f) / l : 0.f;
            bf16* y = reinterpret_cast<bf16*>(p.out) + orow * p.H * p.V + (size_t)h * p.V + v0;
#pragma unroll 1
            for (int c = 0; c < DV / 16; ++c) {
                uint32_t v[16];
                __syncwarp();
                tc_ld16(to + 16u * c, v);
                tc_ld_wait();
                if (row < p.T) {
#pragma unroll
                    for (int u = 0; u < 2; ++u)
                        if (v0 + 16 * c + 8 * u < p.V) {
                            uint32_t w[4];
#pragma unroll
                            for (int i = 0; i < 4; ++i)
                                w[i] = pack_bf2(__uint_as_float(v[8 * u + 2 * i]) * inv, __uint_as_float(v[8 * u + 2 * i + 1]) * inv);
                            *reinterpret_cast<uint4*>(y + 16 * c + 8 * u) = make_uint4(w[0], w[1], w[2], w[3]);
                        }
                }
            }
        }
        tc_fence_before();
    }
    __syncthreads();
    if (warp == 9) {
        tc_fence_after();
        tc_dealloc(tmem, 512);
    }
}

}  // namespace glq
