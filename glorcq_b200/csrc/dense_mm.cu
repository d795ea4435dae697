// Products with unquantized row-major weights, y = alpha * act(x . W^T), plain or over a device-side list of problems
// (the experts of a mixture), in three forms:
//   * few rows per problem (a decode step): a streaming kernel in the manner of the output projection (lm_head.cu):
//     16 weight rows per warp tile, k split over the warps of a CTA, up to 8 activation rows as the columns of the
//     tensor-core op; the first weight loads are issued before the kernel waits for its predecessor;
//   * many rows: a persistent tcgen05 kernel; activation and weight tiles arrive by TMA (128-byte swizzle), the
//     accumulator is double-buffered in tensor memory so that the epilogue of a tile overlaps the next tile's products;
//   * float32, or rows that are no multiple of 16 bytes: a tiled kernel on the CUDA cores.
// Rows sums are taken in a fixed order in all three: results do not depend on what else is in the batch.
#include "tma.cuh"

namespace glq {
thread_local int g_dense_cuda_error = 0;

struct DmParams {
    const void* x;
    const void* W;
    void* y;
    float* y32;
    const int* slot_index;
    const int* n_slots;
    const int* slot_count;
    const int* slot_offset;
    const int* entry_row;
    long long ldx, ldy, ldy32, ldw;
    int N, K, rows, slots, split, act;
    float alpha;
    int vec_y, vec_y32;
    int xrows;                       // streaming kernel: activation rows staged, one of zeros behind fewer than eight
    const float* hn_o;               // streaming kernel: rows made from a recurrence's output (see glq_dense_mm_t)
    const void* hn_g;
    const float* hn_w;
    long long hn_ldg;
    int hn_heads;
    float hn_eps;
    const void* mul;
    const int64_t* mul_row;
    long long ldmul;
    int mul_rows, residual, vec_mul;
};

struct DmSlot {
    int mat, off, cnt;
};
__device__ __forceinline__ DmSlot dm_slot(const DmParams& p, int s) {
    if (!p.slot_index) return {0, 0, p.rows};
    if (s >= __ldg(p.n_slots)) return {0, 0, 0};
    return {__ldg(p.slot_index + s), __ldg(p.slot_offset + s), __ldg(p.slot_count + s)};
}

template <typename T> __device__ __forceinline__ const T* dm_mul_row(const DmParams& p, int row) {
    long long r = row;
    if (p.mul_row) {
        r = p.mul_row[row];
        r = r < 0 ? 0 : (r >= p.mul_rows ? p.mul_rows - 1 : r);
    }
    return reinterpret_cast<const T*>(p.mul) + r * p.ldmul;
}
template <typename T, bool MUL = true> __device__ __forceinline__ void dm_store(const DmParams& p, int row, int n, float v) {
    if (MUL && p.mul) v *= to_f(dm_mul_row<T>(p, row)[n]);
    if (p.residual) {
        float* x = p.y32 + (size_t)row * p.ldy32 + n;
        v += *x;
        *x = v;
        if (p.y) reinterpret_cast<T*>(p.y)[(size_t)row * p.ldy + n] = from_f<T>(v);
        return;
    }
    if (n < p.split) reinterpret_cast<T*>(p.y)[(size_t)row * p.ldy + n] = from_f<T>(v);
    else p.y32[(size_t)row * p.ldy32 + (n - p.split)] = v;
}

template <typename T> __device__ __forceinline__ float dm_glu(float gate, float other) { return gate * sigmoid_t<T>(gate) * other; }

// =====================================================================================================
// streaming kernel: up to 8 rows per slot
// =====================================================================================================
__device__ __forceinline__ uint4 dm_ldg(const uint4* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.L2::256B.v4.u32 {%0,%1,%2,%3}, [%4];"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
                 : "l"(p));
    return v;
}
// parts of at most 128 U values, which are requested before the sum and stay in registers
template <int WARPS, int U>
__device__ __forceinline__ void stage_parts(const DmParams& p, bf16* xs, int XS, int units, int share, int len, float* s_part) {
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, heads = p.hn_heads, V = p.K / heads;
    const bf16* gates = reinterpret_cast<const bf16*>(p.hn_g);
    for (int i = w; i < units * share; i += WARPS) {
        const int u = i / share, row = u / heads, h = u % heads;
        const int lo = (i % share) * len, hi = min(V, lo + len);
        const float* o = p.hn_o + (size_t)row * p.K + (size_t)h * V;
        float4 x[U];
        uint2 gv[U];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < U; ++j) {
            const int k = lo + 128 * j + 4 * lane;
            x[j] = k < hi ? *reinterpret_cast<const float4*>(o + k) : make_float4(0, 0, 0, 0);
            if (k < hi) gv[j] = *reinterpret_cast<const uint2*>(gates + (size_t)row * p.hn_ldg + (size_t)h * V + k);
        }
#pragma unroll
        for (int j = 0; j < U; ++j) ss += x[j].x * x[j].x + x[j].y * x[j].y + x[j].z * x[j].z + x[j].w * x[j].w;
        ss = warp_sum(ss);
        if (share > 1) {             // one round: every warp has at most one part
            if (lane == 0) s_part[w] = ss;
            asm volatile("bar.sync 1, %0;" ::"r"(units * share * 32) : "memory");
            ss = 0.f;
            for (int j = 0; j < share; ++j) ss += s_part[u * share + j];
        }
        const float inv = 1.f / sqrtf(ss / V + p.hn_eps);
#pragma unroll
        for (int j = 0; j < U; ++j) {
            const int k = lo + 128 * j + 4 * lane;
            if (k >= hi) continue;
            const float4 nw = *reinterpret_cast<const float4*>(p.hn_w + (size_t)h * V + k);
            const float4 v = make_float4(x[j].x * inv * nw.x * sigmoid_fast_f(bf_lo(gv[j].x)), x[j].y * inv * nw.y * sigmoid_fast_f(bf_hi(gv[j].x)),
                                         x[j].z * inv * nw.z * sigmoid_fast_f(bf_lo(gv[j].y)), x[j].w * inv * nw.w * sigmoid_fast_f(bf_hi(gv[j].y)));
            *reinterpret_cast<uint2*>(xs + (size_t)row * XS + (size_t)h * V + k) = make_uint2(pack_bf2(v.x, v.y), pack_bf2(v.z, v.w));
        }
    }
}
// Activation rows made from hn_o: RMS norm over each of hn_heads parts, times its weight, times the sigmoid of the gate.  Warps take
// (row, part) pairs, several to a pair when there are few; the values stay in registers between the sum and the product.
template <int WARPS>
__device__ __forceinline__ void stage_normed(const DmParams& p, bf16* xs, int XS, int cnt, float* s_part) {
    const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, heads = p.hn_heads, V = p.K / heads, units = cnt * heads;
    const bf16* gates = reinterpret_cast<const bf16*>(p.hn_g);
    for (int i = threadIdx.x; i < (p.xrows - cnt) * (p.K / 8); i += WARPS * 32)          // rows past the last: zeros
        *reinterpret_cast<uint4*>(xs + (size_t)(cnt + i / (p.K / 8)) * XS + 8 * (i % (p.K / 8))) = make_uint4(0, 0, 0, 0);
    int share = 1;
    while (2 * share * units <= WARPS) share *= 2;
    const int len = ((V + share - 1) / share + 3) / 4 * 4;                               // of a warp's part
    if (V % 4 == 0 && len <= 512 && p.hn_ldg % 4 == 0 && (reinterpret_cast<uintptr_t>(gates) & 7) == 0 &&
        (reinterpret_cast<uintptr_t>(p.hn_w) & 15) == 0) {
        if (len <= 256) stage_parts<WARPS, 2>(p, xs, XS, units, share, len, s_part);
        else stage_parts<WARPS, 4>(p, xs, XS, units, share, len, s_part);
        return;
    }
    for (int u = w; u < units; u += WARPS) {
        const int row = u / heads, h = u % heads;
        const float* o = p.hn_o + (size_t)row * p.K + (size_t)h * V;
        float ss = 0.f;
        for (int k = lane; k < V; k += 32) ss += o[k] * o[k];
        const float inv = 1.f / sqrtf(warp_sum(ss) / V + p.hn_eps);
        for (int k = lane; k < V; k += 32) {
            const float v = o[k] * inv * p.hn_w[(size_t)h * V + k] * sigmoid_fast_f(to_f(gates[(size_t)row * p.hn_ldg + (size_t)h * V + k]));
            xs[(size_t)row * XS + (size_t)h * V + k] = from_f<bf16>(v);
        }
    }
}

// WARPS warps a CTA, SPLIT of them share one 16-row tile; DEPTH 16-byte loads per lane and row are in flight.
// EXT: rows made from hn_o, or a product added to the residual.
template <int WARPS, int SPLIT, int DEPTH, int CTAS, bool EXT>
__global__ void __launch_bounds__(WARPS * 32, CTAS) dense_stream_kernel(const DmParams p) {
    constexpr int TILES = WARPS / SPLIT, THREADS = WARPS * 32;
    extern __shared__ __align__(16) unsigned char dm_smem[];
    const int K = p.K, tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
    const int g = lane >> 2, t = lane & 3;
    const int tw = w / SPLIT, s = w % SPLIT;
    const int chunks = (K + 31) / 32;                              // of 32 channels
    const int c_lo = (int)((long)s * chunks / SPLIT), c_hi = (int)((long)(s + 1) * chunks / SPLIT);
    const int XS = (chunks + 1) * 32;                              // padded activation rows: distinct banks
    bf16* xs = reinterpret_cast<bf16*>(dm_smem);
    float4* red = reinterpret_cast<float4*>(dm_smem + (size_t)p.xrows * XS * 2);
    __shared__ float s_part[WARPS];
    const int ntiles = (p.N + 15) / 16;
    const bool plain = p.slot_index == nullptr;
    DmSlot sl{0, 0, p.rows};
    if (!plain) {
        pdl_wait();
        pdl_release();
        sl = dm_slot(p, blockIdx.y);
        if (sl.cnt == 0) return;
    }
    const bf16* Wm = reinterpret_cast<const bf16*>(p.W) + (size_t)sl.mat * p.N * p.ldw;
    const int iters = (ntiles + TILES * (int)gridDim.x - 1) / (TILES * (int)gridDim.x);
    for (int it = 0; it < iters; ++it) {
        const int tile = (it * (int)gridDim.x + (int)blockIdx.x) * TILES + tw;
        const bool live = tile < ntiles;
        const int r0 = min(tile * 16 + g, p.N - 1), r1 = min(tile * 16 + g + 8, p.N - 1);
        const bf16* w0 = Wm + (size_t)r0 * p.ldw + t * 8;
        const bf16* w1 = Wm + (size_t)r1 * p.ldw + t * 8;
        const int lim = K - 8 - t * 8;      // this lane's 8 channels of chunk c exist when 32 c <= lim
        uint4 qa[DEPTH], qb[DEPTH];
        auto fetch = [&](int c, int d) {
            const bool ok = live && c < c_hi && 32 * c <= lim;
            qa[d] = ok ? dm_ldg(reinterpret_cast<const uint4*>(w0 + 32 * c)) : make_uint4(0, 0, 0, 0);
            qb[d] = ok ? dm_ldg(reinterpret_cast<const uint4*>(w1 + 32 * c)) : make_uint4(0, 0, 0, 0);
        };
#pragma unroll
        for (int d = 0; d < DEPTH; ++d) fetch(c_lo + d, d);
        if (it == 0) {
            if (plain) {
                pdl_wait();
                pdl_release();
            }
            if (EXT && p.hn_o) {
                stage_normed<WARPS>(p, xs, XS, sl.cnt, s_part);
                for (int i = tid; i < p.xrows * 32; i += THREADS) {  // channels past K of the last chunk
                    const int k = K + (i & 31);
                    if (k < chunks * 32) xs[(size_t)(i >> 5) * XS + k] = from_f<bf16>(0.f);
                }
            } else {
                for (int i = tid; i < p.xrows * chunks * 4; i += THREADS) {
                    const int row = i / (chunks * 4), c = i % (chunks * 4), k = c * 8;
                    uint4 v = make_uint4(0, 0, 0, 0);
                    if (row < sl.cnt && k < K) {
                        const int e = sl.off + row;
                        const long long xr = p.entry_row ? p.entry_row[e] : e;
                        v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p.x) + xr * p.ldx + k);
                    }
                    *reinterpret_cast<uint4*>(xs + (size_t)row * XS + c * 8) = v;
                }
            }
            __syncthreads();
        }
        float prev[4] = {0.f, 0.f, 0.f, 0.f};                      // the residual's values, requested ahead of the product
        if (EXT && p.residual && s == 0 && live) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int n = tile * 16 + g + 8 * (i >> 1), row = 2 * t + (i & 1);
                if (row < sl.cnt && n < p.N) prev[i] = p.y32[(size_t)row * p.ldy32 + n];
            }
        }
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        const uint4* xb = reinterpret_cast<const uint4*>(xs + (size_t)min(g, p.xrows - 1) * XS) + t;   // past the rows: zeros
        for (int c0 = c_lo; c0 < c_hi; c0 += DEPTH) {
#pragma unroll
            for (int d = 0; d < DEPTH; ++d) {
                const int c = c0 + d;
                if (c < c_hi) {
                    const uint4 a = qa[d], b = qb[d];
                    fetch(c + DEPTH, d);
                    const uint4 xv = xb[c * 4];
                    mma_bf16(acc, a.x, b.x, a.y, b.y, xv.x, xv.y);
                    mma_bf16(acc, a.z, b.z, a.w, b.w, xv.z, xv.w);
                }
            }
        }
        if (s != 0) red[w * 32 + lane] = make_float4(acc[0], acc[1], acc[2], acc[3]);
        __syncthreads();
        if (s == 0) {
            for (int s2 = 1; s2 < SPLIT; ++s2) {
                const float4 v = red[(w + s2) * 32 + lane];
                acc[0] += v.x;
                acc[1] += v.y;
                acc[2] += v.z;
                acc[3] += v.w;
            }
        }
        if (s == 0 && live && p.act == GLQ_ACT_SILU_GLU) {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int n = tile * 8 + g, row = 2 * t + i;
                if (row < sl.cnt && 2 * n < p.N) dm_store<bf16, false>(p, sl.off + row, n, p.alpha * dm_glu<bf16>(acc[i], acc[2 + i]));
            }
        } else if (s == 0 && live) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int n = tile * 16 + g + 8 * (i >> 1), row = 2 * t + (i & 1);
                if (row >= sl.cnt || n >= p.N) continue;
                const float v = p.alpha * act_dyn(p.act, acc[i]);
                if (!EXT || !p.residual) {
                    dm_store<bf16>(p, sl.off + row, n, v);
                } else {
                    p.y32[(size_t)row * p.ldy32 + n] = prev[i] + v;
                    if (p.y) reinterpret_cast<bf16*>(p.y)[(size_t)row * p.ldy + n] = from_f<bf16>(prev[i] + v);
                }
            }
        }
        if (it + 1 < iters) __syncthreads();
    }
}

// =====================================================================================================
// generic kernel: any type, any size
// =====================================================================================================
template <typename T>
__global__ void __launch_bounds__(256) dense_generic_kernel(const DmParams p) {
    __shared__ float xs[16][65], ws[16][65];
    pdl_wait();
    pdl_release();
    const DmSlot sl = dm_slot(p, blockIdx.z);
    const int n0 = blockIdx.x * 64;
    const T* Wm = reinterpret_cast<const T*>(p.W) + (size_t)sl.mat * p.N * p.ldw;
    const T* X = reinterpret_cast<const T*>(p.x);
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    for (int m0 = blockIdx.y * 64; m0 < sl.cnt; m0 += gridDim.y * 64) {
        float acc[4][4] = {};
        for (int k0 = 0; k0 < p.K; k0 += 16) {
            __syncthreads();
            for (int i = threadIdx.x; i < 64 * 16; i += 256) {
                const int r = i >> 4, kk = i & 15;
                const bool kin = k0 + kk < p.K;
                float xv = 0.f, wv = 0.f;
                if (kin && m0 + r < sl.cnt) {
                    const int e = sl.off + m0 + r;
                    const long long xr = p.entry_row ? p.entry_row[e] : e;
                    xv = to_f(X[xr * p.ldx + k0 + kk]);
                }
                if (kin && n0 + r < p.N) wv = to_f(Wm[(size_t)(n0 + r) * p.ldw + k0 + kk]);
                xs[kk][r] = xv;
                ws[kk][r] = wv;
            }
            __syncthreads();
#pragma unroll
            for (int kk = 0; kk < 16; ++kk)
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int j = 0; j < 4; ++j) acc[i][j] += xs[kk][ty + 16 * i] * ws[kk][tx + 16 * j];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int m = m0 + ty + 16 * i, n = n0 + tx + 16 * j;
                if (p.act == GLQ_ACT_SILU_GLU) {
                    const float other = __shfl_xor_sync(0xffffffffu, acc[i][j], 8);
                    if (tx < 8 && m < sl.cnt && n < p.N) dm_store<T>(p, sl.off + m, (n0 >> 1) + 8 * j + tx, p.alpha * dm_glu<T>(acc[i][j], other));
                } else if (m < sl.cnt && n < p.N) {
                    dm_store<T>(p, sl.off + m, n, p.alpha * act_dyn(p.act, acc[i][j]));
                }
            }
    }
}

// entry rows of x -> consecutive rows (the token operand of the grouped tensor-core kernel)
__global__ void __launch_bounds__(256) dense_gather_kernel(const DmParams p, bf16* __restrict__ out) {
    pdl_wait();
    pdl_release();
    const int last = __ldg(p.n_slots) - 1;
    const int total = last < 0 ? 0 : __ldg(p.slot_offset + last) + __ldg(p.slot_count + last);
    const int vec = p.K / 8;
    for (int e = blockIdx.x; e < total; e += gridDim.x) {
        const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(p.x) + (long long)p.entry_row[e] * p.ldx);
        uint4* dst = reinterpret_cast<uint4*>(out + (size_t)e * p.K);
        for (int i = threadIdx.x; i < vec; i += 256) dst[i] = src[i];
    }
}

// =====================================================================================================
// tcgen05 kernel: 128 rows x TN features per tile
// =====================================================================================================
constexpr int kDtThreads = 320;        // warp 0: TMA, warp 1: MMA, warps 2..9: epilogue
constexpr int kDtMaxSlots = 1024;

template <int TN> struct DtCfg {
    static constexpr int A_BYTES = 128 * 128, B_BYTES = TN * 128, STAGE = A_BYTES + B_BYTES;
    static constexpr int S = (208 * 1024) / STAGE > 6 ? 6 : (208 * 1024) / STAGE;
    static constexpr size_t SMEM = (size_t)S * STAGE + 1024;
};

template <int TN>
__global__ void __launch_bounds__(kDtThreads, 1) dense_tc_kernel(const __grid_constant__ CUtensorMap ma,
                                                                const __grid_constant__ CUtensorMap mb, const DmParams p) {
    using C = DtCfg<TN>;
    constexpr int S = C::S;
    extern __shared__ unsigned char dt_smem_raw[];
    __shared__ __align__(8) unsigned long long bars[2 * S + 4];
    __shared__ uint32_t s_tmem;
    __shared__ int s_dead;
    __shared__ int s_pre[kDtMaxSlots + 1];      // row tiles before each slot
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t sbase = (smem_u32(dt_smem_raw) + 1023u) & ~1023u;
    const uint32_t full = smem_u32(bars), empty = full + 8 * S, afull = full + 16 * S, aempty = afull + 16;
    volatile int* dead = &s_dead;
    if (threadIdx.x == 0) {
        for (int s = 0; s < S; ++s) {
            mbar_init(full + 8 * s, 1);
            mbar_init(empty + 8 * s, 1);
        }
        for (int b = 0; b < 2; ++b) {
            mbar_init(afull + 8 * b, 1);
            mbar_init(aempty + 8 * b, 8);
        }
        s_dead = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tc_alloc(smem_u32(&s_tmem), 2 * TN);
    pdl_wait();
    pdl_release();
    const int nslots = p.slot_index ? min(__ldg(p.n_slots), p.slots) : 1;
    if (warp == 0) {
        int base = 0;
        for (int s0 = 0; s0 < nslots; s0 += 32) {
            const int s = s0 + lane;
            int v = 0;
            if (s < nslots) v = ((p.slot_index ? __ldg(p.slot_count + s) : p.rows) + 127) / 128;
            int inc = v;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int u = __shfl_up_sync(0xffffffffu, inc, o);
                if (lane >= o) inc += u;
            }
            if (s < nslots) s_pre[s + 1] = base + inc;
            base += __shfl_sync(0xffffffffu, inc, 31);
        }
        if (lane == 0) s_pre[0] = 0;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    const int nft = (p.N + TN - 1) / TN;
    const int total = s_pre[nslots] * nft;
    const int nk = (p.K + 63) / 64;
    // tile -> (slot, row tile, feature tile): row tiles of a slot run fastest, so that they share a weight tile
    auto locate = [&](int tile, int& slot, int& mt, int& ft) {
        int lo = 0, hi = nslots;
        while (hi - lo > 1) {
            const int mid = (lo + hi) >> 1;
            if (s_pre[mid] * nft <= tile) lo = mid;
            else hi = mid;
        }
        slot = lo;
        const int m = s_pre[lo + 1] - s_pre[lo], l = tile - s_pre[lo] * nft;
        ft = l / m;
        mt = l - ft * m;
    };

    if (warp == 0) {
        if (lane == 0) {
            int s = 0, issued = 0;
            uint32_t ph = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
                int slot, mt, ft;
                locate(tile, slot, mt, ft);
                const DmSlot sl = dm_slot(p, slot);
                const int row = sl.off + mt * 128, wrow = sl.mat * p.N + ft * TN;
                for (int k = 0; k < nk; ++k) {
                    ok = tc_wait(empty + 8 * s, ph ^ 1u, dead, 110);
                    if (!ok) break;
                    const uint32_t a = sbase + (uint32_t)s * C::STAGE;
                    mbar_expect_tx(full + 8 * s, C::STAGE);
                    tma_load_2d(a, &ma, k * 64, row, full + 8 * s);
                    tma_load_2d(a + C::A_BYTES, &mb, k * 64, wrow, full + 8 * s);
                    ++issued;
                    if (++s == S) {
                        s = 0;
                        ph ^= 1u;
                    }
                }
            }
            if (*dead) {   // copies in flight must land before the CTA leaves (bounded)
                for (int i = 0; i < S && i < issued; ++i) {
                    if (--s < 0) {
                        s = S - 1;
                        ph ^= 1u;
                    }
                    const unsigned long long t0 = global_ns();
                    while (!mbar_test_wait(full + 8 * s, ph) && global_ns() - t0 < 2000000ull) __nanosleep(64);
                }
            }
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            int s = 0, buf = 0;
            uint32_t ph = 0, aph = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < total && ok; tile += gridDim.x) {
                ok = tc_wait(aempty + 8 * buf, aph ^ 1u, dead, 111);
                if (!ok) break;
                tc_fence_after();
                for (int k = 0; k < nk; ++k) {
                    ok = tc_wait(full + 8 * s, ph, dead, 112);
                    if (!ok) break;
                    tc_fence_after();
                    const uint32_t a = sbase + (uint32_t)s * C::STAGE;
#pragma unroll
                    for (int kk = 0; kk < 4; ++kk)
                        tc_mma_f16(tmem + (uint32_t)(buf * TN), tc_smem_desc(a + 32u * kk), tc_smem_desc(a + C::A_BYTES + 32u * kk),
                                   dt_idesc(TN), (k | kk) != 0);
                    tc_commit(empty + 8 * s);
                    if (++s == S) {
                        s = 0;
                        ph ^= 1u;
                    }
                }
                if (ok) tc_commit(afull + 8 * buf);
                buf ^= 1;
                if (buf == 0) aph ^= 1u;
            }
        }
        __syncwarp();
    } else {
        const int q = warp & 3;              // tensor memory lanes 32 q .. 32 q + 31
        const int half = (warp - 2) >> 2;    // left or right half of the tile's columns
        int buf = 0;
        uint32_t aph = 0;
        for (int tile = blockIdx.x; tile < total; tile += gridDim.x) {
            int slot, mt, ft;
            locate(tile, slot, mt, ft);
            const DmSlot sl = dm_slot(p, slot);
            if (!tc_wait_warp(afull + 8 * buf, aph, dead, 113)) break;
            tc_fence_after();
            const int r = mt * 128 + q * 32 + lane;
            const bool rin = r < sl.cnt;
            const size_t orow = (size_t)(sl.off + r);
#pragma unroll 1
            for (int c0 = half * (TN / 2); c0 < (half + 1) * (TN / 2); c0 += 16) {
                const int n0 = ft * TN + c0;
                if (n0 >= p.N) break;
                uint32_t v[16];
                __syncwarp();
                tc_ld16(tmem + (uint32_t)(buf * TN + c0) + ((uint32_t)(q * 32) << 16), v);
                tc_ld_wait();
                if (!rin) continue;
                float f[16];
                if (p.act == GLQ_ACT_SILU_GLU) {
#pragma unroll
                    for (int j = 0; j < 8; ++j) f[j] = p.alpha * dm_glu<bf16>(__uint_as_float(v[j]), __uint_as_float(v[j + 8]));
                    const int m0 = n0 >> 1;
                    if (p.vec_y)
                        *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.y) + orow * p.ldy + m0) =
                            make_uint4(pack_bf2(f[0], f[1]), pack_bf2(f[2], f[3]), pack_bf2(f[4], f[5]), pack_bf2(f[6], f[7]));
                    else
#pragma unroll
                        for (int j = 0; j < 8; ++j) dm_store<bf16>(p, (int)orow, m0 + j, f[j]);
                    continue;
                }
#pragma unroll
                for (int j = 0; j < 16; ++j) f[j] = p.alpha * act_dyn(p.act, __uint_as_float(v[j]));
                if (p.mul) {
                    const bf16* mr = dm_mul_row<bf16>(p, (int)orow) + n0;
                    if (n0 + 16 <= p.N && p.vec_mul) {
                        const uint4 m0 = reinterpret_cast<const uint4*>(mr)[0], m1 = reinterpret_cast<const uint4*>(mr)[1];
                        const uint32_t mw[8] = {m0.x, m0.y, m0.z, m0.w, m1.x, m1.y, m1.z, m1.w};
#pragma unroll
                        for (int j = 0; j < 8; ++j) {
                            f[2 * j] *= bf_lo(mw[j]);
                            f[2 * j + 1] *= bf_hi(mw[j]);
                        }
                    } else {
#pragma unroll
                        for (int j = 0; j < 16; ++j)
                            if (n0 + j < p.N) f[j] *= to_f(mr[j]);
                    }
                }
                if (p.residual && n0 + 16 <= p.N && p.vec_y32 && (!p.y || p.vec_y)) {
                    float4* dst = reinterpret_cast<float4*>(p.y32 + orow * p.ldy32 + n0);
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        const float4 x = dst[j];
                        f[4 * j] += x.x;
                        f[4 * j + 1] += x.y;
                        f[4 * j + 2] += x.z;
                        f[4 * j + 3] += x.w;
                        dst[j] = make_float4(f[4 * j], f[4 * j + 1], f[4 * j + 2], f[4 * j + 3]);
                    }
                    if (p.y) {
                        uint4* yd = reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.y) + orow * p.ldy + n0);
                        yd[0] = make_uint4(pack_bf2(f[0], f[1]), pack_bf2(f[2], f[3]), pack_bf2(f[4], f[5]), pack_bf2(f[6], f[7]));
                        yd[1] = make_uint4(pack_bf2(f[8], f[9]), pack_bf2(f[10], f[11]), pack_bf2(f[12], f[13]), pack_bf2(f[14], f[15]));
                    }
                } else if (n0 + 16 <= p.split && p.vec_y) {
                    uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.y) + orow * p.ldy + n0);
                    dst[0] = make_uint4(pack_bf2(f[0], f[1]), pack_bf2(f[2], f[3]), pack_bf2(f[4], f[5]), pack_bf2(f[6], f[7]));
                    dst[1] = make_uint4(pack_bf2(f[8], f[9]), pack_bf2(f[10], f[11]), pack_bf2(f[12], f[13]), pack_bf2(f[14], f[15]));
                } else if (!p.residual && n0 >= p.split && n0 + 16 <= p.N && p.vec_y32) {
                    float4* dst = reinterpret_cast<float4*>(p.y32 + orow * p.ldy32 + (n0 - p.split));
#pragma unroll
                    for (int j = 0; j < 4; ++j) dst[j] = make_float4(f[4 * j], f[4 * j + 1], f[4 * j + 2], f[4 * j + 3]);
                } else {
#pragma unroll
                    for (int j = 0; j < 16; ++j)
                        if (n0 + j < p.N) dm_store<bf16, false>(p, (int)orow, n0 + j, f[j]);
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(aempty + 8 * buf);
            buf ^= 1;
            if (buf == 0) aph ^= 1u;
        }
    }
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tc_dealloc(tmem, 2 * TN);
    }
}

// ---- host ---------------------------------------------------------------------------------------------
template <int TN>
static int launch_dt(const DmParams& p, const void* xa, long xrows, long ldx, long nmat, long tiles, void* stream) {
    CUtensorMap ma, mb;
    if (!make_map(&ma, xa, xrows, p.K, ldx, 128) || !make_map(&mb, p.W, nmat * p.N, p.K, p.ldw, TN)) return GLQ_ERR_UNSUPPORTED;
    const int grid = (int)std::max<long>(1, std::min<long>(tiles, dn_sms()));
    return dn_launch(dense_tc_kernel<TN>, dim3(grid), kDtThreads, DtCfg<TN>::SMEM, stream, ma, mb, p);
}

}  // namespace glq

using namespace glq;

extern "C" const char* glq_dense_status_string(int status) {
    switch (status) {
        case GLQ_OK: return "ok";
        case GLQ_ERR_ARG: return "invalid argument";
        case GLQ_ERR_ALIGN: return "misaligned pointer or leading dimension";
        case GLQ_ERR_UNSUPPORTED: return "unsupported shape";
        case GLQ_ERR_CUDA: return "CUDA error";
        case GLQ_ERR_WORKSPACE: return "workspace too small";
    }
    return "unknown status";
}
extern "C" int glq_dense_last_cuda_error(void) { return g_dense_cuda_error; }
extern "C" int glq_dense_debug_error(unsigned long long* out4, int clear) {
    DN_CUDA(cudaMemcpyFromSymbol(out4, g_glq_err, 4 * sizeof(unsigned long long)));
    if (clear) {
        const unsigned long long z[4] = {0, 0, 0, 0};
        DN_CUDA(cudaMemcpyToSymbol(g_glq_err, z, sizeof(z)));
    }
    return GLQ_OK;
}

// rows per problem up to which the streaming kernel runs (weights are read once per 8 rows)
static constexpr int kStreamRows = 8;
static size_t stream_row_bytes(int K) { return (size_t)(cdiv_i(K, 32) + 1) * 64; }
static int stream_rows(const glq_dense_mm_t* a) { return std::min(8, (a->slot_index ? a->max_slot_rows : a->rows) + 1); }

extern "C" int glq_dense_matmul_path(const glq_dense_mm_t* a) {
    if (a->dtype != GLQ_DT_BF16 || a->K % 8 || a->ldw % 8 || (!a->hn_o && (a->ldx % 8 || !al16(a->x))) || !al16(a->W)) return 0;
    const int rows = a->slot_index ? a->max_slot_rows : a->rows;
    if (rows <= kStreamRows && stream_row_bytes(a->K) * stream_rows(a) <= 200 * 1024) return 1;
    if ((a->slot_index && a->max_slots > kDtMaxSlots) || (a->entry_row && !a->gather) || !encode_tiled()) return 0;
    return 2;
}

extern "C" int glq_dense_matmul(const glq_dense_mm_t* a, void* stream) {
    if (!a || a->N <= 0 || a->K <= 0 || a->rows < 0 || a->split < 0 || a->split > a->N) return GLQ_ERR_ARG;
    if (a->dtype != GLQ_DT_BF16 && a->dtype != GLQ_DT_F32) return GLQ_ERR_ARG;
    if (a->ldw && a->ldw < a->K) return GLQ_ERR_ARG;
    if (a->rows == 0) return GLQ_OK;
    const bool grouped = a->slot_index != nullptr;
    if ((!a->x && !a->hn_o) || !a->W || (a->split > 0 && !a->y) || (a->split < a->N && !a->y32)) return GLQ_ERR_ARG;
    if (a->act == GLQ_ACT_SILU_GLU && (a->N % 16 || a->split != a->N)) return GLQ_ERR_ARG;
    if (a->residual && (a->split != 0 || grouped || a->mul)) return GLQ_ERR_ARG;
    if (a->mul && a->act == GLQ_ACT_SILU_GLU) return GLQ_ERR_ARG;
    if (a->mul_row && a->mul_rows <= 0) return GLQ_ERR_ARG;
    if (grouped && (!a->n_slots || !a->slot_count || !a->slot_offset || a->max_slots <= 0 || a->max_slot_rows <= 0 || a->n_matrices <= 0))
        return GLQ_ERR_ARG;
    if (!grouped && a->entry_row) return GLQ_ERR_ARG;
    DmParams p{};
    p.x = a->x;
    p.W = a->W;
    p.y = a->y;
    p.y32 = a->y32;
    p.slot_index = a->slot_index;
    p.n_slots = a->n_slots;
    p.slot_count = a->slot_count;
    p.slot_offset = a->slot_offset;
    p.entry_row = a->entry_row;
    p.ldx = a->ldx;
    p.ldw = a->ldw ? a->ldw : a->K;
    p.ldy = a->ldy;
    p.ldy32 = a->ldy32;
    p.N = a->N;
    p.K = a->K;
    p.rows = a->rows;
    p.slots = grouped ? a->max_slots : 1;
    p.split = a->split;
    p.act = a->act;
    p.alpha = a->alpha;
    p.mul = a->mul;
    p.ldmul = a->ldmul;
    p.mul_row = a->mul_row;
    p.mul_rows = a->mul_rows;
    p.vec_mul = a->mul && al16(a->mul) && a->ldmul % 8 == 0;
    p.residual = a->residual;
    p.vec_y = a->y && al16(a->y) && a->ldy % 8 == 0;
    p.vec_y32 = a->y32 && al16(a->y32) && a->ldy32 % 4 == 0 && a->split % 4 == 0;
    const int path = glq_dense_matmul_path(a);
    if (a->hn_o) {
        if (path != 1 || grouped || a->hn_heads <= 0 || a->K % a->hn_heads || !a->hn_g || !a->hn_w || !al16(a->hn_o)) return GLQ_ERR_ARG;
        p.hn_o = a->hn_o;
        p.hn_g = a->hn_g;
        p.hn_w = a->hn_w;
        p.hn_ldg = a->hn_ldg;
        p.hn_heads = a->hn_heads;
        p.hn_eps = a->hn_eps;
    }
    const int rows_max = grouped ? a->max_slot_rows : a->rows;
    if (path == 1) {
        const int tiles = cdiv_i(a->N, 16), sms = dn_sms();
        p.xrows = stream_rows(a);
        auto go = [&](auto kern, int warps, int grid) {
            const size_t smem = stream_row_bytes(a->K) * p.xrows + (size_t)warps * 32 * sizeof(float4);
            return dn_launch(kern, dim3(grid, p.slots), warps * 32, smem, stream, p);
        };
        // measured on 1 x N x K products of 6 to 25 MB: many tiles walk over resident CTAs; a few per SM fit one wave of
        // small CTAs; less than one per SM takes deep loads, with sixteen warps on a tile when rows are long
        const long work = (long)tiles * p.slots;
        auto pick = [&](auto ext) {
            constexpr bool EXT = decltype(ext)::value;
            if (work > 12L * sms) return go(dense_stream_kernel<8, 4, 8, 2, EXT>, 8, std::min(cdiv_i(tiles, 2), 2 * sms));
            if (work > 3L * sms && a->K < 4096) return go(dense_stream_kernel<4, 4, 8, 4, EXT>, 4, tiles);
            if (work > sms) return go(dense_stream_kernel<8, 8, 4, 3, EXT>, 8, tiles);
            if (a->K >= 2304) return go(dense_stream_kernel<16, 16, 8, 1, EXT>, 16, tiles);
            return go(dense_stream_kernel<8, 8, 8, 2, EXT>, 8, tiles);
        };
        return a->hn_o || a->residual ? pick(std::true_type()) : pick(std::false_type());
    }
    if (path == 2) {
        const void* xa = a->x;
        long ldx = a->ldx;
        if (a->entry_row) {
            if (!al16(a->gather)) return GLQ_ERR_ALIGN;
            const int st = dn_launch(dense_gather_kernel, dim3(std::min(a->rows, 8 * dn_sms())), 256, 0, stream, p,
                                     reinterpret_cast<bf16*>(a->gather));
            if (st != GLQ_OK) return st;
            xa = a->gather;
            ldx = a->K;
            p.entry_row = nullptr;
        }
        const long mt = grouped ? a->rows / 128 + p.slots : cdiv_i(a->rows, 128);
        const long sms = dn_sms();
        const long nmat = grouped ? a->n_matrices : 1;
        // feature tile of the shortest estimate: rounds over the SMs times a tile's cost, which grows slowly with its width
        // (measured 0.33 and 0.45 us per 64 channels at 64 and 256 features)
        auto cost = [&](int tn) { return cdiv_i(mt * cdiv_i(a->N, tn), sms) * (0.28 + 0.17 * tn / 256); };
        const double c64 = cost(64), c128 = a->N > 64 ? cost(128) : 1e30, c256 = a->N > 128 ? cost(256) : 1e30;
        if (c256 <= c128 && c256 <= c64) return launch_dt<256>(p, xa, a->rows, ldx, nmat, mt * cdiv_i(a->N, 256), stream);
        if (c128 <= c64) return launch_dt<128>(p, xa, a->rows, ldx, nmat, mt * cdiv_i(a->N, 128), stream);
        return launch_dt<64>(p, xa, a->rows, ldx, nmat, mt * cdiv_i(a->N, 64), stream);
    }
    const dim3 grid(cdiv_i(a->N, 64), std::min(cdiv_i(rows_max, 64), 1024), p.slots);
    if (grid.z > 65535) return GLQ_ERR_UNSUPPORTED;
    if (a->dtype == GLQ_DT_F32) return dn_launch(dense_generic_kernel<float>, grid, 256, 0, stream, p);
    return dn_launch(dense_generic_kernel<bf16>, grid, 256, 0, stream, p);
}
