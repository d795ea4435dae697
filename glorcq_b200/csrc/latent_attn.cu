// Latent attention: keys and values of a position are projections of one latent vector (plus a rotated key part that
// all heads share), and the cache holds only the latent and that part.
//   * the norm of the new latents, the rotation of the shared key part and of every head's rotated query part, and the
//     cache write are a launch of their own before the prompt form and part of the absorbed form's first launch;
//   * absorbed form (decode steps, short portions): the query is taken through the key projection once
//     (q' = W_uk^T q), scores and the weighted sum run over the cached latents of all heads at once on the tensor
//     cores, and the value projection follows for the sum; positions are split over CTAs;
//   * prompt form: causal attention over keys and values that products have expanded from the cached latents, on tcgen05
//     (values expanded in transposed form) or, for head sizes that form does not cover, on mma.sync.
// Scores, softmax weights and sums are float; where a float operand enters a tensor-core product (q', the weights) it
// goes in as a sum of two bf16 numbers.
#include "attn_tc.cuh"

namespace glq {

struct LaParams {
    void* q;
    const float* ckr;
    const float* gate;
    const float* norm_w;
    const float* cos_t;
    const float* sin_t;
    void* cache;
    const void* ukt;
    const void* uv;
    void* out;
    const void* kv;
    const long long* start;
    long long ldq, ldk, ldc, ldkv;
    int B, T, H, D, R, V, K, rot_dims, max_len, S;
    float scale, eps;
    // absorbed form
    void* qa;            // bf16: two planes (B, rows16, KRp); generic: float (B, rows16, K + R)
    float* po;           // (B, tiles, splits, 16, K)
    float* pm;           // (B, tiles, splits, 16)
    float* pl;
    float* ol;           // (B * T, H, K) weighted latents
    int KRp, rows16, splits;
};

template <typename T> __device__ __forceinline__ void rotate_part(T* x, const float* cs, const float* sn, int half, int lane) {
    for (int i = lane; i < half; i += 32) {
        const float u = to_f(x[i]), v = to_f(x[i + half]), c = cs[i], s = sn[i];
        x[i] = from_f<T>(u * c - v * s);
        x[i + half] = from_f<T>(v * c + u * s);
    }
}

// one new position: its latent normed, its key part turned, both into the cache
template <typename T>
__device__ __forceinline__ void cache_row(const LaParams& p, size_t row, long long pos, float* red) {
    const int b = (int)(row / p.T), half = p.rot_dims / 2;
    const float* c = p.ckr + row * p.ldk;
    const float* kr = c + p.K;
    T* dst = reinterpret_cast<T*>(p.cache) + ((size_t)b * p.max_len + pos) * p.ldc;
    const float* cs = p.cos_t + (size_t)pos * half;
    const float* sn = p.sin_t + (size_t)pos * half;
    float ss = 0.f;
    for (int i = threadIdx.x; i < p.K; i += blockDim.x) ss += c[i] * c[i];
    const float inv = 1.f / sqrtf(block_sum(ss, red) / p.K + p.eps);
    for (int i = threadIdx.x; i < p.K; i += blockDim.x) dst[i] = from_f<T>(c[i] * inv * p.norm_w[i]);
    for (int i = threadIdx.x; i < p.R; i += blockDim.x) {
        float v = kr[i];
        if (i < half) v = kr[i] * cs[i] - kr[i + half] * sn[i];
        else if (i < 2 * half) v = kr[i] * cs[i - half] + kr[i - half] * sn[i - half];
        dst[p.K + i] = from_f<T>(v);
    }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LaParams p) {
    __shared__ float red[32];
    pdl_wait();
    pdl_release();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const size_t row = blockIdx.x;
    const long long pos = *p.start + (long long)(row % p.T);
    if (pos < 0 || pos >= p.max_len) return;
    cache_row<T>(p, row, pos, red);
    const int half = p.rot_dims / 2;
    for (int h = warp; h < p.H; h += 4)
        rotate_part(reinterpret_cast<T*>(p.q) + row * p.ldq + (size_t)h * (p.D + p.R) + p.D, p.cos_t + (size_t)pos * half,
                    p.sin_t + (size_t)pos * half, half, lane);
}

// 8 consecutive values from global memory
__device__ __forceinline__ void ld8(const bf16* p, float (&v)[8]) {
    const uint4 w = *reinterpret_cast<const uint4*>(p);
    v[0] = bf_lo(w.x), v[1] = bf_hi(w.x), v[2] = bf_lo(w.y), v[3] = bf_hi(w.y);
    v[4] = bf_lo(w.z), v[5] = bf_hi(w.z), v[6] = bf_lo(w.w), v[7] = bf_hi(w.w);
}
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = p[i];
}

constexpr int kHmRows = 8;       // activation rows staged at a time

// out[r, n] = sum_k W[n, k] xs[r, k] for `nr` staged rows and output rows n = n_lo .. n_hi of one head's matrix;
// lanes of a group share an output row, eight k values each
template <typename T, typename F>
__device__ __forceinline__ void head_products(const T* __restrict__ W, int n_lo, int n_hi, int Kd, bool vec, const float* xs, int ldxs,
                                              int nr, F emit) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    int gl = 1;                                             // lanes per output row
    while (gl < 32 && gl * 8 < Kd) gl <<= 1;
    const int gi = lane / gl, li = lane % gl, per = 32 / gl;
    for (int n0 = n_lo + warp * per; n0 < n_hi; n0 += 8 * per) {
        const int n = n0 + gi;
        float acc[kHmRows];
#pragma unroll
        for (int r = 0; r < kHmRows; ++r) acc[r] = 0.f;
        if (n < n_hi) {
            for (int k = li * 8; k < Kd; k += gl * 8) {
                float w[8];
                if (vec) {
                    ld8(W + (size_t)n * Kd + k, w);
                } else {
#pragma unroll
                    for (int i = 0; i < 8; ++i) w[i] = k + i < Kd ? to_f(W[(size_t)n * Kd + k + i]) : 0.f;
                }
#pragma unroll
                for (int r = 0; r < kHmRows; ++r)
                    if (r < nr)
#pragma unroll
                        for (int i = 0; i < 8; ++i) acc[r] += w[i] * xs[r * ldxs + k + i];
            }
        }
#pragma unroll
        for (int r = 0; r < kHmRows; ++r)
            if (r < nr) {
                float a = acc[r];
                for (int o = gl >> 1; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
                if (li == 0 && n < n_hi) emit(r, n, a);
            }
    }
}

// q' of a head: (K, D) times the unrotated query, then the rotated query, all times scale * log2(e); the blocks behind
// the last head write the cache rows of the new positions
template <typename T, bool SPLIT>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const LaParams p) {
    extern __shared__ float xs[];
    __shared__ float red[32];
    const int Dp = (p.D + 7) / 8 * 8;
    pdl_wait();
    pdl_release();
    const int h = blockIdx.x, rows = p.B * p.T, half = p.rot_dims / 2;
    const long long start = *p.start;
    if (h == p.H) {
        for (int row = blockIdx.z * gridDim.y + blockIdx.y; row < rows; row += gridDim.y * gridDim.z) {
            const long long pos = start + row % p.T;
            if (pos >= 0 && pos < p.max_len) cache_row<T>(p, row, pos, red);
        }
        return;
    }
    const int per = (p.K + gridDim.y - 1) / gridDim.y, n_lo = blockIdx.y * per, n_hi = min(p.K, n_lo + per);
    const float sc = p.scale * 1.4426950408889634f;
    const int ld = SPLIT ? p.KRp : p.K + p.R;
    const size_t plane = (size_t)p.B * p.rows16 * p.KRp;
    auto put = [&](int row, int n, float v) {
        const size_t o = ((size_t)(row / p.T) * p.rows16 + (size_t)(row % p.T) * p.H + h) * ld + n;
        if constexpr (SPLIT) {
            const bf16 hi = __float2bfloat16_rn(v);
            reinterpret_cast<bf16*>(p.qa)[o] = hi;
            reinterpret_cast<bf16*>(p.qa)[plane + o] = __float2bfloat16_rn(v - __bfloat162float(hi));
        } else {
            reinterpret_cast<float*>(p.qa)[o] = v;
        }
    };
    for (int r0 = blockIdx.z * kHmRows; r0 < rows; r0 += gridDim.z * kHmRows) {
        const int nr = min(kHmRows, rows - r0);
        __syncthreads();
        for (int i = threadIdx.x; i < nr * Dp; i += 256) {
            const int r = i / Dp, d = i % Dp;
            xs[i] = d < p.D ? to_f(reinterpret_cast<const T*>(p.q)[(size_t)(r0 + r) * p.ldq + (size_t)h * (p.D + p.R) + d]) : 0.f;
        }
        __syncthreads();
        head_products(reinterpret_cast<const T*>(p.ukt) + (size_t)h * p.K * p.D, n_lo, n_hi, p.D, p.D % 8 == 0, xs, Dp, nr,
                      [&](int r, int n, float v) { put(r0 + r, n, v * sc); });
        if (blockIdx.y == 0) {
            const int tail = ld - p.K;               // rotated part, then the padding
            for (int i = threadIdx.x; i < nr * tail; i += 256) {
                const int r = i / tail, j = i % tail;
                float v = 0.f;
                if (j < p.R) {
                    const T* q = reinterpret_cast<const T*>(p.q) + (size_t)(r0 + r) * p.ldq + (size_t)h * (p.D + p.R) + p.D;
                    const long long pos = min((long long)p.max_len - 1, max(0LL, start + (r0 + r) % p.T));
                    v = to_f(q[j]);
                    if (j < half) v = v * p.cos_t[pos * half + j] - to_f(q[j + half]) * p.sin_t[pos * half + j];
                    else if (j < 2 * half) v = v * p.cos_t[pos * half + j - half] + to_f(q[j - half]) * p.sin_t[pos * half + j - half];
                }
                put(r0 + r, p.K + j, v * sc);
            }
        }
    }
}

constexpr int kMaxSplits = 128;
constexpr int kAbPos = 64;       // positions per stage of the absorbed form

// stages of split z for `total` positions, and how many splits have any
struct SplitRange {
    int lo, hi, used;
};
__device__ __forceinline__ SplitRange split_range(const LaParams& p, int z, int total) {
    const int ntile = (total + kAbPos - 1) / kAbPos, per = (ntile + p.splits - 1) / p.splits;
    return {z * per, min(ntile, (z + 1) * per), (ntile + per - 1) / per};
}

// weighted latent of a (row, head): the splits' sums combined; grid (rows, heads, column parts)
__global__ void __launch_bounds__(512) latent_combine_kernel(const LaParams p) {
    __shared__ float sw[kMaxSplits], part[4][128];
    pdl_wait();
    pdl_release();
    const int row = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31;
    const int rr = (row % p.T) * p.H + h;
    // splits behind the last position left their sums unwritten
    const int used = p.splits > 1 ? split_range(p, 0, (int)min((long long)p.max_len, *p.start + p.T)).used : 1;
    const size_t first = (((size_t)(row / p.T) * (p.rows16 / 16) + rr / 16) * p.splits) * 16 + rr % 16;     // split z: + 16 z
    if (threadIdx.x < 32) {
        float mz[kMaxSplits / 32], lz[kMaxSplits / 32], m = -INFINITY;
#pragma unroll
        for (int u = 0; u < kMaxSplits / 32; ++u) {
            const int z = lane + 32 * u;
            mz[u] = z < p.splits ? p.pm[first + 16 * z] : -INFINITY;
            lz[u] = z < p.splits ? p.pl[first + 16 * z] : 0.f;
            m = fmaxf(m, mz[u]);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        float l = 0.f;
#pragma unroll
        for (int u = 0; u < kMaxSplits / 32; ++u) {
            mz[u] = exp2f(mz[u] - m);
            l += mz[u] * lz[u];
        }
        const float inv = 1.f / warp_sum(l);
#pragma unroll
        for (int u = 0; u < kMaxSplits / 32; ++u) sw[lane + 32 * u] = mz[u] * inv;
    }
    __syncthreads();
    // 128 columns at a time, four groups of threads over the splits
    const int per = (p.K + gridDim.z - 1) / gridDim.z, k_hi = min(p.K, (int)(blockIdx.z + 1) * per);
    const int zq = (used + 3) / 4, grp = threadIdx.x >> 7, z0 = grp * zq, z1 = min(used, z0 + zq);
    for (int kb = blockIdx.z * per; kb < k_hi; kb += 128) {
        const int k = kb + (threadIdx.x & 127);
        float v = 0.f;
        if (k < k_hi) {
            const float* po = p.po + first * p.K + k;
#pragma unroll 16
            for (int z = z0; z < z1; ++z) {
                v += sw[z] * po[(size_t)16 * z * p.K];
            }
        }
        part[grp][threadIdx.x & 127] = v;
        __syncthreads();
        if (grp == 0 && k < k_hi)
            p.ol[((size_t)row * p.H + h) * p.K + k] =
                (part[0][threadIdx.x] + part[1][threadIdx.x]) + (part[2][threadIdx.x] + part[3][threadIdx.x]);
        __syncthreads();
    }
}

// the head's value matrix times the weighted latent, times the head's gate
template <typename T>
__global__ void __launch_bounds__(256) latent_value_kernel(const LaParams p) {
    extern __shared__ float xs[];
    const int Kp = (p.K + 7) / 8 * 8;
    pdl_wait();
    pdl_release();
    const int h = blockIdx.x, rows = p.B * p.T;
    const int per = (p.V + gridDim.y - 1) / gridDim.y, n_lo = blockIdx.y * per, n_hi = min(p.V, n_lo + per);
    for (int r0 = blockIdx.z * kHmRows; r0 < rows; r0 += gridDim.z * kHmRows) {
        const int nr = min(kHmRows, rows - r0);
        __syncthreads();
        for (int i = threadIdx.x; i < nr * Kp; i += 256) {
            const int r = i / Kp, k = i % Kp;
            xs[i] = k < p.K ? p.ol[((size_t)(r0 + r) * p.H + h) * p.K + k] : 0.f;
        }
        __syncthreads();
        head_products(reinterpret_cast<const T*>(p.uv) + (size_t)h * p.V * p.K, n_lo, n_hi, p.K, p.K % 8 == 0, xs, Kp, nr,
                      [&](int r, int n, float v) {
                          const size_t row = r0 + r;
                          reinterpret_cast<T*>(p.out)[row * p.H * p.V + (size_t)h * p.V + n] =
                              from_f<T>(v * sigmoid_f(p.gate[row * p.ldk + h]));
                      });
    }
}

// ---- attention over the cached latents, tensor cores ----------------------------------------------------

constexpr int kAbThreads = 512;

// 16 rows (query position, head) against one split of the positions; NT: 8-column tiles of the latent per warp
template <int NT>
__global__ void __launch_bounds__(kAbThreads) latent_absorbed_kernel(const LaParams p) {
    extern __shared__ __align__(16) unsigned char la_raw[];
    const int KRp = p.KRp, LD = KRp + 8;
    bf16* qh = reinterpret_cast<bf16*>(la_raw);              // [16][LD]
    bf16* ql = qh + 16 * LD;                                 // [16][LD]
    bf16* cs = ql + 16 * LD;                                 // [2][kAbPos][LD]
    bf16* ph = cs + 2 * kAbPos * LD;                         // [16][kAbPos + 8]
    bf16* pl = ph + 16 * (kAbPos + 8);
    __shared__ float sc[4][16][kAbPos + 1], s_m[16], s_l[16], s_f[16];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    const int rt = blockIdx.x, z = blockIdx.y, b = blockIdx.z, tiles = gridDim.x;
    const int KR = p.K + p.R;
    pdl_wait();
    pdl_release();
    const long long start = *p.start;
    const int total = (int)min((long long)p.max_len, start + p.T);
    const SplitRange sr = split_range(p, z, total);
    const int c_lo = sr.lo, c_hi = sr.hi;
    const bf16* cache = reinterpret_cast<const bf16*>(p.cache) + (size_t)b * p.max_len * p.ldc;
    auto load = [&](int c, int buf) {        // warp = rows warp, warp + 16, ..
        const uint32_t dst = smem_u32(cs + (size_t)buf * kAbPos * LD);
#pragma unroll 4
        for (int r = warp; r < kAbPos; r += kAbThreads / 32) {
            const int pos = c * kAbPos + r;
            const bf16* src = cache + (size_t)(pos < total ? pos : 0) * p.ldc;
            for (int cc = 8 * lane; cc < KRp; cc += 256) cpa16(dst + (r * LD + cc) * 2, cc < KR ? src + cc : src, pos < total && cc < KR);
        }
        cpa_commit();
    };
    if (c_lo < c_hi) {      // the queries' copies join the first stage's group
        const bf16* src = reinterpret_cast<const bf16*>(p.qa) + ((size_t)b * p.rows16 + rt * 16) * KRp;
        const size_t plane = (size_t)p.B * p.rows16 * KRp;
        const int vec = KRp / 8;
        for (int i = tid; i < 16 * vec; i += kAbThreads) {
            const int r = i / vec, cc = (i % vec) * 8;
            const bool live = rt * 16 + r < p.T * p.H;
            const bf16* q = live ? src + (size_t)r * KRp + cc : src;
            cpa16(smem_u32(qh + r * LD + cc), q, live);
            cpa16(smem_u32(ql + r * LD + cc), q + plane, live);
        }
        load(c_lo, 0);
    }
    if (tid < 16) {
        s_m[tid] = -INFINITY;
        s_l[tid] = 0.f;
    }
    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    for (int c = c_lo; c < c_hi; ++c) {
        const int buf = (c - c_lo) & 1;
        if (c + 1 < c_hi) {
            load(c + 1, buf ^ 1);
            cpa_wait<1>();
        } else {
            cpa_wait<0>();
        }
        __syncthreads();
        const bf16* ct = cs + (size_t)buf * kAbPos * LD;
        // scores: warp = 16 positions, a quarter of the columns (every fourth step of 32)
        float s[4][4];                       // query part x 8-position tile
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[u][e] = 0.f;
        const int wp = warp & 3, wk = warp >> 2;
        const uint32_t ba = smem_u32(ct + (16 * wp + (lane & 7) + (lane >> 4) * 8) * LD + ((lane >> 3) & 1) * 8);
        const uint32_t qo = (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * LD + (lane >> 4) * 8) * 2;
        const uint32_t qha = smem_u32(qh) + qo, qla = smem_u32(ql) + qo;
#pragma unroll 2
        for (int k0 = 32 * wk; k0 < KRp; k0 += 128) {
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const uint32_t o = (uint32_t)(k0 + 16 * u) * 2;
                uint32_t b0, b1, b2, b3, a0, a1, a2, a3;
                ldsm4(ba + o, b0, b1, b2, b3);
                ldsm4(qha + o, a0, a1, a2, a3);
                mma_bf16(s[0], a0, a1, a2, a3, b0, b1);
                mma_bf16(s[1], a0, a1, a2, a3, b2, b3);
                ldsm4(qla + o, a0, a1, a2, a3);
                mma_bf16(s[2], a0, a1, a2, a3, b0, b1);
                mma_bf16(s[3], a0, a1, a2, a3, b2, b3);
            }
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) sc[wk][g + 8 * (e >> 1)][16 * wp + 8 * n + 2 * t4 + (e & 1)] = s[n][e] + s[2 + n][e];
        __syncthreads();
        // softmax: warp = a row, lane = positions lane and lane + 32
        {
            const int r = warp, row = rt * 16 + r;
            const long long lim = row < p.T * p.H ? min((long long)total - 1, start + row / p.H) - c * kAbPos : -1;   // last position seen
            float v[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) v[u] = lane + 32 * u <= lim ? (sc[0][r][lane + 32 * u] + sc[1][r][lane + 32 * u]) + (sc[2][r][lane + 32 * u] + sc[3][r][lane + 32 * u])
                                                                          : -INFINITY;
            float mx = fmaxf(v[0], v[1]);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mo = s_m[r], mn = fmaxf(mo, mx);
            const float f = mn == -INFINITY ? 1.f : exp2f(mo - mn);
            float sum = 0.f;
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const float pv = lane + 32 * u <= lim ? exp2f(v[u] - mn) : 0.f;
                sum += pv;
                const bf16 hi = __float2bfloat16_rn(pv);
                ph[r * (kAbPos + 8) + lane + 32 * u] = hi;
                pl[r * (kAbPos + 8) + lane + 32 * u] = __float2bfloat16_rn(pv - __bfloat162float(hi));
            }
            sum = warp_sum(sum);
            __syncwarp();
            if (lane == 0) {
                s_m[r] = mn;
                s_l[r] = s_l[r] * f + sum;
                s_f[r] = f;
            }
        }
        __syncthreads();
        const float f0 = s_f[g], f1 = s_f[g + 8];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            acc[j][0] *= f0;
            acc[j][1] *= f0;
            acc[j][2] *= f1;
            acc[j][3] *= f1;
        }
        // weighted latents: warp = NT column tiles
#pragma unroll
        for (int kk = 0; kk < kAbPos / 16; ++kk) {
            const int off = ((lane & 7) + ((lane >> 3) & 1) * 8) * (kAbPos + 8) + 16 * kk + (lane >> 4) * 8;
            uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
            ldsm4(smem_u32(ph + off), h0, h1, h2, h3);
            ldsm4(smem_u32(pl + off), l0, l1, l2, l3);
#pragma unroll
            for (int jp = 0; jp < NT / 2; ++jp) {
                const int col = (warp * NT + 2 * jp) * 8;
                if (col >= p.K) continue;
                uint32_t b0, b1, b2, b3;
                ldsm4_t(smem_u32(ct + (16 * kk + (lane & 7) + ((lane >> 3) & 1) * 8) * LD + col + (lane >> 4) * 8), b0, b1, b2, b3);
                mma_bf16(acc[2 * jp], h0, h1, h2, h3, b0, b1);
                mma_bf16(acc[2 * jp], l0, l1, l2, l3, b0, b1);
                mma_bf16(acc[2 * jp + 1], h0, h1, h2, h3, b2, b3);
                mma_bf16(acc[2 * jp + 1], l0, l1, l2, l3, b2, b3);
            }
        }
        __syncthreads();
    }
    __syncthreads();
    const size_t pi = (((size_t)b * tiles + rt) * p.splits + z) * 16;
    if (tid < 16) {
        p.pm[pi + tid] = s_m[tid];
        p.pl[pi + tid] = s_l[tid];
    }
    if (c_lo >= c_hi) return;        // nothing to add: weight zero, the sums are not read
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        const int col = (warp * NT + j) * 8 + 2 * t4;
        if (col < p.K) {
            *reinterpret_cast<float2*>(p.po + (pi + g) * p.K + col) = make_float2(acc[j][0], acc[j][1]);
            *reinterpret_cast<float2*>(p.po + (pi + g + 8) * p.K + col) = make_float2(acc[j][2], acc[j][3]);
        }
    }
}

// the same for any type and size: one row per CTA, one split
template <typename T>
__global__ void __launch_bounds__(128) latent_absorbed_generic_kernel(const LaParams p) {
    extern __shared__ float ga[];
    const int KR = p.K + p.R;
    float* qs = ga;                  // [KR]
    float* ps = qs + KR;             // [128]
    float* os = ps + 128;            // [K]
    __shared__ float red[32];
    pdl_wait();
    pdl_release();
    const int row = blockIdx.x, b = blockIdx.y, tiles = p.rows16 / 16;
    const long long start = *p.start;
    const int total = (int)min((long long)p.max_len, start + row / p.H + 1);
    const T* cache = reinterpret_cast<const T*>(p.cache) + (size_t)b * p.max_len * p.ldc;
    const float* q = reinterpret_cast<const float*>(p.qa) + ((size_t)b * p.rows16 + row) * KR;
    for (int i = threadIdx.x; i < KR; i += 128) qs[i] = q[i];
    for (int i = threadIdx.x; i < p.K; i += 128) os[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int c0 = 0; c0 < total; c0 += 128) {
        __syncthreads();
        const int pos = c0 + threadIdx.x;
        float s = -INFINITY;
        if (pos < total) {
            const T* c = cache + (size_t)pos * p.ldc;
            float a = 0.f;
            for (int k = 0; k < KR; ++k) a += qs[k] * to_f(c[k]);
            s = a;
        }
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float mn = fmaxf(m, mx), f = exp2f(m - mn);
        ps[threadIdx.x] = pos < total ? exp2f(s - mn) : 0.f;
        l = l * f + block_sum(ps[threadIdx.x], red);
        m = mn;
        __syncthreads();
        const int n = min(128, total - c0);
        for (int k = threadIdx.x; k < p.K; k += 128) {
            float a = os[k] * f;
            for (int j = 0; j < n; ++j) a += ps[j] * to_f(cache[(size_t)(c0 + j) * p.ldc + k]);
            os[k] = a;
        }
    }
    const size_t pi = (((size_t)b * tiles + row / 16) * p.splits) * 16 + row % 16;
    for (int k = threadIdx.x; k < p.K; k += 128) p.po[pi * p.K + k] = os[k];
    if (threadIdx.x == 0) {
        p.pm[pi] = m;
        p.pl[pi] = l;
    }
}

// ---- prompt form -------------------------------------------------------------------------------------------
template <int DK, int DV> struct LpCfg {
    static constexpr int LK = DK + 8, LV = DV + 8, STAGE = 64 * (LK + LV);
    static constexpr size_t SMEM = (size_t)2 * STAGE * 2;
};

template <int DK, int DV>
__global__ void __launch_bounds__(128) latent_prefill_kernel(const LaParams p) {
    using C = LpCfg<DK, DV>;
    constexpr int LK = C::LK, LV = C::LV, KS = DK / 16, NT = DV / 8;
    extern __shared__ __align__(16) unsigned char lp_raw[];
    bf16* sm = reinterpret_cast<bf16*>(lp_raw);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_release();
    // work order: the query blocks with the most keys first, over all heads and sequences
    const int n_hb = p.H * p.B;
    const int qb = (int)(gridDim.x / n_hb) - 1 - (int)(blockIdx.x / n_hb);
    const int h = (int)(blockIdx.x % n_hb) % p.H, b = (int)(blockIdx.x % n_hb) / p.H;
    const int start = p.S - p.T;
    const int q0 = qb * 64 + 16 * warp;                     // first query row of the warp
    const int DR = p.D + p.R;
    const bf16* kv = reinterpret_cast<const bf16*>(p.kv) + (size_t)b * p.S * p.ldkv;
    const bf16* rot = reinterpret_cast<const bf16*>(p.cache) + (size_t)b * p.max_len * p.ldc + p.K;
    auto load = [&](int kb, int buf) {
        bf16* ks = sm + (size_t)buf * C::STAGE;
        bf16* vs = ks + 64 * LK;
        for (int i = tid; i < 64 * (DK / 8); i += 128) {
            const int r = i / (DK / 8), cc = (i % (DK / 8)) * 8, key = kb * 64 + r;
            const bool live = key < p.S && cc < DR;
            const bf16* src = !live ? kv : (cc < p.D ? kv + (size_t)key * p.ldkv + (size_t)h * p.D + cc
                                                     : rot + (size_t)key * p.ldc + (cc - p.D));
            cpa16(smem_u32(ks + r * LK + cc), src, live);
        }
        for (int i = tid; i < 64 * (DV / 8); i += 128) {
            const int r = i / (DV / 8), cc = (i % (DV / 8)) * 8, key = kb * 64 + r;
            const bool live = key < p.S && cc < p.V;
            cpa16(smem_u32(vs + r * LV + cc), live ? kv + (size_t)key * p.ldkv + (size_t)p.H * p.D + (size_t)h * p.V + cc : kv, live);
        }
        cpa_commit();
    };
    const int last = min(p.S, start + min(p.T, qb * 64 + 64)) - 1;      // last key any row of the block sees
    const int nkb = last / 64 + 1;
    load(0, 0);
    uint32_t qf[KS][4];
    {
        const int r0 = q0 + g, r1 = q0 + g + 8;
        const bf16* qp = reinterpret_cast<const bf16*>(p.q) + (size_t)h * DR;
        const bf16* p0 = qp + ((size_t)b * p.T + min(r0, p.T - 1)) * p.ldq;
        const bf16* p1 = qp + ((size_t)b * p.T + min(r1, p.T - 1)) * p.ldq;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int col = 16 * ks + 8 * u + 2 * t;
                qf[ks][2 * u] = col < DR ? *reinterpret_cast<const uint32_t*>(p0 + col) : 0u;
                qf[ks][2 * u + 1] = col < DR ? *reinterpret_cast<const uint32_t*>(p1 + col) : 0u;
            }
    }
    float o[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    const float sc = p.scale * 1.4426950408889634f;
    for (int kb = 0; kb < nkb; ++kb) {
        if (kb + 1 < nkb) {
            load(kb + 1, (kb + 1) & 1);
            cpa_wait<1>();
        } else {
            cpa_wait<0>();
        }
        __syncthreads();
        const bf16* ks_ = sm + (size_t)(kb & 1) * C::STAGE;
        const bf16* vs_ = ks_ + 64 * LK;
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            if (16 * ks >= DR) continue;
#pragma unroll
            for (int jp = 0; jp < 4; ++jp) {
                uint32_t b0, b1, b2, b3;
                ldsm4(smem_u32(ks_ + (16 * jp + (lane & 7) + (lane >> 4) * 8) * LK + 16 * ks + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
                mma_bf16(s[2 * jp], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b0, b1);
                mma_bf16(s[2 * jp + 1], qf[ks][0], qf[ks][1], qf[ks][2], qf[ks][3], b2, b3);
            }
        }
        const bool edge = kb * 64 + 63 > start + q0;         // some key of the block lies after some row of the warp
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float v = s[j][e] * sc;
                if (edge) {
                    const int key = kb * 64 + 8 * j + 2 * t + (e & 1), row = start + q0 + g + 8 * (e >> 1);
                    if (key > row || key >= p.S) v = -INFINITY;
                }
                s[j][e] = v;
                if (e < 2) mx0 = fmaxf(mx0, v);
                else mx1 = fmaxf(mx1, v);
            }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);
        const float f0 = n0 == -INFINITY ? 0.f : n0, f1 = n1 == -INFINITY ? 0.f : n1;
        const float a0 = ex2(m0 - f0), a1 = ex2(m1 - f1);
        m0 = n0;
        m1 = n1;
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            s[j][0] = ex2(s[j][0] - f0);
            s[j][1] = ex2(s[j][1] - f0);
            s[j][2] = ex2(s[j][2] - f1);
            s[j][3] = ex2(s[j][3] - f1);
            s0 += s[j][0] + s[j][1];
            s1 += s[j][2] + s[j][3];
        }
        l0 = l0 * a0 + s0;
        l1 = l1 * a1 + s1;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            o[j][0] *= a0;
            o[j][1] *= a0;
            o[j][2] *= a1;
            o[j][3] *= a1;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t hi[4], lo[4];
            split_bf2(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
            split_bf2(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
            split_bf2(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
            split_bf2(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
            const int vrow = 16 * kk + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int jp = 0; jp < NT / 2; ++jp) {
                uint32_t b0, b1, b2, b3;
                ldsm4_t(smem_u32(vs_ + vrow * LV + 16 * jp + (lane >> 4) * 8), b0, b1, b2, b3);
                mma_bf16(o[2 * jp], hi[0], hi[1], hi[2], hi[3], b0, b1);
                mma_bf16(o[2 * jp], lo[0], lo[1], lo[2], lo[3], b0, b1);
                mma_bf16(o[2 * jp + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
                mma_bf16(o[2 * jp + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
            }
        }
        __syncthreads();
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int r = q0 + g + 8 * e;
        if (r >= p.T) continue;
        const size_t row = (size_t)b * p.T + r;
        const float inv = sigmoid_f(p.gate[row * p.ldk + h]) / (e ? l1 : l0);
        bf16* y = reinterpret_cast<bf16*>(p.out) + row * p.H * p.V + (size_t)h * p.V;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const int v = 8 * j + 2 * t;
            if (v < p.V) *reinterpret_cast<uint32_t*>(y + v) = pack_bf2(o[j][2 * e] * inv, o[j][2 * e + 1] * inv);
        }
    }
}

}  // namespace glq

using namespace glq;

static LaParams la_params(const glq_latent_t* a) {
    LaParams p{};
    p.q = a->q;
    p.ckr = a->ckr;
    p.gate = a->gate;
    p.norm_w = a->norm_w;
    p.cos_t = a->cos_t;
    p.sin_t = a->sin_t;
    p.cache = a->cache;
    p.ukt = a->ukt;
    p.uv = a->uv;
    p.out = a->out;
    p.kv = a->kv;
    p.start = reinterpret_cast<const long long*>(a->start);
    p.ldq = a->ldq;
    p.ldk = a->ldk;
    p.ldc = a->ldc;
    p.ldkv = a->ldkv;
    p.B = a->B;
    p.T = a->T;
    p.H = a->H;
    p.D = a->D;
    p.R = a->R;
    p.V = a->V;
    p.K = a->K;
    p.rot_dims = a->rot_dims;
    p.max_len = a->max_len;
    p.S = a->S;
    p.scale = a->scale;
    p.eps = a->eps;
    p.KRp = (a->K + a->R + 31) / 32 * 32;
    p.rows16 = (a->T * a->H + 15) / 16 * 16;
    return p;
}
static bool la_sizes_ok(const glq_latent_t* a) {
    return a && a->B > 0 && a->T >= 0 && a->H > 0 && a->D > 0 && a->R >= 0 && a->V > 0 && a->K > 0 && a->rot_dims >= 0 &&
           a->rot_dims % 2 == 0 && a->rot_dims <= a->R && a->max_len > 0 && (a->dtype == GLQ_DT_BF16 || a->dtype == GLQ_DT_F32);
}
static size_t la_absorbed_smem(const LaParams& p) {
    return (size_t)(32 + 2 * kAbPos) * (p.KRp + 8) * 2 + (size_t)2 * 16 * (kAbPos + 8) * 2;
}
// tensor-core form of the absorbed attention: 16-byte rows, latents of up to 512 columns
static bool la_tensor(const glq_latent_t* a) {
    return a->dtype == GLQ_DT_BF16 && a->K % 16 == 0 && a->K <= 512 && a->R % 8 == 0 && a->ldc % 8 == 0 && al16(a->cache) &&
           la_absorbed_smem(la_params(a)) <= 208 * 1024;
}
static int la_splits(const glq_latent_t* a) {
    if (!la_tensor(a)) return 1;
    const long ctas = (long)a->B * ((a->T * a->H + 15) / 16);
    const long want = std::max<long>(1, dn_sms() / ctas), tiles = cdiv_i(a->max_len, kAbPos);
    const long cap = a->max_splits > 0 ? std::min(a->max_splits, kMaxSplits) : kMaxSplits;
    return (int)std::min(std::min(want, tiles), cap);
}
struct LaWs {
    size_t qa, po, pm, pl, ol, total;
};
static LaWs la_ws(const glq_latent_t* a) {
    const LaParams p = la_params(a);
    const size_t rows = (size_t)a->B * p.rows16, parts = rows * la_splits(a);
    auto up = [](size_t v) { return (v + 255) / 256 * 256; };
    LaWs w{};
    w.qa = 0;
    w.po = up(la_tensor(a) ? rows * p.KRp * 4 : rows * (a->K + a->R) * 4);
    w.pm = w.po + up(parts * a->K * 4);
    w.pl = w.pm + up(parts * 4);
    w.ol = w.pl + up(parts * 4);
    w.total = w.ol + up((size_t)a->B * a->T * a->H * a->K * 4);
    return w;
}

extern "C" int glq_latent_prep(const glq_latent_t* a, void* stream) {
    if (!la_sizes_ok(a) || !a->q || !a->ckr || !a->norm_w || !a->cache || !a->start || (a->rot_dims && (!a->cos_t || !a->sin_t)))
        return GLQ_ERR_ARG;
    if (a->T == 0) return GLQ_OK;
    const LaParams p = la_params(a);
    const dim3 grid(a->B * a->T);
    if (a->dtype == GLQ_DT_BF16) return dn_launch(latent_prep_kernel<bf16>, grid, 128, 0, stream, p);
    return dn_launch(latent_prep_kernel<float>, grid, 128, 0, stream, p);
}

extern "C" size_t glq_latent_absorbed_workspace_bytes(const glq_latent_t* a) { return la_sizes_ok(a) ? la_ws(a).total : 0; }

template <typename T> static int la_absorbed(const glq_latent_t* a, void* stream) {
    LaParams p = la_params(a);
    const LaWs w = la_ws(a);
    if (a->workspace_bytes < w.total) return GLQ_ERR_WORKSPACE;
    char* ws = reinterpret_cast<char*>(a->workspace);
    p.qa = ws + w.qa;
    p.po = reinterpret_cast<float*>(ws + w.po);
    p.pm = reinterpret_cast<float*>(ws + w.pm);
    p.pl = reinterpret_cast<float*>(ws + w.pl);
    p.ol = reinterpret_cast<float*>(ws + w.ol);
    p.splits = la_splits(a);
    const bool tensor = la_tensor(a);
    const int rb = std::min(cdiv_i((long)a->B * a->T, kHmRows), 512);
    // output rows of a head are split over CTAs until the machine is covered
    auto parts = [&](int n, int lanes_k, long want) {
        int gl = 1;
        while (gl < 32 && gl * 8 < lanes_k) gl <<= 1;
        const int step = 8 * (32 / gl);                      // output rows a CTA takes at a time
        return std::max(1, std::min(cdiv_i(n, step), cdiv_i(want, (long)a->H * rb)));
    };
    const size_t xa = (size_t)kHmRows * ((a->D + 7) / 8 * 8) * 4, xv = (size_t)kHmRows * ((a->K + 7) / 8 * 8) * 4;
    int st;
    if (tensor) {
        st = dn_launch(latent_absorb_kernel<T, true>, dim3(a->H + 1, parts(a->K, a->D, 4L * dn_sms()), rb), 256, xa, stream, p);
        if (st != GLQ_OK) return st;
        const dim3 grid(p.rows16 / 16, p.splits, a->B);
        const size_t smem = la_absorbed_smem(p);
        if (a->K <= 256) st = dn_launch(latent_absorbed_kernel<2>, grid, kAbThreads, smem, stream, p);
        else st = dn_launch(latent_absorbed_kernel<4>, grid, kAbThreads, smem, stream, p);
    } else {
        st = dn_launch(latent_absorb_kernel<T, false>, dim3(a->H + 1, parts(a->K, a->D, 4L * dn_sms()), rb), 256, xa, stream, p);
        if (st != GLQ_OK) return st;
        const size_t smem = (size_t)(2 * a->K + a->R + 128) * 4;
        st = dn_launch(latent_absorbed_generic_kernel<T>, dim3(a->T * a->H, a->B), 128, smem, stream, p);
    }
    if (st != GLQ_OK) return st;
    const long rh = (long)a->B * a->T * a->H;
    const int kp = (int)std::max<long>(1, std::min<long>(cdiv_i(a->K, 128), cdiv_i(2L * dn_sms(), rh)));
    st = dn_launch(latent_combine_kernel, dim3(a->B * a->T, a->H, kp), 512, 0, stream, p);
    if (st != GLQ_OK) return st;
    return dn_launch(latent_value_kernel<T>, dim3(a->H, parts(a->V, a->K, 2L * dn_sms()), rb), 256, xv, stream, p);
}

extern "C" int glq_latent_absorbed(const glq_latent_t* a, void* stream) {
    if (!la_sizes_ok(a) || !a->q || !a->ckr || !a->norm_w || !a->cache || !a->start || (a->rot_dims && (!a->cos_t || !a->sin_t)) || !a->ukt || !a->uv || !a->gate ||
        !a->out || !a->workspace)
        return GLQ_ERR_ARG;
    // matrices with rows of whole vectors are read eight values at a time, others one by one
    if (!al16(a->workspace) || (a->D % 8 == 0 && !al16(a->ukt)) || (a->K % 8 == 0 && !al16(a->uv))) return GLQ_ERR_ALIGN;
    if (a->K > 4096 || a->D > 4096 || a->R > 4096 || a->B > 65535 || a->H > 65534) return GLQ_ERR_UNSUPPORTED;
    if (a->T == 0) return GLQ_OK;
    return a->dtype == GLQ_DT_BF16 ? la_absorbed<bf16>(a, stream) : la_absorbed<float>(a, stream);
}

static size_t lt_smem(const glq_latent_t* a) {
    return at_smem((a->D + 63) / 64 + (a->R + 63) / 64, a->V <= 64 ? 64 : 128);
}
extern "C" int glq_latent_prefill_form(const glq_latent_t* a) {
    if (!la_sizes_ok(a) || a->dtype != GLQ_DT_BF16 || a->D % 8 || a->R % 8 || a->V % 8 || a->K % 8 || a->ldc % 8 || a->ldq % 8 || a->V > 128)
        return 0;
    static const bool mma_only = std::getenv("GLQ_NO_TC") != nullptr;
    if (!mma_only && lt_smem(a) <= 226 * 1024 && encode_tiled()) return 2;
    return a->D + a->R <= 256 ? 1 : 0;
}

static int latent_prefill_tc(const glq_latent_t* a, void* stream) {
    AtParams p{};
    p.gate = a->gate;
    p.out = a->out;
    p.ldg = a->ldk;
    p.B = a->B;
    p.T = a->T;
    p.H = a->H;
    p.V = a->V;
    p.S = a->S;
    p.krows = a->S;
    p.rrows = a->max_len;
    p.group = 1;
    p.scale = a->scale;
    AtGeom g{};
    g.cd = cdiv_i(a->D, 64);
    g.nc = g.cd + cdiv_i(a->R, 64);
    g.steps_last_d = cdiv_i(a->D - 64 * (g.cd - 1), 16);
    g.steps_last_r = a->R ? cdiv_i(a->R - 64 * (g.nc - g.cd - 1), 16) : 0;
    const int dv = a->V <= 64 ? 64 : 128, dr = a->D + a->R;
    AtMaps m{};
    const bf16* q = reinterpret_cast<const bf16*>(a->q);
    const long rows = (long)a->B * a->T;
    const long qs[3] = {1, dr, (long)a->ldq}, ks[3] = {1, a->D, (long)a->ldkv};
    const long qn[3] = {a->D, a->H, rows}, qr[3] = {a->R, a->H, rows}, kn[3] = {a->D, a->H, (long)a->B * a->S};
    const int bq[3] = {64, 1, 128}, bk[3] = {64, 1, 64};
    bool ok = make_map_nd(&m.qn, q, 3, qn, qs, bq) && make_map_nd(&m.kn, a->kv, 3, kn, ks, bk);
    if (ok && a->R)
        ok = make_map_nd(&m.qr, q + a->D, 3, qr, qs, bq) &&
             make_map(&m.kr, reinterpret_cast<const bf16*>(a->cache) + a->K, (long)a->B * a->max_len, a->R, (long)a->ldc, 64);
    ok = ok && make_map(&m.vt, a->vt, (long)a->B * a->H * a->V, a->S, (long)a->ldvt, dv);
    if (!ok) return GLQ_ERR_UNSUPPORTED;
    const dim3 grid((unsigned)((long)cdiv_i(a->T, 256) * a->H * a->B));
    if (dv == 64) return dn_launch(causal_attn_tc_kernel<64, false>, grid, kAtThreads, lt_smem(a), stream, m, p, g);
    return dn_launch(causal_attn_tc_kernel<128, false>, grid, kAtThreads, lt_smem(a), stream, m, p, g);
}

extern "C" int glq_latent_prefill(const glq_latent_t* a, void* stream) {
    const int form = glq_latent_prefill_form(a);
    if (form == 0) return GLQ_ERR_UNSUPPORTED;
    if (!a->q || !a->cache || !a->kv || !a->gate || !a->out || a->S < a->T || a->S > a->max_len || (form == 2 && !a->vt)) return GLQ_ERR_ARG;
    if (!al16(a->kv) || !al16(a->cache) || !al16(a->q) || !al16(a->out) || a->ldkv % 8) return GLQ_ERR_ALIGN;
    if (form == 2 && (!al16(a->vt) || a->ldvt % 8 || a->ldvt < a->S)) return GLQ_ERR_ALIGN;
    if (a->T == 0) return GLQ_OK;
    if (form == 2) return latent_prefill_tc(a, stream);
    const LaParams p = la_params(a);
    const dim3 grid((unsigned)((long)cdiv_i(a->T, 64) * a->H * a->B));
    const int dk = a->D + a->R;
#define LP(DK, DV) return dn_launch(latent_prefill_kernel<DK, DV>, grid, 128, LpCfg<DK, DV>::SMEM, stream, p)
    if (a->V <= 64) {
        if (dk <= 64) LP(64, 64);
        if (dk <= 128) LP(128, 64);
        if (dk <= 192) LP(192, 64);
        LP(256, 64);
    }
    if (dk <= 64) LP(64, 128);
    if (dk <= 128) LP(128, 128);
    if (dk <= 192) LP(192, 128);
    LP(256, 128);
#undef LP
}
