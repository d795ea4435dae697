// Grouped-query attention over cached keys and values.  Queries and keys may be turned by their position and then divided
// by their root mean square; the values are a projection of their own or the keys as projected.
//   * prep + prompt form: queries turned and normed in place, new keys and values into the cache, then causal attention on
//     tcgen05 over the cache itself (attn_tc.cuh);
//   * decode form (few positions): one launch prepares the new rows, reads the cache in position splits and weighs the
//     values, with all query heads of a key head as the rows of the tensor-core ops; a second merges the splits;
//   * generic form (float32, sizes that are no multiple of eight): prep, then one CTA per query and head.
// Scores, weights and sums are float; a float operand of a tensor-core product goes in as a sum of two bf16 numbers.
#include "attn_tc.cuh"
#include "recurrent.cuh"

namespace glq {

struct GaParams {
    void* q;                         // (B * T, ldp): H x D
    const void* k;                   // G x D
    const void* v;                   // G x V
    const float* cos_t;
    const float* sin_t;
    const long long* start;
    void* kc;                        // (B, max_len, G, D)
    void* vc;                        // (B, max_len, G, V)
    void* out;                       // (B * T, H * V)
    long long ldp;
    int B, T, H, G, D, V, group, rot_dims, rot_pairs, qk_norm, max_len, state_idle;
    float scale, eps;
    // decode form
    float* po;                       // (B, G, tiles, splits, 16, V)
    float2* pml;                     // (B, G, tiles, splits, 16): maximum, sum
    int splits, tiles;
};

__device__ __forceinline__ void gld8(const bf16* p, float (&v)[8]) {
    const uint4 w = *reinterpret_cast<const uint4*>(p);
    v[0] = bf_lo(w.x), v[1] = bf_hi(w.x), v[2] = bf_lo(w.y), v[3] = bf_hi(w.y);
    v[4] = bf_lo(w.z), v[5] = bf_hi(w.z), v[6] = bf_lo(w.w), v[7] = bf_hi(w.w);
}

// A group of `gl` lanes (a power of two, 8 gl >= D, D % 8 == 0) makes one head's row: this lane's elements e .. e + 7
__device__ __forceinline__ void head_row8(const GaParams& p, const bf16* x, int e, int gl, size_t pos, float (&v)[8]) {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.f;
    if (e < p.D) {
        gld8(x + e, v);
        if (e < p.rot_dims) {
            const int half = p.rot_dims >> 1;
            const float* cs = p.cos_t + pos * half;
            const float* sn = p.sin_t + pos * half;
            if (p.rot_pairs) {
                float c[4] = {1.f, 1.f, 1.f, 1.f}, s[4] = {0.f, 0.f, 0.f, 0.f};
                if (half % 4 == 0) {       // whole vectors: all four pairs are turned
                    ld4(cs + e / 2, c);
                    ld4(sn + e / 2, s);
                } else {
#pragma unroll
                    for (int j = 0; j < 4; ++j)
                        if (e + 2 * j < p.rot_dims) c[j] = cs[e / 2 + j], s[j] = sn[e / 2 + j];
                }
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float a = v[2 * j], o = v[2 * j + 1];
                    v[2 * j] = a * c[j] - o * s[j];
                    v[2 * j + 1] = o * c[j] + a * s[j];
                }
            } else if (half % 8 == 0) {
                const bool second = e >= half;
                float u[8], c[4], s[4];
                gld8(x + (second ? e - half : e + half), u);
#pragma unroll
                for (int q = 0; q < 2; ++q) {
                    ld4(cs + (second ? e - half : e) + 4 * q, c);
                    ld4(sn + (second ? e - half : e) + 4 * q, s);
#pragma unroll
                    for (int j = 0; j < 4; ++j) v[4 * q + j] = v[4 * q + j] * c[j] + (second ? u[4 * q + j] : -u[4 * q + j]) * s[j];
                }
            } else {
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] = rotated(x, e + j, p.rot_dims, 0, cs, sn);
            }
        }
    }
    if (p.qk_norm) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
        for (int o = gl >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.f / sqrtf(ss / p.D + p.eps);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= inv;
    }
}
__device__ __forceinline__ uint4 pack8(const float (&v)[8]) {
    return make_uint4(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]), pack_bf2(v[4], v[5]), pack_bf2(v[6], v[7]));
}

// prompt: rows of H query heads (in place) and G key heads (into the cache), 16-byte accesses; a warp takes 32 / gl heads of
// a row at a time, the key heads' values on the way.  Work is row by row over (row, heads) tasks.
__global__ void __launch_bounds__(256, 5) gqa_prep_vec_kernel(const GaParams p, int gl) {
    pdl_wait();
    pdl_release();
    const int lane = threadIdx.x & 31, per = 32 / gl, li = lane % gl, e = 8 * li;
    const int heads = p.H + p.G, tasks = (heads + per - 1) / per;
    const long long start = *p.start, total = (long long)p.B * p.T * tasks;
    for (long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5); i < total; i += (long long)gridDim.x * 8) {
        const size_t row = (size_t)(i / tasks), b = row / p.T;
        const int h = (int)(i % tasks) * per + lane / gl;
        const long long pos = start + (long long)(row % p.T);
        if (pos < 0 || pos >= p.max_len) continue;
        const bool live = h < heads, isq = h < p.H;
        const bf16* src = reinterpret_cast<const bf16*>(isq || !live ? p.q : p.k) + row * p.ldp + (size_t)(!live ? 0 : (isq ? h : h - p.H)) * p.D;
        float v[8];
        head_row8(p, src, e, gl, (size_t)pos, v);
        __syncwarp();                      // all lanes have read the row that is replaced
        if (!live) continue;
        if (isq) {
            if (e < p.D) *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.q) + row * p.ldp + (size_t)h * p.D + e) = pack8(v);
            continue;
        }
        const size_t crow = (b * p.max_len + pos) * p.G + h - p.H;
        if (e < p.D) *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.kc) + crow * p.D + e) = pack8(v);
        const bf16* vs = reinterpret_cast<const bf16*>(p.v) + row * p.ldp + (size_t)(h - p.H) * p.V;
        for (int c = e; c < p.V; c += 8 * gl)
            *reinterpret_cast<uint4*>(reinterpret_cast<bf16*>(p.vc) + crow * p.V + c) = *reinterpret_cast<const uint4*>(vs + c);
    }
}

// the same for any type and size: one warp per head, its row staged in shared memory
template <typename T>
__global__ void __launch_bounds__(128) gqa_prep_kernel(const GaParams p) {
    extern __shared__ float gp_smem[];
    pdl_wait();
    pdl_release();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = p.rot_dims >> 1;
    float* buf = gp_smem + (size_t)warp * p.D;
    const size_t row = blockIdx.x, b = row / p.T;
    const long long pos = *p.start + (long long)(row % p.T);
    if (pos < 0 || pos >= p.max_len) return;
    const size_t crow = (b * p.max_len + pos) * p.G;
    for (int h = warp; h < p.H + p.G; h += 4) {
        const bool isq = h < p.H;
        const T* src = isq ? reinterpret_cast<const T*>(p.q) + row * p.ldp + (size_t)h * p.D
                           : reinterpret_cast<const T*>(p.k) + row * p.ldp + (size_t)(h - p.H) * p.D;
        float ss = 0.f;
        for (int d = lane; d < p.D; d += 32) {
            const float v = rotated(src, d, p.rot_dims, p.rot_pairs, p.cos_t + (size_t)pos * half, p.sin_t + (size_t)pos * half);
            buf[d] = v;
            ss += v * v;
        }
        const float inv = p.qk_norm ? 1.f / sqrtf(warp_sum(ss) / p.D + p.eps) : 1.f;
        __syncwarp();
        T* dst = isq ? reinterpret_cast<T*>(p.q) + row * p.ldp + (size_t)h * p.D : reinterpret_cast<T*>(p.kc) + (crow + h - p.H) * p.D;
        for (int d = lane; d < p.D; d += 32) dst[d] = from_f<T>(buf[d] * inv);
    }
    const T* vs = reinterpret_cast<const T*>(p.v) + row * p.ldp;
    T* vd = reinterpret_cast<T*>(p.vc) + crow * p.V;
    for (int i = threadIdx.x; i < p.G * p.V; i += 128) vd[i] = vs[i];
}

// one query of one head; prep has run
template <typename T>
__global__ void __launch_bounds__(128) gqa_generic_kernel(const GaParams p) {
    extern __shared__ float gg_smem[];
    float* sq = gg_smem;                 // [D]
    float* so = sq + p.D;                // [V]
    __shared__ float pr[128], red[32];
    pdl_wait();
    pdl_release();
    const int tid = threadIdx.x;
    const size_t row = blockIdx.x, b = row / p.T;
    const int h = blockIdx.y, kh = h / p.group;
    const long long pos = *p.start + (long long)(row % p.T);
    if (pos < 0 || pos >= p.max_len) return;
    const T* q = reinterpret_cast<const T*>(p.q) + row * p.ldp + (size_t)h * p.D;
    const T* kc = reinterpret_cast<const T*>(p.kc) + (b * p.max_len * p.G + kh) * p.D;
    const T* vc = reinterpret_cast<const T*>(p.vc) + (b * p.max_len * p.G + kh) * p.V;
    for (int d = tid; d < p.D; d += 128) sq[d] = to_f(q[d]);
    for (int v = tid; v < p.V; v += 128) so[v] = 0.f;
    float m = -INFINITY, l = 0.f;
    const int total = (int)pos + 1;
    for (int k0 = 0; k0 < total; k0 += 128) {
        const int key = k0 + tid, nk = min(128, total - k0);
        __syncthreads();
        float s = -INFINITY;
        if (key < total) {
            const T* kr = kc + (size_t)key * p.G * p.D;
            float a = 0.f;
            for (int d = 0; d < p.D; ++d) a += sq[d] * to_f(kr[d]);
            s = a * p.scale;
        }
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        if ((tid & 31) == 0) red[tid >> 5] = mx;
        __syncthreads();
        const float mn = fmaxf(fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3])), m);
        const float f = expf(m - mn), w = key < total ? expf(s - mn) : 0.f;
        m = mn;
        pr[tid] = w;
        l = l * f + block_sum(w, red);
        for (int v = tid; v < p.V; v += 128) {
            float a = so[v] * f;
            const T* vr = vc + (size_t)k0 * p.G * p.V + v;
            for (int j = 0; j < nk; ++j) a += pr[j] * to_f(vr[(size_t)j * p.G * p.V]);
            so[v] = a;
        }
    }
    for (int v = tid; v < p.V; v += 128) reinterpret_cast<T*>(p.out)[row * p.H * p.V + (size_t)h * p.V + v] = from_f<T>(so[v] / l);
}

// ---- decode form ---------------------------------------------------------------------------------------------
constexpr int kGdWarps = 4, kGdStages = 3, kGdTile = 16 * kGdWarps;     // positions of a CTA's round, 16 a warp
struct GdSizes {
    int LD, LV;                          // row strides (bf16) of staged keys and values
    size_t q_bytes, stage, ring;
};
__host__ __device__ inline GdSizes gd_sizes(int D, int DV) {
    GdSizes s;
    s.LD = (D + 15) / 16 * 16 + 8;
    s.LV = DV + 8;
    s.q_bytes = (size_t)2 * 16 * s.LD * 2;
    s.stage = (size_t)16 * (s.LD + s.LV) * 2;
    s.ring = s.stage * kGdStages * kGdWarps;
    const size_t merge = (size_t)kGdWarps * 16 * (DV + 4) * 4;
    if (s.ring < merge) s.ring = merge;
    return s;
}

// 16 rows (query position, head of the group) of a key head against one split of the positions
template <int DV>
__global__ void __launch_bounds__(kGdWarps * 32) gqa_decode_kernel(const GaParams p, int gl) {
    constexpr int NV = DV / 8;
    extern __shared__ __align__(16) unsigned char gd_raw[];
    __shared__ float s_m[kGdWarps][16], s_l[kGdWarps][16];
    const GdSizes z = gd_sizes(p.D, DV);
    bf16* qh = reinterpret_cast<bf16*>(gd_raw);              // [16][LD]
    bf16* ql = qh + 16 * z.LD;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    unsigned char* ring = gd_raw + z.q_bytes;
    const int kh = blockIdx.x / p.tiles, rt = blockIdx.x % p.tiles, sp = blockIdx.y, b = blockIdx.z;
    const int D = p.D, V = p.V, Dp = z.LD - 8;
    if (!p.state_idle) pdl_wait();
    const int start = (int)min(max(*p.start, 0ll), (long long)p.max_len - p.T), total = start + p.T;
    const int nt = (total + kGdTile - 1) / kGdTile, per = (nt + p.splits - 1) / p.splits;
    const int lo = sp * per, hi = min(nt, lo + per);
    const bf16* kc = reinterpret_cast<const bf16*>(p.kc) + ((size_t)b * p.max_len * p.G + kh) * D;
    const bf16* vc = reinterpret_cast<const bf16*>(p.vc) + ((size_t)b * p.max_len * p.G + kh) * V;
    auto load = [&](int i) {             // the warp's 16 positions of round lo + i
        if (lo + i < hi) {
            const uint32_t ks = smem_u32(ring + (size_t)(warp * kGdStages + i % kGdStages) * z.stage), vs = ks + 16 * z.LD * 2;
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (lane >> 2) + 8 * u, pos = (lo + i) * kGdTile + 16 * warp + r;
                const bool live = pos < total;
                const bf16* kr = kc + (size_t)(live ? pos : 0) * p.G * D;
                const bf16* vr = vc + (size_t)(live ? pos : 0) * p.G * V;
                for (int cc = 8 * t4; cc < Dp; cc += 32) cpa16(ks + (r * z.LD + cc) * 2, cc < D ? kr + cc : kr, live && cc < D);
                for (int cc = 8 * t4; cc < V; cc += 32) cpa16(vs + (r * z.LV + cc) * 2, vr + cc, live);
            }
        }
        cpa_commit();
    };
    // positions that were cached by earlier calls are requested before the wait for this step's projections
    int issued = 0;
    if (p.state_idle)
        while (issued < kGdStages - 1 && lo + issued < hi && (lo + issued + 1) * kGdTile <= start) load(issued++);
    pdl_wait();
    pdl_release();
    const int rows = p.T * p.group;
    if (lo < hi) {
        const int per_w = 32 / gl, li = lane % gl, e = 8 * li;
        // queries of this tile
        for (int r0 = warp * per_w; r0 < 16; r0 += kGdWarps * per_w) {
            const int r = r0 + lane / gl, ri = min(rt * 16 + r, rows - 1), t = ri / p.group, h = kh * p.group + ri % p.group;
            float v[8];
            head_row8(p, reinterpret_cast<const bf16*>(p.q) + ((size_t)b * p.T + t) * p.ldp + (size_t)h * D, e, gl, (size_t)start + t, v);
            if (r < 16 && e < Dp) {
                uint32_t hw[4], lw[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) split_bf2(v[2 * j], v[2 * j + 1], hw[j], lw[j]);
                *reinterpret_cast<uint4*>(qh + r * z.LD + e) = make_uint4(hw[0], hw[1], hw[2], hw[3]);
                *reinterpret_cast<uint4*>(ql + r * z.LD + e) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
            }
        }
        // new positions that lie in this split (every row tile of the head writes the same values)
        for (int i0 = 0; i0 < p.T && total > lo * kGdTile && start < hi * kGdTile; i0 += kGdWarps * per_w) {
            const int i = i0 + warp * per_w + lane / gl, pos = start + i;
            const bool live = i < p.T && pos >= lo * kGdTile && pos < hi * kGdTile;
            const size_t row = (size_t)b * p.T + (i < p.T ? i : 0);
            float v[8];
            head_row8(p, reinterpret_cast<const bf16*>(p.k) + row * p.ldp + (size_t)kh * D, e, gl, (size_t)(i < p.T ? pos : start), v);
            if (live) {
                if (e < D) *reinterpret_cast<uint4*>(const_cast<bf16*>(kc) + (size_t)pos * p.G * D + e) = pack8(v);
                const bf16* src = reinterpret_cast<const bf16*>(p.v) + row * p.ldp + (size_t)kh * V;
                for (int c = e; c < V; c += 8 * gl)
                    *reinterpret_cast<uint4*>(const_cast<bf16*>(vc) + (size_t)pos * p.G * V + c) = *reinterpret_cast<const uint4*>(src + c);
            }
        }
    }
    __syncthreads();
    while (issued < kGdStages - 1) load(issued++);
    float o[NV][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < NV; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
    int seen[2];                         // last position that rows g, g + 8 of the tile see
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int r = rt * 16 + g + 8 * e;
        seen[e] = r < rows ? start + r / p.group : -1;
    }
    const float sc = p.scale * 1.4426950408889634f;
    for (int i = 0; lo + i < hi; ++i) {
        cpa_wait<kGdStages - 2>();
        __syncwarp();
        const uint32_t ks = smem_u32(ring + (size_t)(warp * kGdStages + i % kGdStages) * z.stage), vs = ks + 16 * z.LD * 2;
        float s[2][4];
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[nb][e] = 0.f;
        for (int c = 0; c < Dp; c += 16) {
            uint32_t a[4], a2[4], k0, k1, k2, k3;
            const uint32_t off = (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * z.LD + c + (lane >> 4) * 8) * 2;
            ldsm4(smem_u32(qh) + off, a[0], a[1], a[2], a[3]);
            ldsm4(smem_u32(ql) + off, a2[0], a2[1], a2[2], a2[3]);
            ldsm4(ks + (uint32_t)(((lane & 7) + (lane >> 4) * 8) * z.LD + c + ((lane >> 3) & 1) * 8) * 2, k0, k1, k2, k3);
            mma_bf16(s[0], a[0], a[1], a[2], a[3], k0, k1);
            mma_bf16(s[1], a[0], a[1], a[2], a[3], k2, k3);
            mma_bf16(s[0], a2[0], a2[1], a2[2], a2[3], k0, k1);
            mma_bf16(s[1], a2[0], a2[1], a2[2], a2[3], k2, k3);
        }
        const int base = (lo + i) * kGdTile + 16 * warp;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int pos = base + 8 * nb + 2 * t4 + (e & 1);
                s[nb][e] = pos <= seen[e >> 1] ? s[nb][e] * sc : -INFINITY;
                mx[e >> 1] = fmaxf(mx[e >> 1], s[nb][e]);
            }
        float f[2], sh[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
            mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
            const float mn = fmaxf(m[e], mx[e]);
            sh[e] = mn == -INFINITY ? 0.f : mn;
            f[e] = ex2(m[e] - sh[e]);
            m[e] = mn;
            l[e] *= f[e];
        }
#pragma unroll
        for (int nb = 0; nb < 2; ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[nb][e] = ex2(s[nb][e] - sh[e >> 1]);
                l[e >> 1] += s[nb][e];
            }
        if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                o[j][0] *= f[0];
                o[j][1] *= f[0];
                o[j][2] *= f[1];
                o[j][3] *= f[1];
            }
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
            split_bf2(s[nb][0], s[nb][1], ph[2 * nb], pl[2 * nb]);
            split_bf2(s[nb][2], s[nb][3], ph[2 * nb + 1], pl[2 * nb + 1]);
        }
        const int vrow = (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
        for (int jp = 0; jp < NV / 2; ++jp) {
            if (16 * jp >= V) break;
            uint32_t b0, b1, b2, b3;
            ldsm4_t(vs + (uint32_t)(vrow * z.LV + 16 * jp + (lane >> 4) * 8) * 2, b0, b1, b2, b3);
            mma_bf16(o[2 * jp], ph[0], ph[1], ph[2], ph[3], b0, b1);
            mma_bf16(o[2 * jp], pl[0], pl[1], pl[2], pl[3], b0, b1);
            mma_bf16(o[2 * jp + 1], ph[0], ph[1], ph[2], ph[3], b2, b3);
            mma_bf16(o[2 * jp + 1], pl[0], pl[1], pl[2], pl[3], b2, b3);
        }
        __syncwarp();                    // the stage of round i - 1 has been read by all lanes
        load(i + kGdStages - 1);
    }
    cpa_wait<0>();
    __syncthreads();
    float* mo = reinterpret_cast<float*>(ring);              // [warp][16][DV + 4]
    constexpr int LO = DV + 4;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        if (t4 == 0) {
            s_m[warp][g + 8 * e] = m[e];
            s_l[warp][g + 8 * e] = l[e];
        }
    }
#pragma unroll
    for (int j = 0; j < NV; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e)
            *reinterpret_cast<float2*>(mo + (size_t)(warp * 16 + g + 8 * e) * LO + 8 * j + 2 * t4) = make_float2(o[j][2 * e], o[j][2 * e + 1]);
    __syncthreads();
    const size_t part = (((size_t)b * p.G + kh) * p.tiles + rt) * p.splits + sp;
    for (int i = tid; i < 16 * (V / 4); i += kGdWarps * 32) {
        const int r = i / (V / 4), v = (i % (V / 4)) * 4;
        float mm = s_m[0][r];
#pragma unroll
        for (int w = 1; w < kGdWarps; ++w) mm = fmaxf(mm, s_m[w][r]);
        float ll = 0.f;
        float4 a = make_float4(0, 0, 0, 0);
#pragma unroll
        for (int w = 0; w < kGdWarps; ++w) {
            const float wt = s_m[w][r] == -INFINITY ? 0.f : ex2(s_m[w][r] - mm);
            const float4 x = *reinterpret_cast<const float4*>(mo + (size_t)(w * 16 + r) * LO + v);
            ll += wt * s_l[w][r];
            a.x += wt * x.x;
            a.y += wt * x.y;
            a.z += wt * x.z;
            a.w += wt * x.w;
        }
        if (p.splits == 1) {
            const int ri = rt * 16 + r;
            if (ri < rows) {
                const float inv = 1.f / ll;
                bf16* y = reinterpret_cast<bf16*>(p.out) + ((size_t)b * p.T + ri / p.group) * p.H * V + (size_t)(kh * p.group + ri % p.group) * V + v;
                *reinterpret_cast<uint2*>(y) = make_uint2(pack_bf2(a.x * inv, a.y * inv), pack_bf2(a.z * inv, a.w * inv));
            }
        } else if (mm != -INFINITY) {    // a split without weight is recognised by its maximum
            *reinterpret_cast<float4*>(p.po + (part * 16 + r) * V + v) = a;
            if (v == 0) p.pml[part * 16 + r] = make_float2(mm, ll);
        } else if (v == 0) {
            p.pml[part * 16 + r] = make_float2(-INFINITY, 0.f);
        }
    }
}

// merges the splits of one row
constexpr int kGdMaxSplits = 128;
constexpr int kGcThreads = 256;
__global__ void __launch_bounds__(kGcThreads) gqa_combine_kernel(const GaParams p) {
    __shared__ float sw[kGdMaxSplits], red[32];
    __shared__ __align__(16) float part[kGcThreads * 4];
    pdl_wait();
    pdl_release();
    const int tid = threadIdx.x, h = blockIdx.y, kh = h / p.group;
    const size_t row = blockIdx.x, b = row / p.T;
    const int ri = (int)(row % p.T) * p.group + h % p.group, r = ri % 16;
    const size_t first = (((size_t)b * p.G + kh) * p.tiles + ri / 16) * p.splits;
    const float2 ml = tid < p.splits ? p.pml[(first + tid) * 16 + r] : make_float2(-INFINITY, 0.f);
    float mx = ml.x;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if ((tid & 31) == 0) red[tid >> 5] = mx;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < kGcThreads / 32; ++i) mx = fmaxf(mx, red[i]);
    const float w = ml.x == -INFINITY ? 0.f : ex2(ml.x - mx);
    const float inv = 1.f / block_sum(w * ml.y, red);
    if (tid < kGdMaxSplits) sw[tid] = w * inv;
    __syncthreads();
    // four columns a thread, the groups of threads share the splits; a split without weight has not been written
    const int vq = p.V / 4, groups = kGcThreads / vq, grp = tid / vq, v = 4 * (tid % vq);
    float4 a = make_float4(0, 0, 0, 0);
    if (grp < groups) {
        const float* po = p.po + (first * 16 + r) * p.V + v;
        for (int s0 = grp; s0 < p.splits; s0 += 8 * groups) {
            float4 x[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int s = min(s0 + i * groups, p.splits - 1);
                x[i] = *reinterpret_cast<const float4*>(po + (size_t)16 * s * p.V);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int s = s0 + i * groups;
                const float ws = s < p.splits ? sw[s] : 0.f;
                if (ws != 0.f) {
                    a.x += ws * x[i].x;
                    a.y += ws * x[i].y;
                    a.z += ws * x[i].z;
                    a.w += ws * x[i].w;
                }
            }
        }
    }
    *reinterpret_cast<float4*>(part + 4 * tid) = a;
    __syncthreads();
    if (tid < vq) {
        for (int i = 1; i < groups; ++i) {
            const float4 x = *reinterpret_cast<const float4*>(part + 4 * (tid + i * vq));
            a.x += x.x;
            a.y += x.y;
            a.z += x.z;
            a.w += x.w;
        }
        *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(p.out) + row * p.H * p.V + (size_t)h * p.V + v) =
            make_uint2(pack_bf2(a.x, a.y), pack_bf2(a.z, a.w));
    }
}

}  // namespace glq

using namespace glq;

static bool ga_sizes_ok(const glq_gqa_t* a) {
    return a && a->B > 0 && a->T >= 0 && a->H > 0 && a->G > 0 && a->H % a->G == 0 && a->D > 0 && a->V > 0 && a->rot_dims >= 0 &&
           a->rot_dims % 2 == 0 && a->rot_dims <= a->D && a->max_len > 0 && (a->dtype == GLQ_DT_BF16 || a->dtype == GLQ_DT_F32);
}
// rows of whole 16-byte vectors
static bool ga_vec(const glq_gqa_t* a) {
    return a->dtype == GLQ_DT_BF16 && a->D % 8 == 0 && a->V % 8 == 0 && a->D <= 256 && a->ldp % 8 == 0 && al16(a->q) && al16(a->k) && al16(a->cos_t) && al16(a->sin_t) &&
           al16(a->v) && al16(a->kc) && al16(a->vc) && al16(a->out);
}
static int ga_lanes(int D) {
    int gl = 1;
    while (8 * gl < (D + 15) / 16 * 16) gl <<= 1;            // the padding of odd multiples of eight is written too
    return gl;
}
static GaParams ga_params(const glq_gqa_t* a) {
    GaParams p{};
    p.q = a->q;
    p.k = a->k;
    p.v = a->v;
    p.cos_t = a->cos_t;
    p.sin_t = a->sin_t;
    p.start = reinterpret_cast<const long long*>(a->start);
    p.kc = a->kc;
    p.vc = a->vc;
    p.out = a->out;
    p.ldp = a->ldp;
    p.B = a->B;
    p.T = a->T;
    p.H = a->H;
    p.G = a->G;
    p.D = a->D;
    p.V = a->V;
    p.group = a->H / a->G;
    p.rot_dims = a->rot_dims;
    p.rot_pairs = a->rot_pairs;
    p.qk_norm = a->qk_norm;
    p.max_len = a->max_len;
    p.state_idle = a->state_idle;
    p.scale = a->scale;
    p.eps = a->eps;
    p.tiles = cdiv_i((long)a->T * p.group, 16);
    const long ctas = (long)a->B * a->G * std::max(1, p.tiles);
    const long want = std::max<long>(1, 2L * dn_sms() / ctas), most = cdiv_i(a->max_len, kGdTile);
    p.splits = (int)std::min<long>(std::min(want, most), kGdMaxSplits);
    return p;
}
static int ga_dv(int V) { return V <= 64 ? 64 : (V <= 128 ? 128 : 256); }

extern "C" size_t glq_gqa_decode_workspace_bytes(const glq_gqa_t* a) {
    if (!ga_sizes_ok(a)) return 0;
    const GaParams p = ga_params(a);
    return p.splits == 1 ? 0 : (size_t)a->B * a->G * p.tiles * p.splits * 16 * ((size_t)a->V * 4 + 8);
}

extern "C" int glq_gqa_form(const glq_gqa_t* a) {
    if (!ga_sizes_ok(a) || !ga_vec(a)) return 0;
    if (a->T <= 8 && a->V <= 256) return 1;
    return at_smem((a->D + 63) / 64, a->V <= 64 ? 64 : 128) <= 226 * 1024 && encode_tiled() ? 2 : 0;
}

static int gqa_prompt(const glq_gqa_t* a, const GaParams& gp, void* stream) {
    AtParams p{};
    p.out = a->out;
    p.B = a->B;
    p.T = a->T;
    p.H = a->H;
    p.V = a->V;
    p.S = a->S;
    p.krows = a->max_len;
    p.group = gp.group;
    p.scale = a->scale;
    AtGeom g{};
    g.cd = g.nc = cdiv_i(a->D, 64);
    g.steps_last_d = cdiv_i(a->D - 64 * (g.cd - 1), 16);
    const int dv = a->V <= 64 ? 64 : 128;
    AtMaps m{};
    const long rows = (long)a->B * a->T, crows = (long)a->B * a->max_len;
    const long qn[3] = {a->D, a->H, rows}, qs[3] = {1, a->D, (long)a->ldp};
    const long kn[3] = {a->D, a->G, crows}, ks[3] = {1, a->D, (long)a->G * a->D};
    const long vn[3] = {a->V, a->G, crows}, vs[3] = {1, a->V, (long)a->G * a->V};
    const int bq[3] = {64, 1, 128}, bk[3] = {64, 1, 64};
    if (!make_map_nd(&m.qn, a->q, 3, qn, qs, bq) || !make_map_nd(&m.kn, a->kc, 3, kn, ks, bk) || !make_map_nd(&m.vt, a->vc, 3, vn, vs, bk))
        return GLQ_ERR_UNSUPPORTED;
    const dim3 grid((unsigned)((long)cdiv_i(a->T, 256) * a->H * a->B), cdiv_i(a->V, dv));
    const size_t smem = at_smem(g.nc, dv);
    if (dv == 64) return dn_launch(causal_attn_tc_kernel<64, true>, grid, kAtThreads, smem, stream, m, p, g);
    return dn_launch(causal_attn_tc_kernel<128, true>, grid, kAtThreads, smem, stream, m, p, g);
}

extern "C" int glq_gqa(const glq_gqa_t* a, void* stream) {
    if (!ga_sizes_ok(a) || !a->q || !a->k || !a->v || !a->start || !a->kc || !a->vc || !a->out || (a->rot_dims && (!a->cos_t || !a->sin_t)))
        return GLQ_ERR_ARG;
    if (a->T > a->max_len) return GLQ_ERR_ARG;
    if (a->B > 65535 || a->H > 65535 || a->D > 2048 || a->V > 8192) return GLQ_ERR_UNSUPPORTED;
    if (a->T == 0) return GLQ_OK;
    const int form = glq_gqa_form(a);
    GaParams p = ga_params(a);
    int st;
    if (form == 1) {
        if (p.splits > 1) {
            const size_t parts = (size_t)a->B * a->G * p.tiles * p.splits * 16;
            if (!a->workspace || a->workspace_bytes < parts * ((size_t)a->V * 4 + 8)) return GLQ_ERR_WORKSPACE;
            if (!al16(a->workspace)) return GLQ_ERR_ALIGN;
            p.po = reinterpret_cast<float*>(a->workspace);
            p.pml = reinterpret_cast<float2*>(p.po + parts * a->V);
        }
        const dim3 grid(a->G * p.tiles, p.splits, a->B);
        const int dv = ga_dv(a->V), gl = ga_lanes(a->D);
        const GdSizes z = gd_sizes(a->D, dv);
        if (dv == 64) st = dn_launch(gqa_decode_kernel<64>, grid, kGdWarps * 32, z.q_bytes + z.ring, stream, p, gl);
        else if (dv == 128) st = dn_launch(gqa_decode_kernel<128>, grid, kGdWarps * 32, z.q_bytes + z.ring, stream, p, gl);
        else st = dn_launch(gqa_decode_kernel<256>, grid, kGdWarps * 32, z.q_bytes + z.ring, stream, p, gl);
        if (st != GLQ_OK || p.splits == 1) return st;
        return dn_launch(gqa_combine_kernel, dim3(a->B * a->T, a->H), kGcThreads, 0, stream, p);
    }
    const dim3 rows(a->B * a->T);
    if (form == 2) {
        if (a->S < a->T || a->S > a->max_len) return GLQ_ERR_ARG;
        if ((st = dn_launch(gqa_prep_vec_kernel, dim3(std::min<long>(5L * dn_sms(), cdiv_i((long)a->B * a->T * (a->H + a->G), 8))), 256, 0, stream, p, ga_lanes(a->D))) != GLQ_OK) return st;
        return gqa_prompt(a, p, stream);
    }
    const size_t ps = (size_t)4 * a->D * 4, gs = (size_t)(a->D + a->V) * 4;
    if (a->dtype == GLQ_DT_BF16) {
        if ((st = dn_launch(gqa_prep_kernel<bf16>, rows, 128, ps, stream, p)) != GLQ_OK) return st;
        return dn_launch(gqa_generic_kernel<bf16>, dim3(a->B * a->T, a->H), 128, gs, stream, p);
    }
    if ((st = dn_launch(gqa_prep_kernel<float>, rows, 128, ps, stream, p)) != GLQ_OK) return st;
    return dn_launch(gqa_generic_kernel<float>, dim3(a->B * a->T, a->H), 128, gs, stream, p);
}
