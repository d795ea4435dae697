// Linear attention with decay: per head, S (D, V) float, carried from call to call,
//     S_t = diag(alpha_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t,   out = rms_norm_per_head(o) * norm_w * gate(g)
// with alpha_t one constant per head (retention; Sun et al., "Retentive Network: A Successor to Transformer for Large
// Language Models") or one value per key channel and position, alpha = sigmoid(z)^(1 / tau), z = a2 . a + a2b (gated
// linear attention; Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training").  Queries and
// keys may be turned by their position and scaled first; everything behind the projections is float.
// Two forms of the same recurrence:
//   * step: the recurrence itself, one position after the other; a CTA owns 32 value columns of a head, and the CTAs of a
//     head are a cluster that norms and gates its output (heads of up to 512 columns; else a launch of its own).
//   * chunk: 64 positions at a time on the tensor cores.  With b_t the running sum of log alpha inside a chunk,
//       o_t = (q_t e^{b_t})^T S_start + sum_{s <= t} A_ts v_s,  A_ts = sum_d q_td k_sd e^{b_td - b_sd},
//       S_end = diag(e^{b_end}) S_start + sum_s (k_s e^{b_end - b_s}) v_s^T.
//     prep makes the three operands of every chunk, state chains the chunks, out forms the outputs.  No factor is larger
//     than one: decays per channel reach A through 16 x 16 blocks whose two sides are measured from the end of the block
//     before the queries, and through the exponent's difference itself on the diagonal.  Every float operand of a
//     tensor-core product goes in as a sum of two bf16 numbers.
// State layout: S (B, H, slices, D, 32).
#include "recurrent.cuh"

namespace glq {

struct DaParams {
    const void* q;
    const void* k;
    const void* v;
    const void* g;
    const float* decay;            // per head, or NULL: per channel from a, a2, a2b
    const float* a;
    const void* a2;
    const float* a2b;
    const float* cos_t;
    const float* sin_t;
    const long long* start;
    const float* norm_w;
    float* S;
    float* o;                      // (B * Tall, H * V)
    void* out;
    long long ldp, lda;
    int B, T, H, D, V, slices, rank, rot_dims, rot_pairs, max_len, norm_stride, gate;
    int state_idle, vec4;
    int t0, Tall;                  // this call's positions: t0 .. t0 + T - 1 of the Tall rows of a sequence
    float q_scale, k_scale, eps, inv_tau;
    // chunk form
    uint4 *Qb, *Kb, *Ab, *Sb;
    float* keep;                   // (bh, nc, Dp): what a chunk leaves of the state it started from
    int nc, Dp, Vp;
};

// log2 of sigmoid(z)^(1 / tau)
__device__ __forceinline__ float log2_alpha(float z, float inv_tau) {
    return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau * 1.4426950408889634f;
}
__device__ __forceinline__ float ex2f(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
constexpr int kMaxCluster = 16;
// a float into the shared memory of CTA `rank` of the cluster, at this CTA's address `addr`
__device__ __forceinline__ void st_cluster(uint32_t addr, int rank, float v) {
    asm volatile("{\n .reg .b32 r;\n mapa.shared::cluster.u32 r, %0, %1;\n st.shared::cluster.f32 [r], %2;\n}\n" ::"r"(addr), "r"(rank), "f"(v)
                 : "memory");
}
__device__ __forceinline__ size_t da_pos(const DaParams& p, int t) {
    const long long pos = *p.start + t;
    return (size_t)(pos < 0 ? 0 : (pos >= p.max_len ? p.max_len - 1 : pos));
}

template <typename T>
__device__ __forceinline__ void da_norm_gate(const DaParams& p, size_t row, int h, int lane) {
    norm_gate<T>(p.o + row * p.H * p.V + (size_t)h * p.V, reinterpret_cast<const T*>(p.g) + row * p.ldp + (size_t)h * p.V,
                 p.norm_w ? p.norm_w + (size_t)h * p.norm_stride : nullptr, p.gate,
                 reinterpret_cast<T*>(p.out) + row * p.H * p.V + (size_t)h * p.V, p.V, p.eps, p.vec4, lane);
}

// CL: the slices of a head are one cluster, which norms and gates the head's output and stores it in T
template <typename T, bool CL>
__global__ void __launch_bounds__(256) decay_step_kernel(const DaParams p) {
    extern __shared__ float da_smem[];
    float* sq = da_smem;                 // [D]
    float* sk = sq + p.D;                // [D]
    float* sa = sk + p.D;                // [D]
    __shared__ float sv[kSl], part[8][kSl], s_ss[2][kMaxCluster];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int sl = blockIdx.x, h = blockIdx.y % p.H, b = blockIdx.y / p.H;
    const int D = p.D, V = p.V, v0 = sl * kSl, vw = min(kSl, V - v0);
    float* S = p.S + (((size_t)b * p.H + h) * p.slices + sl) * (size_t)D * kSl;
    const int rr = warp * 4 + (lane >> 3), cc = (lane & 7) * 4;
    constexpr int U = 8;
    float4 pre[U];
    const bool held = D <= 32 * U;       // the slice stays in registers from step to step
    // a state that the preceding launch does not touch is requested before the wait for the projections
    if (!p.state_idle) pdl_wait();
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int d = rr + 32 * u;
        pre[u] = d < D ? *reinterpret_cast<const float4*>(S + (size_t)d * kSl + cc) : make_float4(0, 0, 0, 0);
    }
    const float fixed = p.decay ? p.decay[h] : 0.f;
    pdl_wait();
    pdl_release();
    const T* a2 = reinterpret_cast<const T*>(p.a2) + (size_t)h * D * p.rank;
    for (int t = 0; t < p.T; ++t) {
        const size_t row = (size_t)b * p.Tall + p.t0 + t;
        const T* q = reinterpret_cast<const T*>(p.q) + row * p.ldp + (size_t)h * D;
        const T* k = reinterpret_cast<const T*>(p.k) + row * p.ldp + (size_t)h * D;
        const T* v = reinterpret_cast<const T*>(p.v) + row * p.ldp + (size_t)h * V + v0;
        const float *cs = nullptr, *sn = nullptr;
        if (p.rot_dims) {
            const size_t at = da_pos(p, p.t0 + t) * (p.rot_dims / 2);
            cs = p.cos_t + at;
            sn = p.sin_t + at;
        }
        __syncthreads();
        for (int d = tid; d < D; d += 256) {
            sq[d] = rotated(q, d, p.rot_dims, p.rot_pairs, cs, sn) * p.q_scale;
            sk[d] = rotated(k, d, p.rot_dims, p.rot_pairs, cs, sn) * p.k_scale;
            float al = fixed;
            if (!p.decay) {
                float z = p.a2b[(size_t)h * D + d];
                const float* ar = p.a + row * p.lda;
                for (int r = 0; r < p.rank; ++r) z += ar[r] * to_f(a2[(size_t)d * p.rank + r]);
                al = exp2f(log2_alpha(z, p.inv_tau));
            }
            sa[d] = al;
        }
        if (tid < kSl) sv[tid] = tid < vw ? to_f(v[tid]) : 0.f;
        __syncthreads();
        const float4 vv = make_float4(sv[cc], sv[cc + 1], sv[cc + 2], sv[cc + 3]);
        float4 acc = make_float4(0, 0, 0, 0);
        for (int d0 = 0; d0 < D; d0 += 32 * U) {
            if (!held && (t > 0 || d0 > 0)) {
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const int d = d0 + rr + 32 * u;
                    pre[u] = d < D ? *reinterpret_cast<const float4*>(S + (size_t)d * kSl + cc) : make_float4(0, 0, 0, 0);
                }
            }
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const int d = d0 + rr + 32 * u;
                if (d < D) {
                    const float al = sa[d], kd = sk[d], qd = sq[d];
                    float4 s = pre[u];
                    s.x = al * s.x + kd * vv.x;
                    s.y = al * s.y + kd * vv.y;
                    s.z = al * s.z + kd * vv.z;
                    s.w = al * s.w + kd * vv.w;
                    pre[u] = s;
                    if (!held || t == p.T - 1) *reinterpret_cast<float4*>(S + (size_t)d * kSl + cc) = s;
                    acc.x += s.x * qd;
                    acc.y += s.y * qd;
                    acc.z += s.z * qd;
                    acc.w += s.w * qd;
                }
            }
        }
#pragma unroll
        for (int o = 8; o < 32; o <<= 1) {
            acc.x += __shfl_xor_sync(0xffffffffu, acc.x, o);
            acc.y += __shfl_xor_sync(0xffffffffu, acc.y, o);
            acc.z += __shfl_xor_sync(0xffffffffu, acc.z, o);
            acc.w += __shfl_xor_sync(0xffffffffu, acc.w, o);
        }
        if (lane < 8) *reinterpret_cast<float4*>(&part[warp][cc]) = acc;
        __syncthreads();
        if constexpr (!CL) {
            if (tid < vw) {
                float num = 0.f;
#pragma unroll
                for (int w = 0; w < 8; ++w) num += part[w][tid];
                p.o[row * p.H * V + (size_t)h * V + v0 + tid] = num;
            }
        } else {
            float num = 0.f, gv = 0.f, nw = 1.f;
            if (warp == 0) {
                if (tid < vw) {
                    gv = to_f(reinterpret_cast<const T*>(p.g)[row * p.ldp + (size_t)h * V + v0 + tid]);
                    if (p.norm_w) nw = p.norm_w[(size_t)h * p.norm_stride + v0 + tid];
#pragma unroll
                    for (int w = 0; w < 8; ++w) num += part[w][tid];
                }
                const float ss = warp_sum(num * num);
                if (lane < p.slices) st_cluster(smem_u32(&s_ss[t & 1][sl]), lane, ss);     // to the CTA of every slice
            }
            // a slot is written again two positions later, behind a barrier that follows its reads
            asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
            if (tid < vw) {
                float ss = 0.f;
                for (int i = 0; i < p.slices; ++i) ss += s_ss[t & 1][i];
                const float inv = 1.f / sqrtf(ss / V + p.eps);
                reinterpret_cast<T*>(p.out)[row * p.H * V + (size_t)h * V + v0 + tid] = from_f<T>(num * inv * nw * gate_f<T>(p.gate, gv));
            }
        }
    }
}

// ---- chunk form ------------------------------------------------------------------------------------------
// Operand layouts (uint4 per lane; the first and the second bf16 part 32 uint4 apart):
//   Qb [chunk][16 positions][d / 16]  queries as left operand (row position, column d), times e^b per channel
//   Kb [chunk][d / 16][16 positions]  keys as left operand of the state's products (row d), times what remains of them
//   Ab [chunk][block (i, j <= i)]     weights of 16 x 16 positions as left operand
//   Sb [chunk][d / 16][v / 8]         state at the chunk's start as right operand (both parts in one uint4)
constexpr int kBlocks = 10;              // 16 x 16 blocks on and below the diagonal

template <bool CH> struct DpCfg {
    static constexpr int LF = CH ? 68 : 72;
    static constexpr size_t SMEM = (size_t)((CH ? 3 : 2) * 64 * LF + (CH ? 2 * 64 * 20 : 0)) * 4;
};

// CH: decay per channel
template <bool CH>
__global__ void __launch_bounds__(256, 2) decay_prep_kernel(const DaParams p) {
    constexpr int LF = DpCfg<CH>::LF;
    extern __shared__ __align__(16) float dp_smem[];
    float* qf = dp_smem;                 // [64][LF] queries, later the weights
    float* kf = qf + 64 * LF;
    float* bf = kf + 64 * LF;            // running sums of log2 alpha (CH)
    float* a1s = bf + 64 * LF;           // [64][20]
    float* a2s = a1s + 64 * 20;          // [64][20]
    __shared__ float seg[4][64], pw[kL + 1];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    const int c = blockIdx.x, h = blockIdx.y % p.H, b = blockIdx.y / p.H;
    const size_t bc = (size_t)blockIdx.y * p.nc + c;
    const int n = min(kL, p.T - c * kL);                     // live positions
    const size_t row0 = (size_t)b * p.Tall + p.t0 + c * kL;
    pdl_wait();
    pdl_release();
    const float dec = CH ? 0.f : p.decay[h];
    if (!CH && tid <= kL) pw[tid] = powf(dec, (float)tid);

    auto load_tile = [&](const void* src, float scale, float* dst, int d0) {
        for (int i = tid; i < kL * 8; i += 256) {
            const int s = i >> 3, cc = (i & 7) * 8, d = d0 + cc;
            float v[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = 0.f;
            if (s < n && d < p.D) {
                const bf16* x = reinterpret_cast<const bf16*>(src) + (row0 + s) * p.ldp + (size_t)h * p.D;
                const uint4 w = *reinterpret_cast<const uint4*>(x + d);
                v[0] = bf_lo(w.x), v[1] = bf_hi(w.x), v[2] = bf_lo(w.y), v[3] = bf_hi(w.y);
                v[4] = bf_lo(w.z), v[5] = bf_hi(w.z), v[6] = bf_lo(w.w), v[7] = bf_hi(w.w);
                if (d < p.rot_dims) {
                    const int half = p.rot_dims >> 1;
                    const size_t at = da_pos(p, p.t0 + c * kL + s) * half;
                    const float* cs = p.cos_t + at;
                    const float* sn = p.sin_t + at;
                    if (!p.rot_pairs && half % 8 == 0) {
                        const bool second = d >= half;
                        const int e = second ? d - half : d;
                        const uint4 o = *reinterpret_cast<const uint4*>(x + (second ? d - half : d + half));
                        const float u[8] = {bf_lo(o.x), bf_hi(o.x), bf_lo(o.y), bf_hi(o.y), bf_lo(o.z), bf_hi(o.z), bf_lo(o.w), bf_hi(o.w)};
#pragma unroll
                        for (int q4 = 0; q4 < 2; ++q4) {
                            float cv[4], sv[4];
                            ld4(cs + e + 4 * q4, cv);
                            ld4(sn + e + 4 * q4, sv);
#pragma unroll
                            for (int j = 0; j < 4; ++j) {
                                const float uu = u[4 * q4 + j] * sv[j];
                                v[4 * q4 + j] = v[4 * q4 + j] * cv[j] + (second ? uu : -uu);
                            }
                        }
                    } else {
#pragma unroll
                        for (int j = 0; j < 8; ++j) v[j] = rotated(x, d + j, p.rot_dims, p.rot_pairs, cs, sn);
                    }
                }
            }
            st4(dst + s * LF + cc, v[0] * scale, v[1] * scale, v[2] * scale, v[3] * scale);
            st4(dst + s * LF + cc + 4, v[4] * scale, v[5] * scale, v[6] * scale, v[7] * scale);
        }
    };

    float acc[4][4];                     // fixed decay: 16 x 32 weights of a warp; CH: 16 x 16 of a block (first two)
    float diag[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    const int wi = CH ? (warp < 1 ? 1 : (warp < 3 ? 2 : 3)) : (warp & 3);          // block row of this warp's weights
    const int wj = CH ? warp - wi * (wi - 1) / 2 : 2 * (warp >> 2);                // first block column
    // CH, on the diagonal of 16 x 16 blocks: warps 6 and 7 take the lower left quarters (queries 8 .. 15, keys 0 .. 7) of two
    // blocks each; of the 8 x 8 blocks left, a thread takes 2 x 2 pairs over half the channels
    const int db8 = (tid >> 4) & 7, du = (tid >> 2) & 3, dt = tid & 3, dh = tid >> 7;

    for (int d0 = 0; d0 < p.Dp; d0 += 64) {
        __syncthreads();
        load_tile(p.q, p.q_scale, qf, d0);
        load_tile(p.k, p.k_scale, kf, d0);
        if (CH) {
            const int d = tid & 63, tg = tid >> 6;
            float z[16];
            const float bias = d0 + d < p.D ? p.a2b[(size_t)h * p.D + d0 + d] : 0.f;
#pragma unroll
            for (int j = 0; j < 16; ++j) z[j] = bias;
            for (int r0 = 0; r0 < p.rank; r0 += 16) {
                if (r0) __syncthreads();
                for (int i = tid; i < 64 * 16; i += 256) {
                    const int s = i >> 4, r = i & 15;
                    a1s[s * 20 + r] = s < n && r0 + r < p.rank ? p.a[(row0 + s) * p.lda + r0 + r] : 0.f;
                    a2s[s * 20 + r] = d0 + s < p.D && r0 + r < p.rank
                                          ? to_f(reinterpret_cast<const bf16*>(p.a2)[((size_t)h * p.D + d0 + s) * p.rank + r0 + r]) : 0.f;
                }
                __syncthreads();
#pragma unroll
                for (int r = 0; r < 16; r += 4) {
                    float w[4];
                    ld4(a2s + d * 20 + r, w);
#pragma unroll
                    for (int j = 0; j < 16; ++j) {
                        float a[4];
                        ld4(a1s + (tg * 16 + j) * 20 + r, a);
                        z[j] += a[0] * w[0] + a[1] * w[1] + a[2] * w[2] + a[3] * w[3];
                    }
                }
            }
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                if (tg * 16 + j < n) sum += log2_alpha(z[j], p.inv_tau);
                z[j] = sum;
            }
            seg[tg][d] = sum;
            __syncthreads();
            float before = 0.f;
            for (int u = 0; u < tg; ++u) before += seg[u][d];
#pragma unroll
            for (int j = 0; j < 16; ++j) bf[(tg * 16 + j) * LF + d] = before + z[j];
        }
        __syncthreads();
        // queries and keys as operands
#pragma unroll 1
        for (int blk = warp; blk < 16; blk += 8) {
            uint32_t hi[4], lo[4];
            {
                const int rb = blk >> 2, db = blk & 3;
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int at = (16 * rb + g + 8 * (i & 1)) * LF + 16 * db + 2 * t4 + 8 * (i >> 1);
                    float2 x = *reinterpret_cast<const float2*>(qf + at);
                    if (CH) {
                        const float2 e = *reinterpret_cast<const float2*>(bf + at);
                        x.x *= ex2f(e.x);
                        x.y *= ex2f(e.y);
                    }
                    split_bf2(x.x, x.y, hi[i], lo[i]);
                }
                uint4* dst = p.Qb + ((bc * 4 + rb) * (p.Dp / 16) + d0 / 16 + db) * 64 + lane;
                dst[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                dst[32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
            {
                const int db = blk >> 2, kk = blk & 3;
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int d = 16 * db + g + 8 * (i & 1), s = 16 * kk + 2 * t4 + 8 * (i >> 1);
                    float x = kf[s * LF + d], y = kf[(s + 1) * LF + d];
                    if (CH) {
                        const float e = bf[63 * LF + d];
                        x *= ex2f(e - bf[s * LF + d]);
                        y *= ex2f(e - bf[(s + 1) * LF + d]);
                    } else {
                        x *= pw[max(n - 1 - s, 0)];          // keys past the sequence are zero
                        y *= pw[max(n - 2 - s, 0)];
                    }
                    split_bf2(x, y, hi[i], lo[i]);
                }
                uint4* dst = p.Kb + ((bc * (p.Dp / 16) + d0 / 16 + db) * 4 + kk) * 64 + lane;
                dst[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                dst[32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
        }
        if (tid < 64) p.keep[bc * p.Dp + d0 + tid] = CH ? ex2f(bf[63 * LF + tid]) : pw[n];
        // weights
        if (CH ? warp < 6 : 16 * wi + 15 >= 16 * wj) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t ah[4], al[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int col = 16 * kk + 2 * t4 + 8 * (i >> 1), at = (16 * wi + g + 8 * (i & 1)) * LF + col;
                    float2 x = *reinterpret_cast<const float2*>(qf + at);
                    if (CH) {                                // measured from the end of the block before
                        const float2 e = *reinterpret_cast<const float2*>(bf + at);
                        const float2 r = *reinterpret_cast<const float2*>(bf + (16 * wi - 1) * LF + col);
                        x.x *= ex2f(e.x - r.x);
                        x.y *= ex2f(e.y - r.y);
                    }
                    split_bf2(x.x, x.y, ah[i], al[i]);
                }
#pragma unroll
                for (int nb = 0; nb < (CH ? 2 : 4); ++nb) {
                    uint32_t bh[2], bl[2];
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const int col = 16 * kk + 2 * t4 + 8 * i, at = (16 * wj + 8 * nb + g) * LF + col;
                        float2 x = *reinterpret_cast<const float2*>(kf + at);
                        if (CH) {
                            const float2 e = *reinterpret_cast<const float2*>(bf + at);
                            const float2 r = *reinterpret_cast<const float2*>(bf + (16 * wi - 1) * LF + col);
                            x.x *= ex2f(r.x - e.x);
                            x.y *= ex2f(r.y - e.y);
                        }
                        split_bf2(x.x, x.y, bh[i], bl[i]);
                    }
                    mma_bf16(acc[nb], ah[0], ah[1], ah[2], ah[3], bh[0], bh[1]);
                    mma_bf16(acc[nb], ah[0], ah[1], ah[2], ah[3], bl[0], bl[1]);
                    mma_bf16(acc[nb], al[0], al[1], al[2], al[3], bh[0], bh[1]);
                }
            }
        } else if (CH) {
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int base = 16 * (2 * (warp - 6) + u);
#pragma unroll 1
                for (int kk = 0; kk < 4; ++kk) {
                    uint32_t ah[2], al[2], bh[2], bl[2];
#pragma unroll
                    for (int i = 0; i < 2; ++i) {            // measured from the quarter's last key
                        const int col = 16 * kk + 2 * t4 + 8 * i, aq = (base + 8 + g) * LF + col, ak = (base + g) * LF + col;
                        const float2 r = *reinterpret_cast<const float2*>(bf + (base + 7) * LF + col);
                        float2 x = *reinterpret_cast<const float2*>(qf + aq), e = *reinterpret_cast<const float2*>(bf + aq);
                        split_bf2(x.x * ex2f(e.x - r.x), x.y * ex2f(e.y - r.y), ah[i], al[i]);
                        x = *reinterpret_cast<const float2*>(kf + ak);
                        e = *reinterpret_cast<const float2*>(bf + ak);
                        split_bf2(x.x * ex2f(r.x - e.x), x.y * ex2f(r.y - e.y), bh[i], bl[i]);
                    }
                    // rows 0 .. 7 of the operand are zero
                    mma_bf16(acc[u], 0u, ah[0], 0u, ah[1], bh[0], bh[1]);
                    mma_bf16(acc[u], 0u, ah[0], 0u, ah[1], bl[0], bl[1]);
                    mma_bf16(acc[u], 0u, al[0], 0u, al[1], bh[0], bh[1]);
                }
            }
        }
        if (CH && dt <= du) {
            // 2 x 2 pairs of an 8 x 8 block on the diagonal, half of the channels
            const int tr = (8 * db8 + 2 * du) * LF + 32 * dh, sr = (8 * db8 + 2 * dt) * LF + 32 * dh;
#pragma unroll 2
            for (int d = 0; d < 32; d += 4) {
                float x[2][4], y[2][4], e[2][4], f[2][4];
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    ld4(qf + tr + u * LF + d, x[u]);
                    ld4(kf + sr + u * LF + d, y[u]);
                    ld4(bf + tr + u * LF + d, e[u]);
                    ld4(bf + sr + u * LF + d, f[u]);
                }
#pragma unroll
                for (int u = 0; u < 2; ++u)
#pragma unroll
                    for (int w = 0; w < 2; ++w)
#pragma unroll
                        for (int j = 0; j < 4; ++j)          // (a key after its query is weighed here and dropped below)
                            diag[2 * u + w] += x[u][j] * y[w][j] * ex2f(fminf(e[u][j] - f[w][j], 0.f));
            }
        }
    }
    __syncthreads();
    float* sc = qf;
    if (CH ? warp < 6 : 16 * wi + 15 >= 16 * wj) {
#pragma unroll
        for (int nb = 0; nb < (CH ? 2 : 4); ++nb)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = 16 * wi + g + 8 * (e >> 1), s = 16 * wj + 8 * nb + 2 * t4 + (e & 1);
                sc[t * LF + s] = CH ? acc[nb][e] : (s <= t ? acc[nb][e] * pw[t - s] : 0.f);
            }
    }
    if (CH) {
        // the diagonal: quarters above it are zero, the halves of the channels meet here
        if (warp >= 6)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int base = 16 * (2 * (warp - 6) + u);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    sc[(base + 8 + g) * LF + base + 2 * t4 + e] = acc[u][2 + e];
                    sc[(base + g) * LF + base + 8 + 2 * t4 + e] = 0.f;
                }
            }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            if (half) __syncthreads();
            if (dh == half)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = 2 * du + (e >> 1), s = 2 * dt + (e & 1);
                    float* at = sc + (8 * db8 + t) * LF + 8 * db8 + s;
                    if (s > t) *at = 0.f;
                    else *at = half ? *at + diag[e] : diag[e];
                }
        }
    }
    __syncthreads();
    for (int blk = warp; blk < kBlocks; blk += 8) {
        const int i = blk < 1 ? 0 : (blk < 3 ? 1 : (blk < 6 ? 2 : 3)), j = blk - i * (i + 1) / 2;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float2 x = *reinterpret_cast<const float2*>(sc + (16 * i + g + 8 * (e & 1)) * LF + 16 * j + 2 * t4 + 8 * (e >> 1));
            split_bf2(x.x, x.y, hi[e], lo[e]);
        }
        uint4* dst = p.Ab + (bc * kBlocks + blk) * 64 + lane;
        dst[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        dst[32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
}

constexpr int kTd = 64, kLd = 72;        // tile width, row stride of a 64-wide shared-memory tile (bf16)
constexpr int kKbBytes = 4 * 4 * 64 * 16;     // bytes of a chunk's key operand for 64 channels
constexpr int kDsStages = 4;
constexpr int kDsStage = kKbBytes + kL * kLd * 2 + kTd * 4;   // bytes: key operand, values, keep

// state at every chunk's start (as sums of two bf16 parts) and after the last chunk; one CTA owns 64 x 64 of a head's S:
// warp = 16 rows x 32 columns
__global__ void __launch_bounds__(256) decay_state_kernel(const DaParams p) {
    extern __shared__ __align__(16) unsigned char da_raw[];
    const int tid = threadIdx.x, lane = tid & 31, warp = (tid >> 5) & 3, wv = tid >> 7, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.z % p.H, b = blockIdx.z / p.H;
    const int d0 = blockIdx.x * kTd, v0 = blockIdx.y * kTd;
    const size_t bh = blockIdx.z;
    const bf16* vb = reinterpret_cast<const bf16*>(p.v) + (size_t)h * p.V;
    auto load = [&](int c) {
        if (c < p.nc) {
            const uint32_t st = smem_u32(da_raw) + (uint32_t)(c % kDsStages) * kDsStage;
            const uint4* ka = p.Kb + ((bh * p.nc + c) * (p.Dp / 16) + d0 / 16) * 256;
#pragma unroll
            for (int i = 0; i < kKbBytes / 16 / 256; ++i) cpa16(st + 16 * (tid + 256 * i), ka + tid + 256 * i, true);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int s = (tid >> 3) + 32 * i, cc = (tid & 7) * 8, tt = c * kL + s;
                const bool vl = tt < p.T && v0 + cc < p.V;
                cpa16(st + kKbBytes + (s * kLd + cc) * 2, vl ? vb + ((size_t)b * p.Tall + p.t0 + tt) * p.ldp + v0 + cc : vb, vl);
            }
            if (tid < kTd / 4) cpa16(st + kKbBytes + kL * kLd * 2 + 16 * tid, p.keep + (bh * p.nc + c) * p.Dp + d0 + 4 * tid, true);
        }
        cpa_commit();
    };
    const int dr[2] = {d0 + 16 * warp + g, d0 + 16 * warp + g + 8};
    float acc[4][4];
    pdl_wait();
    pdl_release();
    for (int c = 0; c < kDsStages - 1; ++c) load(c);
    const size_t slb = bh * p.slices;
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = v0 + 32 * wv + 8 * j + 2 * t + (e & 1), d = dr[e >> 1];
            acc[j][e] = d < p.D && v < p.V ? p.S[((slb + v / kSl) * p.D + d) * kSl + v % kSl] : 0.f;
        }
    for (int c = 0; c < p.nc; ++c) {
        const size_t bc = bh * p.nc + c;
        cpa_wait<kDsStages - 2>();
        __syncthreads();                 // chunk c has landed; nobody still reads the stage that is loaded next
        load(c + kDsStages - 1);
        const unsigned char* st = da_raw + (size_t)(c % kDsStages) * kDsStage;
        const uint32_t ka = smem_u32(st) + (uint32_t)(warp * 256 + lane) * 16, va = smem_u32(st) + kKbBytes;
        const float* keep = reinterpret_cast<const float*>(st + kKbBytes + kL * kLd * 2) + 16 * warp + g;
        float add[2][4][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) add[u][j][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            const uint4 hi = lds128(ka + kk * 1024), lo = lds128(ka + kk * 1024 + 512);
            uint32_t vf[2][4];
#pragma unroll
            for (int jp = 0; jp < 2; ++jp)
                ldsm4_t(va + ((16 * kk + (lane & 7) + ((lane >> 3) & 1) * 8) * kLd + 32 * wv + 16 * jp + (lane >> 4) * 8) * 2, vf[jp][0], vf[jp][1],
                        vf[jp][2], vf[jp][3]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                mma_bf16(add[0][j], hi.x, hi.y, hi.z, hi.w, vf[j >> 1][2 * (j & 1)], vf[j >> 1][2 * (j & 1) + 1]);
                mma_bf16(add[1][j], lo.x, lo.y, lo.z, lo.w, vf[j >> 1][2 * (j & 1)], vf[j >> 1][2 * (j & 1) + 1]);
            }
        }
        // the state this chunk starts from
        uint4* sb = p.Sb + ((bc * (p.Dp / 16) + d0 / 16 + warp) * (p.Vp / 8) + v0 / 8 + 4 * wv) * 32 + lane;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            uint32_t h0, l0, h1, l1;
            split_bf2(acc[j][0], acc[j][1], h0, l0);
            split_bf2(acc[j][2], acc[j][3], h1, l1);
            sb[j * 32] = make_uint4(transpose8(h0), transpose8(h1), transpose8(l0), transpose8(l1));
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[j][e] = keep[8 * (e >> 1)] * acc[j][e] + (add[0][j][e] + add[1][j][e]);
    }
    cpa_wait<0>();
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = v0 + 32 * wv + 8 * j + 2 * t + (e & 1), d = dr[e >> 1];
            if (d < p.D && v < p.V) p.S[((slb + v / kSl) * p.D + d) * kSl + v % kSl] = acc[j][e];
        }
}

// outputs of a chunk: 64 positions x VT value columns of a head; the rows of the state come in steps of 32, two buffered.
// A head that fits VT columns is normed, gated and stored here.
template <int VT> struct DoCfg {
    static constexpr int LV = VT + 8, NV = VT / 8;
    static constexpr int STAGE = 2 * NV * 32 * 16;           // bytes of 32 rows of state fragments
    static constexpr size_t SMEM = (size_t)2 * STAGE + (size_t)kL * LV * 2;
};

template <int VT>
__global__ void __launch_bounds__(128, 3) decay_out_kernel(const DaParams p) {
    using C = DoCfg<VT>;
    constexpr int LV = C::LV, NV = C::NV;
    extern __shared__ __align__(16) unsigned char da_raw[];
    bf16* vs = reinterpret_cast<bf16*>(da_raw + 2 * C::STAGE);      // [64][LV]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.z % p.H, b = blockIdx.z / p.H, c = blockIdx.y, v0 = blockIdx.x * VT;
    const size_t bc = (size_t)blockIdx.z * p.nc + c, row0 = (size_t)b * p.Tall + p.t0 + c * kL;
    const bf16* vb = reinterpret_cast<const bf16*>(p.v) + (size_t)h * p.V;
    pdl_wait();
    pdl_release();
    auto load = [&](int k, int buf) {
        const uint4* sb = p.Sb + (bc * (p.Dp / 16) + 2 * k) * (size_t)(p.Vp / 8) * 32;
        const uint32_t dst = smem_u32(da_raw + (size_t)buf * C::STAGE);
        for (int i = tid; i < 2 * NV * 32; i += 128) {
            const int r = i / (NV * 32), j = i % (NV * 32);
            const bool live = v0 / 8 + j / 32 < p.Vp / 8;
            cpa16(dst + 16 * i, live ? sb + (size_t)r * (p.Vp / 8) * 32 + (size_t)(v0 / 8) * 32 + j : sb, live);
        }
        cpa_commit();
    };
    for (int i = tid; i < kL * (VT / 8); i += 128) {
        const int s = i / (VT / 8), cc = (i % (VT / 8)) * 8;
        const bool live = c * kL + s < p.T && v0 + cc < p.V;
        cpa16(smem_u32(vs + s * LV + cc), live ? vb + (row0 + s) * p.ldp + v0 + cc : vb, live);
    }
    load(0, 0);
    const uint4* qb = p.Qb + (bc * 4 + warp) * (size_t)(p.Dp / 16) * 64 + lane;
    const int nk = p.Dp / 32;
    uint4 qn[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) qn[i] = qb[32 * i];
    float acc[NV][4];
#pragma unroll
    for (int j = 0; j < NV; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    for (int k = 0; k < nk; ++k) {
        uint4 qc[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) qc[i] = qn[i];
        if (k + 1 < nk) {
            load(k + 1, (k + 1) & 1);
#pragma unroll
            for (int i = 0; i < 4; ++i) qn[i] = qb[(size_t)128 * (k + 1) + 32 * i];
            cpa_wait<1>();
        } else {
            cpa_wait<0>();
        }
        __syncthreads();
        const uint32_t sb = smem_u32(da_raw + (size_t)(k & 1) * C::STAGE);
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
            const uint4 hi = qc[2 * kk], lo = qc[2 * kk + 1];
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const uint4 f = lds128(sb + (uint32_t)((kk * NV + j) * 32 + lane) * 16);
                mma_bf16(acc[j], hi.x, hi.y, hi.z, hi.w, f.x, f.y);
                mma_bf16(acc[j], hi.x, hi.y, hi.z, hi.w, f.z, f.w);
                mma_bf16(acc[j], lo.x, lo.y, lo.z, lo.w, f.x, f.y);
            }
        }
        __syncthreads();
    }
    const int tr[2] = {16 * warp + g, 16 * warp + g + 8};
    if (p.decay) {
        const float dec = p.decay[h], s0 = powf(dec, (float)(tr[0] + 1)), s1 = powf(dec, (float)(tr[1] + 1));
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            acc[j][0] *= s0;
            acc[j][1] *= s0;
            acc[j][2] *= s1;
            acc[j][3] *= s1;
        }
    }
    const uint4* ab = p.Ab + (bc * kBlocks + warp * (warp + 1) / 2) * 64 + lane;
#pragma unroll 1
    for (int kk = 0; kk <= warp; ++kk) {
        const uint4 hi = ab[64 * kk], lo = ab[64 * kk + 32];
        const int srow = 16 * kk + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
        for (int jp = 0; jp < NV / 2; ++jp) {
            uint32_t b0, b1, b2, b3;
            ldsm4_t(smem_u32(vs + srow * LV + 16 * jp + (lane >> 4) * 8), b0, b1, b2, b3);
            mma_bf16(acc[2 * jp], hi.x, hi.y, hi.z, hi.w, b0, b1);
            mma_bf16(acc[2 * jp], lo.x, lo.y, lo.z, lo.w, b0, b1);
            mma_bf16(acc[2 * jp + 1], hi.x, hi.y, hi.z, hi.w, b2, b3);
            mma_bf16(acc[2 * jp + 1], lo.x, lo.y, lo.z, lo.w, b2, b3);
        }
    }
    const bool whole = p.V <= VT;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) ss += acc[j][2 * e] * acc[j][2 * e] + acc[j][2 * e + 1] * acc[j][2 * e + 1];
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        if (c * kL + tr[e] >= p.T) continue;
        const size_t row = row0 + tr[e], at = row * p.H * p.V + (size_t)h * p.V;
        if (whole) {
            const float inv = 1.f / sqrtf(ss / p.V + p.eps);
            const bf16* gr = reinterpret_cast<const bf16*>(p.g) + row * p.ldp + (size_t)h * p.V;
            const float* w = p.norm_w ? p.norm_w + (size_t)h * p.norm_stride : nullptr;
            bf16* out = reinterpret_cast<bf16*>(p.out) + at;
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int v = 8 * j + 2 * t;
                if (v < p.V) {
                    const uint32_t gv = *reinterpret_cast<const uint32_t*>(gr + v);
                    const float w0 = w ? w[v] : 1.f, w1 = w ? w[v + 1] : 1.f;
                    *reinterpret_cast<uint32_t*>(out + v) = pack_bf2(acc[j][2 * e] * inv * w0 * gate_f<bf16>(p.gate, bf_lo(gv)),
                                                                     acc[j][2 * e + 1] * inv * w1 * gate_f<bf16>(p.gate, bf_hi(gv)));
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int v = v0 + 8 * j + 2 * t;
                if (v < p.V) *reinterpret_cast<float2*>(p.o + at + v) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
            }
        }
    }
}

// one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) decay_norm_kernel(const DaParams p) {
    pdl_wait();
    pdl_release();
    const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= (long long)p.B * p.T * p.H) return;
    const int h = (int)(i % p.H);
    const long long bt = i / p.H;
    da_norm_gate<T>(p, (size_t)(bt / p.T) * p.Tall + p.t0 + bt % p.T, h, threadIdx.x & 31);
}

}  // namespace glq

using namespace glq;

struct DaWs {
    size_t qb, kb, ab, sb, keep, total;
};
static DaWs da_ws(const glq_decay_t* a) {
    DaWs w{};
    size_t at = 0;
    auto take = [&](size_t bytes) {
        const size_t v = at;
        at += (bytes + 255) / 256 * 256;
        return v;
    };
    const size_t chunks = (size_t)a->B * a->H * cdiv_i(std::min(a->T, kSegment), kL), Dp = (a->D + 63) / 64 * 64, Vp = (a->V + 63) / 64 * 64;
    w.qb = take(chunks * kL * Dp * 4);
    w.kb = take(chunks * kL * Dp * 4);
    w.ab = take(chunks * kBlocks * 64 * 16);
    w.sb = take(chunks * Dp * Vp * 4);
    w.keep = take(chunks * Dp * 4);
    w.total = at;
    return w;
}
extern "C" int glq_decay_slices(int V) { return (V + kSl - 1) / kSl; }
extern "C" size_t glq_decay_workspace_bytes(const glq_decay_t* a) { return da_ws(a).total; }

static int da_params(const glq_decay_t* a, DaParams& p) {
    if (!a || a->B <= 0 || a->T < 0 || a->H <= 0 || a->D <= 0 || a->V <= 0 || a->rot_dims < 0 || a->rot_dims % 2 || a->rot_dims > a->D)
        return GLQ_ERR_ARG;
    if (!a->q || !a->k || !a->v || !a->g || !a->S || !a->o || !a->out) return GLQ_ERR_ARG;
    if (!a->decay && (!a->a || !a->a2 || !a->a2b || a->rank <= 0 || !(a->tau > 0.f))) return GLQ_ERR_ARG;
    if (a->rot_dims && (!a->start || !a->cos_t || !a->sin_t || a->max_len <= 0)) return GLQ_ERR_ARG;
    if (a->dtype != GLQ_DT_BF16 && a->dtype != GLQ_DT_F32) return GLQ_ERR_ARG;
    if (!al16(a->S) || !al16(a->o)) return GLQ_ERR_ALIGN;
    if (a->D > 8192 || (long)a->B * a->H > 65535) return GLQ_ERR_UNSUPPORTED;
    p.q = a->q;
    p.k = a->k;
    p.v = a->v;
    p.g = a->g;
    p.decay = a->decay;
    p.a = a->a;
    p.a2 = a->a2;
    p.a2b = a->a2b;
    p.cos_t = a->cos_t;
    p.sin_t = a->sin_t;
    p.start = reinterpret_cast<const long long*>(a->start);
    p.norm_w = a->norm_w;
    p.S = a->S;
    p.o = a->o;
    p.out = a->out;
    p.ldp = a->ldp;
    p.lda = a->lda;
    p.B = a->B;
    p.T = p.Tall = a->T;
    p.H = a->H;
    p.D = a->D;
    p.V = a->V;
    p.slices = glq_decay_slices(a->V);
    p.rank = a->rank;
    p.rot_dims = a->rot_dims;
    p.rot_pairs = a->rot_pairs;
    p.max_len = a->max_len;
    p.norm_stride = a->norm_stride;
    p.gate = a->gate;
    p.state_idle = a->state_idle;
    p.vec4 = al16(a->g) && al16(a->out) && al16(a->norm_w) && a->ldp % 4 == 0 && a->norm_stride % 4 == 0;
    p.q_scale = a->q_scale;
    p.k_scale = a->k_scale;
    p.eps = a->eps;
    p.inv_tau = a->decay ? 0.f : 1.f / a->tau;
    return GLQ_OK;
}
static int da_norm(const DaParams& p, int dtype, void* stream) {
    const dim3 grid(cdiv_i((long)p.B * p.T * p.H, 8));
    if (dtype == GLQ_DT_BF16) return dn_launch(decay_norm_kernel<bf16>, grid, 256, 0, stream, p);
    return dn_launch(decay_norm_kernel<float>, grid, 256, 0, stream, p);
}

constexpr int kClusterSteps = 64;        // longer passes norm all rows in a launch of their own
extern "C" int glq_decay_step(const glq_decay_t* a, void* stream) {
    DaParams p{};
    int st = da_params(a, p);
    if (st != GLQ_OK) return st;
    if (p.T == 0) return GLQ_OK;
    const dim3 grid(p.slices, p.B * p.H);
    const size_t smem = (size_t)3 * p.D * 4;
    if (p.slices <= kMaxCluster && p.T <= kClusterSteps) {
        if (a->dtype == GLQ_DT_BF16) return dn_launch_cluster(p.slices, decay_step_kernel<bf16, true>, grid, 256, smem, stream, p);
        return dn_launch_cluster(p.slices, decay_step_kernel<float, true>, grid, 256, smem, stream, p);
    }
    if (a->dtype == GLQ_DT_BF16) st = dn_launch(decay_step_kernel<bf16, false>, grid, 256, smem, stream, p);
    else st = dn_launch(decay_step_kernel<float, false>, grid, 256, smem, stream, p);
    if (st != GLQ_OK) return st;
    return da_norm(p, a->dtype, stream);
}

extern "C" int glq_decay_chunk_supported(const glq_decay_t* a) {
    return a && a->dtype == GLQ_DT_BF16 && a->D % 8 == 0 && a->V % 8 == 0 && a->ldp % 8 == 0 && al16(a->q) && al16(a->k) && al16(a->v) &&
           al16(a->g) && (!a->rot_dims || (al16(a->cos_t) && al16(a->sin_t)));
}

extern "C" int glq_decay_chunk(const glq_decay_t* a, void* stream) {
    if (!glq_decay_chunk_supported(a)) return GLQ_ERR_UNSUPPORTED;
    DaParams p{};
    int st = da_params(a, p);
    if (st != GLQ_OK) return st;
    if (p.T == 0) return GLQ_OK;
    const DaWs w = da_ws(a);
    if (!a->workspace) return GLQ_ERR_ARG;
    if (a->workspace_bytes < w.total) return GLQ_ERR_WORKSPACE;
    if (!al16(a->workspace) || !al16(a->out)) return GLQ_ERR_ALIGN;
    char* ws = reinterpret_cast<char*>(a->workspace);
    p.Qb = reinterpret_cast<uint4*>(ws + w.qb);
    p.Kb = reinterpret_cast<uint4*>(ws + w.kb);
    p.Ab = reinterpret_cast<uint4*>(ws + w.ab);
    p.Sb = reinterpret_cast<uint4*>(ws + w.sb);
    p.keep = reinterpret_cast<float*>(ws + w.keep);
    p.Dp = (a->D + 63) / 64 * 64;
    p.Vp = (a->V + 63) / 64 * 64;
    const int bh = p.B * p.H;
    for (p.t0 = 0; p.t0 < p.Tall; p.t0 += kSegment) {
        p.T = std::min(kSegment, p.Tall - p.t0);
        p.nc = cdiv_i(p.T, kL);
        const dim3 pg(p.nc, bh);
        if (p.decay) st = dn_launch(decay_prep_kernel<false>, pg, 256, DpCfg<false>::SMEM, stream, p);
        else st = dn_launch(decay_prep_kernel<true>, pg, 256, DpCfg<true>::SMEM, stream, p);
        if (st != GLQ_OK) return st;
        // (waiting CTAs of the next two would take room from the running kernel)
        if ((st = dn_launch_if(false, decay_state_kernel, dim3(p.Dp / 64, p.Vp / 64, bh), 256, (size_t)kDsStages * kDsStage, stream, p)) != GLQ_OK) return st;
        if (p.V > 64) st = dn_launch_if(false, decay_out_kernel<128>, dim3(cdiv_i(p.V, 128), p.nc, bh), 128, DoCfg<128>::SMEM, stream, p);
        else st = dn_launch_if(false, decay_out_kernel<64>, dim3(1, p.nc, bh), 128, DoCfg<64>::SMEM, stream, p);
        if (st != GLQ_OK) return st;
        if (p.V > 128 && (st = da_norm(p, a->dtype, stream)) != GLQ_OK) return st;
    }
    return GLQ_OK;
}
