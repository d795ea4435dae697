// Matrix-memory recurrence with exponential gates and a running log maximum (mLSTM; Beck et al., "xLSTM: Extended Long
// Short-Term Memory").  Per head, S (D, V), n (D) and m are float and carried from call to call:
//     m' = max(f + m, i);  S' = e^(f+m-m') S + e^(i-m') k v^T;  n' = e^(f+m-m') n + e^(i-m') k
//     o = S'^T q / (max(|n'.q|, e^-m') + 1e-6)
// Two forms of the same recurrence:
//   * step: the recurrence itself, one position after the other; a CTA owns 32 value columns of a head.  The per-head
//     norm and output gate that follow go into the staging of the output product of a decode step (dense_mm.cu), or are
//     a launch of their own.
//   * chunk: 64 positions at a time on the tensor cores.  With b the running sum of f inside a chunk, a_s = i_s - b_s
//     and r_t = b_t - m_t, position s reaches position t of its chunk with weight e^(r_t + a_s) and the state at the
//     chunk's start with e^(r_t + m_start); m_t = b_t + max(m_start, max_{s<=t} a_s) is the recurrence's own maximum.
//     Every float operand of a tensor-core product (scaled keys, state, weights) goes in as a sum of two bf16 numbers.
// State layout: S (B, H, slices, D, 32), n (B, H, slices, D) and m (B, H, slices), the last two once per 32-column
// slice, so that no CTA reads what another one is about to write.
#include "recurrent.cuh"

namespace glq {

struct MlParams {
    const void* qkvg;
    const float* gates;
    const float* bias_i;
    const float* bias_f;
    const float* norm_w;
    float* S;
    float* n;
    float* m;
    void* out;
    float* o;                      // (B * Tall, H * V)
    long long ldp, ldg;
    int B, T, H, D, V, slices;
    int state_idle, vec4;          // vec4: gates, norm weights and outputs allow reads of four values
    int t0, Tall;                  // this call's positions: t0 .. t0 + T - 1 of the Tall rows of a sequence
    float cap, eps, scale;
    // chunk form
    float *bs, *as, *cm, *tot, *m0, *min_, *nbuf, *ksum;
    uint32_t *Sb, *Kb;
    int nc, Dp, Vp;
};

__device__ __forceinline__ float log_i(const MlParams& p, size_t row, int h) {
    return p.cap * tanhf((p.gates[row * p.ldg + h] + p.bias_i[h]) / p.cap);
}
__device__ __forceinline__ float log_f(const MlParams& p, size_t row, int h) {
    const float z = p.cap * tanhf((p.gates[row * p.ldg + p.H + h] + p.bias_f[h]) / p.cap);
    return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// one row of head h: out = rms_norm(o) * w * sigmoid(g); one warp
template <typename T>
__device__ __forceinline__ void head_norm_gate(const MlParams& p, size_t row, int h, int lane) {
    const float* o = p.o + row * p.H * p.V + (size_t)h * p.V;
    const T* g = reinterpret_cast<const T*>(p.qkvg) + row * p.ldp + (size_t)p.H * (2 * p.D + p.V) + (size_t)h * p.V;
    T* out = reinterpret_cast<T*>(p.out) + row * p.H * p.V + (size_t)h * p.V;
    norm_gate<T>(o, g, p.norm_w + (size_t)h * p.V, GLQ_GATE_SIGMOID, out, p.V, p.eps, p.vec4, lane);
}

template <typename T>
__global__ void __launch_bounds__(256) mlstm_step_kernel(const MlParams p) {
    extern __shared__ float ml_smem[];
    float* sq = ml_smem;                 // [D]
    float* sk = sq + p.D;                // [D]
    __shared__ float sv[kSl], part[8][kSl], dpart[8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int sl = blockIdx.x, h = blockIdx.y % p.H, b = blockIdx.y / p.H;
    const int D = p.D, V = p.V, v0 = sl * kSl, vw = min(kSl, V - v0);
    const size_t bh = (size_t)b * p.H + h;
    float* S = p.S + (bh * p.slices + sl) * (size_t)D * kSl;
    float* n = p.n + (bh * p.slices + sl) * (size_t)D;
    float* mp = p.m + bh * p.slices + sl;
    const int rr = warp * 4 + (lane >> 3), cc = (lane & 7) * 4;
    constexpr int U = 8;
    float4 pre[U];
    // a state that the preceding launch does not touch is requested before the wait for the projections
    if (!p.state_idle) pdl_wait();
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int d = rr + 32 * u;
        pre[u] = d < D ? *reinterpret_cast<const float4*>(S + (size_t)d * kSl + cc) : make_float4(0, 0, 0, 0);
    }
    float m = *mp;
    pdl_wait();
    pdl_release();
    for (int t = 0; t < p.T; ++t) {
        const size_t row = (size_t)b * p.Tall + p.t0 + t;
        const T* q = reinterpret_cast<const T*>(p.qkvg) + row * p.ldp + (size_t)h * D;
        const T* k = q + (size_t)p.H * D;
        const T* v = reinterpret_cast<const T*>(p.qkvg) + row * p.ldp + (size_t)2 * p.H * D + (size_t)h * V + v0;
        __syncthreads();
        for (int d = tid; d < D; d += 256) {
            sq[d] = to_f(q[d]) * p.scale;
            sk[d] = to_f(k[d]);
        }
        if (tid < kSl) sv[tid] = tid < vw ? to_f(v[tid]) : 0.f;
        const float li = log_i(p, row, h), lf = log_f(p, row, h);
        const float mn = fmaxf(lf + m, li);
        const float keep = expf(lf + m - mn), add = expf(li - mn);
        m = mn;
        __syncthreads();
        const float4 vv = make_float4(sv[cc], sv[cc + 1], sv[cc + 2], sv[cc + 3]);
        float4 acc = make_float4(0, 0, 0, 0);
        for (int d0 = 0; d0 < D; d0 += 32 * U) {
            if (t > 0 || d0 > 0) {
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
                    const float kd = add * sk[d], qd = sq[d];
                    float4 s = pre[u];
                    s.x = keep * s.x + kd * vv.x;
                    s.y = keep * s.y + kd * vv.y;
                    s.z = keep * s.z + kd * vv.z;
                    s.w = keep * s.w + kd * vv.w;
                    *reinterpret_cast<float4*>(S + (size_t)d * kSl + cc) = s;
                    acc.x += s.x * qd;
                    acc.y += s.y * qd;
                    acc.z += s.z * qd;
                    acc.w += s.w * qd;
                }
            }
        }
        float den = 0.f;
        for (int d = tid; d < D; d += 256) {
            const float nn = keep * n[d] + add * sk[d];
            n[d] = nn;
            den += nn * sq[d];
        }
#pragma unroll
        for (int o = 8; o < 32; o <<= 1) {
            acc.x += __shfl_xor_sync(0xffffffffu, acc.x, o);
            acc.y += __shfl_xor_sync(0xffffffffu, acc.y, o);
            acc.z += __shfl_xor_sync(0xffffffffu, acc.z, o);
            acc.w += __shfl_xor_sync(0xffffffffu, acc.w, o);
        }
        den = warp_sum(den);
        if (lane < 8) *reinterpret_cast<float4*>(&part[warp][cc]) = acc;
        if (lane == 0) dpart[warp] = den;
        __syncthreads();
        if (tid < vw) {
            float num = 0.f, dd = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                num += part[w][tid];
                dd += dpart[w];
            }
            p.o[row * p.H * V + (size_t)h * V + v0 + tid] = num / (fmaxf(fabsf(dd), expf(-m)) + 1e-6f);
        }
    }
    if (tid == 0) *mp = m;
}

// ---- chunk form ------------------------------------------------------------------------------------------
// Per chunk and head, one CTA.  Gates: running sum of f (bs), i - bs (as) and its running maximum (cm) for every position,
// sum and maximum of the chunk (tot); positions past T weigh nothing.  Keys: k e^(as - maximum) as the left operand of the
// state's products, [d / 16][16 positions][part][lane] of uint4 (part: the two bf16 parts), and their sum over the chunk.
constexpr int kGd = 128;                 // keys of 128 channels at a time: warp = 16 of them
__global__ void __launch_bounds__(256) mlstm_gate_kernel(const MlParams p) {
    __shared__ __align__(16) bf16 ks[kL * (kGd + 8)];
    __shared__ float ws[kL];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, t4 = lane & 3;
    const int c = blockIdx.x, h = blockIdx.y % p.H, b = blockIdx.y / p.H;
    const size_t bh = blockIdx.y, bc = bh * p.nc + c;
    const bf16* kb = reinterpret_cast<const bf16*>(p.qkvg) + (size_t)p.H * p.D + (size_t)h * p.D;
    pdl_wait();
    pdl_release();
    auto load = [&](int d0) {
        for (int i = tid; i < kL * (kGd / 8); i += 256) {
            const int s = i / (kGd / 8), cc = (i % (kGd / 8)) * 8, tt = c * kL + s;
            const bool live = tt < p.T && d0 + cc < p.D;
            cpa16(smem_u32(ks + s * (kGd + 8) + cc), live ? kb + ((size_t)b * p.Tall + p.t0 + tt) * p.ldp + d0 + cc : kb, live);
        }
        cpa_commit();
    };
    load(0);
    if (warp == 0) {
        // the maximum the sequence starts from, before the state kernel replaces it
        if (c == 0 && lane == 0) p.m0[bh] = p.m[bh * p.slices];
        float f[2], li[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = c * kL + 2 * lane + e;
            const size_t row = (size_t)b * p.Tall + p.t0 + t;
            f[e] = t < p.T ? log_f(p, row, h) : 0.f;
            li[e] = t < p.T ? log_i(p, row, h) : -INFINITY;
        }
        float sum = f[0] + f[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += u;
        }
        const float b1 = sum, b0 = sum - f[1];
        const float a0 = li[0] - b0, a1 = li[1] - b1;
        float mx = fmaxf(a0, a1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float u = __shfl_up_sync(0xffffffffu, mx, o);
            if (lane >= o) mx = fmaxf(mx, u);
        }
        const float prev = __shfl_up_sync(0xffffffffu, mx, 1), top = __shfl_sync(0xffffffffu, mx, 31);
        const size_t i = bc * kL + 2 * lane;
        *reinterpret_cast<float2*>(p.bs + i) = make_float2(b0, b1);
        *reinterpret_cast<float2*>(p.as + i) = make_float2(a0, a1);
        *reinterpret_cast<float2*>(p.cm + i) = make_float2(lane ? fmaxf(prev, a0) : a0, mx);
        if (lane == 31) *reinterpret_cast<float2*>(p.tot + bc * 2) = make_float2(b1, mx);
        ws[2 * lane] = expf(a0 - top);
        ws[2 * lane + 1] = expf(a1 - top);
    }
    for (int d0 = 0; d0 < p.Dp; d0 += kGd) {
        cpa_wait<0>();
        __syncthreads();
        if (d0 + 16 * warp < p.Dp) {
            uint4* dst = reinterpret_cast<uint4*>(p.Kb) + (bc * (p.Dp / 16) + d0 / 16 + warp) * 256 + lane;
            float ns[2] = {0.f, 0.f};
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t a[4], hi[4], lo[4];
                ldsm4_t(smem_u32(ks + (16 * kk + (lane >> 4) * 8 + (lane & 7)) * (kGd + 8) + 16 * warp + ((lane >> 3) & 1) * 8), a[0], a[1],
                        a[2], a[3]);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int s = 16 * kk + 2 * t4 + 8 * (i >> 1);
                    const float x = bf_lo(a[i]) * ws[s], y = bf_hi(a[i]) * ws[s + 1];
                    ns[i & 1] += x + y;
                    split_bf2(x, y, hi[i], lo[i]);
                }
                dst[kk * 64] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
                dst[kk * 64 + 32] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                ns[e] += __shfl_xor_sync(0xffffffffu, ns[e], 1);
                ns[e] += __shfl_xor_sync(0xffffffffu, ns[e], 2);
                if (t4 == 0) p.ksum[bc * p.Dp + d0 + 16 * warp + (lane >> 2) + 8 * e] = ns[e];
            }
        }
        __syncthreads();
        if (d0 + kGd < p.Dp) load(d0 + kGd);
    }
}

constexpr int kTd = 64, kLd = 72;        // tile width, row stride of a 64-wide shared-memory tile (bf16)
constexpr int kKb = 4 * 4 * 64 * 16;     // bytes of a chunk's key operand for 64 channels
constexpr int kStStages = 4;
constexpr int kStStage = kKb + kL * kLd * 2 + kTd * 4;   // bytes: key operand, values, key sums

// Scratch layout of a chunk's starting state: blocks of 16 rows (d) x 8 columns (v) as the fragments the output kernel's
// products take, [d / 16][v / 8][lane] of uint4 = (first part rows 0-7, rows 8-15, second part rows 0-7, rows 8-15).

// state at every chunk's start (as sums of two bf16 parts, and n) and after the last chunk; one CTA owns 64 x 64 of a
// head's S: warp = 16 rows x 32 columns
__global__ void __launch_bounds__(256) mlstm_state_kernel(const MlParams p) {
    extern __shared__ __align__(16) unsigned char ml_raw[];
    __shared__ float2 s_tot[kSegment / kL];
    const int tid = threadIdx.x, lane = tid & 31, warp = (tid >> 5) & 3, wv = tid >> 7, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.z % p.H, b = blockIdx.z / p.H;
    const int d0 = blockIdx.x * kTd, v0 = blockIdx.y * kTd;
    const size_t bh = blockIdx.z;
    const bf16* vb = reinterpret_cast<const bf16*>(p.qkvg) + (size_t)2 * p.H * p.D + (size_t)h * p.V;
    auto load = [&](int c) {
        if (c < p.nc) {
            const uint32_t st = smem_u32(ml_raw) + (uint32_t)(c % kStStages) * kStStage;
            const unsigned char* ka = reinterpret_cast<const unsigned char*>(p.Kb) + ((bh * p.nc + c) * (p.Dp / 16) + d0 / 16) * 4096;
#pragma unroll
            for (int i = 0; i < kKb / 16 / 256; ++i) cpa16(st + 16 * (tid + 256 * i), ka + 16 * (tid + 256 * i), true);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int s = (tid >> 3) + 32 * i, cc = (tid & 7) * 8, tt = c * kL + s;
                const bool vl = tt < p.T && v0 + cc < p.V;
                cpa16(st + kKb + (s * kLd + cc) * 2, vl ? vb + ((size_t)b * p.Tall + p.t0 + tt) * p.ldp + v0 + cc : vb, vl);
            }
            if (tid < kTd / 4) cpa16(st + kKb + kL * kLd * 2 + 16 * tid, p.ksum + (bh * p.nc + c) * p.Dp + d0 + 4 * tid, true);
        }
        cpa_commit();
    };
    const int dr[2] = {d0 + 16 * warp + g, d0 + 16 * warp + g + 8};
    float acc[4][4], nacc[2];
    pdl_wait();
    pdl_release();
    for (int c = 0; c < kStStages - 1; ++c) load(c);
    const size_t slb = bh * p.slices;
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = v0 + 32 * wv + 8 * j + 2 * t + (e & 1), d = dr[e >> 1];
            acc[j][e] = d < p.D && v < p.V ? p.S[((slb + v / kSl) * p.D + d) * kSl + v % kSl] : 0.f;
        }
#pragma unroll
    for (int e = 0; e < 2; ++e) nacc[e] = dr[e] < p.D ? p.n[(slb + v0 / kSl) * p.D + dr[e]] : 0.f;
    float m = p.m0[bh];
    for (int c = tid; c < p.nc; c += 256) s_tot[c] = *reinterpret_cast<const float2*>(p.tot + (bh * p.nc + c) * 2);
    for (int c = 0; c < p.nc; ++c) {
        const size_t bc = bh * p.nc + c;
        cpa_wait<kStStages - 2>();
        __syncthreads();                 // chunk c has landed; nobody still reads the stage that is loaded next
        load(c + kStStages - 1);
        const unsigned char* st = ml_raw + (size_t)(c % kStStages) * kStStage;
        const uint32_t ka = smem_u32(st) + (uint32_t)(warp * 256 + lane) * 16, va = smem_u32(st) + kKb;
        const float* ksum = reinterpret_cast<const float*>(st + kKb + kL * kLd * 2);
        // the chunk's end: b_L = tot.x, m_L = b_L + max(m, tot.y); keys carry e^(as - tot.y)
        const float2 tot = s_tot[c];
        const float m_end = tot.x + fmaxf(m, tot.y), rl = tot.x - m_end, keep = expf(rl + m), fac = expf(rl + tot.y);
        if (blockIdx.x == 0 && blockIdx.y == 0 && tid == 0) p.min_[bc] = m;
        m = m_end;
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
        uint4* sb = reinterpret_cast<uint4*>(p.Sb) + ((bc * (p.Dp / 16) + d0 / 16 + warp) * (p.Vp / 8) + v0 / 8 + 4 * wv) * 32 + lane;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            uint32_t h0, l0, h1, l1;
            split_bf2(acc[j][0], acc[j][1], h0, l0);
            split_bf2(acc[j][2], acc[j][3], h1, l1);
            sb[j * 32] = make_uint4(transpose8(h0), transpose8(h1), transpose8(l0), transpose8(l1));
        }
        if (blockIdx.y == 0 && wv == 0 && t == 0) {
            p.nbuf[bc * p.Dp + dr[0]] = nacc[0];
            p.nbuf[bc * p.Dp + dr[1]] = nacc[1];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[j][e] = keep * acc[j][e] + fac * (add[0][j][e] + add[1][j][e]);
#pragma unroll
        for (int e = 0; e < 2; ++e) nacc[e] = keep * nacc[e] + fac * ksum[16 * warp + g + 8 * e];
    }
    cpa_wait<0>();
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int v = v0 + 32 * wv + 8 * j + 2 * t + (e & 1), d = dr[e >> 1];
            if (d < p.D && v < p.V) p.S[((slb + v / kSl) * p.D + d) * kSl + v % kSl] = acc[j][e];
        }
    for (int s = v0 / kSl; s < min(p.slices, (v0 + kTd) / kSl); ++s) {
        if (t == 0 && wv == 0)
#pragma unroll
            for (int e = 0; e < 2; ++e)
                if (dr[e] < p.D) p.n[(slb + s) * p.D + dr[e]] = nacc[e];
        if (blockIdx.x == 0 && tid == 0) p.m[slb + s] = m;
    }
}

// outputs of a chunk: 64 positions x VT value columns of a head; the rows of the state come in steps of 32, two buffered
template <int VT> struct MoCfg {
    static constexpr int LV = VT + 8, NV = VT / 8, LQ = 40;
    static constexpr int QK = kL * LQ * 2;                   // bytes of 64 x 32 queries (or keys)
    static constexpr int SB = 2 * NV * 32 * 16;              // bytes of 32 rows of state fragments
    static constexpr int STAGE = 2 * QK + SB;
    static constexpr size_t SMEM = (size_t)2 * STAGE + (size_t)kL * LV * 2;
};

template <int VT>
__global__ void __launch_bounds__(128, 3) mlstm_out_kernel(const MlParams p) {
    using C = MoCfg<VT>;
    constexpr int LV = C::LV, NV = C::NV, LQ = C::LQ;
    extern __shared__ __align__(16) unsigned char ml_raw[];
    bf16* vs = reinterpret_cast<bf16*>(ml_raw + 2 * C::STAGE);      // [64][LV]
    __shared__ float sa[kL], sr[kL], sm[kL], sqn[kL];
    __shared__ __align__(16) float sn[2][32];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.z % p.H, b = blockIdx.z / p.H, c = blockIdx.y, v0 = blockIdx.x * VT;
    const size_t bc = (size_t)blockIdx.z * p.nc + c;
    const bf16* base = reinterpret_cast<const bf16*>(p.qkvg);
    pdl_wait();
    pdl_release();
    auto row_of = [&](int s) { return ((size_t)b * p.Tall + p.t0 + c * kL + s) * p.ldp; };
    auto load = [&](int k, int buf) {
        unsigned char* st = ml_raw + (size_t)buf * C::STAGE;
        bf16* qs = reinterpret_cast<bf16*>(st);
        bf16* ks = qs + kL * LQ;
        const int d0 = 32 * k;
        for (int i = tid; i < kL * 4; i += 128) {
            const int s = i >> 2, cc = (i & 3) * 8;
            const bool live = c * kL + s < p.T && d0 + cc < p.D;
            const bf16* src = live ? base + row_of(s) + (size_t)h * p.D + d0 + cc : base;
            cpa16(smem_u32(qs + s * LQ + cc), src, live);
            cpa16(smem_u32(ks + s * LQ + cc), live ? src + (size_t)p.H * p.D : base, live);
        }
        const uint4* sb = reinterpret_cast<const uint4*>(p.Sb) + (bc * (p.Dp / 16) + d0 / 16) * (size_t)(p.Vp / 8) * 32;
        const uint32_t dst = smem_u32(st + 2 * C::QK);
        for (int i = tid; i < 2 * NV * 32; i += 128) {
            const int r = i / (NV * 32), j = i % (NV * 32);
            const bool live = v0 / 8 + j / 32 < p.Vp / 8;
            cpa16(dst + 16 * i, live ? sb + (size_t)r * (p.Vp / 8) * 32 + (size_t)(v0 / 8) * 32 + j : sb, live);
        }
        if (tid < 8) cpa16(smem_u32(&sn[buf][4 * tid]), p.nbuf + bc * p.Dp + d0 + 4 * tid, true);
        cpa_commit();
    };
    for (int i = tid; i < kL * (VT / 8); i += 128) {
        const int s = i / (VT / 8), cc = (i % (VT / 8)) * 8;
        const bool live = c * kL + s < p.T && v0 + cc < p.V;
        cpa16(smem_u32(vs + s * LV + cc), live ? base + row_of(s) + (size_t)2 * p.H * p.D + (size_t)h * p.V + v0 + cc : base, live);
    }
    load(0, 0);
    const float m0 = p.min_[bc];
    if (tid < kL) {
        const float bb = p.bs[bc * kL + tid], mm = bb + fmaxf(m0, p.cm[bc * kL + tid]);
        sa[tid] = p.as[bc * kL + tid];
        sr[tid] = bb - mm;
        sm[tid] = mm;
    }
    float qk[8][4], acc[NV][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) qk[j][e] = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] = 0.f;
    float qn = 0.f;                                      // row tid / 2, half tid % 2 of q . n
    const int nk = p.Dp / 32;
    for (int k = 0; k < nk; ++k) {
        if (k + 1 < nk) {
            load(k + 1, (k + 1) & 1);
            cpa_wait<1>();
        } else {
            cpa_wait<0>();
        }
        __syncthreads();
        const unsigned char* st = ml_raw + (size_t)(k & 1) * C::STAGE;
        const bf16* qs = reinterpret_cast<const bf16*>(st);
        const bf16* ks = qs + kL * LQ;
        const uint32_t sb = smem_u32(st + 2 * C::QK);
        {
            const bf16* qr = qs + (tid >> 1) * LQ + (tid & 1) * 16;
            const float* nr = sn[k & 1] + (tid & 1) * 16;
#pragma unroll
            for (int i = 0; i < 16; i += 2) {
                const uint32_t w = *reinterpret_cast<const uint32_t*>(qr + i);
                qn += bf_lo(w) * nr[i] + bf_hi(w) * nr[i + 1];
            }
        }
#pragma unroll
        for (int kk = 0; kk < 2; ++kk) {
            uint32_t a0, a1, a2, a3;
            ldsm4(smem_u32(qs + (16 * warp + (lane & 7) + ((lane >> 3) & 1) * 8) * LQ + 16 * kk + (lane >> 4) * 8), a0, a1, a2, a3);
#pragma unroll
            for (int jp = 0; jp < 4; ++jp) {
                if (jp > warp) continue;                 // keys after every query of this warp
                uint32_t b0, b1, b2, b3;
                ldsm4(smem_u32(ks + (16 * jp + (lane & 7) + (lane >> 4) * 8) * LQ + 16 * kk + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
                mma_bf16(qk[2 * jp], a0, a1, a2, a3, b0, b1);
                mma_bf16(qk[2 * jp + 1], a0, a1, a2, a3, b2, b3);
            }
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const uint4 f = lds128(sb + (uint32_t)((kk * NV + j) * 32 + lane) * 16);
                mma_bf16(acc[j], a0, a1, a2, a3, f.x, f.y);
                mma_bf16(acc[j], a0, a1, a2, a3, f.z, f.w);
            }
        }
        __syncthreads();
    }
    qn += __shfl_xor_sync(0xffffffffu, qn, 1);
    if ((tid & 1) == 0) sqn[tid >> 1] = qn;
    __syncthreads();
    const int tr[2] = {16 * warp + g, 16 * warp + g + 8};
    float den[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const float w = expf(sr[tr[e]] + m0) * p.scale;
        den[e] = 0.f;
#pragma unroll
        for (int j = 0; j < NV; ++j) {
            acc[j][2 * e] *= w;
            acc[j][2 * e + 1] *= w;
        }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int s = 8 * j + 2 * t + (e & 1), tt = tr[e >> 1];
            const float v = s <= tt ? qk[j][e] * p.scale * expf(sr[tt] + sa[s]) : 0.f;
            qk[j][e] = v;
            den[e >> 1] += v;
        }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
        if (kk > warp) continue;
        uint32_t hi[4], lo[4];
        split_bf2(qk[2 * kk][0], qk[2 * kk][1], hi[0], lo[0]);
        split_bf2(qk[2 * kk][2], qk[2 * kk][3], hi[1], lo[1]);
        split_bf2(qk[2 * kk + 1][0], qk[2 * kk + 1][1], hi[2], lo[2]);
        split_bf2(qk[2 * kk + 1][2], qk[2 * kk + 1][3], hi[3], lo[3]);
        const int srow = 16 * kk + (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
        for (int jp = 0; jp < NV / 2; ++jp) {
            uint32_t b0, b1, b2, b3;
            ldsm4_t(smem_u32(vs + srow * LV + 16 * jp + (lane >> 4) * 8), b0, b1, b2, b3);
            mma_bf16(acc[2 * jp], hi[0], hi[1], hi[2], hi[3], b0, b1);
            mma_bf16(acc[2 * jp], lo[0], lo[1], lo[2], lo[3], b0, b1);
            mma_bf16(acc[2 * jp + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
            mma_bf16(acc[2 * jp + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
        }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        den[e] += __shfl_xor_sync(0xffffffffu, den[e], 1);
        den[e] += __shfl_xor_sync(0xffffffffu, den[e], 2);
        const int tt = tr[e];
        den[e] += expf(sr[tt] + m0) * p.scale * sqn[tt];
        const float inv = 1.f / (fmaxf(fabsf(den[e]), expf(-sm[tt])) + 1e-6f);
        if (c * kL + tt < p.T) {
            float* o = p.o + ((size_t)b * p.Tall + p.t0 + c * kL + tt) * p.H * p.V + (size_t)h * p.V;
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int v = v0 + 8 * j + 2 * t;
                if (v < p.V) *reinterpret_cast<float2*>(o + v) = make_float2(acc[j][2 * e] * inv, acc[j][2 * e + 1] * inv);
            }
        }
    }
}

// one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) mlstm_norm_kernel(const MlParams p) {
    pdl_wait();
    pdl_release();
    const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (i >= (long long)p.B * p.T * p.H) return;
    const int h = (int)(i % p.H);
    const long long bt = i / p.H;
    head_norm_gate<T>(p, (size_t)(bt / p.T) * p.Tall + p.t0 + bt % p.T, h, threadIdx.x & 31);
}

}  // namespace glq

using namespace glq;

extern "C" int glq_mlstm_slices(int V) { return (V + kSl - 1) / kSl; }

static inline size_t up256d(size_t v) { return (v + 255) / 256 * 256; }

struct MlWs {
    size_t bs, as, cm, tot, m0, min_, nbuf, ksum, sb, kb, total;
};
static MlWs ml_ws(const glq_mlstm_t* a) {
    MlWs w{};
    size_t at = 0;
    auto take = [&](size_t bytes) {
        const size_t v = at;
        at += up256d(bytes);
        return v;
    };
    const size_t bh = (size_t)a->B * a->H, nc = cdiv_i(std::min(a->T, kSegment), kL), Dp = (a->D + 63) / 64 * 64, Vp = (a->V + 63) / 64 * 64;
    w.bs = take(bh * nc * kL * 4);
    w.as = take(bh * nc * kL * 4);
    w.cm = take(bh * nc * kL * 4);
    w.tot = take(bh * nc * 8);
    w.m0 = take(bh * 4);
    w.min_ = take(bh * nc * 4);
    w.nbuf = take(bh * nc * Dp * 4);
    w.ksum = take(bh * nc * Dp * 4);
    w.sb = take(bh * nc * Dp * Vp * 4);
    w.kb = take(bh * nc * Dp * kL * 4);
    w.total = at;
    return w;
}
extern "C" size_t glq_mlstm_workspace_bytes(const glq_mlstm_t* a) { return ml_ws(a).total; }

static int ml_params(const glq_mlstm_t* a, MlParams& p) {
    if (!a || a->B <= 0 || a->T < 0 || a->H <= 0 || a->D <= 0 || a->V <= 0 || !(a->gate_cap > 0.f)) return GLQ_ERR_ARG;
    if (!a->qkvg || !a->gates || !a->bias_i || !a->bias_f || !a->norm_w || !a->S || !a->n || !a->m || !a->o) return GLQ_ERR_ARG;
    if (a->dtype != GLQ_DT_BF16 && a->dtype != GLQ_DT_F32) return GLQ_ERR_ARG;
    if (!al16(a->S) || !al16(a->o)) return GLQ_ERR_ALIGN;
    if (a->D > 8192 || (long)a->B * a->H > 65535) return GLQ_ERR_UNSUPPORTED;
    p.qkvg = a->qkvg;
    p.gates = a->gates;
    p.bias_i = a->bias_i;
    p.bias_f = a->bias_f;
    p.norm_w = a->norm_w;
    p.S = a->S;
    p.n = a->n;
    p.m = a->m;
    p.o = a->o;
    p.out = a->out;
    p.ldp = a->ldp;
    p.ldg = a->ldg;
    p.B = a->B;
    p.T = p.Tall = a->T;
    p.H = a->H;
    p.D = a->D;
    p.V = a->V;
    p.slices = glq_mlstm_slices(a->V);
    p.state_idle = a->state_idle;
    p.vec4 = al16(a->qkvg) && al16(a->out) && al16(a->norm_w) && a->ldp % 4 == 0 && a->H * (2 * a->D + a->V) % 4 == 0;
    p.cap = a->gate_cap;
    p.eps = a->eps;
    p.scale = (float)(1.0 / sqrt((double)a->D));
    return GLQ_OK;
}
static int ml_norm(const MlParams& p, int dtype, void* stream) {
    const dim3 grid(cdiv_i((long)p.B * p.T * p.H, 8));
    if (dtype == GLQ_DT_BF16) return dn_launch(mlstm_norm_kernel<bf16>, grid, 256, 0, stream, p);
    return dn_launch(mlstm_norm_kernel<float>, grid, 256, 0, stream, p);
}

extern "C" int glq_mlstm_step(const glq_mlstm_t* a, void* stream) {
    MlParams p{};
    int st = ml_params(a, p);
    if (st != GLQ_OK) return st;
    if (p.T == 0) return GLQ_OK;
    const dim3 grid(p.slices, p.B * p.H);
    const size_t smem = (size_t)2 * p.D * 4;
    if (a->dtype == GLQ_DT_BF16) st = dn_launch(mlstm_step_kernel<bf16>, grid, 256, smem, stream, p);
    else st = dn_launch(mlstm_step_kernel<float>, grid, 256, smem, stream, p);
    if (st != GLQ_OK || !p.out) return st;
    return ml_norm(p, a->dtype, stream);
}

extern "C" int glq_mlstm_chunk(const glq_mlstm_t* a, void* stream) {
    if (!a || a->dtype != GLQ_DT_BF16) return GLQ_ERR_ARG;
    if (a->D % 8 || a->V % 8 || a->ldp % 8) return GLQ_ERR_UNSUPPORTED;
    MlParams p{};
    int st = ml_params(a, p);
    if (st != GLQ_OK) return st;
    const MlWs w = ml_ws(a);
    if (!a->out || !a->workspace) return GLQ_ERR_ARG;
    if (a->workspace_bytes < w.total) return GLQ_ERR_WORKSPACE;
    if (!al16(a->qkvg) || !al16(a->workspace)) return GLQ_ERR_ALIGN;
    char* ws = reinterpret_cast<char*>(a->workspace);
    p.bs = reinterpret_cast<float*>(ws + w.bs);
    p.as = reinterpret_cast<float*>(ws + w.as);
    p.cm = reinterpret_cast<float*>(ws + w.cm);
    p.tot = reinterpret_cast<float*>(ws + w.tot);
    p.m0 = reinterpret_cast<float*>(ws + w.m0);
    p.min_ = reinterpret_cast<float*>(ws + w.min_);
    p.nbuf = reinterpret_cast<float*>(ws + w.nbuf);
    p.ksum = reinterpret_cast<float*>(ws + w.ksum);
    p.Sb = reinterpret_cast<uint32_t*>(ws + w.sb);
    p.Kb = reinterpret_cast<uint32_t*>(ws + w.kb);
    p.Dp = (a->D + 63) / 64 * 64;
    p.Vp = (a->V + 63) / 64 * 64;
    const int bh = p.B * p.H;
    for (p.t0 = 0; p.t0 < p.Tall; p.t0 += kSegment) {
        p.T = std::min(kSegment, p.Tall - p.t0);
        p.nc = cdiv_i(p.T, kL);
        if ((st = dn_launch(mlstm_gate_kernel, dim3(p.nc, bh), 256, 0, stream, p)) != GLQ_OK) return st;
        if ((st = dn_launch_if(false, mlstm_state_kernel, dim3(p.Dp / 64, p.Vp / 64, bh), 256, (size_t)kStStages * kStStage, stream, p)) != GLQ_OK) return st;
        if (p.V > 64) st = dn_launch_if(false, mlstm_out_kernel<128>, dim3(cdiv_i(p.V, 128), p.nc, bh), 128, MoCfg<128>::SMEM, stream, p);
        else st = dn_launch_if(false, mlstm_out_kernel<64>, dim3(1, p.nc, bh), 128, MoCfg<64>::SMEM, stream, p);
        if (st != GLQ_OK) return st;
        if ((st = ml_norm(p, a->dtype, stream)) != GLQ_OK) return st;
    }
    return GLQ_OK;
}
