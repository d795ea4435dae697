// Row kernels of the unquantized decoders: embedding, residual add with the layer norm of the sublayer's output or with
// RMS norms on either side of the add, softmax routing with a correction term and its entry lists, and the weighted sum of the experts' outputs fused with
// the norm and the residual add that follow it.  One CTA per row; the residual stream and all statistics are float.
#include "dense_common.cuh"
#include "moe_plan.cuh"

namespace glq {

constexpr int kRowThreads = 256;
constexpr int kMaxC = 32768;          // row length; a row is staged in shared memory as float

template <typename T>
__global__ void __launch_bounds__(kRowThreads) dense_embed_kernel(const int64_t* __restrict__ ids, const T* __restrict__ table,
                                                                  int C, int vocab, const float* __restrict__ hw, float eps,
                                                                  float* __restrict__ x, T* __restrict__ h) {
    __shared__ float red[32];
    pdl_wait();
    pdl_release();
    const size_t row = blockIdx.x;
    long long id = ids[row];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    float s = 0.f;
    for (int c = threadIdx.x; c < C; c += kRowThreads) {
        const T v = table[(size_t)id * C + c];
        x[row * C + c] = to_f(v);
        if (!hw) h[row * C + c] = v;
        s += to_f(v) * to_f(v);
    }
    if (!hw) return;
    const float inv = 1.f / sqrtf(block_sum(s, red) / C + eps);
    for (int c = threadIdx.x; c < C; c += kRowThreads) h[row * C + c] = from_f<T>(to_f(table[(size_t)id * C + c]) * inv * hw[c]);
}

// ys: the sublayer's output row.  x += norm(ys) * w; h = x, or norm(x) * final_w
template <typename T>
__device__ __forceinline__ void norm_add_row(float* ys, float* red, const float* __restrict__ w, const float* __restrict__ fw,
                                             float eps, int C, float* __restrict__ x, T* __restrict__ h) {
    float s = 0.f;
    for (int c = threadIdx.x; c < C; c += kRowThreads) s += ys[c];
    const float mean = block_sum(s, red) / C;
    s = 0.f;
    for (int c = threadIdx.x; c < C; c += kRowThreads) {
        const float d = ys[c] - mean;
        s += d * d;
    }
    const float inv = 1.f / sqrtf(block_sum(s, red) / C + eps);
    for (int c = threadIdx.x; c < C; c += kRowThreads) {
        const float v = x[c] + (ys[c] - mean) * inv * w[c];
        x[c] = v;
        ys[c] = v;
        if (!fw) h[c] = from_f<T>(v);
    }
    if (!fw) return;
    s = 0.f;
    for (int c = threadIdx.x; c < C; c += kRowThreads) s += ys[c];
    const float mean2 = block_sum(s, red) / C;
    s = 0.f;
    for (int c = threadIdx.x; c < C; c += kRowThreads) {
        const float d = ys[c] - mean2;
        s += d * d;
    }
    const float inv2 = 1.f / sqrtf(block_sum(s, red) / C + eps);
    for (int c = threadIdx.x; c < C; c += kRowThreads) h[c] = from_f<T>((ys[c] - mean2) * inv2 * fw[c]);
}

// The same with the row in registers: 8 consecutive values per thread and step, STEPS * 8 * kRowThreads values at most.
// load(c, v): the sublayer's output at columns c .. c + 7, given x there
template <typename T> __device__ __forceinline__ void st8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void st8<float>(float* p, const float (&v)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void st8<bf16>(bf16* p, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf2(v[0], v[1]), pack_bf2(v[2], v[3]), pack_bf2(v[4], v[5]), pack_bf2(v[6], v[7]));
}
__device__ __forceinline__ void ld8(const float* p, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
__device__ __forceinline__ void ld8(const bf16* p, float (&v)[8]) {
    const uint4 w = *reinterpret_cast<const uint4*>(p);
    v[0] = bf_lo(w.x), v[1] = bf_hi(w.x), v[2] = bf_lo(w.y), v[3] = bf_hi(w.y);
    v[4] = bf_lo(w.z), v[5] = bf_hi(w.z), v[6] = bf_lo(w.w), v[7] = bf_hi(w.w);
}
template <typename T, int STEPS, typename F>
__device__ __forceinline__ void norm_add_row_regs(float* red, const float* __restrict__ w, const float* __restrict__ fw, float eps, int C,
                                                  float* __restrict__ x, T* __restrict__ h, F load) {
    float xv[STEPS][8], yv[STEPS][8];
    float s = 0.f;
#pragma unroll
    for (int u = 0; u < STEPS; ++u) {
        const int c = (u * kRowThreads + threadIdx.x) * 8;
        if (c < C) {
            ld8(x + c, xv[u]);
            load(c, xv[u], yv[u]);
#pragma unroll
            for (int i = 0; i < 8; ++i) s += yv[u][i];
        }
    }
    const float mean = block_sum(s, red) / C;
    s = 0.f;
#pragma unroll
    for (int u = 0; u < STEPS; ++u)
        if ((u * kRowThreads + threadIdx.x) * 8 < C)
#pragma unroll
            for (int i = 0; i < 8; ++i) s += (yv[u][i] - mean) * (yv[u][i] - mean);
    const float inv = 1.f / sqrtf(block_sum(s, red) / C + eps);
    s = 0.f;
#pragma unroll
    for (int u = 0; u < STEPS; ++u) {
        const int c = (u * kRowThreads + threadIdx.x) * 8;
        if (c < C) {
            float wv[8];
            ld8(w + c, wv);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                xv[u][i] += (yv[u][i] - mean) * inv * wv[i];
                s += xv[u][i];
            }
            st8<float>(x + c, xv[u]);
            if (!fw) st8<T>(h + c, xv[u]);
        }
    }
    if (!fw) return;
    const float mean2 = block_sum(s, red) / C;
    s = 0.f;
#pragma unroll
    for (int u = 0; u < STEPS; ++u)
        if ((u * kRowThreads + threadIdx.x) * 8 < C)
#pragma unroll
            for (int i = 0; i < 8; ++i) s += (xv[u][i] - mean2) * (xv[u][i] - mean2);
    const float inv2 = 1.f / sqrtf(block_sum(s, red) / C + eps);
#pragma unroll
    for (int u = 0; u < STEPS; ++u) {
        const int c = (u * kRowThreads + threadIdx.x) * 8;
        if (c < C) {
            float wv[8];
            ld8(fw + c, wv);
#pragma unroll
            for (int i = 0; i < 8; ++i) wv[i] *= (xv[u][i] - mean2) * inv2;
            st8<T>(h + c, wv);
        }
    }
}

// STEPS 0: any width, through shared memory
template <typename T, int STEPS>
__global__ void __launch_bounds__(kRowThreads) dense_add_norm_kernel(const float* __restrict__ y, const float* __restrict__ w,
                                                                     const float* __restrict__ fw, float eps, int C,
                                                                     float* __restrict__ x, T* __restrict__ h) {
    extern __shared__ float ys[];
    __shared__ float red[32];
    pdl_wait();
    pdl_release();
    const size_t o = (size_t)blockIdx.x * C;
    if constexpr (STEPS > 0) {
        norm_add_row_regs<T, STEPS>(red, w, fw, eps, C, x + o, h + o, [&](int c, const float (&)[8], float (&v)[8]) { ld8(y + o + c, v); });
    } else {
        for (int c = threadIdx.x; c < C; c += kRowThreads) ys[c] = y[o + c];
        norm_add_row<T>(ys, red, w, fw, eps, C, x + o, h + o);
    }
}

// x += alpha * (rms(y) * w + rms(y2) * w2); h = rms(x) * hw.  y2 may be missing, y too (nothing is added); without w, y is
// added as it is, and without hw, h = x.
struct RmsParams {
    const float* y;
    const float* w;
    const float* y2;
    const float* w2;
    const float* hw;
    long long ldy, ldy2;
    float eps, alpha;
    int C;
};
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();
    if (lane == 0) red[warp] = make_float2(a, b);
    __syncthreads();
    const float2 v = lane < kRowThreads / 32 ? red[lane] : make_float2(0.f, 0.f);
    return make_float2(warp_sum(v.x), warp_sum(v.y));
}
// STEPS 0: any width, one value per thread and step; else the row in registers, 8 values per thread and step
template <typename T, int STEPS>
__global__ void __launch_bounds__(kRowThreads) dense_rms_add_kernel(const RmsParams p, float* __restrict__ xg, T* __restrict__ hg) {
    __shared__ float2 red[32];
    pdl_wait();
    pdl_release();
    const int C = p.C;
    const size_t row = blockIdx.x;
    float* x = xg + row * C;
    T* h = hg ? hg + row * C : nullptr;
    const float* y = p.y ? p.y + row * p.ldy : nullptr;
    const float* y2 = p.y2 ? p.y2 + row * p.ldy2 : nullptr;
    if constexpr (STEPS > 0) {
        float xv[STEPS][8], yv[STEPS][8], zv[STEPS][8];
        float s = 0.f, s2 = 0.f;
#pragma unroll
        for (int u = 0; u < STEPS; ++u) {
            const int c = (u * kRowThreads + threadIdx.x) * 8;
            if (c >= C) continue;
            ld8(x + c, xv[u]);
            if (y) {
                ld8(y + c, yv[u]);
#pragma unroll
                for (int i = 0; i < 8; ++i) s += yv[u][i] * yv[u][i];
            }
            if (y2) {
                ld8(y2 + c, zv[u]);
#pragma unroll
                for (int i = 0; i < 8; ++i) s2 += zv[u][i] * zv[u][i];
            }
        }
        float f = p.alpha, f2 = p.alpha;
        if (p.w) {
            const float2 t = block_sum2(s, s2, red);
            f *= 1.f / sqrtf(t.x / C + p.eps);
            f2 *= 1.f / sqrtf(t.y / C + p.eps);
        }
        s = 0.f;
#pragma unroll
        for (int u = 0; u < STEPS; ++u) {
            const int c = (u * kRowThreads + threadIdx.x) * 8;
            if (c >= C) continue;
            float wv[8];
            if (y) {
                if (p.w) ld8(p.w + c, wv);
#pragma unroll
                for (int i = 0; i < 8; ++i) xv[u][i] += yv[u][i] * f * (p.w ? wv[i] : 1.f);
            }
            if (y2) {
                if (p.w2) ld8(p.w2 + c, wv);
#pragma unroll
                for (int i = 0; i < 8; ++i) xv[u][i] += zv[u][i] * f2 * (p.w2 ? wv[i] : 1.f);
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) s += xv[u][i] * xv[u][i];
            if (y) st8<float>(x + c, xv[u]);
            if (h && !p.hw) st8<T>(h + c, xv[u]);
        }
        if (!h || !p.hw) return;
        const float inv = 1.f / sqrtf(block_sum2(s, 0.f, red).x / C + p.eps);
#pragma unroll
        for (int u = 0; u < STEPS; ++u) {
            const int c = (u * kRowThreads + threadIdx.x) * 8;
            if (c >= C) continue;
            float wv[8];
            ld8(p.hw + c, wv);
#pragma unroll
            for (int i = 0; i < 8; ++i) wv[i] *= xv[u][i] * inv;
            st8<T>(h + c, wv);
        }
    } else {
        float f = p.alpha, f2 = p.alpha;
        if (p.w) {
            float s = 0.f, s2 = 0.f;
            for (int c = threadIdx.x; c < C; c += kRowThreads) {
                if (y) s += y[c] * y[c];
                if (y2) s2 += y2[c] * y2[c];
            }
            const float2 t = block_sum2(s, s2, red);
            f *= 1.f / sqrtf(t.x / C + p.eps);
            f2 *= 1.f / sqrtf(t.y / C + p.eps);
        }
        float s = 0.f;
        for (int c = threadIdx.x; c < C; c += kRowThreads) {
            float v = x[c];
            if (y) v += y[c] * f * (p.w ? p.w[c] : 1.f);
            if (y2) v += y2[c] * f2 * (p.w2 ? p.w2[c] : 1.f);
            if (y) x[c] = v;
            if (h && !p.hw) h[c] = from_f<T>(v);
            s += v * v;
        }
        if (!h || !p.hw) return;
        const float inv = 1.f / sqrtf(block_sum2(s, 0.f, red).x / C + p.eps);
        for (int c = threadIdx.x; c < C; c += kRowThreads) h[c] = from_f<T>(x[c] * inv * p.hw[c]);   // x: own writes
    }
}

// experts' outputs of a token in slot order; a slot without an entry passes the layer's input through
template <typename T, int STEPS>
__global__ void __launch_bounds__(kRowThreads) dense_combine_norm_kernel(const T* __restrict__ eo, long long lde,
                                                                         const int* __restrict__ tok_entries,
                                                                         const float* __restrict__ wts, int top,
                                                                         const float* __restrict__ w, const float* __restrict__ fw,
                                                                         float eps, int C, float* __restrict__ x, T* __restrict__ h) {
    extern __shared__ float ys[];
    __shared__ float red[32];
    pdl_wait();
    pdl_release();
    const size_t row = blockIdx.x, o = row * C;
    if constexpr (STEPS > 0) {
        norm_add_row_regs<T, STEPS>(red, w, fw, eps, C, x + o, h + o, [&](int c, const float (&xv)[8], float (&v)[8]) {
#pragma unroll
            for (int i = 0; i < 8; ++i) v[i] = 0.f;
#pragma unroll 4
            for (int j = 0; j < top; ++j) {
                const int e = __ldg(tok_entries + row * top + j);
                const float g = __ldg(wts + row * top + j);
                float u[8];
                if (e >= 0) {
                    ld8(eo + (size_t)e * lde + c, u);
                } else {
#pragma unroll
                    for (int i = 0; i < 8; ++i) u[i] = xv[i];
                }
#pragma unroll
                for (int i = 0; i < 8; ++i) v[i] += g * u[i];
            }
        });
    } else {
        for (int c = threadIdx.x; c < C; c += kRowThreads) {
            float a = 0.f;
            for (int j = 0; j < top; ++j) {
                const int e = tok_entries[row * top + j];
                a += wts[row * top + j] * (e >= 0 ? to_f(eo[(size_t)e * lde + c]) : x[o + c]);
            }
            ys[c] = a;
        }
        norm_add_row<T>(ys, red, w, fw, eps, C, x + o, h + o);
    }
}

// ---- routing -------------------------------------------------------------------------------------------
struct RtParams {
    const float* logits;
    const float* correction;
    long long ldl;
    int n, E, A, top, chunk;      // A: experts and pass-through experts
    int* sel;
    float* wts;
    float* entry_scale;
    int* tok_entries;
    int* entry_row;
    int* active;
    int* slot_count;
    int* slot_offset;
    int* n_active;
    int max_slots;
};

// one token by one warp: s = softmax(logits); `top` times the largest remaining s + correction, lowest index on ties.
// sc: 2 * A floats of shared memory of this warp; s_sel, s_wts: the token's choices in shared memory as well, or NULL
__device__ __forceinline__ void route_corrected(const RtParams& p, int t, int lane, float* sc, int* s_sel, float* s_wts) {
    const float* row = p.logits + (size_t)t * p.ldl;
    float* score = sc + p.A;
    float mx = -INFINITY;
    for (int e = lane; e < p.A; e += 32) {
        const float v = row[e];
        score[e] = v;
        sc[e] = p.correction[e];
        mx = fmaxf(mx, v);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.f;
    for (int e = lane; e < p.A; e += 32) {
        const float v = expf(score[e] - mx);
        score[e] = v;
        sum += v;
    }
    sum = warp_sum(sum);
    for (int e = lane; e < p.A; e += 32) {
        score[e] /= sum;
        sc[e] += score[e];
    }
    __syncwarp();
    for (int j = 0; j < p.top; ++j) {
        float best = -INFINITY;
        int be = 0x7fffffff;
        for (int e = lane; e < p.A; e += 32)
            if (sc[e] > best) best = sc[e], be = e;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oe = __shfl_xor_sync(0xffffffffu, be, o);
            if (ob > best || (ob == best && oe < be)) best = ob, be = oe;
        }
        // nothing comparable left (scores that are no numbers): a pass-through slot of weight zero
        const bool none = be == 0x7fffffff;
        if (lane == 0) {
            const int sel = none ? p.A : be;
            const float wt = none ? 0.f : score[be];
            p.sel[(size_t)t * p.top + j] = sel;
            p.wts[(size_t)t * p.top + j] = wt;
            p.tok_entries[(size_t)t * p.top + j] = -1;
            if (s_sel) {
                s_sel[t * p.top + j] = sel;
                s_wts[t * p.top + j] = wt;
            }
            if (!none) sc[be] = -INFINITY;
        }
        __syncwarp();
    }
}

__global__ void __launch_bounds__(256) dense_route_kernel(const RtParams p) {
    extern __shared__ float rt_sc[];
    pdl_wait();
    pdl_release();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = blockIdx.x * 8 + warp;
    if (t < p.n) route_corrected(p, t, lane, rt_sc + (size_t)warp * 2 * p.A, nullptr, nullptr);
}

// few entries: routing and lists in one CTA
constexpr int kRouteOneCta = 1024;
__global__ void __launch_bounds__(1024) dense_route_plan_kernel(const RtParams p) {
    extern __shared__ float rt_sc[];
    __shared__ int s_sel[kRouteOneCta];
    __shared__ float s_wts[kRouteOneCta];
    int* cnt = reinterpret_cast<int*>(rt_sc + (size_t)16 * p.A);
    pdl_wait();
    pdl_release();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (warp < 8)       // the lists take all warps
        for (int t = warp; t < p.n; t += 8) route_corrected(p, t, lane, rt_sc + (size_t)warp * 2 * p.A, s_sel, s_wts);
    __syncthreads();
    const int ms = p.max_slots;
    plan_entries<float>(cnt, p.n, p.E, p.top, p.chunk, 0, 1, s_sel, s_wts, p.active, p.n_active, p.slot_count, p.slot_offset,
                        p.entry_row, p.entry_scale, p.tok_entries, p.active + ms, p.n_active + 1, p.slot_count + ms,
                        p.slot_offset + ms);
}

}  // namespace glq

using namespace glq;

template <typename F> static int by_dtype(int dtype, F f) {
    if (dtype == GLQ_DT_BF16) return f(bf16());
    if (dtype == GLQ_DT_F32) return f(float());
    return GLQ_ERR_ARG;
}

extern "C" int glq_dense_embed(int dtype, const int64_t* ids, const void* table, int rows, int C, int vocab, const float* hw, float eps,
                               float* x, void* h, void* stream) {
    if (!ids || !table || !x || !h || rows < 0 || C <= 0 || vocab <= 0) return GLQ_ERR_ARG;
    if (rows == 0) return GLQ_OK;
    return by_dtype(dtype, [&](auto z) {
        using T = decltype(z);
        return dn_launch(dense_embed_kernel<T>, dim3(rows), kRowThreads, 0, stream, ids, (const T*)table, C, vocab, hw, eps, x, (T*)h);
    });
}

extern "C" int glq_dense_add_norm(int dtype, const float* y, const float* w, const float* final_w, float eps, int rows, int C,
                                  float* x, void* h, void* stream) {
    if (!y || !w || !x || !h || rows < 0 || C <= 0) return GLQ_ERR_ARG;
    if (C > kMaxC) return GLQ_ERR_UNSUPPORTED;
    if (rows == 0) return GLQ_OK;
    return by_dtype(dtype, [&](auto z) {
        using T = decltype(z);
        const bool vec = C % 8 == 0 && al16(y) && al16(w) && al16(x) && al16(h) && al16(final_w);
        if (vec && C <= 8 * kRowThreads)
            return dn_launch(dense_add_norm_kernel<T, 1>, dim3(rows), kRowThreads, 0, stream, y, w, final_w, eps, C, x, (T*)h);
        if (vec && C <= 16 * kRowThreads)
            return dn_launch(dense_add_norm_kernel<T, 2>, dim3(rows), kRowThreads, 0, stream, y, w, final_w, eps, C, x, (T*)h);
        if (vec && C <= 32 * kRowThreads)
            return dn_launch(dense_add_norm_kernel<T, 4>, dim3(rows), kRowThreads, 0, stream, y, w, final_w, eps, C, x, (T*)h);
        return dn_launch(dense_add_norm_kernel<T, 0>, dim3(rows), kRowThreads, (size_t)C * 4, stream, y, w, final_w, eps, C, x, (T*)h);
    });
}

extern "C" int glq_dense_rms_add(int dtype, const float* y, int64_t ldy, const float* w, const float* y2, int64_t ldy2, const float* w2,
                                 float alpha, const float* hw, float eps, int rows, int C, float* x, void* h, void* stream) {
    if (!x || rows < 0 || C <= 0 || (!y && y2) || (y2 && !w != !w2) || (!y && !h)) return GLQ_ERR_ARG;
    if (rows == 0) return GLQ_OK;
    const RmsParams p{y, w, y2, w2, hw, (long long)ldy, (long long)ldy2, eps, alpha, C};
    return by_dtype(dtype, [&](auto z) {
        using T = decltype(z);
        const bool vec = C % 8 == 0 && al16(x) && al16(h) && al16(y) && al16(y2) && al16(w) && al16(w2) && al16(hw) && (!y || ldy % 4 == 0) &&
                         (!y2 || ldy2 % 4 == 0);
        auto go = [&](auto kern) { return dn_launch(kern, dim3(rows), kRowThreads, 0, stream, p, x, (T*)h); };
        if (vec && C <= 8 * kRowThreads) return go(dense_rms_add_kernel<T, 1>);
        if (vec && C <= 16 * kRowThreads) return go(dense_rms_add_kernel<T, 2>);
        return go(dense_rms_add_kernel<T, 0>);
    });
}

extern "C" int glq_dense_combine_norm(int dtype, const void* entry_out, int64_t lde, const int32_t* tok_entries, const float* wts,
                                      int top, const float* w, const float* final_w, float eps, int rows, int C, float* x, void* h,
                                      void* stream) {
    if (!entry_out || !tok_entries || !wts || !w || !x || !h || top <= 0 || rows < 0 || C <= 0) return GLQ_ERR_ARG;
    if (C > kMaxC) return GLQ_ERR_UNSUPPORTED;
    if (rows == 0) return GLQ_OK;
    return by_dtype(dtype, [&](auto z) {
        using T = decltype(z);
        const bool vec = C % 8 == 0 && lde % 8 == 0 && al16(entry_out) && al16(w) && al16(x) && al16(h) && al16(final_w);
        auto go = [&](auto kern, size_t smem) {
            return dn_launch(kern, dim3(rows), kRowThreads, smem, stream, (const T*)entry_out, (long long)lde, tok_entries, wts, top, w,
                             final_w, eps, C, x, (T*)h);
        };
        if (vec && C <= 8 * kRowThreads) return go(dense_combine_norm_kernel<T, 1>, 0);
        if (vec && C <= 16 * kRowThreads) return go(dense_combine_norm_kernel<T, 2>, 0);
        if (vec && C <= 32 * kRowThreads) return go(dense_combine_norm_kernel<T, 4>, 0);
        return go(dense_combine_norm_kernel<T, 0>, (size_t)C * 4);
    });
}

extern "C" int glq_route_max_slots(int n, int E, int top, int chunk) {
    const long nk = (long)n * top;
    const long m = std::min<long>(E, nk) + (chunk > 0 ? nk / chunk : 0);
    return (int)std::max<long>(1, std::min(m, nk));
}

extern "C" int glq_route(const glq_route_t* a, void* stream) {
    if (!a || a->n < 0 || a->E <= 0 || a->identity < 0 || a->top <= 0 || a->top > a->E + a->identity) return GLQ_ERR_ARG;
    if (!a->logits || !a->correction || !a->sel || !a->wts || !a->entry_scale || !a->tok_entries || !a->entry_row || !a->active ||
        !a->slot_count || !a->slot_offset || !a->n_active)
        return GLQ_ERR_ARG;
    if (a->E + a->identity > 2048) return GLQ_ERR_UNSUPPORTED;
    if (a->n == 0) return GLQ_OK;
    if (a->max_slots < glq_route_max_slots(a->n, a->E, a->top, a->chunk)) return GLQ_ERR_WORKSPACE;
    RtParams p{};
    p.logits = a->logits;
    p.correction = a->correction;
    p.ldl = a->ldl;
    p.n = a->n;
    p.E = a->E;
    p.A = a->E + a->identity;
    p.top = a->top;
    p.chunk = a->chunk;
    p.sel = a->sel;
    p.wts = a->wts;
    p.entry_scale = a->entry_scale;
    p.tok_entries = a->tok_entries;
    p.entry_row = a->entry_row;
    p.active = a->active;
    p.slot_count = a->slot_count;
    p.slot_offset = a->slot_offset;
    p.n_active = a->n_active;
    p.max_slots = a->max_slots;
    const int nk = a->n * a->top;
    const size_t sc = (size_t)16 * p.A * 4;
    if (nk <= kRouteOneCta && a->n <= 128) return dn_launch(dense_route_plan_kernel, dim3(1), 1024, sc + (size_t)2 * p.E * 4, stream, p);
    if (!a->block_counts) return GLQ_ERR_ARG;
    int st = dn_launch(dense_route_kernel, dim3(cdiv_i(a->n, 8)), 256, sc, stream, p);
    if (st != GLQ_OK) return st;
    // the list kernels are plain launches: they start when their predecessor is done
    cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
    const int nb = cdiv_i(nk, kPlanChunk), ms = p.max_slots;
    moe_plan_count_kernel<<<nb, 32, p.E * sizeof(int), s>>>(p.sel, nk, p.E, a->block_counts);
    moe_plan_lists_kernel<<<1, 1024, 2 * p.E * sizeof(int), s>>>(a->block_counts, nb, nk, p.E, p.chunk, 0, 1, p.active, p.n_active,
                                                                 p.slot_count, p.slot_offset, p.active + ms, p.n_active + 1,
                                                                 p.slot_count + ms, p.slot_offset + ms);
    moe_plan_scatter_kernel<float><<<nb, 32, p.E * sizeof(int), s>>>(p.sel, p.wts, nk, p.E, p.top, a->block_counts, p.entry_row,
                                                                     p.entry_scale, p.tok_entries);
    DN_CUDA(cudaGetLastError());
    return GLQ_OK;
}
