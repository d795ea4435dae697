// What the recurrent mixers share: the slices and chunks of their states, the rotation of queries and keys, and the
// per-head norm with output gate behind the recurrence.
#pragma once

#include "dense_common.cuh"

namespace glq {

constexpr int kSl = 32;            // value columns of a state slice
constexpr int kL = 64;             // positions of a chunk
constexpr int kSegment = 4096;     // positions the chunk forms take at a time (bounds their workspace)

__device__ __forceinline__ void ld4(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w;
}
__device__ __forceinline__ void ld4(const bf16* p, float (&v)[4]) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    v[0] = bf_lo(a.x), v[1] = bf_hi(a.x), v[2] = bf_lo(a.y), v[3] = bf_hi(a.y);
}
__device__ __forceinline__ void st4(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void st4(bf16* p, float a, float b, float c, float d) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf2(a, b), pack_bf2(c, d));
}

// element d of x (one head) turned: the first rot_dims elements pair up as (i, i + rot_dims / 2), or with `pairs` as
// (2i, 2i + 1); cs, sn: cosines and sines of the row's position
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int d, int rot_dims, int pairs, const float* cs, const float* sn) {
    const float v = to_f(x[d]);
    if (d >= rot_dims) return v;
    const int half = rot_dims >> 1;
    const bool second = pairs ? d & 1 : d >= half;
    const int i = pairs ? d >> 1 : (second ? d - half : d);
    const float o = to_f(x[pairs ? d ^ 1 : (second ? d - half : d + half)]);
    return second ? v * cs[i] + o * sn[i] : v * cs[i] - o * sn[i];
}

// one warp: out = rms_norm(o) * w * gate(g) for V <= 128 U values, four per lane and step, all requested before the sum
template <typename T, int U>
__device__ __forceinline__ void norm_gate_row(const float* __restrict__ o, const T* __restrict__ g, const float* __restrict__ w,
                                              int gate, T* __restrict__ out, int V, float eps, int lane) {
    float4 x[U];
    float gv[U][4], ss = 0.f;
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int v = (u * 32 + lane) * 4;
        x[u] = v < V ? *reinterpret_cast<const float4*>(o + v) : make_float4(0, 0, 0, 0);
        if (v < V) ld4(g + v, gv[u]);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) ss += x[u].x * x[u].x + x[u].y * x[u].y + x[u].z * x[u].z + x[u].w * x[u].w;
    const float inv = 1.f / sqrtf(warp_sum(ss) / V + eps);
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int v = (u * 32 + lane) * 4;
        if (v < V) {
            const float4 wv = w ? *reinterpret_cast<const float4*>(w + v) : make_float4(1.f, 1.f, 1.f, 1.f);
            st4(out + v, x[u].x * inv * wv.x * gate_f<T>(gate, gv[u][0]), x[u].y * inv * wv.y * gate_f<T>(gate, gv[u][1]),
                x[u].z * inv * wv.z * gate_f<T>(gate, gv[u][2]), x[u].w * inv * wv.w * gate_f<T>(gate, gv[u][3]));
        }
    }
}
// one warp, any size; vec4: all pointers allow accesses of four values.  w may be NULL
template <typename T>
__device__ __forceinline__ void norm_gate(const float* o, const T* g, const float* w, int gate, T* out, int V, float eps, bool vec4, int lane) {
    if (V % 4 == 0 && V <= 512 && vec4) return norm_gate_row<T, 4>(o, g, w, gate, out, V, eps, lane);
    float ss = 0.f;
    for (int v = lane; v < V; v += 32) {
        const float x = o[v];
        ss += x * x;
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / V + eps);
    for (int v = lane; v < V; v += 32) out[v] = from_f<T>(o[v] * inv * (w ? w[v] : 1.f) * gate_f<T>(gate, to_f(g[v])));
}

// 8x8 block of 16-bit values held row-wise across a warp -> column-wise
__device__ __forceinline__ uint32_t transpose8(uint32_t v) {
    uint32_t r;
    asm("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
    return r;
}

}  // namespace glq
