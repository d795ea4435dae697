// Helpers of the unquantized kernels: storage types, 16-byte vectors of bfloat16, the bf16 tensor-core op.
#pragma once

#include <cuda_bf16.h>

#include <cstdlib>

#include "../../include/glorcq_b200_dense.h"
#include "tc_mm.cuh"

namespace glq {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ uint32_t pack_bf2(float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float bf_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float bf_hi(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }
// two floats as the sum of two bf16 pairs: the second holds what the first's rounding lost
__device__ __forceinline__ void split_bf2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf2(a, b);
    lo = pack_bf2(a - bf_lo(hi), b - bf_hi(hi));
}

// D(16x8, f32) += A(16x16, bf16, row) * B(16x8, bf16, col); fragment ownership as mma16816
__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
                 : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
                 : "r"(addr));
}
// 16 bytes global -> shared; not live: zeros, nothing is read
__device__ __forceinline__ void cpa16(uint32_t dst, const void* src, bool live) {
    const int bytes = live ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cpa_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cpa_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_release() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }

// the same to a few units in the last place, for results that are stored as bf16
__device__ __forceinline__ float sigmoid_fast_f(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
template <typename T> __device__ __forceinline__ float sigmoid_t(float v) { return sizeof(T) == 2 ? sigmoid_fast_f(v) : sigmoid_f(v); }
template <typename T> __device__ __forceinline__ float gate_f(int gate, float v) {
    const float s = sigmoid_t<T>(v);
    return gate == GLQ_GATE_SILU ? v * s : s;
}

template <int ACT> __device__ __forceinline__ float act_f(float z) {
    if (ACT == GLQ_ACT_RELU2) {
        const float r = fmaxf(z, 0.f);
        return r * r;
    }
    if (ACT == GLQ_ACT_GELU_ERF) return 0.5f * z * (1.f + erff(z * 0.70710678118654752f));
    if (ACT == GLQ_ACT_GELU_TANH) return 0.5f * z * (1.f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
    return z;
}
__device__ __forceinline__ float act_dyn(int act, float z) {
    if (act == GLQ_ACT_RELU2) return act_f<GLQ_ACT_RELU2>(z);
    if (act == GLQ_ACT_GELU_ERF) return act_f<GLQ_ACT_GELU_ERF>(z);
    if (act == GLQ_ACT_GELU_TANH) return act_f<GLQ_ACT_GELU_TANH>(z);
    return z;
}

// block-wide sum, every thread gets it; red: 32 floats of shared memory
__device__ __forceinline__ float block_sum(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float s = lane < nw ? red[lane] : 0.f;
    return warp_sum(s);
}

// ---- host side ---------------------------------------------------------------------------------------
extern thread_local int g_dense_cuda_error;
inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }
inline int cdiv_i(long a, long b) { return (int)((a + b - 1) / b); }
#define DN_CUDA(call)                          \
    do {                                       \
        const cudaError_t e_ = (call);         \
        if (e_ != cudaSuccess) {               \
            g_dense_cuda_error = (int)e_;      \
            return GLQ_ERR_CUDA;               \
        }                                      \
    } while (0)

inline int dn_sms() {
    static int sms[64] = {0};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 148;
    if (sms[dev] == 0) {
        int v = 0;
        if (cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || v <= 0) v = 148;
        sms[dev] = v;
    }
    return sms[dev];
}

// Launch that may start while its predecessor drains: every kernel here calls pdl_wait() before it touches anything a
// predecessor wrote.
// (early = false: an ordinary launch, for a kernel whose waiting CTAs would only take room from its predecessor)
// cluster: CTAs along x that form a cluster (1: none)
template <typename... KArgs, typename... Args>
inline int dn_launch_as(bool early, int cluster, void (*kern)(KArgs...), dim3 grid, int block, size_t smem, void* stream, Args... args) {
    static const bool pdl = std::getenv("GLQ_NO_PDL") == nullptr;
    // 48 KB without opting in is dynamic plus static shared memory; no kernel here has more than 24 KB of the latter
    if (smem > 24 * 1024) DN_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(block);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = reinterpret_cast<cudaStream_t>(stream);
    cudaLaunchAttribute attr[2]{};
    int n = 0;
    if (pdl && early) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (cluster > 1) {
        if (cluster > 8) DN_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = (unsigned)cluster;
        attr[n].val.clusterDim.y = attr[n].val.clusterDim.z = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    DN_CUDA(cudaLaunchKernelEx(&cfg, kern, KArgs(args)...));
    return GLQ_OK;
}
template <typename... KArgs, typename... Args>
inline int dn_launch_if(bool early, void (*kern)(KArgs...), dim3 grid, int block, size_t smem, void* stream, Args... args) {
    return dn_launch_as(early, 1, kern, grid, block, smem, stream, args...);
}
template <typename... KArgs, typename... Args>
inline int dn_launch_cluster(int cluster, void (*kern)(KArgs...), dim3 grid, int block, size_t smem, void* stream, Args... args) {
    return dn_launch_as(true, cluster, kern, grid, block, smem, stream, args...);
}
template <typename... KArgs, typename... Args>
inline int dn_launch(void (*kern)(KArgs...), dim3 grid, int block, size_t smem, void* stream, Args... args) {
    return dn_launch_if(true, kern, grid, block, smem, stream, args...);
}

}  // namespace glq
