// Entry lists of a mixture-of-experts call on the device, shared by the quantized and the dense experts: entries
// (token, slot) sorted by expert in token order, and the compacted list of live experts ("slots").  WT is the type
// of the routing weights.
#pragma once

#include "glq_common.cuh"

namespace glq {

// Warp 0 of a CTA: exclusive prefix of the per-expert counts in sm_cnt (entry offsets are global: every rank
// numbers the entries alike) into sm_off, and the compacted lists of the live experts this rank holds.
__device__ __forceinline__ void plan_lists(int lane, const int* sm_cnt, int* sm_off, int E, int nk, int chunk, int ep_rank,
                                           int ep_world, int* __restrict__ active, int* __restrict__ n_active,
                                           int* __restrict__ slot_count, int* __restrict__ slot_offset,
                                           int* __restrict__ active2, int* __restrict__ n_active2,
                                           int* __restrict__ slot_count2, int* __restrict__ slot_offset2) {
    int base = 0, j = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
        const int e = e0 + lane;
        const int c = e < E ? sm_cnt[e] : 0;
        int v = c;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int tv = __shfl_up_sync(0xffffffffu, v, o);
            if (lane >= o) v += tv;
        }
        const int off = base + v - c;
        if (e < E) sm_off[e] = off;
        const bool act = e < E && c > 0 && e % ep_world == ep_rank;
        // slots of this expert: one, or ceil(c / chunk) of at most `chunk` consecutive entries each
        const int ns = act ? (chunk > 0 ? (c + chunk - 1) / chunk : 1) : 0;
        int sv = ns;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int tv = __shfl_up_sync(0xffffffffu, sv, o);
            if (lane >= o) sv += tv;
        }
        for (int i = 0; i < ns; ++i) {
            const int pos = j + sv - ns + i;
            const int cc = chunk > 0 ? min(chunk, c - i * chunk) : c;
            const int oo = off + (chunk > 0 ? i * chunk : 0);
            active[pos] = e;
            slot_count[pos] = cc;
            slot_offset[pos] = oo;
            // the same lists twice, for gate (table entry e, entries 0..nk) and up (entry E+e, entries nk..2nk)
            active2[pos] = e;
            slot_count2[pos] = cc;
            slot_offset2[pos] = oo;
        }
        j += __shfl_sync(0xffffffffu, sv, 31);
        base += __shfl_sync(0xffffffffu, v, 31);
    }
    __syncwarp();
    for (int i = lane; i < j; i += 32) {
        active2[j + i] = E + active[i];
        slot_count2[j + i] = slot_count[i];
        slot_offset2[j + i] = nk + slot_offset[i];
    }
    if (lane == 0) {
        *n_active = j;
        *n_active2 = 2 * j;
    }
}

// Phase B of the one-CTA plan, called by all warps of a CTA after sel / wts of all tokens are written and the CTA
// has synchronised: per-expert counts, lists, and each expert's entries in token order (ballot scans: deterministic).
// sm_cnt: 2 * E ints of shared memory.  A selection outside [0, E) has no entry.
template <typename WT>
__device__ __forceinline__ void plan_entries(int* sm_cnt, int n, int E, int k, int chunk, int ep_rank, int ep_world,
                                             const int* __restrict__ sel, const WT* __restrict__ wts, int* __restrict__ active,
                                             int* __restrict__ n_active, int* __restrict__ slot_count,
                                             int* __restrict__ slot_offset, int* __restrict__ entry_row,
                                             WT* __restrict__ entry_scale, int* __restrict__ tok_entries,
                                             int* __restrict__ active2, int* __restrict__ n_active2,
                                             int* __restrict__ slot_count2, int* __restrict__ slot_offset2) {
    int* sm_off = sm_cnt + E;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    const int nk = n * k;
    const unsigned lt = (1u << lane) - 1u;
    // Phase B1: entries per expert, one warp per expert (ballot counts: no atomics, any order gives the same sum)
    for (int e = warp; e < E; e += nwarps) {
        int c = 0;
        for (int i0 = 0; i0 < nk; i0 += 32) {
            const int i = i0 + lane;
            c += __popc(__ballot_sync(0xffffffffu, i < nk && sel[i] == e));
        }
        if (lane == 0) sm_cnt[e] = c;
    }
    __syncthreads();
    // Phase B2, warp 0: exclusive prefix of the counts (entry offsets are global: every rank numbers the
    // entries alike) and the compacted list of live experts this rank holds (e mod world == rank)
    if (warp == 0)
        plan_lists(lane, sm_cnt, sm_off, E, nk, chunk, ep_rank, ep_world, active, n_active, slot_count, slot_offset, active2,
                   n_active2, slot_count2, slot_offset2);
    __syncthreads();
    // Phase B3: each expert's entries in token order, one warp per expert
    for (int e = warp; e < E; e += nwarps) {
        if (sm_cnt[e] == 0) continue;
        int pos = sm_off[e];
        for (int i0 = 0; i0 < nk; i0 += 32) {
            const int i = i0 + lane;
            const bool hit = i < nk && sel[i] == e;
            const unsigned m = __ballot_sync(0xffffffffu, hit);
            if (hit) {
                const int q = pos + __popc(m & lt);
                entry_row[q] = i / k;
                entry_row[nk + q] = i / k;
                entry_scale[q] = wts[i];
                tok_entries[i] = q;
            }
            pos += __popc(m);
        }
    }
}

constexpr int kPlanChunk = 512;
constexpr long long kPlanParallelFrom = 2048;   // entries (tokens x top-k) from which the plan runs as four launches

// one warp per block: blk[b][e] = entries of expert e among the block's kPlanChunk entries
static __global__ void __launch_bounds__(32) moe_plan_count_kernel(const int* __restrict__ sel, int nk, int E, int* __restrict__ blk) {
    extern __shared__ int sm_c[];
    const int lane = threadIdx.x, b = blockIdx.x;
    for (int e = lane; e < E; e += 32) sm_c[e] = 0;
    __syncwarp();
    const int i_end = min(nk, (b + 1) * kPlanChunk);
    for (int i0 = b * kPlanChunk; i0 < i_end; i0 += 32) {
        const int i = i0 + lane;
        const int e = i < i_end ? sel[i] : -1;
        const bool valid = e >= 0 && e < E;
        const unsigned m = __match_any_sync(0xffffffffu, valid ? e : E + lane);
        if (valid && lane == __ffs(m) - 1) sm_c[e] += __popc(m);
        __syncwarp();
    }
    for (int e = lane; e < E; e += 32) blk[(size_t)b * E + e] = sm_c[e];
}

static __global__ void __launch_bounds__(1024) moe_plan_lists_kernel(int* __restrict__ blk, int nb, int nk, int E, int chunk, int ep_rank,
                                                              int ep_world, int* __restrict__ active, int* __restrict__ n_active,
                                                              int* __restrict__ slot_count, int* __restrict__ slot_offset,
                                                              int* __restrict__ active2, int* __restrict__ n_active2,
                                                              int* __restrict__ slot_count2, int* __restrict__ slot_offset2) {
    extern __shared__ int sm_cnt[];  // [E] counts, then [E] offsets
    int* sm_off = sm_cnt + E;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int e = threadIdx.x; e < E; e += blockDim.x) {
        int c = 0;
        for (int b = 0; b < nb; ++b) c += blk[(size_t)b * E + e];
        sm_cnt[e] = c;
    }
    __syncthreads();
    if (warp == 0)
        plan_lists(lane, sm_cnt, sm_off, E, nk, chunk, ep_rank, ep_world, active, n_active, slot_count, slot_offset, active2,
                   n_active2, slot_count2, slot_offset2);
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += blockDim.x) {   // counts -> first entry number of (block, expert)
        int run = sm_off[e];
        for (int b = 0; b < nb; ++b) {
            const int c = blk[(size_t)b * E + e];
            blk[(size_t)b * E + e] = run;
            run += c;
        }
    }
}

template <typename WT>
__global__ void __launch_bounds__(32) moe_plan_scatter_kernel(const int* __restrict__ sel, const WT* __restrict__ wts, int nk,
                                                              int E, int k, const int* __restrict__ blk,
                                                              int* __restrict__ entry_row, WT* __restrict__ entry_scale,
                                                              int* __restrict__ tok_entries) {
    extern __shared__ int sm_b[];
    const int lane = threadIdx.x, b = blockIdx.x;
    const unsigned lt = (1u << lane) - 1u;
    for (int e = lane; e < E; e += 32) sm_b[e] = blk[(size_t)b * E + e];
    __syncwarp();
    const int i_end = min(nk, (b + 1) * kPlanChunk);
    for (int i0 = b * kPlanChunk; i0 < i_end; i0 += 32) {
        const int i = i0 + lane;
        const int e = i < i_end ? sel[i] : -1;
        const bool valid = e >= 0 && e < E;
        const unsigned m = __match_any_sync(0xffffffffu, valid ? e : E + lane);
        if (valid) {
            const int q = sm_b[e] + __popc(m & lt);
            entry_row[q] = i / k;
            entry_row[nk + q] = i / k;
            entry_scale[q] = wts[i];
            tok_entries[i] = q;
        }
        __syncwarp();
        if (valid && lane == __ffs(m) - 1) sm_b[e] += __popc(m);
        __syncwarp();
    }
}

}  // namespace glq
