// Activation rows of the bf16-weight projections.
//
// A projection reads one or two segments per row; a segment is a slice of an fp32 buffer that may be RMS-normalised in
// groups (the slice is cut into `groups` equal consecutive parts, each divided by its own sqrt(mean(part²) + eps), the
// whole multiplied by `gamma`) and multiplied by sigmoid(gate).  Everything here is fp32.  The second segment starts at
// the next multiple of eight columns of the weight; the columns between hold zeros on both sides.
#pragma once
#include <cuda_bf16.h>

#include "kernels.h"
#include "q8_common.cuh"

namespace dj {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
// min(g, limit)·sigmoid(1.702·min(g, limit))·(clamp(u, ±limit) + 1)
__device__ __forceinline__ float gated_clamp_f(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return (g * sigmoid_f(1.702f * g)) * (u + 1.0f);
}
__device__ __forceinline__ float softcap_f(float v, float cap) { return cap > 0.0f ? cap * tanhf(v / cap) : v; }

constexpr int kMaxNormGroups = 512;
struct RowScratch { float part[kMaxNormGroups + 32]; float scale[kMaxNormGroups]; };

// Stages one segment of row m with the whole block (blockDim.x a multiple of 32): put(k, v) receives every element
// k < seg.k after norm and gate; raw(k) / get(k) address the same storage between the passes.  `Store` needs
// operator()(int k) → float& (fp32 storage).  Ends with every element written, NOT with a barrier.
template <typename Store>
__device__ __forceinline__ void stage_segment(const RowOperand& seg, int m, RowScratch& sc, Store at) {
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, nw = nt >> 5;
    const float* x = seg.x + (size_t)m * seg.ldx;
    const float* gate = seg.gate ? seg.gate + (size_t)m * seg.ldg : nullptr;
    if (seg.groups == 0) {
        for (int k = tid; k < seg.k; k += nt) {
            const float v = x[k];
            at(k) = gate ? v * sigmoid_f(gate[k]) : v;
        }
        return;
    }
    const int len = seg.k / seg.groups;
    const int parts = seg.groups >= nw ? 1 : (nw + seg.groups - 1) / seg.groups;      // warps that share a group
    for (int u = warp; u < seg.groups * parts; u += nw) {
        const int g = u / parts, q = u - g * parts;
        const int lo = g * len + (int)((long long)q * len / parts), hi = g * len + (int)((long long)(q + 1) * len / parts);
        float ss = 0.0f;
        for (int k = lo + lane; k < hi; k += 32) { const float v = x[k]; at(k) = v; ss = fmaf(v, v, ss); }
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (lane == 0) sc.part[u] = ss;
    }
    __syncthreads();
    for (int g = tid; g < seg.groups; g += nt) {
        float ss = 0.0f;
        for (int q = 0; q < parts; q++) ss += sc.part[g * parts + q];
        sc.scale[g] = 1.0f / sqrtf(ss / (float)len + seg.eps);
    }
    __syncthreads();
    for (int k = tid; k < seg.k; k += nt) {
        float v = (at(k) * sc.scale[k / len]) * seg.gamma[k];
        if (gate) v *= sigmoid_f(gate[k]);
        at(k) = v;
    }
}

__host__ __device__ __forceinline__ int pad8(int k) { return (k + 7) & ~7; }

}  // namespace dj
