// Activation rows of the bf16-weight projections.
//
// A projection reads one or two segments per row; a segment is a slice of an fp32 buffer that may be RMS-normalised in
// groups (the slice is cut into `groups` equal consecutive parts, each divided by its own sqrt(mean(part²) + eps), the
// whole multiplied by `gamma`) and multiplied by sigmoid(gate), or added to a row of the residual stream (`base`).
// Everything here is fp32.  The second segment starts at
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
__device__ __forceinline__ float pair_f(float g, float u, float limit, int pair) { return pair == kPairSilu ? (g * sigmoid_f(g)) * u : gated_clamp_f(g, u, limit); }
__device__ __forceinline__ float softcap_f(float v, float cap) { return cap > 0.0f ? cap * tanhf(v / cap) : v; }

constexpr int kMaxNormGroups = 512;
struct RowScratch { float part[kMaxNormGroups + 32]; float scale[kMaxNormGroups]; };

// Stages one segment of row m with the whole block (blockDim.x a multiple of 32).  `at(k)` is the fp32 storage of column k;
// four columns from a multiple of four on are contiguous in it.  Ends with every element written, NOT with a barrier.
// The loads of a pass are issued in batches of four 16-byte pieces per thread: a block stages a row of thousands of
// values, and what it waits for is the round trip to L2.  `keep`: this block writes the sum of a row with a base.
template <typename Store>
__device__ __forceinline__ void stage_segment(const RowOperand& seg, int m, RowScratch& sc, Store at, bool keep = false) {
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, nw = nt >> 5;
    const float* x = seg.x + (size_t)m * seg.ldx;
    const float* gate = seg.gate ? seg.gate + (size_t)m * seg.ldg : nullptr;
    const float* base = seg.base ? seg.base + (size_t)m * seg.ldbase : nullptr;
    float* sum = keep && seg.sum ? seg.sum + (size_t)m * seg.ldsum : nullptr;
    const int len = seg.groups > 0 ? seg.k / seg.groups : seg.k;
    const bool vec = (((uintptr_t)x | (uintptr_t)gate | (uintptr_t)seg.gamma | (uintptr_t)base | (uintptr_t)sum) & 15) == 0 && ((seg.k | len) & 3) == 0;
    auto quad = [&](int k) -> float4& { return *reinterpret_cast<float4*>(&at(k)); };
    auto ld4 = [](const float* p) { return *reinterpret_cast<const float4*>(p); };
    auto gated = [](float4 v, float4 g) {
        return make_float4(v.x * sigmoid_f(g.x), v.y * sigmoid_f(g.y), v.z * sigmoid_f(g.z), v.w * sigmoid_f(g.w));
    };
    if (seg.groups == 0) {
        if (vec) {
            for (int k0 = tid * 4; k0 < seg.k; k0 += nt * 16) {
                float4 v[4], g[4];
#pragma unroll
                for (int u = 0; u < 4; u++) {
                    const int k = k0 + u * nt * 4;
                    if (k < seg.k) { v[u] = ld4(x + k); if (gate) g[u] = ld4(gate + k); }
                }
#pragma unroll
                for (int u = 0; u < 4; u++)
                    if (k0 + u * nt * 4 < seg.k) quad(k0 + u * nt * 4) = gate ? gated(v[u], g[u]) : v[u];
            }
        } else {
            for (int k = tid; k < seg.k; k += nt) {
                const float v = x[k];
                at(k) = gate ? v * sigmoid_f(gate[k]) : v;
            }
        }
        return;
    }
    const int parts = seg.groups >= nw ? 1 : (nw + seg.groups - 1) / seg.groups;      // warps that share a group
    for (int u = warp; u < seg.groups * parts; u += nw) {
        const int g = u / parts, q = u - g * parts;
        float ss = 0.0f;
        if (vec) {
            const int n4 = len / 4, lo = g * len + q * n4 / parts * 4, hi = g * len + (q + 1) * n4 / parts * 4;
            for (int k0 = lo + lane * 4; k0 < hi; k0 += 512) {
                float4 v[4];
#pragma unroll
                for (int j = 0; j < 4; j++)
                    if (k0 + j * 128 < hi) v[j] = ld4(x + k0 + j * 128);
#pragma unroll
                for (int j = 0; j < 4; j++)
                    if (k0 + j * 128 < hi) {
                        quad(k0 + j * 128) = v[j];
                        ss = fmaf(v[j].x, v[j].x, ss); ss = fmaf(v[j].y, v[j].y, ss); ss = fmaf(v[j].z, v[j].z, ss); ss = fmaf(v[j].w, v[j].w, ss);
                    }
            }
        } else {
            const int lo = g * len + (int)((long long)q * len / parts), hi = g * len + (int)((long long)(q + 1) * len / parts);
            for (int k = lo + lane; k < hi; k += 32) { const float v = x[k]; at(k) = v; ss = fmaf(v, v, ss); }
        }
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
    if (vec) {
        for (int k0 = tid * 4; k0 < seg.k; k0 += nt * 16) {
            float4 w[4], g[4];
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const int k = k0 + u * nt * 4;
                if (k < seg.k) { w[u] = ld4(seg.gamma + k); if (gate) g[u] = ld4(gate + k); else if (base) g[u] = ld4(base + k); }
            }
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const int k = k0 + u * nt * 4;
                if (k < seg.k) {
                    const float s = sc.scale[k / len];
                    float4 v = quad(k);
                    v = make_float4((v.x * s) * w[u].x, (v.y * s) * w[u].y, (v.z * s) * w[u].z, (v.w * s) * w[u].w);
                    if (base) {
                        v = make_float4(fmaf(seg.mult, v.x, g[u].x), fmaf(seg.mult, v.y, g[u].y), fmaf(seg.mult, v.z, g[u].z), fmaf(seg.mult, v.w, g[u].w));
                        if (sum) *reinterpret_cast<float4*>(sum + k) = v;
                    }
                    quad(k) = gate ? gated(v, g[u]) : v;
                }
            }
        }
    } else {
        for (int k = tid; k < seg.k; k += nt) {
            float v = (at(k) * sc.scale[k / len]) * seg.gamma[k];
            if (gate) v *= sigmoid_f(gate[k]);
            if (base) {
                v = fmaf(seg.mult, v, base[k]);
                if (sum) sum[k] = v;
            }
            at(k) = v;
        }
    }
}

__host__ __device__ __forceinline__ int pad8(int k) { return (k + 7) & ~7; }

}  // namespace dj
