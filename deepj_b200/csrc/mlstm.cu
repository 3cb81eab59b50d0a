// Matrix-memory recurrence with exponential gates and a running maximum, per head:
//     i = cap·tanh(iraw/cap)      f = logsigmoid(cap·tanh(fraw/cap))      m_t = max(f + m_{t-1}, i)
//     S_t = e^{f + m_{t-1} − m_t} S_{t-1} + e^{i − m_t} k vᵀ              n_t likewise with k alone
//     o_t = S_tᵀ q / (max(|n_t·q|, e^{−m_t}) + 1e-6),                     q scaled by `qscale`
// State, normaliser and maximum are fp32 and live in HBM between calls; a sequence at position 0 starts from zeros whatever the
// buffers hold.  S is kept as [sequence][head][value column][key channel]; (n, m) twice, by parity of the position, because
// every block of a step reads them and one writes them.
//
//   k_mlstm_step     one token: a block per (32 value columns, head, sequence), a warp per four columns, key channels over the
//                    lanes; the state is fetched before the dependency wait
//   k_mlstm_gates    several tokens, in blocks of 32 (or 64): with b_t the sum of f within a block and a_s = i_s − b_s, the weight of
//                    token s in the output of token t is e^{(b_t − m_t) + a_s}, that of the state before the block
//                    e^{b_t + m_0 − m_t}.  The sums are formed in double and handed on as two floats: they reach hundreds where
//                    their differences matter to the last bit.
//   k_mlstm_chunk    a block per (kCols value columns, head, sequence) walks the token blocks: outputs from the state before the
//                    block and from the products within it, then the state after it.  fp32 FMA throughout.
// The tensor-core form of the walk is in mlstm_mma.cu.
#include "mlstm.cuh"
#include "row_operand.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr int kTok = kMlTok, kCols = 32, kMaxDim = 512;

__device__ __forceinline__ float warp_sum(float v) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// NE: key channels per lane
template <int NE>
__global__ void __launch_bounds__(256) k_mlstm_step(const MlstmArgs a) {
    __shared__ float qs[32 * NE], ks[32 * NE], red[8];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, b = blockIdx.z;
    if (!a.early) { pdl_wait(); pdl_launch_dependents(); }
    const int pos = (int)a.pos[b], c0 = blockIdx.x * 32 + warp * 4;
    const bool fresh = pos == 0;
    float* st = a.state + (((size_t)b * a.H + h) * a.vdim + c0) * a.dim;
    const size_t slot = (size_t)a.B * a.H * (a.dim + 1), bh = (size_t)b * a.H + h;
    const float* nOld = a.norm + (size_t)(pos & 1) * slot + bh * (a.dim + 1);
    float* nNew = a.norm + (size_t)((pos + 1) & 1) * slot + bh * (a.dim + 1);
    float S[4][NE];
#pragma unroll
    for (int c = 0; c < 4; c++)
#pragma unroll
        for (int e = 0; e < NE; e++) {
            const int i = e * 32 + lane;
            S[c][e] = !fresh && c0 + c < a.vdim && i < a.dim ? st[(size_t)c * a.dim + i] : 0.0f;
        }
    const float m0 = fresh ? 0.0f : nOld[a.dim];
    if (a.early) { pdl_wait(); pdl_launch_dependents(); }
    const float* x = a.proj + (size_t)b * a.ld;
    const float iv = gate_cap_f(x[a.i_off + h], a.cap), fv = log_sigmoid_f(gate_cap_f(x[a.f_off + h], a.cap));
    const float m = fmaxf(fv + m0, iv), keep = expf(fv + m0 - m), add = expf(iv - m);
    float nq = 0.0f;
    for (int i = tid; i < 32 * NE; i += 256) {
        const float q = i < a.dim ? x[a.q_off + h * a.dim + i] * a.qscale : 0.0f, k = i < a.dim ? x[a.k_off + h * a.dim + i] : 0.0f;
        qs[i] = q; ks[i] = k;
        if (i < a.dim) {
            const float n = fmaf(keep, fresh ? 0.0f : nOld[i], add * k);
            nq = fmaf(n, q, nq);
            if (blockIdx.x == 0) nNew[i] = n;
        }
    }
    if (blockIdx.x == 0 && tid == 0) nNew[a.dim] = m;
    nq = warp_sum(nq);
    if (lane == 0) red[warp] = nq;
    __syncthreads();
    nq = ((red[0] + red[1]) + (red[2] + red[3])) + ((red[4] + red[5]) + (red[6] + red[7]));
    const float inv = 1.0f / (fmaxf(fabsf(nq), expf(-m)) + kMlDenEps);
    float o[4];
#pragma unroll
    for (int c = 0; c < 4; c++) {
        const float v = c0 + c < a.vdim ? x[a.v_off + h * a.vdim + c0 + c] * add : 0.0f;
        o[c] = 0.0f;
#pragma unroll
        for (int e = 0; e < NE; e++) {
            const int i = e * 32 + lane;
            S[c][e] = fmaf(keep, S[c][e], v * ks[i]);
            o[c] = fmaf(S[c][e], qs[i], o[c]);
            if (c0 + c < a.vdim && i < a.dim) st[(size_t)c * a.dim + i] = S[c][e];
        }
    }
#pragma unroll
    for (int c = 0; c < 4; c++) {
        const float v = warp_sum(o[c]);
        if (lane == 0 && c0 + c < a.vdim) a.out[(size_t)b * a.ldo + h * a.vdim + c0 + c] = v * inv;
    }
}

__global__ void __launch_bounds__(256) k_mlstm_gates(const MlstmArgs a) {
    extern __shared__ double blk[];
    pdl_wait();
    pdl_launch_dependents();
    ml_gate_block<1>(a, blockIdx.x, blockIdx.y, blk);
}

size_t chunk_smem(int dim) {
    const int P = ((dim + 3) & ~3) + 4;
    return ((size_t)2 * kTok * P + (size_t)(kCols + 1) * P + 2 * (size_t)kTok * (kCols + 4) + (size_t)kTok * (kTok + 1) + 8 * kTok) * 4;
}

// 2 × 2 products of rows (x0, x1) and (y0, y1) over P4 float4s
__device__ __forceinline__ void tile_dot(const float* x0, const float* x1, const float* y0, const float* y1, int P4, float (&d)[4]) {
    d[0] = d[1] = d[2] = d[3] = 0.0f;
#pragma unroll 4
    for (int i = 0; i < P4; i++) {
        const float4 a = reinterpret_cast<const float4*>(x0)[i], b = reinterpret_cast<const float4*>(x1)[i];
        const float4 c = reinterpret_cast<const float4*>(y0)[i], e = reinterpret_cast<const float4*>(y1)[i];
        d[0] = fmaf(a.x, c.x, d[0]); d[1] = fmaf(a.x, e.x, d[1]); d[2] = fmaf(b.x, c.x, d[2]); d[3] = fmaf(b.x, e.x, d[3]);
        d[0] = fmaf(a.y, c.y, d[0]); d[1] = fmaf(a.y, e.y, d[1]); d[2] = fmaf(b.y, c.y, d[2]); d[3] = fmaf(b.y, e.y, d[3]);
        d[0] = fmaf(a.z, c.z, d[0]); d[1] = fmaf(a.z, e.z, d[1]); d[2] = fmaf(b.z, c.z, d[2]); d[3] = fmaf(b.z, e.z, d[3]);
        d[0] = fmaf(a.w, c.w, d[0]); d[1] = fmaf(a.w, e.w, d[1]); d[2] = fmaf(b.w, c.w, d[2]); d[3] = fmaf(b.w, e.w, d[3]);
    }
}

__global__ void __launch_bounds__(256) k_mlstm_chunk(const MlstmArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int dim = a.dim, Dp = (dim + 3) & ~3, P = Dp + 4, P4 = Dp / 4, VP = kCols + 4;
    float* Q = sm;                       // [kTok][P]
    float* K = Q + kTok * P;             // [kTok][P]
    float* S = K + kTok * P;             // [kCols][P]: the state, a row per value column; row kCols: the normaliser
    float* V = S + (kCols + 1) * P;      // [kTok][VP]
    float* W = V + kTok * VP;            // [kTok][VP]: values times their weight in the state after the block
    float* X = W + kTok * VP;            // [kTok][kTok + 1]: weighted products q·k
    float* den = X + kTok * (kTok + 1);  // [kTok] 1 / denominator
    float* gt = den + kTok;              // [7][kTok] gates of the block's tokens
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * kCols, nc = min(kCols, a.vdim - c0);
    const size_t bh = (size_t)b * a.H + h;
    pdl_wait();
    pdl_launch_dependents();
    const int pos = (int)a.pos[b];
    const MlGates g = ml_gates(a.ws, a.B, a.T, a.H, dim, kTok, bh);
    float* st = a.state + (bh * a.vdim + c0) * dim;
    for (int i = tid; i < (kCols + 1) * P; i += 256) {
        const int c = i / P, d = i - c * P;
        S[i] = d < dim ? (c == kCols ? g.n0[d] : pos != 0 && c < nc ? st[(size_t)c * dim + d] : 0.0f) : 0.0f;
    }
    const int tx = tid & 15, ty = tid >> 4, nb = ml_blocks(a.T, kTok);
    for (int j = 0; j < nb; j++) {
        const int t0 = j * kTok, n = min(kTok, a.T - t0);
        __syncthreads();
        for (int i = tid; i < kTok * P; i += 256) {
            const int t = i / P, d = i - t * P;
            const float* x = a.proj + ((size_t)b * a.T + t0 + t) * a.ld + (size_t)h * dim + d;
            const bool on = t < n && d < dim;
            Q[i] = on ? x[a.q_off] * a.qscale : 0.0f;
            K[i] = on ? x[a.k_off] : 0.0f;
        }
        for (int i = tid; i < 7 * kTok; i += 256) {
            const int f = i / kTok, t = i - f * kTok;
            gt[i] = t < n ? g.rowHi[(size_t)f * a.B * a.H * a.T + t0 + t] : f == 0 ? -INFINITY : 0.0f;
        }
        for (int i = tid; i < kTok * kCols; i += 256) {
            const int t = i / kCols, c = i - t * kCols;
            const float v = t < n && c < nc ? a.proj[((size_t)b * a.T + t0 + t) * a.ld + a.v_off + (size_t)h * a.vdim + c0 + c] : 0.0f;
            V[t * VP + c] = v;
            W[t * VP + c] = t < n ? v * g.add[t0 + t] : 0.0f;
        }
        __syncthreads();
        float d[4], o[4];
        tile_dot(Q + ty * P, Q + (ty + 16) * P, K + tx * P, K + (tx + 16) * P, P4, d);
        tile_dot(Q + ty * P, Q + (ty + 16) * P, S + tx * P, S + (tx + 16) * P, P4, o);
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int t = ty + (e >> 1) * 16, s = tx + (e & 1) * 16;
            X[t * (kTok + 1) + s] = s <= t ? d[e] * expf((gt[t] + gt[2 * kTok + s]) + (gt[kTok + t] + gt[3 * kTok + s])) : 0.0f;
            o[e] *= gt[4 * kTok + t];
        }
        __syncthreads();
        for (int t = warp; t < kTok; t += 8) {               // n_t·q_t
            float v = 0.0f;
            for (int i = lane; i < dim; i += 32) v = fmaf(S[kCols * P + i], Q[t * P + i], v);
            v = warp_sum(fmaf(v, gt[4 * kTok + t], X[t * (kTok + 1) + lane]));
            if (lane == 0) den[t] = 1.0f / (fmaxf(fabsf(v), gt[5 * kTok + t]) + kMlDenEps);
        }
#pragma unroll 4
        for (int s = 0; s < kTok; s++) {
            const float x0 = X[ty * (kTok + 1) + s], x1 = X[(ty + 16) * (kTok + 1) + s], v0 = V[s * VP + tx], v1 = V[s * VP + tx + 16];
            o[0] = fmaf(x0, v0, o[0]); o[1] = fmaf(x0, v1, o[1]); o[2] = fmaf(x1, v0, o[2]); o[3] = fmaf(x1, v1, o[3]);
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int t = ty + (e >> 1) * 16, c = tx + (e & 1) * 16;
            if (t < n && c < nc) a.out[((size_t)b * a.T + t0 + t) * a.ldo + (size_t)h * a.vdim + c0 + c] = o[e] * den[t];
        }
        const float keep = g.keep[j];
        for (int u = tid; u < kCols / 4 * P4; u += 256) {    // a thread: four columns, four channels
            const int i = u % P4 * 4, c = u / P4 * 4;
            float4 r[4];
#pragma unroll
            for (int q = 0; q < 4; q++) {
                r[q] = *reinterpret_cast<const float4*>(S + (c + q) * P + i);
                r[q].x *= keep; r[q].y *= keep; r[q].z *= keep; r[q].w *= keep;
            }
#pragma unroll 4
            for (int s = 0; s < kTok; s++) {
                const float4 k = *reinterpret_cast<const float4*>(K + s * P + i), w = *reinterpret_cast<const float4*>(W + s * VP + c);
                const float ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
                for (int q = 0; q < 4; q++) {
                    r[q].x = fmaf(ww[q], k.x, r[q].x); r[q].y = fmaf(ww[q], k.y, r[q].y);
                    r[q].z = fmaf(ww[q], k.z, r[q].z); r[q].w = fmaf(ww[q], k.w, r[q].w);
                }
            }
#pragma unroll
            for (int q = 0; q < 4; q++) *reinterpret_cast<float4*>(S + (c + q) * P + i) = r[q];
        }
        for (int i = tid; i < dim; i += 256) {
            float v = S[kCols * P + i] * keep;
            for (int s = 0; s < kTok; s++) v = fmaf(gt[6 * kTok + s], K[s * P + i], v);
            S[kCols * P + i] = v;
        }
    }
    __syncthreads();
    for (int i = tid; i < nc * dim; i += 256) st[i] = S[i / dim * P + i % dim];
    if (blockIdx.x == 0) {
        float* nNew = a.norm + (size_t)((pos + a.T) & 1) * a.B * a.H * (dim + 1) + bh * (dim + 1);
        for (int i = tid; i < dim; i += 256) nNew[i] = S[kCols * P + i];
    }
}

}  // namespace

const char* mlstm_check(const MlstmArgs& a) {
    if (a.dim > kMaxDim) return "key size not supported";
    if (ml_blocks(a.T, kTok) > 1900) return "too many tokens";
    return nullptr;
}
size_t mlstm_ws_floats(const MlstmArgs& a) {
    if (a.T == 1) return 0;
    return mlstm_mma_fits(a) ? mlstm_mma_ws_floats(a) : ml_gate_floats(a.B, a.T, a.H, a.dim, kTok);
}

void launch_mlstm(const MlstmArgs& a, cudaStream_t s) {
    if (a.T == 1) {
        const dim3 grid((unsigned)((a.vdim + 31) / 32), (unsigned)a.H, (unsigned)a.B);
        if (a.dim <= 64) launch_k(k_mlstm_step<2>, grid, dim3(256), 0, s, true, a);
        else if (a.dim <= 128) launch_k(k_mlstm_step<4>, grid, dim3(256), 0, s, true, a);
        else if (a.dim <= 256) launch_k(k_mlstm_step<8>, grid, dim3(256), 0, s, true, a);
        else launch_k(k_mlstm_step<16>, grid, dim3(256), 0, s, true, a);
        return;
    }
    if (mlstm_mma_fits(a)) { launch_mlstm_mma(a, s); return; }
    static bool attr = false;
    if (!attr) {
        DJ_CUDA_CHECK(cudaFuncSetAttribute(k_mlstm_chunk, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 64));
        attr = true;
    }
    launch_k(k_mlstm_gates, dim3((unsigned)a.H, (unsigned)a.B), dim3(256), (size_t)ml_blocks(a.T, kTok) * 24, s, true, a);
    launch_k(k_mlstm_chunk, dim3((unsigned)((a.vdim + kCols - 1) / kCols), (unsigned)a.H, (unsigned)a.B), dim3(256), chunk_smem(a.dim), s, true, a);
}

}  // namespace dj
