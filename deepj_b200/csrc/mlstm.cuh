// What the gate kernel of the matrix-memory recurrence (mlstm.cu) hands to the kernels that walk the token blocks.
#pragma once
#include "kernels.h"

namespace dj {

constexpr int kMlTok = 32, kMlTokMma = 64;         // tokens per block: FMA form, tensor-core form
constexpr float kMlDenEps = 1e-6f;

__host__ __device__ __forceinline__ int ml_blocks(int T, int tok) { return (T + tok - 1) / tok; }

// Per (sequence, head): arrays of T floats, then one value per token block, then the normaliser.
struct MlGates {
    float* rowHi; float* rowLo;      // b_t − m_t
    float* colHi; float* colLo;      // a_s
    float* carry;                    // e^{b_t + m_0 − m_t}: the state before the block, seen by token t
    float* floor_;                   // e^{−m_t}
    float* add;                      // e^{b_L + a_s − m_L}: token s in the state after the block
    float* keep;                     // [token blocks] e^{b_L + m_0 − m_L}
    float* n0;                       // [dim] normaliser before the call
};
__host__ __device__ __forceinline__ size_t ml_gate_floats(int B, int T, int H, int dim, int tok) {
    return ((size_t)B * H * (7 * (size_t)T + ml_blocks(T, tok) + dim) + 3) & ~(size_t)3;
}
__host__ __device__ __forceinline__ MlGates ml_gates(float* ws, int B, int T, int H, int dim, int tok, size_t bh) {
    const size_t n = (size_t)B * H * T;
    MlGates g;
    float* p = ws + bh * T;
    g.rowHi = p; g.rowLo = p + n; g.colHi = p + 2 * n; g.colLo = p + 3 * n; g.carry = p + 4 * n; g.floor_ = p + 5 * n; g.add = p + 6 * n;
    g.keep = ws + 7 * n + bh * ml_blocks(T, tok);
    g.n0 = ws + 7 * n + (size_t)B * H * ml_blocks(T, tok) + bh * dim;
    return g;
}

__device__ __forceinline__ float gate_cap_f(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }

// The gates of one head of one sequence, by a block of 256 threads: a warp per token block, TPL consecutive tokens per lane.
// blk [3][token blocks] (shared): per token block its sum of f, its largest a_s, and the maximum before it.
template <int TPL>
__device__ __forceinline__ void ml_gate_block(const MlstmArgs& a, int h, int b, double* blk) {
    constexpr int TOK = 32 * TPL;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nb = ml_blocks(a.T, TOK), pos = (int)a.pos[b];
    const size_t bh = (size_t)b * a.H + h, slot = (size_t)a.B * a.H * (a.dim + 1);
    const MlGates g = ml_gates(a.ws, a.B, a.T, a.H, a.dim, TOK, bh);
    const float* nOld = a.norm + (size_t)(pos & 1) * slot + bh * (a.dim + 1);
    const bool fresh = pos == 0;
    for (int i = threadIdx.x; i < a.dim; i += 256) g.n0[i] = fresh ? 0.0f : nOld[i];
    const double start = fresh ? 0.0 : (double)nOld[a.dim];
    double* sum = blk; double* top = blk + nb; double* before = blk + 2 * nb;
    // b_t and a_t of this lane's tokens, and the running maximum of a within the block
    auto scan = [&](int j, double (&bt)[TPL], double (&at)[TPL], double (&mx)[TPL]) {
        float iv[TPL];
        double run = 0.0;
#pragma unroll
        for (int u = 0; u < TPL; u++) {
            const int t = j * TOK + lane * TPL + u;
            float fv = 0.0f;
            iv[u] = 0.0f;
            if (t < a.T) {
                const float* x = a.proj + ((size_t)b * a.T + t) * a.ld;
                iv[u] = gate_cap_f(x[a.i_off + h], a.cap);
                fv = log_sigmoid_f(gate_cap_f(x[a.f_off + h], a.cap));
            }
            run += fv;
            bt[u] = run;
        }
        for (int o = 1; o < 32; o <<= 1) {
            const double u = __shfl_up_sync(0xffffffffu, run, o);
            if (lane >= o) run += u;
        }
        const double ahead = run - bt[TPL - 1];              // of the lanes before
        double best = -1e30;
#pragma unroll
        for (int u = 0; u < TPL; u++) {
            bt[u] += ahead;
            at[u] = j * TOK + lane * TPL + u < a.T ? (double)iv[u] - bt[u] : -1e30;
            best = fmax(best, at[u]);
            mx[u] = best;
        }
        for (int o = 1; o < 32; o <<= 1) {
            const double u = __shfl_up_sync(0xffffffffu, best, o);
            if (lane >= o) best = fmax(best, u);
        }
        const double prev = __shfl_up_sync(0xffffffffu, best, 1);
#pragma unroll
        for (int u = 0; u < TPL; u++)
            if (lane > 0) mx[u] = fmax(mx[u], prev);
    };
    double bt[TPL], at[TPL], mx[TPL];
    for (int j = warp; j < nb; j += 8) {
        scan(j, bt, at, mx);
        if (lane == 31) { sum[j] = bt[TPL - 1]; top[j] = mx[TPL - 1]; }
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        double m = start;
        for (int j = 0; j < nb; j++) { before[j] = m; m = (double)(float)(sum[j] + fmax(m, top[j])); }
        a.norm[(size_t)((pos + a.T) & 1) * slot + bh * (a.dim + 1) + a.dim] = (float)m;
    }
    __syncthreads();
    for (int j = warp; j < nb; j += 8) {
        scan(j, bt, at, mx);
        const double m0 = before[j], end = (double)(float)(sum[j] + fmax(m0, top[j]));      // the maximum after the block
#pragma unroll
        for (int u = 0; u < TPL; u++) {
            const int t = j * TOK + lane * TPL + u;
            if (t >= a.T) break;
            const double m = (double)(float)(bt[u] + fmax(m0, mx[u])), row = bt[u] - m;
            g.rowHi[t] = (float)row; g.rowLo[t] = (float)(row - (double)(float)row);
            g.colHi[t] = (float)at[u]; g.colLo[t] = (float)(at[u] - (double)(float)at[u]);
            g.carry[t] = expf((float)(bt[u] + m0 - m));
            g.floor_[t] = expf((float)-m);
            g.add[t] = expf((float)(sum[j] + at[u] - end));
        }
        if (lane == 0) g.keep[j] = expf((float)(sum[j] + m0 - end));
    }
}

DJ_PART bool mlstm_mma_fits(const MlstmArgs& a);
DJ_PART size_t mlstm_mma_ws_floats(const MlstmArgs& a);
DJ_PART void launch_mlstm_mma(const MlstmArgs& a, cudaStream_t s);

}  // namespace dj
