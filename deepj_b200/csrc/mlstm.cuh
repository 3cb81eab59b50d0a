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

DJ_PART bool mlstm_mma_fits(const MlstmArgs& a);
DJ_PART size_t mlstm_mma_ws_floats(const MlstmArgs& a);          // behind the gates
DJ_PART void launch_mlstm_mma(const MlstmArgs& a, float* rows, cudaStream_t s);

}  // namespace dj
