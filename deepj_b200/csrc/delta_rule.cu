// Generalized delta rule: a linear recurrence with a matrix state per head,
//     u_t = k_t / sqrt(Σ k_t² + ε)                    S_t = diag(w_t) S_{t-1} − (a_t ⊙ u_t)(u_tᵀ S_{t-1}) + k_t v_tᵀ
//     o_t = S_tᵀ r_t
// with a decay w and a removal rate a per key channel,
//     w_t = exp(−exp(−1/2) · sigmoid(W2 tanh(low_t) + w0)),    a_t = sigmoid(araw_t + abias).
// The state is fp32 and lives in HBM between calls, [sequence][head][value column][key channel]; a sequence at position
// 0 starts from zeros whatever the buffer holds.  Prompts and single tokens run the same scan, token by token, so how a
// prompt is cut changes nothing.
//
//   k_delta_prepare   per (token, head): w, b = a ⊙ k / (Σk² + ε) — with b the removal term is b (kᵀS) — and, per block of four
//                     tokens, what relates them: with P_ij = Π_{i<l<j} w_l, the vectors k̃_j = k_j ⊙ Π_{l<j} w_l and the scalars
//                     A_ij = k_jᵀ(P_ij ⊙ b_i), B_ij = k_jᵀ(P_ij ⊙ k_i)
//   k_delta_scan      a block of eight warps per (sequence, head, 16 value columns), a warp per two of them: a lane holds some
//                     key channels of its columns in registers.  The four kᵀS of a token block come out of ONE warp reduction
//                     against the state S_0 before it: k_jᵀS_{j-1} = k̃_jᵀS_0 − Σ_{i<j} A_ij k_iᵀS_{i-1} + Σ_{i<j} B_ij v_i;
//                     then the four updates run on the registers, two channels per instruction, and the outputs share the
//                     next block's reduction.  Tokens stream through a two-stage cp.async ring.  A single token (decode) computes its own w and b and reads
//                     the state before the dependency wait.
#include "row_operand.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr float kUnitEps = 1e-6f;
constexpr int kPrepRows = 8;           // tokens per block of k_delta_prepare: two token blocks
constexpr int kBlk = 4, kPairs = 6;    // tokens per block, pairs i < j of them

struct PrepParams {
    const float* proj; int ld, k_off, a_off, low_off, rank;
    const float* abias; const __nv_bfloat16* w2; int w2p; const float* w0;
    float* wOut; float* bOut; float* ktOut;      // [rows][H·dim]
    float* pairs;                                // [B][token blocks][H][2·kPairs]: A then B, pairs (0,1)(0,2)(1,2)(0,3)(1,3)(2,3)
    int T, H, dim;
};
__device__ __forceinline__ int token_blocks(int T) { return (T + kBlk - 1) / kBlk; }

__global__ void __launch_bounds__(128) k_delta_prepare(const PrepParams p) {
    extern __shared__ __align__(16) float low[];                       // [kPrepRows][w2p], then [kPrepRows] 1 / (Σk² + ε)
    __shared__ float red[4][2 * 2 * kPairs];
    float* inv = low + kPrepRows * p.w2p;
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.x, t0 = blockIdx.y * kPrepRows, n = min(kPrepRows, p.T - t0);
    const size_t r0 = (size_t)blockIdx.z * p.T + t0;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int i = threadIdx.x; i < kPrepRows * p.w2p; i += 128) {
        const int r = i / p.w2p, j = i - r * p.w2p;
        low[i] = (r < n && j < p.rank) ? tanhf(p.proj[(r0 + r) * p.ld + p.low_off + j]) : 0.0f;
    }
    for (int r = warp; r < n; r += 4) {
        const float* k = p.proj + (r0 + r) * p.ld + p.k_off + h * p.dim;
        float ss = 0.0f;
        for (int i = lane; i < p.dim; i += 32) ss = fmaf(k[i], k[i], ss);
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (lane == 0) inv[r] = 1.0f / (ss + kUnitEps);
    }
    __syncthreads();
    const float rate = expf(-0.5f);
    float pr[2][2 * kPairs];
#pragma unroll
    for (int q = 0; q < 2; q++)
#pragma unroll
        for (int j = 0; j < 2 * kPairs; j++) pr[q][j] = 0.0f;
    for (int i = threadIdx.x; i < p.dim; i += 128) {
        const int c = h * p.dim + i;
        float acc[kPrepRows];
#pragma unroll
        for (int r = 0; r < kPrepRows; r++) acc[r] = 0.0f;
        const __nv_bfloat16* w = p.w2 + (size_t)c * p.w2p;
        for (int j = 0; j < p.w2p; j += 8) {
            const uint4 d = __ldg(reinterpret_cast<const uint4*>(w + j));
            const uint32_t u[4] = {d.x, d.y, d.z, d.w};
#pragma unroll
            for (int q = 0; q < 4; q++) {
                const float lo = __uint_as_float(u[q] << 16), hi = __uint_as_float(u[q] & 0xffff0000u);
#pragma unroll
                for (int r = 0; r < kPrepRows; r++) {
                    const float2 l = *reinterpret_cast<const float2*>(low + r * p.w2p + j + 2 * q);
                    acc[r] = fmaf(lo, l.x, acc[r]);
                    acc[r] = fmaf(hi, l.y, acc[r]);
                }
            }
        }
        const float w0 = p.w0[c], ab = p.abias[c];
#pragma unroll
        for (int q = 0; q < 2; q++) {
            float kv[kBlk], wv[kBlk], bv[kBlk];
#pragma unroll
            for (int j = 0; j < kBlk; j++) {
                const int r = q * kBlk + j;
                kv[j] = 0.0f; wv[j] = 1.0f; bv[j] = 0.0f;
                if (r < n) {
                    const float* row = p.proj + (r0 + r) * p.ld;
                    kv[j] = row[p.k_off + c];
                    wv[j] = expf(-rate * sigmoid_f(acc[r] + w0));
                    bv[j] = sigmoid_f(row[p.a_off + c] + ab) * kv[j] * inv[r];
                }
            }
            float run = 1.0f;
            int pair = 0;
#pragma unroll
            for (int j = 0; j < kBlk; j++) {
                if (q * kBlk + j < n) {
                    const size_t o = (r0 + q * kBlk + j) * p.H * p.dim + c;
                    p.wOut[o] = wv[j]; p.bOut[o] = bv[j]; p.ktOut[o] = kv[j] * run;
                }
                run *= wv[j];
#pragma unroll
                for (int e = 0; e < j; e++, pair++) {
                    float x = kv[j];
#pragma unroll
                    for (int l = e + 1; l < j; l++) x *= wv[l];
                    pr[q][pair] = fmaf(x, bv[e], pr[q][pair]);
                    pr[q][kPairs + pair] = fmaf(x, kv[e], pr[q][kPairs + pair]);
                }
            }
        }
    }
#pragma unroll
    for (int q = 0; q < 2; q++)
#pragma unroll
        for (int j = 0; j < 2 * kPairs; j++) {
            float v = pr[q][j];
            for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (lane == 0) red[warp][q * 2 * kPairs + j] = v;
        }
    __syncthreads();
    const int tb = threadIdx.x / (2 * kPairs), j = threadIdx.x % (2 * kPairs), blk = t0 / kBlk + tb;
    if (tb < 2 && blk < token_blocks(p.T))
        p.pairs[(((size_t)blockIdx.z * token_blocks(p.T) + blk) * p.H + h) * 2 * kPairs + j] =
            (red[0][threadIdx.x] + red[1][threadIdx.x]) + (red[2][threadIdx.x] + red[3][threadIdx.x]);
}

struct ScanParams {
    PrepParams in;                 // projections, decay weights; wOut / bOut are read here
    int r_off, v_off;
    float* state; const float* pos;
    float* out; int ldo;
    int T, vec, early;             // vec: every field can be copied in 16-byte pieces; early: the state may be read before the wait
};

// Sums C per-lane values over the warp; lane (group g of 32/C lanes) ends up with the sum of column g.  C a power of two.
template <int C>
__device__ __forceinline__ float reduce_columns(float (&v)[C], int lane) {
#pragma unroll
    for (int half = C / 2, bit = 16; half > 0; half >>= 1, bit >>= 1) {
        const bool up = (lane & bit) != 0;
#pragma unroll
        for (int j = 0; j < half; j++) {
            const float keep = up ? v[j + half] : v[j], send = up ? v[j] : v[j + half];
            v[j] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
        }
    }
#pragma unroll
    for (int bit = 16 / C; bit > 0; bit >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], bit);
    return v[0];
}

// two fp32 lanes per instruction
typedef unsigned long long f2;
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) { f2 d; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c)); return d; }
__device__ __forceinline__ f2 mul2(f2 a, f2 b) { f2 d; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b)); return d; }
__device__ __forceinline__ f2 pack2(float a, float b) { f2 d; asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(a), "f"(b)); return d; }
__device__ __forceinline__ float sum2(f2 v) { float a, b; asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); return a + b; }

// The 2·EP channels of a lane.
template <int EP>
__device__ __forceinline__ void lane_row(const float* row, int lane, f2 (&v)[EP]) {
    if constexpr (EP == 1) v[0] = *reinterpret_cast<const f2*>(row + lane * 2);
    else {
#pragma unroll
        for (int j = 0; j < EP; j += 2) {
            const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(row + lane * 2 * EP + 2 * j);
            v[j] = f.x; v[j + 1] = f.y;
        }
    }
}
template <int EP>
__device__ __forceinline__ float dot_row(const f2 (&a)[EP], const f2 (&S)[EP]) {
    f2 x = mul2(a[0], S[0]);
#pragma unroll
    for (int e = 1; e < EP; e++) x = fma2(a[e], S[e], x);
    return sum2(x);
}
// S ← w ⊙ S + k·v − q·dot for one column; returns the lane's part of rᵀS
template <int EP>
__device__ __forceinline__ float update_row(f2 (&S)[EP], const f2 (&w)[EP], const f2 (&k)[EP], const f2 (&q)[EP], const f2 (&r)[EP], float v, float dot) {
    const f2 vv = pack2(v, v), nd = pack2(-dot, -dot);
    f2 x = 0;
#pragma unroll
    for (int e = 0; e < EP; e++) {
        S[e] = fma2(w[e], S[e], fma2(k[e], vv, mul2(q[e], nd)));
        x = e == 0 ? mul2(r[e], S[e]) : fma2(r[e], S[e], x);
    }
    return sum2(x);
}

constexpr int kScanCols = 2, kScanWarps = 8, kScanThreads = 32 * kScanWarps, kBlockCols = kScanCols * kScanWarps;

// 2·EP key channels per lane (lane·2EP …), kScanCols value columns per warp, TB tokens per stage of the ring.
template <int EP, int TB, bool FUSED>
__global__ void __launch_bounds__(kScanThreads) k_delta_scan(const ScanParams p) {
    constexpr int C = kScanCols, NT = kScanThreads, P = 64 * EP, ROW = 5 * P + kBlockCols;                  // a token: k̃, k, w, b, r of the head, v of the block's columns
    constexpr int STAGE = TB * ROW + TB / kBlk * 2 * kPairs;                // … and the pairs of its token blocks
    extern __shared__ __align__(16) float ring[];                           // [2][STAGE]; FUSED: one token, then low [w2p]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, b = blockIdx.z, dim = p.in.dim, H = p.in.H, HD = H * dim, hd = h * dim;
    const int cb = blockIdx.x * kBlockCols, c0 = cb + warp * C;                  // the block's and this warp's first column
    const size_t row0 = (size_t)b * p.T;
    if (P > dim)                                                            // channels past the head stay zero
        for (int t = 0; t < (FUSED ? 1 : 2 * TB); t++)
            for (int i = tid; i < 5 * (P - dim); i += NT)
                ring[(t / TB) * STAGE + (t % TB) * ROW + i / (P - dim) * P + dim + i % (P - dim)] = 0.0f;
    if (!p.early) pdl_wait();
    const bool fresh = p.pos[b] == 0.0f;
    float* st = p.state + (((size_t)b * H + h) * dim + c0) * dim;
    f2 S[C][EP];
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int e = 0; e < EP; e++) {
            const int i = (lane * EP + e) * 2;
            const bool on = !fresh && c0 + c < dim;
            S[c][e] = pack2(on && i < dim ? st[(size_t)c * dim + i] : 0.0f, on && i + 1 < dim ? st[(size_t)c * dim + i + 1] : 0.0f);
        }
    if constexpr (FUSED) {
        pdl_wait();
        pdl_launch_dependents();
        float* low = ring + ROW;
        const float* x = p.in.proj + row0 * p.in.ld;
        for (int j = tid; j < p.in.w2p; j += NT) low[j] = j < p.in.rank ? tanhf(x[p.in.low_off + j]) : 0.0f;
        float ss = 0.0f;
        for (int i = lane; i < dim; i += 32) { const float k = x[p.in.k_off + hd + i]; ss = fmaf(k, k, ss); }
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.0f / (ss + kUnitEps), rate = expf(-0.5f);
        __syncthreads();
        for (int i = tid; i < dim; i += NT) {
            const float kk = x[p.in.k_off + hd + i];
            ring[P + i] = kk;
            ring[4 * P + i] = x[p.r_off + hd + i];
            float acc = 0.0f;
            const __nv_bfloat16* w = p.in.w2 + (size_t)(hd + i) * p.in.w2p;
            for (int j = 0; j < p.in.w2p; j += 8) {
                const uint4 u4 = __ldg(reinterpret_cast<const uint4*>(w + j));
                const uint32_t u[4] = {u4.x, u4.y, u4.z, u4.w};
#pragma unroll
                for (int q = 0; q < 4; q++) {
                    acc = fmaf(__uint_as_float(u[q] << 16), low[j + 2 * q], acc);
                    acc = fmaf(__uint_as_float(u[q] & 0xffff0000u), low[j + 2 * q + 1], acc);
                }
            }
            ring[2 * P + i] = expf(-rate * sigmoid_f(acc + p.in.w0[hd + i]));
            ring[3 * P + i] = sigmoid_f(x[p.in.a_off + hd + i] + p.in.abias[hd + i]) * kk * inv;
        }
        for (int i = tid; i < kBlockCols; i += NT) ring[5 * P + i] = cb + i < dim ? x[p.v_off + hd + cb + i] : 0.0f;
        __syncthreads();
        f2 k[EP], w[EP], q[EP], r[EP];
        lane_row<EP>(ring + P, lane, k); lane_row<EP>(ring + 2 * P, lane, w); lane_row<EP>(ring + 3 * P, lane, q); lane_row<EP>(ring + 4 * P, lane, r);
        float d[C], o[C];
#pragma unroll
        for (int c = 0; c < C; c++) d[c] = dot_row<EP>(k, S[c]);
        const float ks = reduce_columns<C>(d, lane);
#pragma unroll
        for (int c = 0; c < C; c++) {
            const float dot = __shfl_sync(0xffffffffu, ks, c * (32 / C));
            o[c] = update_row<EP>(S[c], w, k, q, r, ring[5 * P + warp * C + c], dot);
        }
        const float os = reduce_columns<C>(o, lane);
        const int col = c0 + lane / (32 / C);
        if (lane % (32 / C) == 0 && col < dim) p.out[row0 * p.ldo + hd + col] = os;
    } else {
        pdl_wait();
        pdl_launch_dependents();
        const int nv = min(kBlockCols, dim - cb), nBlk = token_blocks(p.T);
        constexpr int BPS = TB / kBlk;                 // token blocks per stage
        auto load = [&](int t0, int stage) {           // a warp copies tokens warp, warp + 8, … of the stage
            float* dst = ring + stage * STAGE;
            const int n = min(TB, p.T - t0);
            for (int t = warp; t < n; t += kScanWarps) {
                const size_t r = row0 + t0 + t;
                const float* row = p.in.proj + r * p.in.ld + hd;
                const float* src[5] = {p.in.ktOut + r * HD + hd, row + p.in.k_off, p.in.wOut + r * HD + hd, p.in.bOut + r * HD + hd, row + p.r_off};
                float* d = dst + t * ROW;
#pragma unroll
                for (int f = 0; f < 5; f++) {
                    if (p.vec) { for (int i = lane * 4; i < dim; i += 128) cp_async16(d + f * P + i, src[f] + i); }
                    else { for (int i = lane; i < dim; i += 32) cp_async4(d + f * P + i, src[f] + i); }
                }
                if (p.vec) { if (lane * 4 < nv) cp_async16(d + 5 * P + lane * 4, row + p.v_off + cb + lane * 4); }
                else if (lane < nv) cp_async4(d + 5 * P + lane, row + p.v_off + cb + lane);
            }
            for (int i = tid; i < BPS * 2 * kPairs; i += NT) {
                const int blk = t0 / kBlk + i / (2 * kPairs);
                if (blk < nBlk) cp_async4(dst + TB * ROW + i, p.in.pairs + (((size_t)b * nBlk + blk) * H + h) * 2 * kPairs + i % (2 * kPairs));
            }
            cp_async_commit();
        };
        constexpr int V = kBlk * C;                    // values per block
        float red[2 * V];                              // [0, V): products of the coming block with S, [V, 2V): outputs of the last one
        auto products = [&](const float* rows) {
#pragma unroll
            for (int j = 0; j < kBlk; j++) {
                f2 kt[EP];
                lane_row<EP>(rows + j * ROW, lane, kt);
#pragma unroll
                for (int c = 0; c < C; c++) red[j * C + c] = dot_row<EP>(kt, S[c]);
            }
        };
        load(0, 0);
        cp_async_wait<0>();
        __syncthreads();
        if (TB < p.T) load(TB, 1);
        const float* rows = ring;
        products(rows);
#pragma unroll
        for (int i = V; i < 2 * V; i++) red[i] = 0.0f;
        constexpr int LPV = 32 / (2 * V);              // lanes per value
        float mine = reduce_columns<2 * V>(red, lane);
        const int oi = lane / LPV - V, oj = oi / C, ocol = c0 + oi % C;      // this lane's output, when oi ≥ 0
        for (int blk = 0; blk < nBlk; blk++) {
            const int slot = blk % BPS, stage = blk / BPS & 1;
            const float* pr = ring + stage * STAGE + TB * ROW + slot * 2 * kPairs;
            const int n = min(kBlk, p.T - blk * kBlk);             // tokens of this block
            float dot[kBlk][C], v[kBlk][C], pair[2 * kPairs];
#pragma unroll
            for (int i = 0; i < kPairs / 2; i++) {                  // pairs: 12 floats, 16-byte aligned
                const float4 f = *reinterpret_cast<const float4*>(pr + 4 * i);
                pair[4 * i] = f.x; pair[4 * i + 1] = f.y; pair[4 * i + 2] = f.z; pair[4 * i + 3] = f.w;
            }
#pragma unroll
            for (int j = 0; j < kBlk; j++) {
                const float2 f = *reinterpret_cast<const float2*>(rows + j * ROW + 5 * P + warp * C);
                v[j][0] = f.x; v[j][1] = f.y;
#pragma unroll
                for (int c = 0; c < C; c++) dot[j][c] = __shfl_sync(0xffffffffu, mine, (j * C + c) * LPV);
            }
            int at = 0;
#pragma unroll
            for (int j = 1; j < kBlk; j++)
#pragma unroll
                for (int i = 0; i < j; i++, at++)
#pragma unroll
                    for (int c = 0; c < C; c++) dot[j][c] = fmaf(pair[kPairs + at], v[i][c], fmaf(-pair[at], dot[i][c], dot[j][c]));
            auto update = [&](int j) {
                f2 k[EP], w[EP], q[EP], r[EP];
                const float* row = rows + j * ROW;
                lane_row<EP>(row + P, lane, k); lane_row<EP>(row + 2 * P, lane, w); lane_row<EP>(row + 3 * P, lane, q); lane_row<EP>(row + 4 * P, lane, r);
#pragma unroll
                for (int c = 0; c < C; c++) red[V + j * C + c] = update_row<EP>(S[c], w, k, q, r, v[j][c], dot[j][c]);
            };
            if (n == kBlk) {
#pragma unroll
                for (int j = 0; j < kBlk; j++) update(j);
            } else {
#pragma unroll
                for (int j = 0; j < kBlk; j++)
                    if (j < n) update(j);
            }
            if (blk + 1 < nBlk) {
                if (slot == BPS - 1) {
                    cp_async_wait<0>();
                    __syncthreads();                   // the next stage has landed, and nobody reads this one any more
                    const int t2 = (blk + 1) * kBlk + TB;
                    if (t2 < p.T) load(t2, stage);
                    rows = ring + (stage ^ 1) * STAGE;
                } else rows += kBlk * ROW;
                products(rows);
            }
            mine = reduce_columns<2 * V>(red, lane);
            if (oi >= 0 && lane % LPV == 0 && oj < n && ocol < dim) p.out[(row0 + blk * kBlk + oj) * p.ldo + hd + ocol] = mine;
        }
    }
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int e = 0; e < EP; e++) {
            const int i = (lane * EP + e) * 2;
            float a, b2;
            asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b2) : "l"(S[c][e]));
            if (i < dim && c0 + c < dim) st[(size_t)c * dim + i] = a;
            if (i + 1 < dim && c0 + c < dim) st[(size_t)c * dim + i + 1] = b2;
        }
}

template <int EP, int TB>
void launch_scan(const ScanParams& p, int B, cudaStream_t s) {
    constexpr int ROW = 5 * 64 * EP + kBlockCols, STAGE = TB * ROW + TB / kBlk * 2 * kPairs;
    const dim3 grid((unsigned)((p.in.dim + kBlockCols - 1) / kBlockCols), (unsigned)p.in.H, (unsigned)B);
    if (p.T == 1) {
        launch_k(k_delta_scan<EP, TB, true>, grid, dim3(kScanThreads), (size_t)(ROW + p.in.w2p) * 4, s, true, p);
        return;
    }
    static bool attr = false;
    if (!attr) {
        DJ_CUDA_CHECK(cudaFuncSetAttribute(k_delta_scan<EP, TB, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024));
        attr = true;
    }
    // blocks that start while an earlier kernel drains would pile up on the SMs that are free first: when everything fits
    // with one or two blocks per SM, ask for as much shared memory as keeps it that way
    size_t smem = (size_t)2 * STAGE * 4;
    const long blocks = (long)grid.x * grid.y * grid.z;
    if (blocks <= g_num_sms) smem = std::max(smem, (size_t)112 * 1024);
    else if (blocks <= 2l * g_num_sms) smem = std::max(smem, (size_t)80 * 1024);
    launch_k(k_delta_scan<EP, TB, false>, grid, dim3(kScanThreads), smem, s, true, p);
}

}  // namespace

constexpr int kDeltaMaxDim = 256;
bool delta_rule_fits(int dim, int rank) { return dim >= 1 && dim <= kDeltaMaxDim && pad8(rank) * kPrepRows * 4 + 64 <= 44 * 1024; }
size_t delta_rule_ws_floats(int B, int T, int H, int dim) {
    return T == 1 ? 0 : 3 * (size_t)B * T * H * dim + (size_t)B * ((T + kBlk - 1) / kBlk) * H * 2 * kPairs;
}

void launch_delta_rule(const DeltaRuleArgs& a, cudaStream_t s) {
    const size_t n = (size_t)a.B * a.T * a.H * a.dim;
    PrepParams q;
    q.proj = a.proj; q.ld = a.ld; q.k_off = a.k_off; q.a_off = a.a_off; q.low_off = a.low_off; q.rank = a.w2.K;
    q.abias = a.abias; q.w2 = a.w2.w; q.w2p = a.w2.Kp; q.w0 = a.w0;
    q.wOut = a.ws; q.bOut = a.ws + n; q.ktOut = a.ws + 2 * n; q.pairs = a.ws + 3 * n;
    q.T = a.T; q.H = a.H; q.dim = a.dim;
    if (a.T > 1)
        launch_k(k_delta_prepare, dim3((unsigned)a.H, (unsigned)((a.T + kPrepRows - 1) / kPrepRows), (unsigned)a.B), dim3(128), (size_t)kPrepRows * (q.w2p + 1) * 4, s,
                 true, q);
    ScanParams p;
    p.in = q; p.r_off = a.r_off; p.v_off = a.v_off;
    p.state = a.state; p.pos = a.pos; p.out = a.out; p.ldo = a.ldo; p.T = a.T;
    p.early = a.early || a.T > 1;             // k_delta_prepare comes before a scan of several tokens
    p.vec = ((a.dim | a.ld | a.r_off | a.k_off | a.v_off) & 3) == 0 && (((uintptr_t)a.proj | (uintptr_t)a.ws) & 15) == 0;
    if (a.dim <= 64) launch_scan<1, 8>(p, a.B, s);
    else if (a.dim <= 128) launch_scan<2, 8>(p, a.B, s);
    else launch_scan<4, 8>(p, a.B, s);
}

}  // namespace dj
