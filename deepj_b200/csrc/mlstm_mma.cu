// Matrix-memory recurrence over many tokens on the tensor cores (the recurrence and its block form are described in mlstm.cu).
//
//   k_mlstm_prepare     the gates (a block per head and sequence), and queries (scaled), keys and values of the chunk as bf16 rows per
//                       (sequence, head), head sizes padded to sixteen (a block per token)
//   k_mlstm_chunk_mma   a block of eight warps per (32 value columns, head, sequence) walks blocks of 64 tokens.  The state lives in
//                       the accumulators of its own update, Sᵀ[column][channel].  Per token block: (1) X = weighted q·k and its row
//                       sums, the values times their weight in the coming state, the state as an operand; (2) outputs
//                       carry ⊙ (Q S) + X V over the denominators, and S ← keep·S + (add ⊙ V)ᵀ K.
// Projections are bf16 operands; everything that the recurrence forms itself — X, the weighted values, the state — enters a
// product as two bf16 halves (16 bits) and is kept and summed in fp32.
#include "mlstm.cuh"
#include "mma_common.cuh"
#include "row_operand.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr int kTok = kMlTokMma, kCols = 32, kThreads = 256;
constexpr int kVP = kCols + 8, kXP = kTok + 8;     // row pitches (halves) of values and of X
constexpr size_t kSmemMax = 227 * 1024 - 64;

__host__ __device__ __forceinline__ int pad16(int n) { return (n + 15) & ~15; }

// B·H blocks for the gates, then one per token: [B·H][T][pad16(dim)] queries, then keys, then [B·H][T][vp] values
__global__ void __launch_bounds__(256) k_mlstm_prepare(const MlstmArgs a, __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ k, __nv_bfloat16* __restrict__ v,
                                                    int dp, int vp) {
    pdl_wait();
    pdl_launch_dependents();
    extern __shared__ double blk[];
    if ((int)blockIdx.x < a.B * a.H) {
        ml_gate_block<kMlTokMma / 32>(a, blockIdx.x % a.H, blockIdx.x / a.H, blk);
        return;
    }
    const int row = blockIdx.x - a.B * a.H, b = row / a.T, t = row - b * a.T;
    const float* x = a.proj + (size_t)row * a.ld;
    const bool pairs = ((a.dim | a.vdim) & 1) == 0 && ((a.ld | a.q_off | a.k_off | a.v_off) & 1) == 0;
    auto copy = [&](int off, int n, int np, float f, __nv_bfloat16* dst) {
        for (int i = threadIdx.x * 2; i < a.H * np; i += 512) {
            const int h = i / np, d = i - h * np;            // np is even: a pair stays within a head
            const float* src = x + off + (size_t)h * n + d;
            float u0 = 0.0f, u1 = 0.0f;
            if (pairs && d + 1 < n) { const float2 p = *reinterpret_cast<const float2*>(src); u0 = p.x; u1 = p.y; }
            else { if (d < n) u0 = src[0]; if (d + 1 < n) u1 = src[1]; }
            *reinterpret_cast<uint32_t*>(dst + (((size_t)b * a.H + h) * a.T + t) * np + d) = pack_bf16(u0 * f, u1 * f);
        }
    };
    copy(a.q_off, a.dim, dp, a.qscale, q);
    copy(a.k_off, a.dim, dp, 1.0f, k);
    copy(a.v_off, a.vdim, vp, 1.0f, v);
}

struct McShape { int LD; size_t stage, total; };
__host__ __device__ __forceinline__ McShape mc_shape(int dp) {
    McShape s;
    s.LD = dp + 8;                                           // rows start in different banks
    s.stage = ((size_t)2 * kTok * s.LD + (size_t)kTok * kVP) * 2;                       // Q, K, V of a token block
    s.total = 2 * s.stage + ((size_t)2 * kCols * s.LD + 2 * kTok * kXP + 2 * kTok * kVP) * 2 + ((size_t)dp + 2 * 7 * kTok + 3 * kTok) * 4;
    return s;
}

// 16 bytes to shared memory, or zeros
__device__ __forceinline__ void cp_async16_or_zero(void* dst, const void* src, bool on) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
constexpr float kLog2e = 1.4426950408889634f;

// NS: n-tiles of the state's channels per warp (four warps share the channels), head size up to 32·NS
template <int NS>
__global__ void __launch_bounds__(kThreads, 1) k_mlstm_chunk_mma(const MlstmArgs a, const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ k,
                                                                 const __nv_bfloat16* __restrict__ v, int dp, int vp) {
    extern __shared__ __align__(16) unsigned char mc_raw[];
    const McShape M = mc_shape(dp);
    const int LD = M.LD;
    __nv_bfloat16* Sh = reinterpret_cast<__nv_bfloat16*>(mc_raw + 2 * M.stage);      // [kCols][LD] state before the block, high halves, then low
    __nv_bfloat16* Xh = Sh + 2 * kCols * LD;                                         // [kTok][kXP], then low
    __nv_bfloat16* Wh = Xh + 2 * kTok * kXP;                                         // [kTok][kVP], then low
    float* nrm = reinterpret_cast<float*>(Wh + 2 * kTok * kVP);                      // [dp]
    float* gates = nrm + dp;                                                         // [2][7][kTok] gates of the tokens of two blocks
    float* rowSum = gates + 2 * 7 * kTok;                                                   // [2][kTok] sums of X by column half
    float* nq = rowSum + 2 * kTok;                                                   // [kTok] normaliser · query
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rl = lane >> 2, t4 = lane & 3;
    const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * kCols, nc = min(kCols, a.vdim - c0), dim = a.dim;
    const size_t bh = (size_t)b * a.H + h;
    q += bh * a.T * dp; k += bh * a.T * dp; v += bh * a.T * vp + c0;
    pdl_wait();
    pdl_launch_dependents();
    const int pos = (int)a.pos[b], nb = ml_blocks(a.T, kTok), dq = dp / 8, vq = (min(kCols, vp - c0)) / 8;
    const MlGates g = ml_gates(a.ws, a.B, a.T, a.H, dim, kTok, bh);
    const int stepT = kThreads / dq, stepC = kThreads - stepT * dq;
    auto load = [&](int j) {
        __nv_bfloat16* Q = reinterpret_cast<__nv_bfloat16*>(mc_raw + (j & 1) * M.stage);
        __nv_bfloat16* K = Q + kTok * LD; __nv_bfloat16* V = K + kTok * LD;
        const int t0 = j * kTok;
        // rows of dq 16-byte pieces: a thread's pieces are kThreads apart
        for (int t = tid / dq, c = tid - t * dq; t < kTok;) {
            const size_t at = (size_t)min(t0 + t, a.T - 1) * dp + c * 8;
            cp_async16_or_zero(Q + t * LD + c * 8, q + at, t0 + t < a.T);
            cp_async16_or_zero(K + t * LD + c * 8, k + at, t0 + t < a.T);
            t += stepT; c += stepC;
            if (c >= dq) { c -= dq; t++; }
        }
        {
            const int t = tid / (kCols / 8), c = tid % (kCols / 8), tt = min(t0 + t, a.T - 1), cc = min(c, vq - 1);
            static_assert(kThreads == kTok * kCols / 8, "one piece of the values per thread");
            cp_async16_or_zero(V + t * kVP + c * 8, v + (size_t)tt * vp + cc * 8, t0 + t < a.T && c < vq);
        }
        float* gt = gates + (j & 1) * 7 * kTok;
        for (int i = tid; i < 7 * kTok; i += kThreads) {
            const int f = i / kTok, t = i % kTok;
            if (t0 + t < a.T) cp_async4(gt + i, g.rowHi + (size_t)f * a.B * a.H * a.T + t0 + t);
            else gt[i] = f == 0 ? -INFINITY : 0.0f;
        }
        cp_async_commit();
    };
    load(0);
    // state fragments: rows (value columns) sm + rl, + 8; channels sn + 8·n + 2·t4, + 1
    const int smr = (warp & 1) * 16, sn = (warp >> 1) * 8 * NS;
    float* st = a.state + (bh * a.vdim + c0) * dim;
    float S[NS][4];
#pragma unroll
    for (int n = 0; n < NS; n++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int c = smr + rl + (e >> 1) * 8, d = sn + 8 * n + 2 * t4 + (e & 1);
            S[n][e] = pos != 0 && c < nc && d < dim ? st[(size_t)c * dim + d] : 0.0f;
        }
    for (int i = tid; i < dp; i += kThreads) nrm[i] = i < dim ? g.n0[i] : 0.0f;
    const int m0 = (warp >> 1) * 16, nh = warp & 1;          // this warp's 16 tokens of X and of the outputs, and its half of their columns
    const int ra = m0 + rl, rb = ra + 8;
    const uint32_t rowLane = (uint32_t)((lane & 15) * 2), colLane = (uint32_t)((lane >> 4) * 16);      // operand A: row, 16-byte column
    const uint32_t bRow = (uint32_t)((lane & 7) + ((lane >> 4) << 3)), bCol = (uint32_t)(((lane >> 3) & 1) * 16);      // operand B from rows [n][k]
    const uint32_t tRow = (uint32_t)((lane & 7) + (((lane >> 3) & 1) << 3)), tCol = (uint32_t)((lane >> 4) * 16);      // operand B from rows [k][n]
    const uint32_t shA = smem_u32(Sh), xhA = smem_u32(Xh), whA = smem_u32(Wh);
    const uint32_t slD = (uint32_t)(kCols * LD * 2), xlD = (uint32_t)(kTok * kXP * 2), wlD = (uint32_t)(kTok * kVP * 2);
    const bool wide = ((a.vdim | a.ldo) & 1) == 0 && ((uintptr_t)a.out & 7) == 0;
    float nextKeep = g.keep[0];
    for (int j = 0; j < nb; j++) {
        const int t0 = j * kTok, n = min(kTok, a.T - t0);
        cp_async_wait<0>();
        __syncthreads();                                     // the block has landed; nobody reads the other stage, X, W, S or the gates any more
        if (j + 1 < nb) load(j + 1);
        const __nv_bfloat16* Q = reinterpret_cast<const __nv_bfloat16*>(mc_raw + (j & 1) * M.stage);
        const __nv_bfloat16* K = Q + kTok * LD; const __nv_bfloat16* V = K + kTok * LD;
        const uint32_t qA = smem_u32(Q), kA = smem_u32(K), vA = smem_u32(V);
        const float* gt = gates + (j & 1) * 7 * kTok;
        const float keep = nextKeep;
        if (j + 1 < nb) nextKeep = g.keep[j + 1];
        // the state before this block as an operand
#pragma unroll
        for (int i = 0; i < NS; i++) {
            const int d = sn + 8 * i + 2 * t4;
            if (d >= dp) continue;
            uint32_t hi, lo;
            split_bf16(S[i][0], S[i][1], hi, lo);
            *reinterpret_cast<uint32_t*>(Sh + (smr + rl) * LD + d) = hi; *reinterpret_cast<uint32_t*>(Sh + (kCols + smr + rl) * LD + d) = lo;
            split_bf16(S[i][2], S[i][3], hi, lo);
            *reinterpret_cast<uint32_t*>(Sh + (smr + rl + 8) * LD + d) = hi; *reinterpret_cast<uint32_t*>(Sh + (kCols + smr + rl + 8) * LD + d) = lo;
        }
        // q·k of this warp's tokens and 32 of the block's
        float x[4][4];
#pragma unroll
        for (int i = 0; i < 4; i++) { x[i][0] = 0.0f; x[i][1] = 0.0f; x[i][2] = 0.0f; x[i][3] = 0.0f; }
        const bool some = nh * 32 <= m0 + 15;                // any of them at or before the tokens
        if (some) {
#pragma unroll 4
            for (int kk = 0; kk < dp / 16; kk++) {
                uint32_t aq[4];
                ldm_x4(aq, qA + (uint32_t)(m0 * LD * 2) + rowLane * LD + colLane + kk * 32);
#pragma unroll
                for (int i = 0; i < 2; i++) {
                    uint32_t bk[4];
                    ldm_x4(bk, kA + (uint32_t)((nh * 32 + i * 16 + bRow) * LD * 2) + bCol + kk * 32);
                    mma_bf16(x[2 * i], aq, bk[0], bk[1]); mma_bf16(x[2 * i + 1], aq, bk[2], bk[3]);
                }
            }
        }
        for (int i = tid; i < kTok * kCols / 2; i += kThreads) {
            const int t = i / (kCols / 2), c = i % (kCols / 2) * 2;
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(V + t * kVP + c));
            uint32_t hi, lo;
            split_bf16(f.x * gt[6 * kTok + t], f.y * gt[6 * kTok + t], hi, lo);
            *reinterpret_cast<uint32_t*>(Wh + t * kVP + c) = hi; *reinterpret_cast<uint32_t*>(Wh + (kTok + t) * kVP + c) = lo;
        }
        {                                                    // four lanes per token, eight channels at a time
            const int t = tid >> 2;
            float s = 0.0f;
            for (int d = (tid & 3) * 8; d < dp; d += 32) {
                const uint4 u = *reinterpret_cast<const uint4*>(Q + t * LD + d);
                const float4 n0 = *reinterpret_cast<const float4*>(nrm + d), n1 = *reinterpret_cast<const float4*>(nrm + d + 4);
                s = fmaf(n0.x, __uint_as_float(u.x << 16), s); s = fmaf(n0.y, __uint_as_float(u.x & 0xffff0000u), s);
                s = fmaf(n0.z, __uint_as_float(u.y << 16), s); s = fmaf(n0.w, __uint_as_float(u.y & 0xffff0000u), s);
                s = fmaf(n1.x, __uint_as_float(u.z << 16), s); s = fmaf(n1.y, __uint_as_float(u.z & 0xffff0000u), s);
                s = fmaf(n1.z, __uint_as_float(u.w << 16), s); s = fmaf(n1.w, __uint_as_float(u.w & 0xffff0000u), s);
            }
            s += __shfl_xor_sync(0xffffffffu, s, 1); s += __shfl_xor_sync(0xffffffffu, s, 2);
            if ((tid & 3) == 0) nq[t] = s;
        }
        float sa = 0.0f, sb = 0.0f;
        const float rha = gt[ra], rla = gt[kTok + ra], rhb = gt[rb], rlb = gt[kTok + rb];
        // the sums cancel before they are scaled to powers of two
#pragma unroll
        for (int i = 0; i < 4; i++) {
            const int s0 = nh * 32 + i * 8 + 2 * t4;
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int s = s0 + e;
                const float ch = gt[2 * kTok + s], cl = gt[3 * kTok + s];
                x[i][e] = s <= ra ? x[i][e] * ex2(((rha + ch) + (rla + cl)) * kLog2e) : 0.0f;
                x[i][2 + e] = s <= rb ? x[i][2 + e] * ex2(((rhb + ch) + (rlb + cl)) * kLog2e) : 0.0f;
                sa += x[i][e]; sb += x[i][2 + e];
            }
            uint32_t hi, lo;
            split_bf16(x[i][0], x[i][1], hi, lo);
            *reinterpret_cast<uint32_t*>(Xh + ra * kXP + s0) = hi; *reinterpret_cast<uint32_t*>(Xh + (kTok + ra) * kXP + s0) = lo;
            split_bf16(x[i][2], x[i][3], hi, lo);
            *reinterpret_cast<uint32_t*>(Xh + rb * kXP + s0) = hi; *reinterpret_cast<uint32_t*>(Xh + (kTok + rb) * kXP + s0) = lo;
        }
        sa += __shfl_xor_sync(0xffffffffu, sa, 1); sa += __shfl_xor_sync(0xffffffffu, sa, 2);
        sb += __shfl_xor_sync(0xffffffffu, sb, 1); sb += __shfl_xor_sync(0xffffffffu, sb, 2);
        if (t4 == 0) { rowSum[nh * kTok + ra] = sa; rowSum[nh * kTok + rb] = sb; }
        __syncthreads();
        // outputs: 16 tokens × 16 columns per warp
        float o[2][4], ol[2][4];
#pragma unroll
        for (int i = 0; i < 2; i++)
#pragma unroll
            for (int e = 0; e < 4; e++) { o[i][e] = 0.0f; ol[i][e] = 0.0f; }
#pragma unroll 4
        for (int kk = 0; kk < dp / 16; kk++) {
            uint32_t aq[4], bs[4], bl[4];
            ldm_x4(aq, qA + (uint32_t)(m0 * LD * 2) + rowLane * LD + colLane + kk * 32);
            const uint32_t at = shA + (uint32_t)((nh * 16 + bRow) * LD * 2) + bCol + kk * 32;
            ldm_x4(bs, at);
            ldm_x4(bl, at + slD);
            mma_bf16(o[0], aq, bs[0], bs[1]); mma_bf16(o[1], aq, bs[2], bs[3]);
            mma_bf16(ol[0], aq, bl[0], bl[1]); mma_bf16(ol[1], aq, bl[2], bl[3]);
        }
        const float ca = gt[4 * kTok + ra], cb = gt[4 * kTok + rb];
#pragma unroll
        for (int i = 0; i < 2; i++) {
            o[i][0] = (o[i][0] + ol[i][0]) * ca; o[i][1] = (o[i][1] + ol[i][1]) * ca;
            o[i][2] = (o[i][2] + ol[i][2]) * cb; o[i][3] = (o[i][3] + ol[i][3]) * cb;
#pragma unroll
            for (int e = 0; e < 4; e++) ol[i][e] = 0.0f;
        }
        for (int kk = 0; kk * 16 <= m0 + 15; kk++) {
            uint32_t xh[4], xl[4], bv[4];
            const uint32_t at = xhA + (uint32_t)(m0 * kXP * 2) + rowLane * kXP + colLane + kk * 32;
            ldm_x4(xh, at);
            ldm_x4(xl, at + xlD);
            ldm_x4_t(bv, vA + (uint32_t)((kk * 16 + tRow) * kVP * 2) + (uint32_t)(nh * 32) + tCol);
            mma_bf16(o[0], xh, bv[0], bv[1]); mma_bf16(o[1], xh, bv[2], bv[3]);
            mma_bf16(ol[0], xl, bv[0], bv[1]); mma_bf16(ol[1], xl, bv[2], bv[3]);
        }
        {
            const float da = 1.0f / (fmaxf(fabsf(fmaf(nq[ra], ca, rowSum[ra] + rowSum[kTok + ra])), gt[5 * kTok + ra]) + kMlDenEps);
            const float db = 1.0f / (fmaxf(fabsf(fmaf(nq[rb], cb, rowSum[rb] + rowSum[kTok + rb])), gt[5 * kTok + rb]) + kMlDenEps);
            float* oa = a.out + ((size_t)b * a.T + t0 + ra) * a.ldo + (size_t)h * a.vdim + c0; float* ob = oa + (size_t)8 * a.ldo;
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int c = nh * 16 + i * 8 + 2 * t4;
                const float2 va = make_float2((o[i][0] + ol[i][0]) * da, (o[i][1] + ol[i][1]) * da), vb = make_float2((o[i][2] + ol[i][2]) * db, (o[i][3] + ol[i][3]) * db);
                if (wide) {                                  // whole pairs of columns at even offsets
                    if (c < nc && ra < n) *reinterpret_cast<float2*>(oa + c) = va;
                    if (c < nc && rb < n) *reinterpret_cast<float2*>(ob + c) = vb;
                } else {
                    if (c < nc && ra < n) oa[c] = va.x;
                    if (c + 1 < nc && ra < n) oa[c + 1] = va.y;
                    if (c < nc && rb < n) ob[c] = vb.x;
                    if (c + 1 < nc && rb < n) ob[c + 1] = vb.y;
                }
            }
        }
        // the state after the block
#pragma unroll
        for (int i = 0; i < NS; i++) { S[i][0] *= keep; S[i][1] *= keep; S[i][2] *= keep; S[i][3] *= keep; }
#pragma unroll
        for (int kk = 0; kk < kTok / 16; kk++) {
            // operand A: (weighted values)ᵀ, 16 columns × 16 tokens, read transposed from rows of tokens
            uint32_t wh[4], wl[4];
            const uint32_t at = whA + (uint32_t)((kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * kVP * 2) + (uint32_t)(smr * 2) + (uint32_t)(((lane >> 3) & 1) * 16);
            ldm_x4_t(wh, at);
            ldm_x4_t(wl, at + wlD);
#pragma unroll
            for (int i = 0; i < NS; i += 2) {
                if (sn + 8 * i >= dp) break;
                uint32_t bk[4];
                ldm_x4_t(bk, kA + (uint32_t)((kk * 16 + tRow) * LD * 2) + (uint32_t)((sn + 8 * i) * 2) + tCol);
                mma_bf16(S[i], wh, bk[0], bk[1]); mma_bf16(S[i + 1], wh, bk[2], bk[3]);
                mma_bf16(S[i], wl, bk[0], bk[1]); mma_bf16(S[i + 1], wl, bk[2], bk[3]);
            }
        }
        for (int p = tid >> 2; p < dp / 2; p += kThreads / 4) {       // the normaliser: two channels per four lanes, which share the tokens
            float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
            for (int u = 0; u < kTok / 4; u++) {
                const int t = u * 4 + (tid & 3);
                const uint32_t kk = *reinterpret_cast<const uint32_t*>(K + t * LD + 2 * p);
                s0 = fmaf(gt[6 * kTok + t], __uint_as_float(kk << 16), s0);
                s1 = fmaf(gt[6 * kTok + t], __uint_as_float(kk & 0xffff0000u), s1);
            }
            s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 1);
            s0 += __shfl_xor_sync(0xffffffffu, s0, 2); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
            if ((tid & 3) == 0) { nrm[2 * p] = fmaf(nrm[2 * p], keep, s0); nrm[2 * p + 1] = fmaf(nrm[2 * p + 1], keep, s1); }
        }
    }
    __syncthreads();                                         // the normaliser is complete
#pragma unroll
    for (int i = 0; i < NS; i++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
            const int c = smr + rl + (e >> 1) * 8, d = sn + 8 * i + 2 * t4 + (e & 1);
            if (c < nc && d < dim) st[(size_t)c * dim + d] = S[i][e];
        }
    if (blockIdx.x == 0) {
        float* nNew = a.norm + (size_t)((pos + a.T) & 1) * a.B * a.H * (dim + 1) + bh * (dim + 1);
        for (int d = tid; d < dim; d += kThreads) nNew[d] = nrm[d];
    }
}

template <int NS>
void run(const MlstmArgs& a, const __nv_bfloat16* q, const __nv_bfloat16* k, const __nv_bfloat16* v, int dp, int vp, cudaStream_t s) {
    static bool done = false;
    if (!done) DJ_CUDA_CHECK(cudaFuncSetAttribute(k_mlstm_chunk_mma<NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    done = true;
    launch_k(k_mlstm_chunk_mma<NS>, dim3((unsigned)((a.vdim + kCols - 1) / kCols), (unsigned)a.H, (unsigned)a.B), dim3(kThreads), mc_shape(dp).total, s, true, a, q, k, v,
             dp, vp);
}

}  // namespace

constexpr int kMmaMinTokens = 16;      // shorter portions take the FMA form
bool mlstm_mma_fits(const MlstmArgs& a) { return !a.exact && a.T >= kMmaMinTokens && pad16(a.dim) <= 256 && mc_shape(pad16(a.dim)).total <= kSmemMax; }
size_t mlstm_mma_ws_floats(const MlstmArgs& a) {
    return ml_gate_floats(a.B, a.T, a.H, a.dim, kTok) + (size_t)a.B * a.H * a.T * (2 * pad16(a.dim) + pad16(a.vdim)) / 2;
}

void launch_mlstm_mma(const MlstmArgs& a, cudaStream_t s) {
    const int dp = pad16(a.dim), vp = pad16(a.vdim);
    const size_t n = (size_t)a.B * a.H * a.T * dp;
    __nv_bfloat16* q = (__nv_bfloat16*)(a.ws + ml_gate_floats(a.B, a.T, a.H, a.dim, kTok)); __nv_bfloat16* k = q + n; __nv_bfloat16* v = k + n;
    launch_k(k_mlstm_prepare, dim3((unsigned)(a.B * (a.H + a.T))), dim3(256), (size_t)ml_blocks(a.T, kTok) * 24, s, true, a, q, k, v, dp, vp);
    if (dp <= 64) run<2>(a, q, k, v, dp, vp, s);
    else if (dp <= 128) run<4>(a, q, k, v, dp, vp, s);
    else run<8>(a, q, k, v, dp, vp, s);
}

}  // namespace dj
