// Generalized delta rule: a linear recurrence with a matrix state per head,
//     u_t = k_t / sqrt(Σ k_t² + ε)                    S_t = diag(w_t) S_{t-1} − (a_t ⊙ u_t)(u_tᵀ S_{t-1}) + k_t v_tᵀ
//     o_t = S_tᵀ r_t
// with a decay w and a removal rate a per key channel,
//     w_t = exp(−exp(−1/2) · sigmoid(W2 tanh(low_t) + w0)),    a_t = sigmoid(araw_t + abias).
// The state is fp32 and lives in HBM between calls, [sequence][head][value column][key channel]; a sequence at position
// 0 starts from zeros whatever the buffer holds.  Prompts and single tokens run the same scan, token by token, so how a
// prompt is cut changes nothing.
//
//   k_delta_prepare   per (token, head): w, and b = a ⊙ k / (Σk² + ε) — with b the removal term is b (kᵀS)
//   k_delta_scan      a block of four warps per (sequence, head, 16 value columns), a warp per four of them: a lane holds some
//                     key channels of its columns in registers, kᵀS and o are warp reductions over all lanes, and the
//                     tokens' vectors stream through a two-stage cp.async ring of shared memory.  A single token computes
//                     its own w and b (no prepare launch) and reads the state before the dependency wait.
#include "row_operand.cuh"

namespace dj {
namespace {

constexpr float kUnitEps = 1e-6f;
constexpr int kPrepRows = 8;

struct PrepParams {
    const float* proj; int ld, k_off, a_off, low_off, rank;
    const float* abias; const __nv_bfloat16* w2; int w2p; const float* w0;
    float* wOut; float* bOut;        // [rows][H·dim]
    int rows, H, dim;
};

__global__ void __launch_bounds__(128) k_delta_prepare(const PrepParams p) {
    extern __shared__ float low[];                       // [kPrepRows][w2p], then [kPrepRows] 1 / (Σk² + ε)
    float* inv = low + kPrepRows * p.w2p;
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.x, r0 = blockIdx.y * kPrepRows, n = min(kPrepRows, p.rows - r0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int i = threadIdx.x; i < kPrepRows * p.w2p; i += 128) {
        const int r = i / p.w2p, j = i - r * p.w2p;
        low[i] = (r < n && j < p.rank) ? tanhf(p.proj[(size_t)(r0 + r) * p.ld + p.low_off + j]) : 0.0f;
    }
    for (int r = warp; r < n; r += 4) {
        const float* k = p.proj + (size_t)(r0 + r) * p.ld + p.k_off + h * p.dim;
        float ss = 0.0f;
        for (int i = lane; i < p.dim; i += 32) ss = fmaf(k[i], k[i], ss);
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (lane == 0) inv[r] = 1.0f / (ss + kUnitEps);
    }
    __syncthreads();
    const float rate = expf(-0.5f);
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
                    acc[r] = fmaf(lo, low[r * p.w2p + j + 2 * q], acc[r]);
                    acc[r] = fmaf(hi, low[r * p.w2p + j + 2 * q + 1], acc[r]);
                }
            }
        }
        const float w0 = p.w0[c], ab = p.abias[c];
        for (int r = 0; r < n; r++) {
            const float* row = p.proj + (size_t)(r0 + r) * p.ld;
            const size_t o = (size_t)(r0 + r) * p.H * p.dim + c;
            float a8 = acc[0];
#pragma unroll
            for (int q = 1; q < kPrepRows; q++) a8 = r == q ? acc[q] : a8;
            p.wOut[o] = expf(-rate * sigmoid_f(a8 + w0));
            p.bOut[o] = sigmoid_f(row[p.a_off + c] + ab) * row[p.k_off + c] * inv[r];
        }
    }
}

struct ScanParams {
    PrepParams in;                 // projections, decay weights; wOut / bOut are read here
    int r_off, v_off;
    float* state; const float* pos;
    float* out; int ldo;
    int T, vec;                    // vec: every field can be copied in 16-byte pieces
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

// E key channels per lane (lane·E …), C value columns per warp, TB tokens per stage of the ring.
template <int E, int C, int TB, bool FUSED>
__global__ void __launch_bounds__(128) k_delta_scan(const ScanParams p) {
    constexpr int P = 32 * E, ROW = 4 * P + 4 * C, STAGE = TB * ROW;        // a token: k, r, w, b of the head, v of the block's columns
    extern __shared__ __align__(16) float ring[];                           // [2][TB][ROW]; FUSED: one token, then low [w2p]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.y, b = blockIdx.z, dim = p.in.dim, H = p.in.H, HD = H * dim, hd = h * dim;
    const int cb = blockIdx.x * 4 * C, c0 = cb + warp * C;                  // the block's and this warp's first column
    const size_t row0 = (size_t)b * p.T;
    if (P > dim)                                                            // channels past the head stay zero
        for (int i = tid; i < (FUSED ? 1 : 2 * TB) * 4 * (P - dim); i += 128)
            ring[(i / (4 * (P - dim))) * ROW + (i / (P - dim)) % 4 * P + dim + i % (P - dim)] = 0.0f;
    // the state was last written several kernels ago: it may be read before the dependency wait
    const bool fresh = p.pos[b] == 0.0f;
    float* st = p.state + (((size_t)b * H + h) * dim + c0) * dim;
    float S[C][E];
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = lane * E + e;
            S[c][e] = (!fresh && i < dim && c0 + c < dim) ? st[(size_t)c * dim + i] : 0.0f;
        }
    auto token = [&](const float* row, int t) {
        float k[E], r[E], w[E], q[E], v[C];
#pragma unroll
        for (int e = 0; e < E; e++) { k[e] = row[lane * E + e]; r[e] = row[P + lane * E + e]; w[e] = row[2 * P + lane * E + e]; q[e] = row[3 * P + lane * E + e]; }
#pragma unroll
        for (int c = 0; c < C; c++) v[c] = row[4 * P + warp * C + c];
        float d[C];
#pragma unroll
        for (int c = 0; c < C; c++) {
            d[c] = k[0] * S[c][0];
#pragma unroll
            for (int e = 1; e < E; e++) d[c] = fmaf(k[e], S[c][e], d[c]);
        }
        const float ks = reduce_columns<C>(d, lane);
        float o[C];
#pragma unroll
        for (int c = 0; c < C; c++) {
            const float dot = __shfl_sync(0xffffffffu, ks, c * (32 / C));
            o[c] = 0.0f;
#pragma unroll
            for (int e = 0; e < E; e++) {
                S[c][e] = fmaf(w[e], S[c][e], fmaf(k[e], v[c], -(q[e] * dot)));
                o[c] = fmaf(r[e], S[c][e], o[c]);
            }
        }
        const float os = reduce_columns<C>(o, lane);
        const int col = c0 + lane / (32 / C);
        if (lane % (32 / C) == 0 && col < dim) p.out[(row0 + t) * p.ldo + hd + col] = os;
    };
    if constexpr (FUSED) {
        pdl_wait();
        pdl_launch_dependents();
        float* low = ring + ROW;
        const float* x = p.in.proj + row0 * p.in.ld;
        for (int j = tid; j < p.in.w2p; j += 128) low[j] = j < p.in.rank ? tanhf(x[p.in.low_off + j]) : 0.0f;
        float ss = 0.0f;
        for (int i = lane; i < dim; i += 32) { const float k = x[p.in.k_off + hd + i]; ss = fmaf(k, k, ss); }
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.0f / (ss + kUnitEps), rate = expf(-0.5f);
        __syncthreads();
        for (int i = tid; i < dim; i += 128) {
            const float k = x[p.in.k_off + hd + i];
            ring[i] = k;
            ring[P + i] = x[p.r_off + hd + i];
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
            ring[3 * P + i] = sigmoid_f(x[p.in.a_off + hd + i] + p.in.abias[hd + i]) * k * inv;
        }
        for (int i = tid; i < 4 * C; i += 128) ring[4 * P + i] = cb + i < dim ? x[p.v_off + hd + cb + i] : 0.0f;
        __syncthreads();
        token(ring, 0);
    } else {
        pdl_wait();
        pdl_launch_dependents();
        const int nv = min(4 * C, dim - cb);
        auto load = [&](int t0, int stage) {
            float* dst = ring + stage * STAGE;
            const int n = min(TB, p.T - t0);
            if (p.vec) {
                const int per = dim / 4, all = 4 * per + nv / 4;
                for (int i = tid; i < n * all; i += 128) {
                    const int t = i / all, j = i - t * all;
                    const float* row = p.in.proj + (row0 + t0 + t) * p.in.ld + hd;
                    const size_t wi = (row0 + t0 + t) * HD + hd;
                    float* d = dst + t * ROW;
                    if (j < per) cp_async16(d + 4 * j, row + p.in.k_off + 4 * j);
                    else if (j < 2 * per) cp_async16(d + P + 4 * (j - per), row + p.r_off + 4 * (j - per));
                    else if (j < 3 * per) cp_async16(d + 2 * P + 4 * (j - 2 * per), p.in.wOut + wi + 4 * (j - 2 * per));
                    else if (j < 4 * per) cp_async16(d + 3 * P + 4 * (j - 3 * per), p.in.bOut + wi + 4 * (j - 3 * per));
                    else cp_async16(d + 4 * P + 4 * (j - 4 * per), row + p.v_off + cb + 4 * (j - 4 * per));
                }
            } else {
                const int all = 4 * dim + nv;
                for (int i = tid; i < n * all; i += 128) {
                    const int t = i / all, j = i - t * all;
                    const float* row = p.in.proj + (row0 + t0 + t) * p.in.ld + hd;
                    const size_t wi = (row0 + t0 + t) * HD + hd;
                    float* d = dst + t * ROW;
                    const int f = j / dim, c = j - f * dim;
                    cp_async4(d + f * P + c, f == 0 ? row + p.in.k_off + c : f == 1 ? row + p.r_off + c : f == 2 ? p.in.wOut + wi + c
                                             : f == 3 ? p.in.bOut + wi + c : row + p.v_off + cb + c);
                }
            }
            cp_async_commit();
        };
        load(0, 0);
        for (int t0 = 0, stage = 0; t0 < p.T; t0 += TB, stage ^= 1) {
            cp_async_wait<0>();
            __syncthreads();                       // this stage has landed, nobody reads the other one any more
            if (t0 + TB < p.T) load(t0 + TB, stage ^ 1);
            const int n = min(TB, p.T - t0);
            const float* rows = ring + stage * STAGE;
            if (n == TB) {
#pragma unroll 2
                for (int t = 0; t < TB; t++) token(rows + t * ROW, t0 + t);
            } else {
                for (int t = 0; t < n; t++) token(rows + t * ROW, t0 + t);
            }
        }
    }
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = lane * E + e;
            if (i < dim && c0 + c < dim) st[(size_t)c * dim + i] = S[c][e];
        }
}

template <int E, int TB>
void launch_scan(const ScanParams& p, int B, cudaStream_t s) {
    constexpr int C = 4, ROW = 4 * 32 * E + 4 * C;
    const dim3 grid((unsigned)((p.in.dim + 4 * C - 1) / (4 * C)), (unsigned)p.in.H, (unsigned)B);
    if (p.T == 1) launch_k(k_delta_scan<E, C, TB, true>, grid, dim3(128), (size_t)(ROW + p.in.w2p) * 4, s, true, p);
    else launch_k(k_delta_scan<E, C, TB, false>, grid, dim3(128), (size_t)2 * TB * ROW * 4, s, true, p);
}

}  // namespace

constexpr int kDeltaMaxDim = 256;
bool delta_rule_fits(int dim, int rank) { return dim >= 1 && dim <= kDeltaMaxDim && pad8(rank) * kPrepRows * 4 + 64 <= 48 * 1024; }
size_t delta_rule_ws_floats(int rows, int H, int dim) { return 2 * (size_t)rows * H * dim; }

void launch_delta_rule(const DeltaRuleArgs& a, cudaStream_t s) {
    const int rows = a.B * a.T;
    PrepParams q;
    q.proj = a.proj; q.ld = a.ld; q.k_off = a.k_off; q.a_off = a.a_off; q.low_off = a.low_off; q.rank = a.w2.K;
    q.abias = a.abias; q.w2 = a.w2.w; q.w2p = a.w2.Kp; q.w0 = a.w0;
    q.wOut = a.ws; q.bOut = a.ws + (size_t)rows * a.H * a.dim;
    q.rows = rows; q.H = a.H; q.dim = a.dim;
    if (a.T > 1)
        launch_k(k_delta_prepare, dim3((unsigned)a.H, (unsigned)((rows + kPrepRows - 1) / kPrepRows)), dim3(128), (size_t)kPrepRows * (q.w2p + 1) * 4, s, true, q);
    ScanParams p;
    p.in = q; p.r_off = a.r_off; p.v_off = a.v_off;
    p.state = a.state; p.pos = a.pos; p.out = a.out; p.ldo = a.ldo; p.T = a.T;
    p.vec = ((a.dim | a.ld | a.r_off | a.k_off | a.v_off) & 3) == 0 && (((uintptr_t)a.proj | (uintptr_t)a.ws) & 15) == 0;
    if (a.dim <= 32) launch_scan<1, 8>(p, a.B, s);
    else if (a.dim <= 64) launch_scan<2, 8>(p, a.B, s);
    else if (a.dim <= 96) launch_scan<3, 8>(p, a.B, s);
    else if (a.dim <= 128) launch_scan<4, 8>(p, a.B, s);
    else launch_scan<8, 4>(p, a.B, s);
}

}  // namespace dj
