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
//   k_delta_scan      one warp per (sequence, head, few value columns): a lane holds the key channels lane, lane + 32, …
//                     of its columns in registers; u·S and o are warp reductions, the next token's vectors are in flight
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
    const float* proj; int ld, r_off, k_off, v_off;
    const float* w; const float* b;
    float* state; const float* pos;
    float* out; int ldo;
    int T, H, dim;
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

// E key channels per lane, C value columns per warp.
template <int E, int C>
__global__ void __launch_bounds__(128) k_delta_scan(const ScanParams p) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int h = blockIdx.y, b = blockIdx.z, dim = p.dim;
    const int c0 = (blockIdx.x * 4 + warp) * C;
    if (c0 >= dim) return;
    const bool fresh = p.pos[b] == 0.0f;
    float* st = p.state + (((size_t)b * p.H + h) * dim + c0) * dim;
    float S[C][E];
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = e * 32 + lane;
            S[c][e] = (!fresh && i < dim && c0 + c < dim) ? st[(size_t)c * dim + i] : 0.0f;
        }
    const size_t row0 = (size_t)b * p.T;
    const int hd = h * dim, HD = p.H * dim;
    float k[E], w[E], q[E], r[E], v;
    auto load = [&](int t, float (&k)[E], float (&w)[E], float (&q)[E], float (&r)[E], float& v) {
        const float* row = p.proj + (row0 + t) * p.ld + hd;
        const size_t wi = (row0 + t) * HD + hd;
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = e * 32 + lane;
            const bool on = i < dim;
            k[e] = on ? row[p.k_off + i] : 0.0f;
            r[e] = on ? row[p.r_off + i] : 0.0f;
            w[e] = on ? p.w[wi + i] : 0.0f;
            q[e] = on ? p.b[wi + i] : 0.0f;
        }
        v = (lane < C && c0 + lane < dim) ? row[p.v_off + c0 + lane] : 0.0f;
    };
    load(0, k, w, q, r, v);
    for (int t = 0; t < p.T; t++) {
        float k2[E], w2[E], q2[E], r2[E], v2;
        if (t + 1 < p.T) load(t + 1, k2, w2, q2, r2, v2);
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
            const float dot = __shfl_sync(0xffffffffu, ks, c * (32 / C)), vc = __shfl_sync(0xffffffffu, v, c);
            o[c] = 0.0f;
#pragma unroll
            for (int e = 0; e < E; e++) {
                S[c][e] = fmaf(w[e], S[c][e], fmaf(k[e], vc, -(q[e] * dot)));
                o[c] = fmaf(r[e], S[c][e], o[c]);
            }
        }
        const float os = reduce_columns<C>(o, lane);
        const int col = c0 + lane / (32 / C);
        if (lane % (32 / C) == 0 && col < dim) p.out[(row0 + t) * p.ldo + hd + col] = os;
        if (t + 1 < p.T) {
#pragma unroll
            for (int e = 0; e < E; e++) { k[e] = k2[e]; w[e] = w2[e]; q[e] = q2[e]; r[e] = r2[e]; }
            v = v2;
        }
    }
#pragma unroll
    for (int c = 0; c < C; c++)
#pragma unroll
        for (int e = 0; e < E; e++) {
            const int i = e * 32 + lane;
            if (i < dim && c0 + c < dim) st[(size_t)c * dim + i] = S[c][e];
        }
}

template <int E>
void launch_scan(const ScanParams& p, int B, cudaStream_t s) {
    constexpr int C = 4;
    launch_k(k_delta_scan<E, C>, dim3((unsigned)((p.dim + 4 * C - 1) / (4 * C)), (unsigned)p.H, (unsigned)B), dim3(128), 0, s, true, p);
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
    launch_k(k_delta_prepare, dim3((unsigned)a.H, (unsigned)((rows + kPrepRows - 1) / kPrepRows)), dim3(128), (size_t)kPrepRows * (q.w2p + 1) * 4, s, true, q);
    ScanParams p;
    p.proj = a.proj; p.ld = a.ld; p.r_off = a.r_off; p.k_off = a.k_off; p.v_off = a.v_off;
    p.w = q.wOut; p.b = q.bOut; p.state = a.state; p.pos = a.pos; p.out = a.out; p.ldo = a.ldo;
    p.T = a.T; p.H = a.H; p.dim = a.dim;
    if (a.dim <= 32) launch_scan<1>(p, a.B, s);
    else if (a.dim <= 64) launch_scan<2>(p, a.B, s);
    else if (a.dim <= 96) launch_scan<3>(p, a.B, s);
    else if (a.dim <= 128) launch_scan<4>(p, a.B, s);
    else launch_scan<8>(p, a.B, s);
}

}  // namespace dj
