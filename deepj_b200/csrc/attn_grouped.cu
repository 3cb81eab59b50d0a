// Grouped attention: query head h reads key/value head h / (H/G).  Per head, queries and keys are RMS-normalised; what a
// score is made of besides the product is given by parameters:
//     s_j = (norm(q)·qtab[i] · norm(k_j)) · scale + rel[h][min(i − j, relLen − 1)]        out = Σ_j softmax_j v_j
// with a query factor by position (or none), a bias by distance (or none), and optionally one more score of 0 in the softmax's
// denominator (a sink without a value).  Where the values are the keys as projected, one row per position serves as both: the
// cache holds the projected key and, beside it, 1 / its root mean square; the key's gain goes into the query.
// A layer may read another layer's cache (nothing is appended then).  Scores, softmax and sums are fp32.
//
//   k_grouped_prepare   norms of the new queries and keys, cache append; queries go to the workspace as rows
//                       [sequence][kv head][token · (H/G) + head in the group]
//   k_grouped_attn      fp32 FMA form, any sizes: a warp per such row, tiles of 32 keys in shared memory shared by eight rows
//   k_grouped_merge     adds the partial results of a split key range
// With a bf16 cache the tensor-core kernels of attn_grouped_mma.cu take over where the sizes allow.
#include "row_operand.cuh"

#include <algorithm>
#include <set>

namespace dj {
namespace {

constexpr int kGaKeys = 32, kGaRows = 8, kGaMaxDim = 512;

template <typename T> __device__ __forceinline__ float widen(T v);
template <> __device__ __forceinline__ float widen<float>(float v) { return v; }
template <> __device__ __forceinline__ float widen<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T narrow(float v);
template <> __device__ __forceinline__ float narrow<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 narrow<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// unit: factor of the scores (1, or log2 e where the exponentials are powers of two).
// a warp per head: H query heads, then (when something is appended) G key/value heads; grid (unit groups, tokens of all sequences)
template <typename CT, typename QT>
__global__ void __launch_bounds__(256) k_grouped_prepare(const GroupedAttnArgs a, QT* __restrict__ qp, int qw, float unit) {
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, u = blockIdx.x * 8 + (threadIdx.x >> 5);
    const int row = blockIdx.y, b = row / a.T, t = row - b * a.T, p = (int)a.pos[b] + t, rep = a.H / a.G;
    if (u >= a.H + (a.k_off >= 0 ? a.G : 0) || p < 0 || p >= a.maxSeq) return;
    const bool query = u < a.H, shared = a.vcache == nullptr;
    const float* x = a.proj + (size_t)row * a.ld + (query ? a.q_off + u * a.dim : a.k_off + (u - a.H) * a.dim);
    const float* gain = query ? a.qgamma : a.kgamma;
    constexpr int NE = 4;                                    // values per lane held in registers; longer heads take another round
    float v[NE], w[NE], ss = 0.0f;
#pragma unroll
    for (int e = 0; e < NE; e++) {
        const int i = e * 32 + lane;
        v[e] = 0.0f; w[e] = 0.0f;
        if (i < a.dim) { v[e] = x[i]; w[e] = gain[i]; ss = fmaf(v[e], v[e], ss); }
    }
    for (int i = NE * 32 + lane; i < a.dim; i += 32) ss = fmaf(x[i], x[i], ss);
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = 1.0f / sqrtf(ss / (float)a.dim + a.eps);
    if (query) {
        const int g = u / rep, hh = u - g * rep;
        QT* dst = qp + (((size_t)b * a.G + g) * a.T * rep + (size_t)t * rep + hh) * qw;
        const float f = a.scale * (a.qtab ? a.qtab[p] : 1.0f) * unit;
        auto put = [&](int i, float xv, float wv) {
            float r = (xv * inv) * wv * f;
            if (shared && i < a.dim) r *= a.kgamma[i];
            dst[i] = narrow<QT>(r);
        };
#pragma unroll
        for (int e = 0; e < NE; e++)
            if (e * 32 + lane < qw) put(e * 32 + lane, v[e], w[e]);
        for (int i = NE * 32 + lane; i < qw; i += 32) put(i, i < a.dim ? x[i] : 0.0f, i < a.dim ? gain[i] : 0.0f);
        return;
    }
    const int g = u - a.H;
    const size_t at = ((size_t)b * a.G + g) * a.maxSeq + p;
    CT* k = (CT*)a.kcache + at * a.kw;
    auto put = [&](int i, float xv, float wv) { k[i] = narrow<CT>(shared ? xv : (xv * inv) * wv); };
#pragma unroll
    for (int e = 0; e < NE; e++)
        if (e * 32 + lane < a.dim) put(e * 32 + lane, v[e], w[e]);
    for (int i = NE * 32 + lane; i < a.dim; i += 32) put(i, x[i], gain[i]);
    if (shared) {
        if (lane == 0) a.kscale[((size_t)b * a.G + g) * a.kpitch + p] = inv;
    } else {
        CT* vd = (CT*)a.vcache + at * a.vw;
        const float* src = a.proj + (size_t)row * a.ld + a.v_off + g * a.vdim;
        for (int i = lane; i < a.vdim; i += 32) vd[i] = narrow<CT>(src[i]);
    }
}

// grid (splits, blocks of eight rows, B·G); NV value columns per lane
template <typename CT, int NV>
__global__ void __launch_bounds__(256) k_grouped_attn(const GroupedAttnArgs a, const float* __restrict__ qp, int qw, float* __restrict__ part, int splits) {
    extern __shared__ __align__(16) float sm[];
    const bool shared = a.vcache == nullptr;
    const int LDK = a.dim | 1, LDV = a.vdim | 1;                 // odd pitches: a lane per key reads without conflicts
    float* qs = sm;                                              // [kGaRows][dim]
    float* ks = qs + kGaRows * a.dim;                            // [kGaKeys][LDK]
    float* vs = shared ? ks : ks + kGaKeys * LDK;                // [kGaKeys][LDV]
    float* sc = (shared ? ks + kGaKeys * LDK : vs + kGaKeys * LDV);      // [kGaKeys]
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, rep = a.H / a.G, rows = a.T * rep;
    const int b = blockIdx.z / a.G, g = blockIdx.z - b * a.G, r0 = blockIdx.y * kGaRows, r = r0 + warp, pos0 = (int)a.pos[b];
    const bool on = r < rows;
    const int t = on ? r / rep : 0, h = g * rep + (on ? r - t * rep : 0), my = on ? pos0 + t : -1;       // this row's position
    const int lastPos = pos0 + min(rows - 1, r0 + kGaRows - 1) / rep;
    if (pos0 < 0 || lastPos >= a.maxSeq) return;
    if (on)
        for (int i = lane; i < a.dim; i += 32) qs[warp * a.dim + i] = qp[((size_t)blockIdx.z * rows + r) * qw + i];
    const int tiles = lastPos / kGaKeys + 1, per = (tiles + splits - 1) / splits, tLo = blockIdx.x * per, tHi = min(tiles, tLo + per);
    float acc[NV];
#pragma unroll
    for (int j = 0; j < NV; j++) acc[j] = 0.0f;
    float mx = -INFINITY, l = 0.0f;
    const CT* kc = (const CT*)a.kcache + (size_t)blockIdx.z * a.maxSeq * a.kw;
    const CT* vc = (const CT*)a.vcache + (size_t)blockIdx.z * a.maxSeq * a.vw;
    for (int tile = tLo; tile < tHi; tile++) {
        __syncthreads();
        const int k0 = tile * kGaKeys, n = min(kGaKeys, lastPos + 1 - k0);
        for (int i = threadIdx.x; i < n * a.dim; i += 256) {
            const int j = i / a.dim, d = i - j * a.dim;
            ks[j * LDK + d] = widen<CT>(kc[(size_t)(k0 + j) * a.kw + d]);
        }
        if (shared) {
            if (threadIdx.x < n) sc[threadIdx.x] = a.kscale[(size_t)blockIdx.z * a.kpitch + k0 + threadIdx.x];
        } else {
            for (int i = threadIdx.x; i < n * a.vdim; i += 256) {
                const int j = i / a.vdim, d = i - j * a.vdim;
                vs[j * LDV + d] = widen<CT>(vc[(size_t)(k0 + j) * a.vw + d]);
            }
        }
        __syncthreads();
        const int seen = min(n, my - k0 + 1);                    // keys of this tile that the row sees
        if (seen <= 0) continue;
        float s = -INFINITY;
        if (lane < seen) {
            const float* k = ks + lane * LDK; const float* q = qs + warp * a.dim;
            float s0 = 0.0f, s1 = 0.0f;
            int d = 0;
            for (; d + 1 < a.dim; d += 2) { s0 = fmaf(q[d], k[d], s0); s1 = fmaf(q[d + 1], k[d + 1], s1); }
            if (d < a.dim) s0 = fmaf(q[d], k[d], s0);
            s = s0 + s1;
            if (shared) s *= sc[lane];
            if (a.rel) s += a.rel[(size_t)h * a.relLen + min(my - k0 - lane, a.relLen - 1)];
        }
        float m2 = s;
        for (int o = 16; o > 0; o >>= 1) m2 = fmaxf(m2, __shfl_xor_sync(0xffffffffu, m2, o));
        m2 = fmaxf(m2, mx);
        const float pr = lane < seen ? expf(s - m2) : 0.0f, corr = mx > -INFINITY ? expf(mx - m2) : 0.0f;
        float sum = pr;
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        l = l * corr + sum;
        mx = m2;
#pragma unroll
        for (int j = 0; j < NV; j++) acc[j] *= corr;
        for (int k = 0; k < seen; k++) {
            const float w = __shfl_sync(0xffffffffu, pr, k);
#pragma unroll
            for (int j = 0; j < NV; j++)
                if (j * 32 + lane < a.vdim) acc[j] = fmaf(w, vs[k * LDV + j * 32 + lane], acc[j]);
        }
    }
    if (!on) return;
    if (splits > 1) {
        float* dst = part + (((size_t)blockIdx.z * rows + r) * splits + blockIdx.x) * (a.vdim + 2);
#pragma unroll
        for (int j = 0; j < NV; j++)
            if (j * 32 + lane < a.vdim) dst[j * 32 + lane] = acc[j];
        if (lane == 0) { dst[a.vdim] = mx; dst[a.vdim + 1] = l; }
        return;
    }
    float mult = 1.0f;
    if (a.sink) {
        const float m2 = fmaxf(mx, 0.0f);
        mult = expf(mx - m2);
        l = l * mult + expf(-m2);
    }
    float* o = a.out + (size_t)(b * a.T + t) * a.ldo + h * a.vdim;
#pragma unroll
    for (int j = 0; j < NV; j++)
        if (j * 32 + lane < a.vdim) o[j * 32 + lane] = acc[j] * mult / l;
}

__global__ void __launch_bounds__(128) k_grouped_merge(const GroupedAttnArgs a, const float* __restrict__ part, int splits) {
    pdl_wait();
    pdl_launch_dependents();
    const int rep = a.H / a.G, rows = a.T * rep, r = blockIdx.x, b = blockIdx.y / a.G, g = blockIdx.y - b * a.G, t = r / rep, h = g * rep + r - t * rep;
    if ((int)a.pos[b] < 0 || (int)a.pos[b] + t >= a.maxSeq) return;
    const float* src = part + ((size_t)blockIdx.y * rows + r) * splits * (a.vdim + 2);
    float m = a.sink ? 0.0f : -INFINITY, l = 0.0f;
    for (int s = 0; s < splits; s++)
        if (src[s * (a.vdim + 2) + a.vdim + 1] > 0.0f) m = fmaxf(m, src[s * (a.vdim + 2) + a.vdim]);
    if (a.sink) l = expf(-m);
    for (int s = 0; s < splits; s++)
        if (src[s * (a.vdim + 2) + a.vdim + 1] > 0.0f) l += src[s * (a.vdim + 2) + a.vdim + 1] * expf(src[s * (a.vdim + 2) + a.vdim] - m);
    for (int i = threadIdx.x; i < a.vdim; i += 128) {
        float v = 0.0f;
        for (int s = 0; s < splits; s++)
            if (src[s * (a.vdim + 2) + a.vdim + 1] > 0.0f) v = fmaf(src[s * (a.vdim + 2) + i], expf(src[s * (a.vdim + 2) + a.vdim] - m), v);
        a.out[(size_t)(b * a.T + t) * a.ldo + h * a.vdim + i] = v / l;
    }
}

size_t fma_smem(const GroupedAttnArgs& a) {
    return ((size_t)kGaRows * a.dim + (size_t)kGaKeys * ((a.dim | 1) + (a.vcache ? (a.vdim | 1) : 0)) + kGaKeys) * 4;
}
int fma_splits(const GroupedAttnArgs& a) {
    const int blocks = (a.T * (a.H / a.G) + kGaRows - 1) / kGaRows * a.B * a.G;
    return std::max(1, std::min(2 * g_num_sms / blocks, (a.maxSeq + 63) / 64));
}
size_t query_floats(const GroupedAttnArgs& a) { return ((size_t)a.B * a.T * a.H * ((a.dim + 15) & ~15) + 3) & ~(size_t)3; }

template <typename CT>
void launch_fma(const GroupedAttnArgs& a, const float* q, int qw, float* part, cudaStream_t s) {
    const int splits = fma_splits(a), rows = a.T * (a.H / a.G);
    const dim3 grid((unsigned)splits, (unsigned)((rows + kGaRows - 1) / kGaRows), (unsigned)(a.B * a.G));
    auto go = [&](auto kernel) {
        static std::set<const void*> raised;
        if (raised.insert((const void*)kernel).second) DJ_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        launch_k(kernel, grid, dim3(256), fma_smem(a), s, true, a, q, qw, part, splits);
    };
    if (a.vdim <= 64) go(k_grouped_attn<CT, 2>);
    else if (a.vdim <= 128) go(k_grouped_attn<CT, 4>);
    else if (a.vdim <= 256) go(k_grouped_attn<CT, 8>);
    else go(k_grouped_attn<CT, 16>);
    if (splits > 1) launch_k(k_grouped_merge, dim3((unsigned)rows, (unsigned)(a.B * a.G)), dim3(128), 0, s, true, a, (const float*)part, splits);
}

}  // namespace

const char* grouped_attn_check(const GroupedAttnArgs& a) {
    if (a.H % a.G != 0) return "the key/value heads must divide the query heads";
    if (a.dim > kGaMaxDim || a.vdim > kGaMaxDim) return "head size not supported";
    if ((long)a.B * a.T > 65535 || (long)a.B * a.G > 65535 || (long)a.T * (a.H / a.G) > 65535l * kGaRows) return "too many rows";
    if (a.B * a.G * ((a.H / a.G + 7) / 8) > kAttnTickets) return "too many heads";
    return nullptr;
}

// the queries as rows, then partials
size_t grouped_attn_ws_floats(const GroupedAttnArgs& a) {
    const size_t rows = (size_t)a.B * a.T * a.H;
    if (grouped_mma_fits(a)) return a.T == 1 ? rows * grouped_mma_splits(a) * ((a.vcache ? a.vw : a.kw) + 4) : query_floats(a);
    const int splits = fma_splits(a);
    return query_floats(a) + (splits > 1 ? rows * splits * (a.vdim + 2) : 0);
}

void launch_grouped_attn(const GroupedAttnArgs& a, cudaStream_t s) {
    const bool mma = grouped_mma_fits(a);
    if (mma && a.T == 1) { launch_grouped_decode(a, s); return; }
    const int qw = (a.dim + 15) & ~15;
    const dim3 grid((unsigned)((a.H + (a.k_off >= 0 ? a.G : 0) + 7) / 8), (unsigned)(a.B * a.T));
    if (mma) {
        launch_k(k_grouped_prepare<__nv_bfloat16, __nv_bfloat16>, grid, dim3(256), 0, s, true, a, (__nv_bfloat16*)a.ws, qw, 1.4426950408889634f);
        launch_grouped_prefill(a, (const __nv_bfloat16*)a.ws, qw, s);
        return;
    }
    float* part = a.ws + query_floats(a);
    if (a.bf16) {
        launch_k(k_grouped_prepare<__nv_bfloat16, float>, grid, dim3(256), 0, s, true, a, a.ws, qw, 1.0f);
        launch_fma<__nv_bfloat16>(a, a.ws, qw, part, s);
    } else {
        launch_k(k_grouped_prepare<float, float>, grid, dim3(256), 0, s, true, a, a.ws, qw, 1.0f);
        launch_fma<float>(a, a.ws, qw, part, s);
    }
}

}  // namespace dj
