// Projections with bf16 weights: out = stage(x) · Wᵀ, W [N][Kp] bf16 row-major (Kp = K rounded up to 8, zero padded).
//
// The reference has no such weights (its Q8 format is this library's own as well); checkpoints that ship in bf16 keep
// their exact values this way.  Activations and accumulation are fp32 everywhere except in the many-row tensor-core
// form (bf16_gemm_tc.cu), which rounds the staged operand to bf16.
//
//   k_bf16_gemv       1-16 rows, passes of up to four: HBM-bound, a warp takes four (or two) weight
//                     rows at a time, the first of them in flight before the dependency wait
//   k_bf16_gemm_f32   many rows, fp32 FMA arithmetic (models run in 32-bit)
//   k_bf16_block      block-diagonal: head h's outputs read head h's slice of the row
//   k_stage_rows      the staged operand of the many-row kernels, as fp32 or bf16 rows in the workspace
#include "row_operand.cuh"

#include <algorithm>
#include <set>

namespace dj {
namespace {

constexpr int kGvThreads = 256, kGvWarps = kGvThreads / 32;
constexpr int kGvRows = 4;                       // weight rows per warp of the expert kernel below
constexpr int kGvSmemMax = 200 * 1024;

// Column k of a staged row: blocks of 256 columns, in which the first and the second half of every group of eight sit in
// separate 128-float planes, so that a warp's two 16-byte reads of its groups are free of bank conflicts.
__device__ __forceinline__ int gv_index(int k) { return (k & ~255) + ((k >> 2) & 1) * 128 + ((k >> 3) & 31) * 4 + (k & 3); }

__device__ __forceinline__ float bf_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf_hi(uint32_t u) { return __uint_as_float(u & 0xffff0000u); }
__device__ __forceinline__ uint4 ld_weight(const __nv_bfloat16* p) { return __ldcs(reinterpret_cast<const uint4*>(p)); }

struct GvParams {
    RowOperand a, b;
    const __nv_bfloat16* w; int N, Kp, K1p;      // K1p: first column of segment b
    const float* residual; int ldr;
    float* out; int ldo;
    int gluRow; float limit; float* glu; int ldglu;
    float softcap; const float* bias; int pair;
    // table-routed experts: blockIdx.y is an entry (token row, slot); the weight rows are those of the entry's expert
    const float* tok; const float* table; int top, vocab, expertRows;
};

// MR activation rows; a warp takes ROWS weight rows at a time and keeps DEPTH K-steps of them in flight
template <int MR, int DEPTH, int ROWS>
__global__ void __launch_bounds__(kGvThreads, MR > 1 ? 1 : DEPTH * ROWS <= 8 ? 3 : 2) k_bf16_gemv(const GvParams p) {
    extern __shared__ __align__(16) float xs[];          // [MR][row]
    __shared__ RowScratch sc;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nIt = (p.Kp + 255) / 256, row = nIt * 256;
    const int tasks = (p.N + ROWS - 1) / ROWS, stride = gridDim.x * kGvWarps;
    int task = blockIdx.x * kGvWarps + warp;
    const __nv_bfloat16* w = p.w;

    uint4 buf[DEPTH][ROWS];
    auto fetch = [&](uint4 (&d)[ROWS], int t, int it) {
        const int k = (it * 32 + lane) * 8;
#pragma unroll
        for (int r = 0; r < ROWS; r++) {
            const int n = t * ROWS + r;
            d[r] = make_uint4(0, 0, 0, 0);
            if (n < p.N && k < p.Kp) d[r] = ld_weight(w + (size_t)n * p.Kp + k);
        }
    };
    // step i of a warp's walk over its tasks is (task + (i / nIt)·stride, i % nIt)
    auto begin = [&] {
#pragma unroll
        for (int j = 0; j < DEPTH - 1; j++) {
            const int t = task + j / nIt * stride;
            if (t < tasks) fetch(buf[j], t, j % nIt);
        }
    };
    if (p.table == nullptr) begin();
    pdl_wait();
    pdl_launch_dependents();
    int xrow = blockIdx.y, orow = blockIdx.y;
    if (p.table != nullptr) {
        xrow = blockIdx.y / p.top;
        const int id = min(max((int)p.tok[xrow], 0), p.vocab - 1);
        w += (size_t)(int)p.table[(size_t)id * p.top + (blockIdx.y - xrow * p.top)] * p.expertRows * p.Kp;
        begin();
    }
#pragma unroll 1
    for (int m = 0; m < MR; m++) {
        float* xr = xs + m * row;
        stage_segment(p.a, xrow + m, sc, [&](int k) -> float& { return xr[gv_index(k)]; }, blockIdx.x == 0);
        if (p.b.k > 0) stage_segment(p.b, xrow + m, sc, [&](int k) -> float& { return xr[gv_index(p.K1p + k)]; });
        for (int k = p.a.k + (int)threadIdx.x; k < (p.b.k > 0 ? p.K1p : row); k += kGvThreads) xr[gv_index(k)] = 0.0f;
        if (p.b.k > 0)
            for (int k = p.K1p + p.b.k + (int)threadIdx.x; k < row; k += kGvThreads) xr[gv_index(k)] = 0.0f;
        if (m + 1 < MR) __syncthreads();                 // the scratch is used again
    }
    __syncthreads();

    float acc[MR][ROWS];
    int it = 0, ahead = (DEPTH - 1) % nIt, aheadTask = task + (DEPTH - 1) / nIt * stride;      // the step being multiplied, the step to request
    while (task < tasks) {
#pragma unroll
      for (int slot = 0; slot < DEPTH; slot++) {
        if (it == 0) {
#pragma unroll
            for (int m = 0; m < MR; m++)
#pragma unroll
                for (int r = 0; r < ROWS; r++) acc[m][r] = 0.0f;
        }
        auto multiply = [&](const uint4 (&d)[ROWS], int it) {
#pragma unroll
            for (int m = 0; m < MR; m++) {
                const float* xb = xs + m * row + it * 256 + lane * 4;
                const float4 x0 = *reinterpret_cast<const float4*>(xb), x1 = *reinterpret_cast<const float4*>(xb + 128);
#pragma unroll
                for (int r = 0; r < ROWS; r++) {
                    float s = acc[m][r];
                    s = fmaf(bf_lo(d[r].x), x0.x, s); s = fmaf(bf_hi(d[r].x), x0.y, s);
                    s = fmaf(bf_lo(d[r].y), x0.z, s); s = fmaf(bf_hi(d[r].y), x0.w, s);
                    s = fmaf(bf_lo(d[r].z), x1.x, s); s = fmaf(bf_hi(d[r].z), x1.y, s);
                    s = fmaf(bf_lo(d[r].w), x1.z, s); s = fmaf(bf_hi(d[r].w), x1.w, s);
                    acc[m][r] = s;
                }
            }
        };
        if (aheadTask < tasks) fetch(buf[(slot + DEPTH - 1) % DEPTH], aheadTask, ahead);
        if (++ahead == nIt) { ahead = 0; aheadTask += stride; }
        multiply(buf[slot], it);
        if (++it < nIt) continue;
        it = 0;
        // lane i = r·MR + m ends up with the sum of (weight row r, activation row m)
        float mine = 0.0f;
#pragma unroll
        for (int r = 0; r < ROWS; r++)
#pragma unroll
            for (int m = 0; m < MR; m++) {
                float v = acc[m][r];
                for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                if (lane == r * MR + m) mine = v;
            }
        const float up = __shfl_down_sync(0xffffffffu, mine, MR);
        const int r = lane / MR, m = lane - r * MR, n = task * ROWS + r;
        if (r < ROWS && n < p.N) {
            const int om = orow + m;
            if (n >= p.gluRow) {
                if (((n - p.gluRow) & 1) == 0) p.glu[(size_t)om * p.ldglu + ((n - p.gluRow) >> 1)] = pair_f(mine, up, p.limit, p.pair);
            } else {
                float v = mine;
                if (p.bias) v += p.bias[n];
                if (p.residual) v += p.residual[(size_t)om * p.ldr + n];
                p.out[(size_t)om * p.ldo + n] = softcap_f(v, p.softcap);
            }
        }
        task += stride;
        if (task >= tasks) break;
      }
    }
}

// out[m] (+)= residual[m] + (1/top) Σ_slots W_expert(slot) · y[m·top + slot]
__global__ void __launch_bounds__(kGvThreads, 2) k_bf16_expert_down(const float* __restrict__ y, int ff, const __nv_bfloat16* __restrict__ w0, int N, int Kp,
                                                                    const float* __restrict__ tok, const float* __restrict__ table, int top, int vocab,
                                                                    const float* residual, int ldr, float* out, int ldo) {
    extern __shared__ __align__(16) float xs[];          // [top][row]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, m = blockIdx.y;
    const int nIt = (Kp + 255) / 256, row = nIt * 256;
    pdl_wait();
    pdl_launch_dependents();
    for (int s = 0; s < top; s++)
        for (int k = threadIdx.x; k < row; k += kGvThreads) xs[s * row + gv_index(k)] = k < ff ? y[((size_t)m * top + s) * ff + k] : 0.0f;
    const int id = min(max((int)tok[m], 0), vocab - 1);
    __syncthreads();
    const int tasks = (N + kGvRows - 1) / kGvRows;
    for (int task = blockIdx.x * kGvWarps + warp; task < tasks; task += gridDim.x * kGvWarps) {
        float acc[kGvRows] = {0.0f, 0.0f, 0.0f, 0.0f};
        for (int s = 0; s < top; s++) {
            const __nv_bfloat16* w = w0 + (size_t)(int)table[(size_t)id * top + s] * N * Kp;
#pragma unroll 2
            for (int it = 0; it < nIt; it++) {
                const int k = (it * 32 + lane) * 8;
                const float* xb = xs + s * row + it * 256 + lane * 4;
                const float4 x0 = *reinterpret_cast<const float4*>(xb), x1 = *reinterpret_cast<const float4*>(xb + 128);
                uint4 d[kGvRows];
#pragma unroll
                for (int r = 0; r < kGvRows; r++) {
                    d[r] = make_uint4(0, 0, 0, 0);
                    if (task * kGvRows + r < N && k < Kp) d[r] = ld_weight(w + (size_t)(task * kGvRows + r) * Kp + k);
                }
#pragma unroll
                for (int r = 0; r < kGvRows; r++) {
                    float v = acc[r];
                    v = fmaf(bf_lo(d[r].x), x0.x, v); v = fmaf(bf_hi(d[r].x), x0.y, v);
                    v = fmaf(bf_lo(d[r].y), x0.z, v); v = fmaf(bf_hi(d[r].y), x0.w, v);
                    v = fmaf(bf_lo(d[r].z), x1.x, v); v = fmaf(bf_hi(d[r].z), x1.y, v);
                    v = fmaf(bf_lo(d[r].w), x1.z, v); v = fmaf(bf_hi(d[r].w), x1.w, v);
                    acc[r] = v;
                }
            }
        }
        float mine = 0.0f;
#pragma unroll
        for (int r = 0; r < kGvRows; r++) {
            float v = acc[r];
            for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (lane == r) mine = v;
        }
        const int n = task * kGvRows + lane;
        if (lane < kGvRows && n < N) out[(size_t)m * ldo + n] = (residual ? residual[(size_t)m * ldr + n] : 0.0f) + mine / (float)top;
    }
}

// One row per block: the staged operand as fp32 or bf16.  With a row map, row i of the output holds source row map[i] / div
// (zeros where map[i] < 0).
template <typename OutT>
__global__ void __launch_bounds__(256) k_stage_rows(const RowOperand a, const RowOperand b, int K1p, int Kp, const int* __restrict__ map, int div,
                                                    OutT* __restrict__ out) {
    extern __shared__ __align__(16) float xs[];
    __shared__ RowScratch sc;
    pdl_wait();
    pdl_launch_dependents();
    int m = blockIdx.x;
    OutT* o = out + (size_t)blockIdx.x * Kp;
    if (map != nullptr) {
        m = map[m];
        if (m < 0) {
            for (int k = threadIdx.x; k < Kp; k += 256) o[k] = (OutT)0.0f;
            return;
        }
        m /= div;
    }
    stage_segment(a, m, sc, [&](int k) -> float& { return xs[k]; }, true);
    if (b.k > 0) {
        __syncthreads();
        stage_segment(b, m, sc, [&](int k) -> float& { return xs[K1p + k]; });
    }
    for (int k = a.k + (int)threadIdx.x; k < (b.k > 0 ? K1p : Kp); k += 256) xs[k] = 0.0f;
    if (b.k > 0)
        for (int k = K1p + b.k + (int)threadIdx.x; k < Kp; k += 256) xs[k] = 0.0f;
    __syncthreads();
    for (int k = (int)threadIdx.x * 2; k < Kp; k += 512) {       // Kp is even
        if constexpr (sizeof(OutT) == 2) *reinterpret_cast<__nv_bfloat162*>(o + k) = __floats2bfloat162_rn(xs[k], xs[k + 1]);
        else *reinterpret_cast<float2*>(o + k) = make_float2(xs[k], xs[k + 1]);
    }
}

// out[m] = base[m] + mult · norm(x[m])·gamma, one row per block; out may be base
__global__ void __launch_bounds__(256) k_norm_add(const RowOperand x, float* out, int ldo) {
    extern __shared__ __align__(16) float xs[];
    __shared__ RowScratch sc;
    pdl_wait();
    pdl_launch_dependents();
    stage_segment(x, blockIdx.x, sc, [&](int k) -> float& { return xs[k]; });
    __syncthreads();
    for (int k = threadIdx.x; k < x.k; k += 256) out[(size_t)blockIdx.x * ldo + k] = xs[k];
}

// out[M × N] = A[M][Kp] (fp32) · W[N][Kp]ᵀ in fp32 FMAs: 64 × 64 tiles, 4 × 4 outputs per thread.
struct F32GemmParams {
    const float* a; const __nv_bfloat16* w; int M, N, Kp;
    const float* residual; int ldr; float* out; int ldo; int gluRow; float limit; float* glu; int ldglu; float softcap;
    const float* bias; int pair;
};
__global__ void __launch_bounds__(256) k_bf16_gemm_f32(const F32GemmParams p) {
    __shared__ float As[16][68], Ws[16][68];
    pdl_wait();
    pdl_launch_dependents();
    const int tid = threadIdx.x, m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    const int tm = (tid >> 4) * 4, tn = (tid & 15) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.Kp; k0 += 16) {
        for (int i = tid; i < 1024; i += 256) {
            const int r = i >> 4, k = i & 15;
            As[k][r] = (m0 + r < p.M && k0 + k < p.Kp) ? p.a[(size_t)(m0 + r) * p.Kp + k0 + k] : 0.0f;
            Ws[k][r] = (n0 + r < p.N && k0 + k < p.Kp) ? __bfloat162float(p.w[(size_t)(n0 + r) * p.Kp + k0 + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; k++) {
            const float4 av = *reinterpret_cast<const float4*>(&As[k][tm]), wv = *reinterpret_cast<const float4*>(&Ws[k][tn]);
            const float a[4] = {av.x, av.y, av.z, av.w}, w[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int m = m0 + tm + i;
        if (m >= p.M) continue;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + tn + j;
            if (n >= p.N) continue;
            if (n >= p.gluRow) {                         // gluRow is even and so is tn: a pair never leaves the thread
                if (((n - p.gluRow) & 1) == 0 && j < 3) p.glu[(size_t)m * p.ldglu + ((n - p.gluRow) >> 1)] = pair_f(acc[i][j], acc[i][j + 1], p.limit, p.pair);
            } else {
                float v = acc[i][j];
                if (p.bias) v += p.bias[n];
                if (p.residual) v += p.residual[(size_t)m * p.ldr + n];
                p.out[(size_t)m * p.ldo + n] = softcap_f(v, p.softcap);
            }
        }
    }
}

// Block-diagonal projection: out[m][h·os + n] = W[h·Nb + n] · x[m][h·xs …].  grid (heads, row tiles, groups of MR rows);
// few rows take one weight row per lane group and block, its first chunk in flight before the dependency wait.
template <int MR>
__global__ void __launch_bounds__(256) k_bf16_block(const float* __restrict__ x, int ldx, int xstr, const __nv_bfloat16* __restrict__ w, int K, int Kp, int Nb,
                                                    float* __restrict__ out, int ldo, int ostr, int M, int tile) {
    extern __shared__ __align__(16) float xs[];          // [MR][Kp]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int h = blockIdx.x, m0 = blockIdx.z * MR;
    const int chunks = Kp / 8;
    int lpr = 1;
    while (lpr < 32 && lpr < chunks) lpr <<= 1;          // lanes per weight row
    const int rpw = 32 / lpr, sub = lane / lpr, l = lane - sub * lpr;
    const int hi = min(Nb, ((int)blockIdx.y + 1) * tile);
    uint4 first = make_uint4(0, 0, 0, 0);
    {
        const int n = blockIdx.y * tile + warp * rpw + sub;
        if (n < hi && l < chunks) first = __ldg(reinterpret_cast<const uint4*>(w + ((size_t)h * Nb + n) * Kp + l * 8));
    }
    pdl_wait();
    pdl_launch_dependents();
#pragma unroll
    for (int m = 0; m < MR; m++)
        for (int k = threadIdx.x; k < Kp; k += 256) xs[m * Kp + k] = (k < K && m0 + m < M) ? x[(size_t)(m0 + m) * ldx + (size_t)h * xstr + k] : 0.0f;
    __syncthreads();
    for (int base = blockIdx.y * tile + warp * rpw; base < hi; base += 8 * rpw) {
        const int n = base + sub;
        float acc[MR];
#pragma unroll
        for (int m = 0; m < MR; m++) acc[m] = 0.0f;
        if (n < hi) {
            const __nv_bfloat16* wr = w + ((size_t)h * Nb + n) * Kp;
            for (int c = l; c < chunks; c += lpr) {
                const uint4 d = c == l && base == (int)blockIdx.y * tile + warp * rpw ? first : __ldg(reinterpret_cast<const uint4*>(wr + c * 8));
#pragma unroll
                for (int m = 0; m < MR; m++) {
                    const float4 x0 = *reinterpret_cast<const float4*>(xs + m * Kp + c * 8), x1 = *reinterpret_cast<const float4*>(xs + m * Kp + c * 8 + 4);
                    float v = acc[m];
                    v = fmaf(bf_lo(d.x), x0.x, v); v = fmaf(bf_hi(d.x), x0.y, v);
                    v = fmaf(bf_lo(d.y), x0.z, v); v = fmaf(bf_hi(d.y), x0.w, v);
                    v = fmaf(bf_lo(d.z), x1.x, v); v = fmaf(bf_hi(d.z), x1.y, v);
                    v = fmaf(bf_lo(d.w), x1.z, v); v = fmaf(bf_hi(d.w), x1.w, v);
                    acc[m] = v;
                }
            }
        }
#pragma unroll
        for (int m = 0; m < MR; m++) {
            for (int o = lpr >> 1; o > 0; o >>= 1) acc[m] += __shfl_xor_sync(0xffffffffu, acc[m], o);
            if (l == 0 && n < hi && m0 + m < M) out[(size_t)(m0 + m) * ldo + (size_t)h * ostr + n] = acc[m];
        }
    }
}

__global__ void __launch_bounds__(256) k_bf16_store(const float* __restrict__ src, int rows, int cols, __nv_bfloat16* __restrict__ dst, long long dst_ld) {
    const long long total = (long long)rows * cols;
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < total; i += (long long)gridDim.x * 256)
        dst[(i / cols) * dst_ld + i % cols] = __float2bfloat16_rn(src[i]);
}

void raise_smem(const void* kernel, size_t bytes) {
    static std::set<const void*> done;
    if (bytes > 40 * 1024 && done.insert(kernel).second)
        DJ_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kGvSmemMax));
}

template <int MR, int DEPTH, int ROWS>
void launch_gv(GvParams p, int m0, unsigned gy, cudaStream_t s) {
    p.a.x += (size_t)m0 * p.a.ldx;
    if (p.a.gate) p.a.gate += (size_t)m0 * p.a.ldg;
    if (p.a.base) p.a.base += (size_t)m0 * p.a.ldbase;
    if (p.a.sum) p.a.sum += (size_t)m0 * p.a.ldsum;
    if (p.b.k > 0) {
        p.b.x += (size_t)m0 * p.b.ldx;
        if (p.b.gate) p.b.gate += (size_t)m0 * p.b.ldg;
    }
    if (p.residual) p.residual += (size_t)m0 * p.ldr;
    if (p.out) p.out += (size_t)m0 * p.ldo;
    if (p.glu) p.glu += (size_t)m0 * p.ldglu;
    const int tiles = (p.N + ROWS * kGvWarps - 1) / (ROWS * kGvWarps);
    const int cap = 2 * g_num_sms;
    const int rounds = (tiles + cap - 1) / cap, gx = (tiles + rounds - 1) / rounds;
    const size_t smem = (size_t)MR * ((p.Kp + 255) / 256) * 1024;
    raise_smem((const void*)k_bf16_gemv<MR, DEPTH, ROWS>, smem);
    launch_k(k_bf16_gemv<MR, DEPTH, ROWS>, dim3((unsigned)gx, gy), dim3(kGvThreads), smem, s, true, p);
}

}  // namespace

void launch_bf16_store(const float* src, int rows, int cols, __nv_bfloat16* dst, long long dst_ld, cudaStream_t s) {
    if (rows <= 0 || cols <= 0) return;
    launch_k(k_bf16_store, dim3((unsigned)std::min<long long>(((long long)rows * cols + 255) / 256, 16ll * g_num_sms)), dim3(256), 0, s, false, src, rows, cols, dst,
             dst_ld);
}

void launch_stage_rows(const RowOperand& a, const RowOperand& b, int Kp, int rows, const int* map, int div, void* out, bool bf16, cudaStream_t s) {
    const int K1p = pad8(a.k);
    const size_t smem = (size_t)Kp * 4;
    if (bf16) {
        raise_smem((const void*)k_stage_rows<__nv_bfloat16>, smem);
        launch_k(k_stage_rows<__nv_bfloat16>, dim3((unsigned)rows), dim3(256), smem, s, true, a, b, K1p, Kp, map, div, (__nv_bfloat16*)out);
    } else {
        raise_smem((const void*)k_stage_rows<float>, smem);
        launch_k(k_stage_rows<float>, dim3((unsigned)rows), dim3(256), smem, s, true, a, b, K1p, Kp, map, div, (float*)out);
    }
}

void launch_norm_add(const RowOperand& x, float* out, int ldo, int rows, cudaStream_t s) {
    const size_t smem = (size_t)pad8(x.k) * 4;
    raise_smem((const void*)k_norm_add, smem);
    launch_k(k_norm_add, dim3((unsigned)rows), dim3(256), smem, s, true, x, out, ldo);
}

constexpr int kGvMaxM = 16;      // up to here passes of the GEMV

size_t bf16_linear_ws_floats(const Bf16LinearArgs& a) {
    return a.M <= kGvMaxM ? 0 : (size_t)a.M * a.w.Kp;
}

const char* bf16_linear_check(const Bf16LinearArgs& a) {
    if ((size_t)a.w.Kp * 4 > (size_t)kGvSmemMax - 1024) return "reduction length too large";
    if (a.a.groups > kMaxNormGroups || a.b.groups > kMaxNormGroups) return "too many norm groups";
    if ((a.a.groups > 0 && a.a.k % a.a.groups != 0) || (a.b.groups > 0 && a.b.k % a.b.groups != 0)) return "norm groups must divide the row";
    return nullptr;
}

void launch_bf16_linear(const Bf16LinearArgs& a, cudaStream_t s) {
    if (a.M <= 0 || a.w.N <= 0) return;
    if (a.M <= kGvMaxM) {
        GvParams p = {};
        p.a = a.a; p.b = a.b; p.w = a.w.w; p.N = a.w.N; p.Kp = a.w.Kp; p.K1p = pad8(a.a.k);
        p.residual = a.residual; p.ldr = a.ldr; p.out = a.out; p.ldo = a.ldo;
        p.gluRow = a.gluRow; p.limit = a.limit; p.glu = a.glu; p.ldglu = a.ldglu; p.softcap = a.softcap; p.bias = a.bias; p.pair = a.pair;
        const size_t perRow = (size_t)((a.w.Kp + 255) / 256) * 1024;
        for (int m0 = 0; m0 < a.M;) {
            int rows = std::min(4, a.M - m0);
            if (rows == 3) rows = 2;
            while (rows > 1 && rows * perRow > (size_t)kGvSmemMax) rows >>= 1;
            // fewer blocks than the SMs hold at a time: two weight rows per warp, twice the blocks
            const bool narrow = (a.w.N + 4 * kGvWarps - 1) / (4 * kGvWarps) <= g_num_sms;
            if (rows == 4) launch_gv<4, 2, 4>(p, m0, 1, s);
            else if (rows == 2) { if (narrow) launch_gv<2, 6, 2>(p, m0, 1, s); else launch_gv<2, 4, 4>(p, m0, 1, s); }
            else if (narrow) launch_gv<1, 8, 2>(p, m0, 1, s);
            else launch_gv<1, 4, 4>(p, m0, 1, s);
            m0 += rows;
        }
        return;
    }
    if (!a.exact && launch_bf16_gemm_tc(a, nullptr, s)) return;
    launch_stage_rows(a.a, a.b, a.w.Kp, a.M, nullptr, 1, a.ws, false, s);
    F32GemmParams p = {a.ws, a.w.w, a.M, a.w.N, a.w.Kp, a.residual, a.ldr, a.out, a.ldo, a.gluRow, a.limit, a.glu, a.ldglu, a.softcap,
                       a.bias, a.pair};
    launch_k(k_bf16_gemm_f32, dim3((a.w.N + 63) / 64, (a.M + 63) / 64), dim3(256), 0, s, true, p);
}

void launch_bf16_block_linear(const float* x, int ldx, int xstr, const Bf16View& w, int heads, float* out, int ldo, int ostr, int M, cudaStream_t s) {
    const int Nb = w.N / heads;
    const dim3 block(256);
    int lpr = 1;
    while (lpr < 32 && lpr < w.Kp / 8) lpr <<= 1;
    const int tile = M <= 4 ? 8 * (32 / lpr) : 64;
    const unsigned tiles = (unsigned)((Nb + tile - 1) / tile);
    auto go = [&](auto kernel, int MR) {
        const size_t smem = (size_t)MR * w.Kp * 4;
        raise_smem((const void*)kernel, smem);
        launch_k(kernel, dim3((unsigned)heads, tiles, (unsigned)((M + MR - 1) / MR)), block, smem, s, true, x, ldx, xstr, w.w, w.K, w.Kp, Nb, out, ldo, ostr, M, tile);
    };
    if (M == 1) go(k_bf16_block<1>, 1);
    else go(k_bf16_block<4>, 4);
}

void launch_bf16_expert_gemv(const Bf16ExpertArgs& e, float* y, cudaStream_t s) {
    GvParams p = {};
    p.a = e.x; p.w = e.up.w; p.N = 2 * e.ff; p.Kp = e.up.Kp; p.K1p = pad8(e.x.k);
    p.gluRow = 0; p.limit = e.limit; p.glu = y; p.ldglu = e.ff;
    p.tok = e.tok; p.table = e.table; p.top = e.top; p.vocab = e.vocab; p.expertRows = 2 * e.ff;
    launch_gv<1, 2, 4>(p, 0, (unsigned)(e.M * e.top), s);       // shallow: more blocks per SM, the entries are many and small
    const int row = (e.down.Kp + 255) / 256 * 256, tiles = (e.d + kGvRows * kGvWarps - 1) / (kGvRows * kGvWarps);
    const size_t smem = (size_t)e.top * row * 4;
    raise_smem((const void*)k_bf16_expert_down, smem);
    launch_k(k_bf16_expert_down, dim3((unsigned)tiles, (unsigned)e.M), dim3(kGvThreads), smem, s, true, (const float*)y, e.ff, e.down.w, e.d, e.down.Kp,
             e.tok, e.table, e.top, e.vocab, e.residual, e.ldr, e.out, e.ldo);
}

}  // namespace dj
