// Latent attention on the tensor cores (bf16 cache).
//
//   k_latent_mma      few tokens: scores and sums in the latent space.  A block takes 32 (token, head) rows — all heads share
//                     the cached rows — and walks its part of the keys in tiles of 64, streamed with cp.async into two
//                     stages.  Eight warps split a tile's keys for Q·Kᵀ and the latent columns for P·V.  A single token
//                     (decode) appends its own row: no append launch, and the older rows are fetched before the dependency wait.
//   k_latent_prefill  prompt chunks: keys and values of the whole context are expanded per head by two projections (bf16,
//                     in the workspace), then 128 query rows per block, 16 per warp, key tiles of 64 in two stages; the
//                     rotated key part is read from the cache.  Per (query, key) pair this costs dim + rot + vdim products
//                     instead of 2·kv_rank + rot.
// Queries, keys and values are bf16 operands with fp32 accumulation; softmax is fp32 and its weights enter the second
// product as two bf16 halves (16 bits).
#include "mma_common.cuh"
#include "row_operand.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr float kLog2e = 1.4426950408889634f;

struct LmParams {
    const float* q; int ldq, dim;
    const float* qc; int ldqc;
    const __nv_bfloat16* cache; int maxSeq, W;
    const float* pos; const float* cosT; const float* sinT;
    float* out; int ldo;
    int T, H, R, rot; float scale;
    float* part; int splits;
    int Wp;                                        // shared-memory columns per row
    // T == 1: the kernel appends the new row itself (norm, rotation, cache write); otherwise kv is null
    const float* kv; int ldkv; const float* gamma; float eps; __nv_bfloat16* append;
    int early;                                     // … and may read positions and older rows before the dependency wait
};

constexpr int kLmRows = 32, kLmKeys = 64, kLmP = kLmKeys + 8;

size_t lm_smem(int Wp) { return (size_t)(kLmRows + 2 * kLmKeys + 1) * (Wp + 8) * 2 + (size_t)2 * kLmRows * kLmP * 2 + (4 * kLmRows + kLmRows) * 4; }

// NT: output n-tiles (eight latent columns each) per warp
template <int NT>
__global__ void __launch_bounds__(256, 1) k_latent_mma(const LmParams p) {
    extern __shared__ __align__(16) unsigned char lm_raw[];
    const int LD = p.Wp + 8;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(lm_raw);        // [32][LD]
    __nv_bfloat16* Ks = Qs + kLmRows * LD;                               // [2][64][LD]
    __nv_bfloat16* Ph = Ks + 2 * kLmKeys * LD;                           // [32][kLmP], then the low halves
    __nv_bfloat16* s_new = Ph + 2 * kLmRows * kLmP;                      // the appended row
    float* s_max = reinterpret_cast<float*>(s_new + LD);                 // [4][32]
    float* s_corr = s_max + 4 * kLmRows;                                 // [32]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    const int b = blockIdx.z, r0 = blockIdx.y * kLmRows, rows = p.T * p.H;
    const __nv_bfloat16* cache = p.cache + (size_t)b * p.maxSeq * p.W;
    // columns past the cached row stay zero
    for (int i = tid; i < 2 * kLmKeys * (LD - p.W); i += 256) Ks[(i / (LD - p.W)) * LD + p.W + i % (LD - p.W)] = __float2bfloat16_rn(0.0f);
    if (p.kv == nullptr || !p.early) { pdl_wait(); pdl_launch_dependents(); }
    const int pos0 = max((int)p.pos[b], 0);
    const int lastKey = min(p.maxSeq - 1, pos0 + min(rows - 1, r0 + kLmRows - 1) / p.H);
    const int tiles = lastKey / kLmKeys + 1, per = (tiles + p.splits - 1) / p.splits;
    const int tLo = blockIdx.x * per, tHi = min(tiles, tLo + per);
    const int chunks = p.W / 8;
    auto load_tile = [&](int tile, int stage) {
        __nv_bfloat16* dst = Ks + stage * kLmKeys * LD;
#pragma unroll 4
        for (int key = warp; key < kLmKeys; key += 8) {
            const __nv_bfloat16* src = cache + (size_t)min(tile * kLmKeys + key, p.maxSeq - 1) * p.W;
            for (int c = lane; c < chunks; c += 32) cp_async16(dst + key * LD + c * 8, src + c * 8);
        }
        cp_async_commit();
    };
    if (tLo < tHi) load_tile(tLo, 0);
    int newTile = -1;                                            // the tile that holds the row this block appends
    if (p.kv != nullptr) {
        pdl_wait();
        pdl_launch_dependents();
        if (pos0 < p.maxSeq && pos0 / kLmKeys >= tLo && pos0 / kLmKeys < tHi) newTile = pos0 / kLmKeys;
    }
    if (newTile >= 0) {
        const float* x = p.kv + (size_t)b * p.ldkv;
        __nv_bfloat16* dst = blockIdx.y == 0 ? p.append + ((size_t)b * p.maxSeq + pos0) * p.W : nullptr;
        float ss = 0.0f;
        for (int i = tid; i < p.R; i += 256) ss = fmaf(x[i], x[i], ss);
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (lane == 0) s_max[warp] = ss;
        __syncthreads();
        ss = 0.0f;
        for (int w = 0; w < 8; w++) ss += s_max[w];
        const float inv = 1.0f / sqrtf(ss / (float)p.R + p.eps);
        for (int i = tid; i < p.R; i += 256) {
            const __nv_bfloat16 v = __float2bfloat16_rn((x[i] * inv) * p.gamma[i]);
            s_new[i] = v;
            if (dst) dst[i] = v;
        }
        for (int i = tid; i < p.rot / 2; i += 256) {
            const float c = p.cosT[(size_t)pos0 * (p.rot / 2) + i], s = p.sinT[(size_t)pos0 * (p.rot / 2) + i], u = x[p.R + 2 * i], v = x[p.R + 2 * i + 1];
            const __nv_bfloat16 a = __float2bfloat16_rn(u * c - v * s), e = __float2bfloat16_rn(v * c + u * s);
            s_new[p.R + 2 * i] = a; s_new[p.R + 2 * i + 1] = e;
            if (dst) { dst[p.R + 2 * i] = a; dst[p.R + 2 * i + 1] = e; }
        }
    }
    const int half = p.rot / 2;
#pragma unroll
    for (int j = 0; j < kLmRows / 8; j++) {                      // query rows, four per warp: latent part, rotated part, zeros
        const int r = warp + 8 * j, row = r0 + r, t = row / p.H, h = row - t * p.H;
        const size_t m = (size_t)b * p.T + t;
        const bool on = row < rows;
        const float* qc = p.qc + m * p.ldqc + (size_t)h * p.R;
#pragma unroll 8
        for (int c = 2 * lane; c < p.R; c += 64)
            *reinterpret_cast<uint32_t*>(Qs + r * LD + c) = on ? pack_bf16(qc[c], qc[c + 1]) : 0u;
        const float* qr = p.q + m * p.ldq + (size_t)h * (p.dim + p.rot) + p.dim;
        const size_t at = (size_t)min(pos0 + t, p.maxSeq - 1) * half;
        for (int i = lane; i < half; i += 32) {
            float a = 0.0f, v = 0.0f;
            if (on) {
                const float co = p.cosT[at + i], si = p.sinT[at + i], x = qr[2 * i], y = qr[2 * i + 1];
                a = x * co - y * si;
                v = y * co + x * si;
            }
            *reinterpret_cast<uint32_t*>(Qs + r * LD + p.R + 2 * i) = pack_bf16(a, v);
        }
        for (int c = p.W + 2 * lane; c < LD; c += 64) *reinterpret_cast<uint32_t*>(Qs + r * LD + c) = 0u;
    }
    const int mt = warp & 1, ng = warp >> 1;                     // Q·Kᵀ: 16 rows × 16 keys per warp
    const int row0 = r0 + mt * 16 + g, row1 = row0 + 8;
    const int lim0 = row0 < rows ? pos0 + row0 / p.H : -1, lim1 = row1 < rows ? pos0 + row1 / p.H : -1;
    const uint32_t qAddr = smem_u32(Qs) + (uint32_t)(((mt * 16 + (lane & 15)) * LD + (lane >> 4) * 8) * 2);
    const uint32_t kAddr = smem_u32(Ks) + (uint32_t)(((ng * 16 + (lane & 7) + ((lane >> 4) << 3)) * LD + ((lane >> 3) & 1) * 8) * 2);
    const uint32_t vAddr = smem_u32(Ks) + (uint32_t)((((lane & 7) + (((lane >> 3) & 1) << 3)) * LD + warp * NT * 8 + (lane >> 4) * 8) * 2);
    const uint32_t pAddr = smem_u32(Ph) + (uint32_t)(((lane & 15) * kLmP + (lane >> 4) * 8) * 2);
    const uint32_t stageBytes = (uint32_t)(kLmKeys * LD * 2), lowBytes = (uint32_t)(kLmRows * kLmP * 2);
    const int kSteps = (p.W + 15) / 16;
    const float sc = p.scale * kLog2e;

    float o[2][NT][4];
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
        for (int j = 0; j < NT; j++) { o[m][j][0] = 0.0f; o[m][j][1] = 0.0f; o[m][j][2] = 0.0f; o[m][j][3] = 0.0f; }
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    for (int tile = tLo; tile < tHi; tile++) {
        const int st = (tile - tLo) & 1;
        cp_async_wait<0>();
        __syncthreads();                                         // the tile is there; the other stage and P are free
        if (tile == newTile) {
            for (int c = tid; c < p.W; c += 256) Ks[(st * kLmKeys + pos0 % kLmKeys) * LD + c] = s_new[c];
            __syncthreads();
        }
        if (tile + 1 < tHi) load_tile(tile + 1, st ^ 1);
        float s[2][4] = {};
#pragma unroll 4
        for (int kk = 0; kk < kSteps; kk++) {
            uint32_t a[4], bq[4];
            ldm_x4(a, qAddr + kk * 32);
            ldm_x4(bq, kAddr + st * stageBytes + kk * 32);
            mma_bf16(s[0], a, bq[0], bq[1]);
            mma_bf16(s[1], a, bq[2], bq[3]);
        }
        float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int key = tile * kLmKeys + ng * 16 + j * 8 + 2 * t4 + e;
                s[j][e] = key <= lim0 ? s[j][e] * sc : -INFINITY;
                s[j][2 + e] = key <= lim1 ? s[j][2 + e] * sc : -INFINITY;
                x0 = fmaxf(x0, s[j][e]); x1 = fmaxf(x1, s[j][2 + e]);
            }
        x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
        x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
        if (t4 == 0) { s_max[ng * kLmRows + mt * 16 + g] = x0; s_max[ng * kLmRows + mt * 16 + g + 8] = x1; }
        __syncthreads();
        float n0 = m0, n1 = m1;
#pragma unroll
        for (int j = 0; j < 4; j++) { n0 = fmaxf(n0, s_max[j * kLmRows + mt * 16 + g]); n1 = fmaxf(n1, s_max[j * kLmRows + mt * 16 + g + 8]); }
        const float c0 = m0 > -INFINITY ? exp2f(m0 - n0) : 1.0f, c1 = m1 > -INFINITY ? exp2f(m1 - n1) : 1.0f;
        float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
        for (int j = 0; j < 2; j++) {
#pragma unroll
            for (int e = 0; e < 2; e++) {
                s[j][e] = s[j][e] > -INFINITY ? exp2f(s[j][e] - n0) : 0.0f;
                s[j][2 + e] = s[j][2 + e] > -INFINITY ? exp2f(s[j][2 + e] - n1) : 0.0f;
                a0 += s[j][e]; a1 += s[j][2 + e];
            }
            uint32_t hi, lo;
            __nv_bfloat16* dst = Ph + (mt * 16 + g) * kLmP + ng * 16 + j * 8 + 2 * t4;
            split_bf16(s[j][0], s[j][1], hi, lo);
            *reinterpret_cast<uint32_t*>(dst) = hi; *reinterpret_cast<uint32_t*>(dst + kLmRows * kLmP) = lo;
            split_bf16(s[j][2], s[j][3], hi, lo);
            *reinterpret_cast<uint32_t*>(dst + 8 * kLmP) = hi; *reinterpret_cast<uint32_t*>(dst + 8 * kLmP + kLmRows * kLmP) = lo;
        }
        l0 = l0 * c0 + a0; l1 = l1 * c1 + a1;                    // this lane's keys only
        m0 = n0; m1 = n1;
        if (ng == 0 && t4 == 0) { s_corr[mt * 16 + g] = c0; s_corr[mt * 16 + g + 8] = c1; }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < 2; m++) {
            const float f0 = s_corr[m * 16 + g], f1 = s_corr[m * 16 + g + 8];
            if (f0 != 1.0f || f1 != 1.0f) {
#pragma unroll
                for (int j = 0; j < NT; j++) { o[m][j][0] *= f0; o[m][j][1] *= f0; o[m][j][2] *= f1; o[m][j][3] *= f1; }
            }
        }
#pragma unroll
        for (int kk = 0; kk < kLmKeys / 16; kk++) {
            uint32_t ph[2][4], pl[2][4];
#pragma unroll
            for (int m = 0; m < 2; m++) {
                ldm_x4(ph[m], pAddr + (uint32_t)(m * 16 * kLmP * 2) + kk * 32);
                ldm_x4(pl[m], pAddr + lowBytes + (uint32_t)(m * 16 * kLmP * 2) + kk * 32);
            }
#pragma unroll
            for (int j = 0; j < NT; j += 2) {
                uint32_t v[4];
                ldm_x4_t(v, vAddr + st * stageBytes + (uint32_t)(kk * 16 * LD * 2) + j * 16);
#pragma unroll
                for (int m = 0; m < 2; m++) { mma_bf16(o[m][j], ph[m], v[0], v[1]); mma_bf16(o[m][j + 1], ph[m], v[2], v[3]); }
#pragma unroll
                for (int m = 0; m < 2; m++) { mma_bf16(o[m][j], pl[m], v[0], v[1]); mma_bf16(o[m][j + 1], pl[m], v[2], v[3]); }
            }
        }
    }
    // row sums: the four key groups of a row, through shared memory; the row maxima travel along
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    __syncthreads();
    if (t4 == 0) { s_max[ng * kLmRows + mt * 16 + g] = l0; s_max[ng * kLmRows + mt * 16 + g + 8] = l1; }
    if (ng == 0 && t4 == 0) { s_corr[mt * 16 + g] = m0; s_corr[mt * 16 + g + 8] = m1; }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < 2; m++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            const int lr = m * 16 + g + 8 * e, row = r0 + lr;
            if (row >= rows) continue;
            const float l = (s_max[lr] + s_max[kLmRows + lr]) + (s_max[2 * kLmRows + lr] + s_max[3 * kLmRows + lr]);
            const int t = row / p.H, h = row - t * p.H;
            float* dst;
            float f = 1.0f;
            if (p.splits == 1) { dst = p.out + ((size_t)b * p.T + t) * p.ldo + (size_t)h * p.R; f = 1.0f / l; }
            else {
                dst = p.part + ((((size_t)b * p.T + t) * p.H + h) * p.splits + blockIdx.x) * (p.R + 2);
                if (warp == 0 && t4 == 0) { dst[p.R] = s_corr[lr]; dst[p.R + 1] = l; }
            }
#pragma unroll
            for (int j = 0; j < NT; j++) {
                const int c = warp * NT * 8 + j * 8 + 2 * t4;
                if (c >= p.R) continue;
                if (p.splits > 1) *reinterpret_cast<float2*>(dst + c) = make_float2(o[m][j][2 * e], o[m][j][2 * e + 1]);      // R + 2 is even
                else { dst[c] = o[m][j][2 * e] * f; dst[c + 1] = o[m][j][2 * e + 1] * f; }
            }
        }
}

// Partials of a split key range → weighted latents; the maxima are in units of log2.
__global__ void __launch_bounds__(128) k_latent_mma_merge(const float* __restrict__ part, int splits, int R, int H, float* __restrict__ out, int ldo) {
    extern __shared__ float wgt[];
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.x, row = blockIdx.y;
    const float* p = part + ((size_t)row * H + h) * splits * (R + 2);
    if (threadIdx.x < 32) {                              // at most 256 splits: eight per lane
        float m[8], l[8], mx = -INFINITY, sum = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; j++) {
            const int s = threadIdx.x + 32 * j;
            m[j] = s < splits ? p[(size_t)s * (R + 2) + R] : -INFINITY;
            l[j] = s < splits ? p[(size_t)s * (R + 2) + R + 1] : 0.0f;
            mx = fmaxf(mx, m[j]);
        }
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
#pragma unroll
        for (int j = 0; j < 8; j++) { m[j] = m[j] > -INFINITY ? exp2f(m[j] - mx) : 0.0f; sum = fmaf(l[j], m[j], sum); }
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
#pragma unroll
        for (int j = 0; j < 8; j++)
            if (threadIdx.x + 32 * j < splits) wgt[threadIdx.x + 32 * j] = m[j] / sum;
    }
    __syncthreads();
    const int i = blockIdx.z * 128 + threadIdx.x;
    if (i < R) {
        float v = 0.0f;
#pragma unroll 16
        for (int s = 0; s < splits; s++) v = fmaf(p[(size_t)s * (R + 2) + i], wgt[s], v);
        out[(size_t)row * ldo + (size_t)h * R + i] = v;
    }
}

int lm_width(int R, int W) {
    const int nt = R <= 128 ? 2 : R <= 256 ? 4 : 8;
    return (std::max(W, nt * 64) + 15) / 16 * 16;
}

template <int NT>
void launch_lm(const LmParams& p, int B, cudaStream_t s) {
    static bool attr = false;
    if (!attr) {
        DJ_CUDA_CHECK(cudaFuncSetAttribute(k_latent_mma<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024));
        attr = true;
    }
    launch_k(k_latent_mma<NT>, dim3((unsigned)p.splits, (unsigned)((p.T * p.H + kLmRows - 1) / kLmRows), (unsigned)B), dim3(256), lm_smem(p.Wp), s, true, p);
}

// ───────────── prompt chunks ─────────────

struct LpParams {
    const float* q; int ldq;                        // [rows][H·(dim + rot)]
    const __nv_bfloat16* k; const __nv_bfloat16* v; // this sequence's expanded keys [maxSeq][H·dim] and values [maxSeq][H·vdim]
    const __nv_bfloat16* cache; int W;              // this sequence's cached rows, the rotated part at column R
    int maxSeq;
    const float* pos; const float* cosT; const float* sinT;
    float* out; int ldo;                            // [rows][H·vdim]
    int T, H, dim, rot, R, vdim; float scale;
};

constexpr int kLpRows = 128, kLpKeys = 64;
template <int KQ, int KV> constexpr size_t lp_smem() { return ((size_t)(kLpRows + 2 * kLpKeys) * (KQ * 16 + 8) + (size_t)2 * kLpKeys * (KV * 16 + 8)) * 2; }

// KQ, KV: 16-wide steps that hold dim + rot and vdim (columns past them are zero)
template <int KQ, int KV>
__global__ void __launch_bounds__(256, 1) k_latent_prefill(const LpParams p) {
    constexpr int LQ = KQ * 16 + 8, LV = KV * 16 + 8;
    extern __shared__ __align__(16) unsigned char lp_raw[];
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(lp_raw);
    __nv_bfloat16* Ks = Qs + kLpRows * LQ;
    __nv_bfloat16* Vs = Ks + 2 * kLpKeys * LQ;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    const int h = blockIdx.y, t0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kLpRows;      // the longest rows first
    const int qk = p.dim + p.rot, half = p.rot / 2;
    {   // the columns that no copy writes stay zero
        const int zq = LQ - qk, zv = LV - p.vdim;
        for (int i = tid; i < 2 * kLpKeys * zq; i += 256) Ks[(i / zq) * LQ + qk + i % zq] = __float2bfloat16_rn(0.0f);
        for (int i = tid; i < 2 * kLpKeys * zv; i += 256) Vs[(i / zv) * LV + p.vdim + i % zv] = __float2bfloat16_rn(0.0f);
    }
    pdl_wait();
    pdl_launch_dependents();
    const int pos0 = max((int)p.pos[0], 0);
    const int lastKey = min(p.maxSeq - 1, pos0 + min(p.T, t0 + kLpRows) - 1);
    const int dc = p.dim / 8, rc = p.rot / 8, vc = p.vdim / 8, kc = dc + rc;
    auto load_tile = [&](int tile, int st) {
        __nv_bfloat16* kd = Ks + st * kLpKeys * LQ;
        __nv_bfloat16* vd = Vs + st * kLpKeys * LV;
        for (int i = tid; i < kLpKeys * (kc + vc); i += 256) {
            const int key = i / (kc + vc), c = i - key * (kc + vc);
            const size_t at = (size_t)min(tile * kLpKeys + key, lastKey);
            if (c < dc) cp_async16(kd + key * LQ + c * 8, p.k + at * p.H * p.dim + (size_t)h * p.dim + c * 8);
            else if (c < kc) cp_async16(kd + key * LQ + c * 8, p.cache + at * p.W + p.R + (c - dc) * 8);
            else cp_async16(vd + key * LV + (c - kc) * 8, p.v + at * p.H * p.vdim + (size_t)h * p.vdim + (c - kc) * 8);
        }
        cp_async_commit();
    };
    load_tile(0, 0);
    for (int i = tid; i < kLpRows * (LQ / 2); i += 256) {
        const int r = i / (LQ / 2), c = (i - r * (LQ / 2)) * 2, t = t0 + r;
        float a = 0.0f, b = 0.0f;
        if (t < p.T && c < qk) {
            const float2 u = *reinterpret_cast<const float2*>(p.q + (size_t)t * p.ldq + (size_t)h * qk + c);
            a = u.x; b = u.y;
            if (c >= p.dim) {
                const int j = (c - p.dim) >> 1, at = min(pos0 + t, p.maxSeq - 1);
                const float co = p.cosT[(size_t)at * half + j], si = p.sinT[(size_t)at * half + j];
                a = u.x * co - u.y * si;
                b = u.y * co + u.x * si;
            }
        }
        *reinterpret_cast<uint32_t*>(Qs + r * LQ + c) = pack_bf16(a, b);
    }
    const int lim0 = pos0 + t0 + warp * 16 + g, lim1 = lim0 + 8;
    const int warpLast = pos0 + t0 + warp * 16 + 15;             // newest key any row of this warp may see
    const uint32_t qAddr = smem_u32(Qs) + (uint32_t)(((warp * 16 + (lane & 15)) * LQ + (lane >> 4) * 8) * 2);
    const uint32_t kAddr = smem_u32(Ks) + (uint32_t)((((lane & 7) + ((lane >> 4) << 3)) * LQ + ((lane >> 3) & 1) * 8) * 2);
    const uint32_t vAddr = smem_u32(Vs) + (uint32_t)((((lane & 7) + (((lane >> 3) & 1) << 3)) * LV + (lane >> 4) * 8) * 2);
    const float sc = p.scale * kLog2e;
    float o[2 * KV][4];
#pragma unroll
    for (int j = 0; j < 2 * KV; j++) { o[j][0] = 0.0f; o[j][1] = 0.0f; o[j][2] = 0.0f; o[j][3] = 0.0f; }
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    const int tiles = lastKey / kLpKeys + 1;
    for (int tile = 0; tile < tiles; tile++) {
        const int st = tile & 1, k0 = tile * kLpKeys;
        cp_async_wait<0>();
        __syncthreads();
        if (tile + 1 < tiles) load_tile(tile + 1, st ^ 1);
        if (k0 > warpLast) continue;                             // every key of the tile lies behind this warp's rows
        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; j++) { s[j][0] = 0.0f; s[j][1] = 0.0f; s[j][2] = 0.0f; s[j][3] = 0.0f; }
#pragma unroll
        for (int kk = 0; kk < KQ; kk++) {
            uint32_t a[4];
            ldm_x4(a, qAddr + kk * 32);
#pragma unroll
            for (int n = 0; n < 4; n++) {
                uint32_t bk[4];
                ldm_x4(bk, kAddr + (uint32_t)((st * kLpKeys + n * 16) * LQ * 2) + kk * 32);
                mma_bf16(s[2 * n], a, bk[0], bk[1]);
                mma_bf16(s[2 * n + 1], a, bk[2], bk[3]);
            }
        }
        const bool edge = k0 + kLpKeys - 1 > pos0 + t0 + warp * 16;
        float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const int key = k0 + j * 8 + 2 * t4 + e;
                s[j][e] = edge && key > lim0 ? -INFINITY : s[j][e] * sc;
                s[j][2 + e] = edge && key > lim1 ? -INFINITY : s[j][2 + e] * sc;
                x0 = fmaxf(x0, s[j][e]); x1 = fmaxf(x1, s[j][2 + e]);
            }
        x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
        x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
        const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);      // finite: key 0 is visible to every row of the first tile
        const float c0 = exp2f(m0 - n0), c1 = exp2f(m1 - n1);
        float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
        for (int j = 0; j < 8; j++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                s[j][e] = exp2f(s[j][e] - n0);
                s[j][2 + e] = exp2f(s[j][2 + e] - n1);
                a0 += s[j][e]; a1 += s[j][2 + e];
            }
        l0 = l0 * c0 + a0; l1 = l1 * c1 + a1;
        m0 = n0; m1 = n1;
        if (c0 != 1.0f || c1 != 1.0f) {
#pragma unroll
            for (int j = 0; j < 2 * KV; j++) { o[j][0] *= c0; o[j][1] *= c0; o[j][2] *= c1; o[j][3] *= c1; }
        }
#pragma unroll
        for (int kk = 0; kk < kLpKeys / 16; kk++) {
            uint32_t ph[4], pl[4];
            split_bf16(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
            split_bf16(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
            split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
            split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int j = 0; j < KV; j++) {
                uint32_t v[4];
                ldm_x4_t(v, vAddr + (uint32_t)((st * kLpKeys + kk * 16) * LV * 2) + j * 32);
                mma_bf16(o[2 * j], ph, v[0], v[1]); mma_bf16(o[2 * j + 1], ph, v[2], v[3]);
                mma_bf16(o[2 * j], pl, v[0], v[1]); mma_bf16(o[2 * j + 1], pl, v[2], v[3]);
            }
        }
    }
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
#pragma unroll
    for (int e = 0; e < 2; e++) {
        const int t = t0 + warp * 16 + g + 8 * e;
        if (t >= p.T) continue;
        const float inv = 1.0f / (e ? l1 : l0);
        float* dst = p.out + (size_t)t * p.ldo + (size_t)h * p.vdim;
#pragma unroll
        for (int j = 0; j < 2 * KV; j++) {
            const int c = j * 8 + 2 * t4;
            if (c < p.vdim) { dst[c] = o[j][2 * e] * inv; dst[c + 1] = o[j][2 * e + 1] * inv; }
        }
    }
}

template <int KQ, int KV>
void launch_lp(const LpParams& p, cudaStream_t s) {
    static bool attr = false;
    if (!attr) {
        DJ_CUDA_CHECK(cudaFuncSetAttribute(k_latent_prefill<KQ, KV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)lp_smem<KQ, KV>()));
        attr = true;
    }
    launch_k(k_latent_prefill<KQ, KV>, dim3((unsigned)((p.T + kLpRows - 1) / kLpRows), (unsigned)p.H), dim3(256), lp_smem<KQ, KV>(), s, true, p);
}

size_t expand_floats(const LatentAttnArgs& a) { return (((size_t)a.maxSeq * a.H * (a.dim + a.vdim) + 1) / 2 + 63) / 64 * 64; }

}  // namespace

// Whether the latent-space form has a tensor-core kernel for these sizes (else the FMA form of attn_latent.cu).
bool latent_mma_fits(const LatentAttnArgs& a) {
    const int W = a.R + a.rot;
    return a.bf16 && W % 8 == 0 && a.R % 2 == 0 && a.R <= 512 && lm_smem(lm_width(a.R, W)) <= 226 * 1024;
}
int latent_mma_splits(const LatentAttnArgs& a) {
    const long ctas = (long)a.B * ((a.T * a.H + kLmRows - 1) / kLmRows);
    const int tiles = (a.maxSeq + kLmKeys - 1) / kLmKeys;
    return (int)std::max(1l, std::min((long)std::min(tiles, 256), g_num_sms / ctas));
}
void launch_latent_mma(const LatentAttnArgs& a, cudaStream_t s) {
    LmParams p;
    p.q = a.q; p.ldq = a.ldq; p.dim = a.dim; p.qc = a.qc; p.ldqc = a.ldqc; p.cache = (const __nv_bfloat16*)a.cache; p.maxSeq = a.maxSeq; p.W = a.R + a.rot;
    p.pos = a.pos; p.cosT = a.cosT; p.sinT = a.sinT; p.out = a.out; p.ldo = a.ldo; p.T = a.T; p.H = a.H; p.R = a.R; p.rot = a.rot; p.scale = a.scale;
    p.part = a.ws; p.splits = latent_mma_splits(a); p.Wp = lm_width(a.R, p.W);
    p.kv = a.T == 1 ? a.kv : nullptr; p.ldkv = a.ldkv; p.gamma = a.gamma; p.eps = a.eps; p.append = (__nv_bfloat16*)a.cache;
    p.early = a.early;
    if (a.R <= 128) launch_lm<2>(p, a.B, s);
    else if (a.R <= 256) launch_lm<4>(p, a.B, s);
    else launch_lm<8>(p, a.B, s);
    if (p.splits > 1)
        launch_k(k_latent_mma_merge, dim3((unsigned)a.H, (unsigned)(a.B * a.T), (unsigned)((a.R + 127) / 128)), dim3(128), (size_t)p.splits * 4, s, true, (const float*)p.part, p.splits, a.R, a.H,
                 a.out, a.ldo);
}

// Prompt chunks over expanded keys and values (op 82); the chunk's rows are in the cache already.
bool latent_prefill_fits(const LatentAttnArgs& a) {
    return a.bf16 && a.dim % 8 == 0 && a.rot % 8 == 0 && a.vdim % 8 == 0 && a.R % 8 == 0 && a.dim + a.rot <= 256 && a.vdim <= 128;
}
size_t latent_prefill_ws_floats(const LatentAttnArgs& a) { return expand_floats(a); }
void launch_latent_prefill(const LatentAttnArgs& a, cudaStream_t s) {
    __nv_bfloat16* k = (__nv_bfloat16*)a.ws;
    __nv_bfloat16* v = k + (size_t)a.maxSeq * a.H * a.dim;
    for (int b = 0; b < a.B; b++) {
        const __nv_bfloat16* cache = (const __nv_bfloat16*)a.cache + (size_t)b * a.maxSeq * (a.R + a.rot);
        launch_bf16_gemm_rows(cache, a.R + a.rot, a.R, a.pos + b, a.T, a.maxSeq, a.uk, k, a.H * a.dim, s);
        launch_bf16_gemm_rows(cache, a.R + a.rot, a.R, a.pos + b, a.T, a.maxSeq, a.uv, v, a.H * a.vdim, s);
        LpParams p;
        p.q = a.q + (size_t)b * a.T * a.ldq; p.ldq = a.ldq; p.k = k; p.v = v; p.cache = cache; p.W = a.R + a.rot; p.maxSeq = a.maxSeq;
        p.pos = a.pos + b; p.cosT = a.cosT; p.sinT = a.sinT; p.out = a.out + (size_t)b * a.T * a.ldo; p.ldo = a.ldo;
        p.T = a.T; p.H = a.H; p.dim = a.dim; p.rot = a.rot; p.R = a.R; p.vdim = a.vdim; p.scale = a.scale;
        const int qk = a.dim + a.rot;
        const bool wide = a.vdim > 64;
        if (qk <= 96) { if (wide) launch_lp<6, 8>(p, s); else launch_lp<6, 4>(p, s); }
        else if (qk <= 192) { if (wide) launch_lp<12, 8>(p, s); else launch_lp<12, 4>(p, s); }
        else { if (wide) launch_lp<16, 8>(p, s); else launch_lp<16, 4>(p, s); }
    }
}

}  // namespace dj
