// Latent attention: every head's keys and values are linear in one latent vector c per position, so the cache holds one
// row per position — [c | rotated key part] — shared by all heads.
//
// Scores are taken in the latent space: with qc = W_ukᵀ q_unrotated (the projection before this op),
//     score = (qc · c_j + rot(q_rotated) · k_rot,j) · scale,    ctx = Σ_j softmax_j · c_j,
// and the head's output is W_uv ctx (the projection behind it).  Scores, softmax and sums are fp32; the cache is fp32 or
// bf16.
//
//   k_latent_append   RMS norm of the latent, rotation of the key part, cache write
//   k_latent_attn     fp32 FMA form, any sizes: a warp per head, tiles of 32 keys in shared memory shared by eight heads
//   k_latent_merge    adds the partial results of a split key range
// With a bf16 cache the tensor-core kernels of attn_latent_mma.cu take over where the sizes allow.
#include "row_operand.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr int kLaKeys = 32, kLaHeads = 8;

template <typename CT> __device__ __forceinline__ float cache_load(const CT* p);
template <> __device__ __forceinline__ float cache_load<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float cache_load<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename CT> __device__ __forceinline__ CT cache_store(float v);
template <> __device__ __forceinline__ float cache_store<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 cache_store<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// one block of 128 threads per token row
template <typename CT>
__global__ void __launch_bounds__(128) k_latent_append(const float* __restrict__ kv, int ld, const float* __restrict__ gamma, float eps, CT* __restrict__ cache,
                                                       int maxSeq, int W, const float* __restrict__ pos, const float* __restrict__ cosT,
                                                       const float* __restrict__ sinT, int T, int R, int rot) {
    __shared__ float part[4];
    pdl_wait();
    pdl_launch_dependents();
    const int row = blockIdx.x, b = row / T, p = (int)pos[b] + row - b * T;
    if (p < 0 || p >= maxSeq) return;
    const float* x = kv + (size_t)row * ld;
    CT* dst = cache + ((size_t)b * maxSeq + p) * W;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < R; i += 128) ss = fmaf(x[i], x[i], ss);
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
    __syncthreads();
    const float inv = 1.0f / sqrtf(((part[0] + part[1]) + (part[2] + part[3])) / (float)R + eps);
    for (int i = threadIdx.x; i < R; i += 128) dst[i] = cache_store<CT>((x[i] * inv) * gamma[i]);
    for (int i = threadIdx.x; i < rot / 2; i += 128) {
        const float c = cosT[(size_t)p * (rot / 2) + i], s = sinT[(size_t)p * (rot / 2) + i], u = x[R + 2 * i], v = x[R + 2 * i + 1];
        dst[R + 2 * i] = cache_store<CT>(u * c - v * s);
        dst[R + 2 * i + 1] = cache_store<CT>(v * c + u * s);
    }
}

struct LaParams {
    const float* q; int ldq, dim;                 // q + h·(dim + rot) + dim: the rotated part
    const float* qc; int ldqc;                    // qc + h·R
    const void* cache; int maxSeq, W;
    const float* pos; const float* cosT; const float* sinT;
    float* out; int ldo;                          // [rows][H·R]
    int T, H, R, rot; float scale;
    float* part; int splits;                      // partials [row][head][split][R + 2]
};

template <typename CT, int NR>
__global__ void __launch_bounds__(256) k_latent_attn(const LaParams p) {
    extern __shared__ float sm[];
    const int W = p.R + p.rot, LD = W | 1;                       // odd row pitch: a lane per key reads without conflicts
    float* qs = sm;                                              // [kLaHeads][W]
    float* ks = qs + kLaHeads * W;                               // [kLaKeys][LD]
    float* ps = ks + kLaKeys * LD;                               // [kLaHeads][kLaKeys]
    pdl_wait();
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int row = blockIdx.y, b = row / p.T, my = (int)p.pos[b] + row - b * p.T;      // this row's position
    const int h = blockIdx.z * kLaHeads + warp;
    if (my < 0 || my >= p.maxSeq) return;
    const int half = p.rot / 2;
    if (h < p.H) {
        for (int i = lane; i < p.R; i += 32) qs[warp * W + i] = p.qc[(size_t)row * p.ldqc + (size_t)h * p.R + i] * p.scale;
        const float* qr = p.q + (size_t)row * p.ldq + (size_t)h * (p.dim + p.rot) + p.dim;
        for (int i = lane; i < half; i += 32) {
            const float c = p.cosT[(size_t)my * half + i], s = p.sinT[(size_t)my * half + i], u = qr[2 * i], v = qr[2 * i + 1];
            qs[warp * W + p.R + 2 * i] = (u * c - v * s) * p.scale;
            qs[warp * W + p.R + 2 * i + 1] = (v * c + u * s) * p.scale;
        }
    }
    const int keys = my + 1, tiles = (keys + kLaKeys - 1) / kLaKeys;
    const int per = (tiles + p.splits - 1) / p.splits;
    const int tLo = blockIdx.x * per, tHi = min(tiles, tLo + per);
    float acc[NR];
#pragma unroll
    for (int j = 0; j < NR; j++) acc[j] = 0.0f;
    float mx = -INFINITY, l = 0.0f;
    const CT* cache = (const CT*)p.cache + (size_t)b * p.maxSeq * p.W;
    for (int tile = tLo; tile < tHi; tile++) {
        __syncthreads();
        const int k0 = tile * kLaKeys, n = min(kLaKeys, keys - k0);
        for (int i = threadIdx.x; i < n * W; i += 256) {
            const int j = i / W, d = i - j * W;
            ks[j * LD + d] = cache_load<CT>(cache + (size_t)(k0 + j) * p.W + d);
        }
        __syncthreads();
        if (h < p.H) {
            float s = -INFINITY;
            if (lane < n) {
                float s0 = 0.0f, s1 = 0.0f;
                const float* kr = ks + lane * LD; const float* q = qs + warp * W;
                int d = 0;
                for (; d + 1 < W; d += 2) { s0 = fmaf(q[d], kr[d], s0); s1 = fmaf(q[d + 1], kr[d + 1], s1); }
                if (d < W) s0 = fmaf(q[d], kr[d], s0);
                s = s0 + s1;
            }
            float m2 = s;
            for (int o = 16; o > 0; o >>= 1) m2 = fmaxf(m2, __shfl_xor_sync(0xffffffffu, m2, o));
            m2 = fmaxf(m2, mx);
            const float pr = lane < n ? expf(s - m2) : 0.0f;
            const float corr = mx > -INFINITY ? expf(mx - m2) : 0.0f;
            float sum = pr;
            for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l = l * corr + sum;
            mx = m2;
            ps[warp * kLaKeys + lane] = pr;
            __syncwarp();
#pragma unroll
            for (int j = 0; j < NR; j++) acc[j] *= corr;
            for (int k = 0; k < n; k++) {
                const float pk = ps[warp * kLaKeys + k];
#pragma unroll
                for (int j = 0; j < NR; j++) {
                    const int i = j * 32 + lane;
                    if (i < p.R) acc[j] = fmaf(pk, ks[k * LD + i], acc[j]);
                }
            }
            __syncwarp();
        }
    }
    if (h >= p.H) return;
    if (p.splits == 1) {
        const float inv = 1.0f / l;
#pragma unroll
        for (int j = 0; j < NR; j++)
            if (j * 32 + lane < p.R) p.out[(size_t)row * p.ldo + (size_t)h * p.R + j * 32 + lane] = acc[j] * inv;
    } else {
        float* o = p.part + (((size_t)row * p.H + h) * p.splits + blockIdx.x) * (p.R + 2);
#pragma unroll
        for (int j = 0; j < NR; j++)
            if (j * 32 + lane < p.R) o[j * 32 + lane] = acc[j];
        if (lane == 0) { o[p.R] = mx; o[p.R + 1] = l; }
    }
}

__global__ void __launch_bounds__(128) k_latent_merge(const float* __restrict__ part, int splits, int R, int H, float* __restrict__ out, int ldo) {
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.x, row = blockIdx.y;
    const float* p = part + ((size_t)row * H + h) * splits * (R + 2);
    float mx = -INFINITY;
    for (int s = 0; s < splits; s++) mx = fmaxf(mx, p[(size_t)s * (R + 2) + R]);
    float l = 0.0f;
    for (int s = 0; s < splits; s++) { const float m = p[(size_t)s * (R + 2) + R]; if (m > -INFINITY) l += p[(size_t)s * (R + 2) + R + 1] * expf(m - mx); }
    for (int i = threadIdx.x; i < R; i += 128) {
        float v = 0.0f;
        for (int s = 0; s < splits; s++) {
            const float m = p[(size_t)s * (R + 2) + R];
            if (m > -INFINITY) v = fmaf(p[(size_t)s * (R + 2) + i], expf(m - mx), v);
        }
        out[(size_t)row * ldo + (size_t)h * R + i] = v / l;
    }
}

size_t la_smem(int W) { return ((size_t)kLaHeads * W + (size_t)kLaKeys * (W | 1) + kLaHeads * kLaKeys) * 4; }

template <typename CT, int NR>
void launch_la(const LaParams& p, int rows, cudaStream_t s) {
    static bool attr = false;
    if (!attr) {
        DJ_CUDA_CHECK(cudaFuncSetAttribute(k_latent_attn<CT, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 1024));
        attr = true;
    }
    launch_k(k_latent_attn<CT, NR>, dim3((unsigned)p.splits, (unsigned)rows, (unsigned)((p.H + kLaHeads - 1) / kLaHeads)), dim3(256), la_smem(p.R + p.rot), s, true, p);
}

template <typename CT>
void append(const LatentAttnArgs& a, cudaStream_t s) {
    launch_k(k_latent_append<CT>, dim3((unsigned)(a.B * a.T)), dim3(128), 0, s, true, a.kv, a.ldkv, a.gamma, a.eps, (CT*)a.cache, a.maxSeq, a.R + a.rot, a.pos,
             a.cosT, a.sinT, a.T, a.R, a.rot);
}

template <typename CT>
void run(const LatentAttnArgs& a, cudaStream_t s) {
    const int rows = a.B * a.T, W = a.R + a.rot;
    LaParams p;
    p.q = a.q; p.ldq = a.ldq; p.dim = a.dim; p.qc = a.qc; p.ldqc = a.ldqc; p.cache = a.cache; p.maxSeq = a.maxSeq; p.W = W;
    p.pos = a.pos; p.cosT = a.cosT; p.sinT = a.sinT; p.out = a.out; p.ldo = a.ldo;
    p.T = a.T; p.H = a.H; p.R = a.R; p.rot = a.rot; p.scale = a.scale;
    p.part = a.ws; p.splits = latent_attn_splits(rows, a.H, a.maxSeq);
    if (a.R <= 64) launch_la<CT, 2>(p, rows, s);
    else if (a.R <= 128) launch_la<CT, 4>(p, rows, s);
    else if (a.R <= 256) launch_la<CT, 8>(p, rows, s);
    else if (a.R <= 512) launch_la<CT, 16>(p, rows, s);
    else launch_la<CT, 32>(p, rows, s);
    if (p.splits > 1)
        launch_k(k_latent_merge, dim3((unsigned)a.H, (unsigned)rows), dim3(128), 0, s, true, (const float*)p.part, p.splits, a.R, a.H, a.out, a.ldo);
}

}  // namespace

int latent_attn_splits(int rows, int H, int maxSeq) {
    const long ctas = (long)rows * ((H + kLaHeads - 1) / kLaHeads);
    const int tiles = (maxSeq + kLaKeys - 1) / kLaKeys;
    return (int)std::max(1l, std::min((long)std::min(tiles, 64), 2l * g_num_sms / ctas));
}
size_t latent_attn_ws_floats(const LatentAttnArgs& a) {
    const int rows = a.B * a.T, splits = latent_mma_fits(a) ? latent_mma_splits(a) : latent_attn_splits(rows, a.H, a.maxSeq);
    return splits > 1 ? (size_t)rows * a.H * splits * (a.R + 2) : 0;
}
bool latent_attn_fits(int R, int rot) { return R >= 1 && R <= 1024 && rot >= 2 && rot % 2 == 0 && la_smem(R + rot) <= 226 * 1024; }

void launch_latent_append(const LatentAttnArgs& a, cudaStream_t s) {
    if (a.bf16) append<__nv_bfloat16>(a, s);
    else append<float>(a, s);
}

void launch_latent_attn(const LatentAttnArgs& a, cudaStream_t s) {
    const bool mma = latent_mma_fits(a);
    if (!mma || a.T > 1) launch_latent_append(a, s);
    if (mma) launch_latent_mma(a, s);
    else if (a.bf16) run<__nv_bfloat16>(a, s);
    else run<float>(a, s);
}

}  // namespace dj
