// Grouped attention on the tensor cores (bf16 cache); what a score is made of is described in attn_grouped.cu.
//
//   k_grouped_decode    one token per sequence.  grid (key splits, blocks of eight query heads of a group, B·G): the heads are the
//                       rows of one 16-row operand, their queries (and softmax weights) as bf16 high halves in rows 0-7 and
//                       low halves in rows 8-15, so one product takes 16 bits of them.  Eight (or four) warps walk tiles
//                       of 16 keys, each through a private ring of tensor copies, as deep as shared memory allows, that starts before the dependency wait; the
//                       block that holds the newest position norms and appends it.  Warps merge
//                       in shared memory, blocks through partials that the last one to finish (a ticket) adds up.
//   k_grouped_prefill   prompt chunks: 128 rows (token, head in the group) per block, 16 per warp, key tiles in three stages.
// Key and value rows travel as 64-column boxes with 128-byte swizzle.
// Waits for copies are bounded (codes 221-223 in the device error word).  Softmax is fp32 and its weights enter the second product as two bf16 halves (16 bits).
#include "mma_common.cuh"
#include "row_operand.cuh"
#include "tc_common.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr float kLog2e = 1.4426950408889634f;
constexpr int kGdKeys = 16, kGpStages = 3, kGdMaxStages = 8, kAlone = 4;
constexpr int kGpRows = 128, kGpThreads = 256;

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float quad_max(float v) {
    v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 1));
    return fmaxf(v, __shfl_xor_sync(0xffffffffu, v, 2));
}
__device__ __forceinline__ float quad_sum(float v) {
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    return v + __shfl_xor_sync(0xffffffffu, v, 2);
}
__device__ __forceinline__ float warp_sum(float v) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// Bias of query rows (table row `rel`, fp32) at distance d, in the exponent's base-2 units.
__device__ __forceinline__ float bias_at(const float* rel, int d, int len) { return __ldg(rel + min(d, len - 1)) * kLog2e; }

struct GdParams {
    GroupedAttnArgs a;
    CUtensorMap k, v;                                        // rows of 64 columns × a tile's keys
    int splits, stages; int* error;
};

// Shared memory: tiles (1024-byte aligned), then queries, the new row, the norms of cached keys.
struct GdShape { int kb, vb, tile, LDQ; };                   // boxes of a key and of a value row, bytes of a stage, query row pitch (halves)
__host__ __device__ __forceinline__ GdShape gd_shape(int kw, int vw, bool shared, int keys) {
    GdShape g;
    g.kb = (kw + 63) / 64; g.vb = shared ? 0 : (vw + 63) / 64;
    g.tile = (g.kb + g.vb) * keys * 128; g.LDQ = g.kb * 64 + 8;
    return g;
}
// Byte offset of 16-byte column c of row r in a tile of boxes: the copy engine swaps the columns of a 128-byte row by its number.
// Columns past a row's width hold zeros, in the boxes and in the query rows.
__device__ __forceinline__ uint32_t swizzled(int r, int c, int keys) { return (uint32_t)((c >> 3) * keys * 128 + r * 128 + (((c & 7) ^ (r & 7)) << 4)); }

size_t gd_smem(const GroupedAttnArgs& a, int warps, int stages) {
    const bool shared = a.vcache == nullptr;
    const GdShape g = gd_shape(a.kw, a.vw, shared, kGdKeys);
    const size_t ring = (size_t)warps * stages * g.tile, merge = (size_t)warps * 8 * ((shared ? a.kw : a.vw) + 4) * 4;
    return 1024 + std::max(ring, merge) + (size_t)16 * g.LDQ * 2 + (size_t)(a.kw + a.vw + 16) * 2 + (size_t)warps * stages * kGdKeys * 4;
}

// VN: most output n-tiles (eight value columns each), NW: warps
template <int VN, int NW>
__global__ void __launch_bounds__(32 * NW, VN <= 8 ? 2 : 1) k_grouped_decode(const __grid_constant__ GdParams p) {
    extern __shared__ __align__(1024) unsigned char gd_raw[];
    __shared__ __align__(8) unsigned long long s_bar[NW * kGdMaxStages];
    __shared__ float s_newScale;
    __shared__ volatile int s_abort;
    __shared__ int s_last;
    const GroupedAttnArgs& a = p.a;
    const int splits = p.splits, stages = p.stages;
    const bool shared = a.vcache == nullptr;
    const GdShape S = gd_shape(a.kw, a.vw, shared, kGdKeys);
    const int Vp = shared ? a.kw : a.vw, vt = Vp / 8;
    const uint32_t raw = smem_u32(gd_raw), skip = ((raw + 1023u) & ~1023u) - raw;
    unsigned char* ring = gd_raw + skip;
    const size_t ringBytes = max((size_t)NW * stages * S.tile, (size_t)NW * 8 * (Vp + 4) * 4);
    __nv_bfloat16* Qh = reinterpret_cast<__nv_bfloat16*>(ring + ringBytes);          // [8][LDQ] high halves, then the low ones
    float* scales = reinterpret_cast<float*>(Qh + 16 * S.LDQ);                   // [warp][stage][16]
    __nv_bfloat16* newK = reinterpret_cast<__nv_bfloat16*>(scales + NW * stages * kGdKeys);
    __nv_bfloat16* newV = newK + a.kw;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rl = lane >> 2, t4 = lane & 3;
    unsigned char* mine = ring + warp * stages * S.tile;
    float* mySc = scales + warp * stages * kGdKeys;
    const int rep = a.H / a.G, b = blockIdx.z / a.G, g = blockIdx.z - b * a.G, h0 = g * rep + blockIdx.y * 8, nrow = min(8, rep - (int)blockIdx.y * 8);
    // The next kernel is not let in early (griddepcontrol.launch_dependents): short contexts keep some SMs busy, and a projection
    // whose blocks all go to the others streams its weights through those alone.
    if (!a.early) pdl_wait();
    const int pos = (int)a.pos[b];
    const bool valid = pos >= 0 && pos < a.maxSeq;
    // a few tiles per warp cost less than adding up the parts of several blocks
    const int tiles = valid ? pos / kGdKeys + 1 : 0, per = tiles <= kAlone * NW ? kAlone * NW : max(NW, (tiles + splits - 1) / splits), active = (tiles + per - 1) / per;
    const int tLo = blockIdx.x * per, tHi = min(tiles, tLo + per);
    const float* ksc = a.kscale + (size_t)blockIdx.z * a.kpitch;
    const int plane = blockIdx.z * a.maxSeq;                 // first row of this head's keys and values
    auto bar = [&](int stage) { return smem_u32(&s_bar[warp * kGdMaxStages + stage]); };
    if (lane == 0) {
        for (int i = 0; i < stages; i++) mbar_init(bar(i), 1);
        if (warp == 0) s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    // rows past the newest key are whatever earlier requests left: finite, and masked
    auto load = [&](int tile, int stage) {
        if (lane != 0) return;
        const int k0 = tile * kGdKeys;
        uint32_t dst = smem_u32(mine + stage * S.tile);
        mbar_arrive_expect_tx(bar(stage), (uint32_t)(S.tile + (shared ? kGdKeys * 4 : 0)));
        for (int c = 0; c < S.kb; c++, dst += kGdKeys * 128) tma_box(dst, &p.k, c * 64, plane + k0, bar(stage));
        for (int c = 0; c < S.vb; c++, dst += kGdKeys * 128) tma_box(dst, &p.v, c * 64, plane + k0, bar(stage));
        if (shared) bulk_g2s(smem_u32(mySc + stage * kGdKeys), ksc + k0, kGdKeys * 4, bar(stage));      // kpitch covers whole tiles
    };
    for (int i = 0; i < stages - 1; i++)
        if (tLo + warp + i * NW < tHi) load(tLo + warp + i * NW, i);
    if (a.early) pdl_wait();
    if (tLo >= tHi) return;

    // A warp norms query rows warp, warp + NW, …; the warp after those with a first row norms the new key.  Rows are loaded to
    // registers together with the gains: one round trip to L2.
    constexpr int NE = VN / 4 > 4 ? 8 : 4;                   // channels per lane (checked against the head size by the launcher)
    const float* x = a.proj + (size_t)b * a.ld;
    const float qf = a.scale * (a.qtab ? __ldg(a.qtab + pos) : 1.0f) * kLog2e;
    const bool append = a.k_off >= 0 && pos / kGdKeys >= tLo && pos / kGdKeys < tHi;
    auto inverse_rms = [&](const float (&v)[NE]) {
        float ss = 0.0f;
#pragma unroll
        for (int e = 0; e < NE; e++) ss = fmaf(v[e], v[e], ss);
        return 1.0f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
    };
    auto fetch = [&](const float* src, int n, float (&v)[NE]) {
#pragma unroll
        for (int e = 0; e < NE; e++) {
            v[e] = 0.0f;
            if (e * 32 + lane < n) v[e] = src[e * 32 + lane];
        }
    };
    if (append && warp == min(nrow, NW - 1)) {
        float k[NE], kg[NE], v[NE];
        fetch(x + a.k_off + (size_t)g * a.dim, a.dim, k);
        fetch(a.kgamma, a.dim, kg);
        if (!shared) fetch(x + a.v_off + (size_t)g * a.vdim, a.vdim, v);
        const float inv = inverse_rms(k);
        __nv_bfloat16* kd = (__nv_bfloat16*)a.kcache + ((size_t)blockIdx.z * a.maxSeq + pos) * a.kw;
        __nv_bfloat16* vd = (__nv_bfloat16*)a.vcache + ((size_t)blockIdx.z * a.maxSeq + pos) * a.vw;
#pragma unroll
        for (int e = 0; e < NE; e++) {
            const int i = e * 32 + lane;
            const __nv_bfloat16 kv = __float2bfloat16_rn(shared ? k[e] : (k[e] * inv) * kg[e]);
            if (i < a.kw) { newK[i] = kv; if (blockIdx.y == 0) kd[i] = kv; }
            if (!shared && i < a.vw) {
                const __nv_bfloat16 vv = __float2bfloat16_rn(v[e]);
                newV[i] = vv;
                if (blockIdx.y == 0) vd[i] = vv;
            }
        }
        if (shared && lane == 0) {
            s_newScale = inv;
            if (blockIdx.y == 0) a.kscale[(size_t)blockIdx.z * a.kpitch + pos] = inv;
        }
    }
    for (int r = warp; r < nrow; r += NW) {
        float q[NE], w[NE], kg[NE];
        fetch(x + a.q_off + (size_t)(h0 + r) * a.dim, a.dim, q);
        fetch(a.qgamma, a.dim, w);
        if (shared) fetch(a.kgamma, a.dim, kg);
        const float inv = inverse_rms(q);
#pragma unroll
        for (int e = 0; e < NE; e++) {
            const int i = e * 32 + lane;
            if (i >= S.kb * 64) break;
            float v = (q[e] * inv) * w[e] * qf;
            if (shared) v *= kg[e];
            const __nv_bfloat16 hi = __float2bfloat16_rn(v);
            Qh[r * S.LDQ + i] = hi;
            Qh[(8 + r) * S.LDQ + i] = __float2bfloat16_rn(v - __bfloat162float(hi));
        }
    }
    for (int i = tid; i < (8 - nrow) * S.LDQ / 2; i += 32 * NW) {        // rows of no head
        reinterpret_cast<uint32_t*>(Qh + nrow * S.LDQ)[i] = 0;
        reinterpret_cast<uint32_t*>(Qh + (8 + nrow) * S.LDQ)[i] = 0;
    }
    __syncthreads();

    const uint32_t qAddr = smem_u32(Qh) + (uint32_t)(((lane & 15) * S.LDQ + (lane >> 4) * 8) * 2);
    uint32_t kOff[4], vOff[4];                               // operand B, columns 16i of a box: from rows of keys, and read transposed
#pragma unroll
    for (int i = 0; i < 4; i++) {
        kOff[i] = swizzled((lane & 7) + ((lane >> 4) << 3), 2 * i + ((lane >> 3) & 1), 0);
        vOff[i] = swizzled((lane & 7) + (((lane >> 3) & 1) << 3), 2 * i + (lane >> 4), 0);
    }
    const float* rel = a.rel ? a.rel + (size_t)(h0 + min(rl, nrow - 1)) * a.relLen : nullptr;
    const float far = a.rel ? bias_at(rel, a.relLen - 1, a.relLen) : 0.0f;
    float o[VN][4];                                          // by the weights' high halves, and by the low ones
#pragma unroll
    for (int j = 0; j < VN; j++) { o[j][0] = 0.0f; o[j][1] = 0.0f; o[j][2] = 0.0f; o[j][3] = 0.0f; }
    float m = -INFINITY, l = 0.0f;
    int stage = 0, phase = 0;
    for (int tile = tLo + warp; tile < tHi; tile += NW) {
        if (!__all_sync(0xffffffffu, mbar_wait(bar(stage), phase, &s_abort, p.error, 221))) {
            // let the copies in flight land before the block goes
            for (unsigned w = 0; w < (1u << 16) && !mbar_try_wait(bar(stage), phase); w++) {}
            for (int t = tile + NW, k = 1; t < tHi && k < stages - 1; t += NW, k++) {
                const int st = (stage + k) % stages, ph = stage + k >= stages ? phase ^ 1 : phase;
                for (unsigned w = 0; w < (1u << 16) && !mbar_try_wait(bar(st), ph); w++) {}
            }
            break;
        }
        const int k0 = tile * kGdKeys;
        unsigned char* K = mine + stage * S.tile;
        unsigned char* V = shared ? K : K + S.kb * kGdKeys * 128;
        float* sc = mySc + stage * kGdKeys;
        if (append && tile == pos / kGdKeys) {               // what was fetched predates the append
            const int r = pos - k0;
            for (int i = lane; i < a.kw; i += 32) *reinterpret_cast<__nv_bfloat16*>(K + swizzled(r, i >> 3, kGdKeys) + (i & 7) * 2) = newK[i];
            if (shared) { if (lane == 0) sc[r] = s_newScale; }
            else { for (int i = lane; i < a.vw; i += 32) *reinterpret_cast<__nv_bfloat16*>(V + swizzled(r, i >> 3, kGdKeys) + (i & 7) * 2) = newV[i]; }
            fence_proxy_async_smem();
            __syncwarp();
        }
        {
            const int next = tile + (stages - 1) * NW;
            if (next < tHi) load(next, stage == 0 ? stages - 1 : stage - 1);
        }
        float bias[2][2] = {{far, far}, {far, far}};
        if (a.rel && pos - (k0 + kGdKeys - 1) < a.relLen - 1) {
#pragma unroll
            for (int j = 0; j < 2; j++)
#pragma unroll
                for (int e = 0; e < 2; e++) bias[j][e] = bias_at(rel, max(pos - k0 - (j * 8 + 2 * t4 + e), 0), a.relLen);
        }
        float s[2][4];                                       // by the queries' high halves, and by the low ones
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int e = 0; e < 4; e++) s[j][e] = 0.0f;
        const uint32_t kAddr = smem_u32(K);
        for (int c = 0; c < S.kb; c++)
#pragma unroll
            for (int kk = 0; kk < 4; kk++) {
                uint32_t aq[4], bk[4];
                ldm_x4(aq, qAddr + c * 128 + kk * 32);
                ldm_x4(bk, kAddr + kOff[kk] + c * (kGdKeys * 128));
                mma_bf16(s[0], aq, bk[0], bk[1]); mma_bf16(s[1], aq, bk[2], bk[3]);
            }
        float w[2][2], mx = -INFINITY;
#pragma unroll
        for (int j = 0; j < 2; j++) {
            w[j][0] = s[j][0] + s[j][2]; w[j][1] = s[j][1] + s[j][3];
            if (shared) {
                const float2 f = *reinterpret_cast<const float2*>(sc + j * 8 + 2 * t4);
                w[j][0] *= f.x; w[j][1] *= f.y;
            }
#pragma unroll
            for (int e = 0; e < 2; e++) {
                w[j][e] = k0 + j * 8 + 2 * t4 + e <= pos ? w[j][e] + bias[j][e] : -INFINITY;
                mx = fmaxf(mx, w[j][e]);
            }
        }
        mx = fmaxf(m, quad_max(mx));                         // finite: a tile's first key is always seen
        const float corr = ex2(m - mx);
        m = mx;
#pragma unroll
        for (int j = 0; j < 2; j++)
#pragma unroll
            for (int e = 0; e < 2; e++) w[j][e] = ex2(w[j][e] - m);
        l = l * corr + ((w[0][0] + w[0][1]) + (w[1][0] + w[1][1]));
        uint32_t pw4[4];                                     // rows 0-7: high halves, rows 8-15: low halves
        split_bf16(w[0][0], w[0][1], pw4[0], pw4[1]); split_bf16(w[1][0], w[1][1], pw4[2], pw4[3]);
        if (__any_sync(0xffffffffu, corr != 1.0f)) {
#pragma unroll
            for (int c = 0; c < VN; c++) { o[c][0] *= corr; o[c][1] *= corr; o[c][2] *= corr; o[c][3] *= corr; }
        }
        const uint32_t vAddr = smem_u32(V);
#pragma unroll
        for (int c = 0; c < VN; c += 4) {
            if (c >= vt) break;
            uint32_t bv[2][4];
            ldm_x4_t(bv[0], vAddr + vOff[(c & 7) / 2] + (c >> 3) * (kGdKeys * 128));
            ldm_x4_t(bv[1], vAddr + vOff[(c & 7) / 2 + 1] + (c >> 3) * (kGdKeys * 128));
            mma_bf16(o[c], pw4, bv[0][0], bv[0][1]); mma_bf16(o[c + 1], pw4, bv[0][2], bv[0][3]);
            mma_bf16(o[c + 2], pw4, bv[1][0], bv[1][1]); mma_bf16(o[c + 3], pw4, bv[1][2], bv[1][3]);
        }
        if (++stage == stages) { stage = 0; phase ^= 1; }
        __syncwarp();
    }
    l = quad_sum(l);
    __syncthreads();                                         // the ring becomes the merge buffer: [warp][8][Vp + 4]
    float* mg = reinterpret_cast<float*>(ring);
    const int mrow = Vp + 4;
    {
        float* dst = mg + (warp * 8 + rl) * mrow;
#pragma unroll
        for (int c = 0; c < VN; c++)
            if (c < vt) *reinterpret_cast<float2*>(dst + c * 8 + 2 * t4) = make_float2(o[c][0] + o[c][2], o[c][1] + o[c][3]);
        if (t4 == 0) { dst[Vp] = m; dst[Vp + 1] = l; }
    }
    __syncthreads();
    // partials: [row][split][pw], the maximum and the sum in the last four floats, the values padded to whole 16-byte pieces
    const int pw = Vp + 4;
    float* part = a.ws + ((size_t)blockIdx.z * rep + blockIdx.y * 8) * splits * pw;
    for (int r = warp; r < nrow; r += NW) {
        float mw[NW], m = active == 1 && a.sink ? 0.0f : -INFINITY;
#pragma unroll
        for (int w = 0; w < NW; w++) { mw[w] = mg[(w * 8 + r) * mrow + Vp]; m = fmaxf(m, mw[w]); }
        float l = active == 1 && a.sink ? ex2(-m) : 0.0f;
#pragma unroll
        for (int w = 0; w < NW; w++) {
            mw[w] = ex2(mw[w] - m);
            l = fmaf(mw[w], mg[(w * 8 + r) * mrow + Vp + 1], l);
        }
        float* dst = active == 1 ? a.out + (size_t)b * a.ldo + (size_t)(h0 + r) * a.vdim : part + ((size_t)r * splits + blockIdx.x) * pw;
        const float norm = active == 1 ? 1.0f / l : 1.0f;
        for (int i = lane; i < (active == 1 ? a.vdim : Vp); i += 32) {
            float v = 0.0f;
#pragma unroll
            for (int w = 0; w < NW; w++) v = fmaf(mw[w], mg[(w * 8 + r) * mrow + i], v);
            dst[i] = v * norm;
        }
        if (active > 1 && lane == 0) { dst[Vp] = m; dst[Vp + 1] = l; }
    }
    if (active == 1) return;
    __syncthreads();
    if (tid == 0) {
        __threadfence();                                     // the block's partials, before its ticket
        int* ticket = a.tickets + blockIdx.z * gridDim.y + blockIdx.y;
        s_last = atomicAdd(ticket, 1) == active - 1;
        if (s_last) *ticket = 0;
        __threadfence();
    }
    __syncthreads();
    if (!s_last) return;
    // a thread: four columns of a row over every `share`-th part, with a running maximum of its own (maximum, sum and values of a
    // part travel together); the shares of a column sit in neighbouring lanes
    const int items = nrow * (Vp / 4);
    int share = 1;
    while (share < 8 && items * share * 2 <= 32 * NW) share <<= 1;
    for (int u = tid / share; u < (items + 31) / 32 * 32; u += 32 * NW / share) {
        const int r = min(u, items - 1) / (Vp / 4), c = min(u, items - 1) % (Vp / 4), first = tid & (share - 1);
        const float* src = part + (size_t)r * splits * pw;
        float M = -INFINITY, L = 0.0f;
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        constexpr int BATCH = 8;
        for (int s0 = first; s0 < active; s0 += share * BATCH) {
            float2 ml[BATCH];
            float4 x4[BATCH];
#pragma unroll
            for (int i = 0; i < BATCH; i++) {
                const int s = s0 + i * share;
                ml[i] = make_float2(-INFINITY, 0.0f); x4[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                if (s < active) {
                    ml[i] = __ldcg(reinterpret_cast<const float2*>(src + (size_t)s * pw + Vp));
                    x4[i] = __ldcg(reinterpret_cast<const float4*>(src + (size_t)s * pw) + c);
                }
            }
            float top = M;
#pragma unroll
            for (int i = 0; i < BATCH; i++) top = fmaxf(top, ml[i].x);
            const float old = ex2(M - top);                  // the batch's first part is there: top is finite
            M = top; L *= old; v.x *= old; v.y *= old; v.z *= old; v.w *= old;
#pragma unroll
            for (int i = 0; i < BATCH; i++) {
                const float f = ex2(ml[i].x - top);
                L = fmaf(f, ml[i].y, L);
                v.x = fmaf(f, x4[i].x, v.x); v.y = fmaf(f, x4[i].y, v.y); v.z = fmaf(f, x4[i].z, v.z); v.w = fmaf(f, x4[i].w, v.w);
            }
        }
        float top = M;
        for (int o2 = 1; o2 < share; o2 <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o2));
        if (a.sink) top = fmaxf(top, 0.0f);
        const float f = ex2(M - top);                        // a share without parts has M = −∞ and adds nothing
        L *= f; v.x *= f; v.y *= f; v.z *= f; v.w *= f;
        for (int o2 = 1; o2 < share; o2 <<= 1) {
            L += __shfl_xor_sync(0xffffffffu, L, o2);
            v.x += __shfl_xor_sync(0xffffffffu, v.x, o2); v.y += __shfl_xor_sync(0xffffffffu, v.y, o2);
            v.z += __shfl_xor_sync(0xffffffffu, v.z, o2); v.w += __shfl_xor_sync(0xffffffffu, v.w, o2);
        }
        if (a.sink) L += ex2(-top);
        if (u < items && first == 0) {
            float* dst = a.out + (size_t)b * a.ldo + (size_t)(h0 + r) * a.vdim + 4 * c;
            const float e[4] = {v.x, v.y, v.z, v.w}, inv = 1.0f / L;
#pragma unroll
            for (int i = 0; i < 4; i++)
                if (4 * c + i < a.vdim) dst[i] = e[i] * inv;
        }
    }
}

size_t gp_smem(const GroupedAttnArgs& a, int keys) {
    const GdShape g = gd_shape(a.kw, a.vw, a.vcache == nullptr, keys);
    return 1024 + (size_t)kGpStages * g.tile + (size_t)kGpRows * g.LDQ * 2 + (size_t)kGpStages * keys * 4;
}

// VN: most output n-tiles, KEYS: keys per tile
template <int VN, int KEYS>
__global__ void __launch_bounds__(kGpThreads, 1) k_grouped_prefill(const __grid_constant__ GdParams p, const __nv_bfloat16* __restrict__ qp) {
    extern __shared__ __align__(1024) unsigned char gd_raw[];
    __shared__ __align__(8) unsigned long long s_bar[2 * kGpStages];
    __shared__ volatile int s_abort;
    constexpr int NT = KEYS / 8;
    const GroupedAttnArgs& a = p.a;
    const bool shared = a.vcache == nullptr;
    const GdShape S = gd_shape(a.kw, a.vw, shared, KEYS);
    const int vt = (shared ? a.kw : a.vw) / 8;
    const uint32_t raw = smem_u32(gd_raw), skip = ((raw + 1023u) & ~1023u) - raw;
    unsigned char* ring = gd_raw + skip;
    __nv_bfloat16* Qs = reinterpret_cast<__nv_bfloat16*>(ring + (size_t)kGpStages * S.tile);        // [kGpRows][LDQ]
    float* scales = reinterpret_cast<float*>(Qs + kGpRows * S.LDQ);                               // [stage][KEYS]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, rl = lane >> 2, t4 = lane & 3;
    const int rep = a.H / a.G, rows = a.T * rep, b = blockIdx.y / a.G, g = blockIdx.y - b * a.G;
    const int r0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kGpRows;         // the rows with the most keys first
    pdl_wait();
    pdl_launch_dependents();
    const int pos0 = (int)a.pos[b];
    if (pos0 < 0 || pos0 + a.T > a.maxSeq) return;
    const int lastKey = pos0 + (min(rows, r0 + kGpRows) - 1) / rep;
    const float* ksc = a.kscale + (size_t)blockIdx.y * a.kpitch;
    const int kq = a.kw / 8, plane = blockIdx.y * a.maxSeq, tiles = lastKey / KEYS + 1;
    auto full = [&](int stage) { return smem_u32(&s_bar[stage]); };
    auto empty = [&](int stage) { return smem_u32(&s_bar[kGpStages + stage]); };
    if (tid == 0) {
        for (int i = 0; i < kGpStages; i++) { mbar_init(full(i), 1); mbar_init(empty(i), kGpThreads / 32); }
        s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    // by one thread; rows past the newest key are whatever earlier requests left: finite, and masked
    auto load = [&](int tile) {
        const int k0 = tile * KEYS, stage = tile % kGpStages;
        uint32_t dst = smem_u32(ring + stage * S.tile);
        mbar_arrive_expect_tx(full(stage), (uint32_t)(S.tile + (shared ? KEYS * 4 : 0)));
        for (int c = 0; c < S.kb; c++, dst += KEYS * 128) tma_box(dst, &p.k, c * 64, plane + k0, full(stage));
        for (int c = 0; c < S.vb; c++, dst += KEYS * 128) tma_box(dst, &p.v, c * 64, plane + k0, full(stage));
        if (shared) bulk_g2s(smem_u32(scales + stage * KEYS), ksc + k0, KEYS * 4, full(stage));
    };
    int issued = 0;
    if (tid == 0)
        for (; issued < min(kGpStages - 1, tiles); issued++) load(issued);
    const __nv_bfloat16* q0 = qp + ((size_t)blockIdx.y * rows + r0) * a.kw;
    for (int i = tid; i < kGpRows * S.kb * 8; i += kGpThreads) {
        const int r = i / (S.kb * 8), c = i - r * (S.kb * 8);
        *reinterpret_cast<uint4*>(Qs + r * S.LDQ + c * 8) =
            r0 + r < rows && c < kq ? *reinterpret_cast<const uint4*>(q0 + (size_t)r * a.kw + c * 8) : make_uint4(0, 0, 0, 0);
    }
    __syncthreads();
    const int w0 = r0 + warp * 16, ra = w0 + rl, rb = ra + 8;
    const int limA = ra < rows ? pos0 + ra / rep : -1, limB = rb < rows ? pos0 + rb / rep : -1;      // newest key of a row
    const int warpLast = w0 < rows ? pos0 + (min(rows, w0 + 16) - 1) / rep : -1, warpFirst = pos0 + w0 / rep;
    const float* relA = a.rel ? a.rel + (size_t)(g * rep + ra % rep) * a.relLen : nullptr;
    const float* relB = a.rel ? a.rel + (size_t)(g * rep + rb % rep) * a.relLen : nullptr;
    const float farA = a.rel ? bias_at(relA, a.relLen - 1, a.relLen) : 0.0f, farB = a.rel ? bias_at(relB, a.relLen - 1, a.relLen) : 0.0f;
    const uint32_t qAddr = smem_u32(Qs) + (uint32_t)(((warp * 16 + (lane & 15)) * S.LDQ + (lane >> 4) * 8) * 2);
    uint32_t kOff[4], vOff[4];                               // operand B, columns 16i of a box: from rows of keys, and read transposed
#pragma unroll
    for (int i = 0; i < 4; i++) {
        kOff[i] = swizzled((lane & 7) + ((lane >> 4) << 3), 2 * i + ((lane >> 3) & 1), 0);
        vOff[i] = swizzled((lane & 7) + (((lane >> 3) & 1) << 3), 2 * i + (lane >> 4), 0);
    }
    float o[VN][4];
#pragma unroll
    for (int j = 0; j < VN; j++) { o[j][0] = 0.0f; o[j][1] = 0.0f; o[j][2] = 0.0f; o[j][3] = 0.0f; }
    float mA = -INFINITY, mB = -INFINITY, lA = 0.0f, lB = 0.0f;
    for (int tile = 0; tile < tiles; tile++) {
        const int stage = tile % kGpStages, k0 = tile * KEYS;
        if (tid == 0 && issued < tiles) {                    // the tile two ahead goes where the last one was
            if (issued < kGpStages || mbar_wait(empty(issued % kGpStages), (issued / kGpStages - 1) & 1, &s_abort, p.error, 223)) load(issued++);
        }
        __syncwarp();
        if (!__all_sync(0xffffffffu, mbar_wait(full(stage), (tile / kGpStages) & 1, &s_abort, p.error, 222))) break;
        auto release = [&] { __syncwarp(); if (lane == 0) mbar_arrive(empty(stage)); };
        if (k0 > warpLast) { release(); continue; }
        const unsigned char* K = ring + stage * S.tile;
        const float* sc = scales + stage * KEYS;
        float s[NT][4];
#pragma unroll
        for (int j = 0; j < NT; j++) { s[j][0] = 0.0f; s[j][1] = 0.0f; s[j][2] = 0.0f; s[j][3] = 0.0f; }
        const uint32_t kAddr = smem_u32(K);
        for (int c = 0; c < S.kb; c++)
#pragma unroll
            for (int kk = 0; kk < 4; kk++) {
                uint32_t aq[4];
                ldm_x4(aq, qAddr + c * 128 + kk * 32);
#pragma unroll
                for (int n = 0; n < NT; n += 2) {
                    uint32_t bk[4];
                    ldm_x4(bk, kAddr + kOff[kk] + c * (KEYS * 128) + n * 8 * 128);
                    mma_bf16(s[n], aq, bk[0], bk[1]); mma_bf16(s[n + 1], aq, bk[2], bk[3]);
                }
            }
        if (shared) {
#pragma unroll
            for (int j = 0; j < NT; j++) {
                const float2 f = *reinterpret_cast<const float2*>(sc + j * 8 + 2 * t4);
                s[j][0] *= f.x; s[j][1] *= f.y; s[j][2] *= f.x; s[j][3] *= f.y;
            }
        }
        const bool whole = k0 + KEYS - 1 <= warpFirst;       // every row of the warp sees the whole tile
        if (whole && (a.rel == nullptr || warpFirst - (k0 + KEYS - 1) >= a.relLen - 1)) {
            if (a.rel) {
#pragma unroll
                for (int j = 0; j < NT; j++) { s[j][0] += farA; s[j][1] += farA; s[j][2] += farB; s[j][3] += farB; }
            }
        } else {
#pragma unroll
            for (int j = 0; j < NT; j++)
#pragma unroll
                for (int e = 0; e < 2; e++) {
                    const int i = j * 8 + 2 * t4 + e, dA = limA - k0 - i, dB = limB - k0 - i;
                    if (a.rel) { s[j][e] += bias_at(relA, max(dA, 0), a.relLen); s[j][2 + e] += bias_at(relB, max(dB, 0), a.relLen); }
                    if (dA < 0) s[j][e] = -INFINITY;
                    if (dB < 0) s[j][2 + e] = -INFINITY;
                }
        }
        float xA = -INFINITY, xB = -INFINITY;
#pragma unroll
        for (int j = 0; j < NT; j++) { xA = fmaxf(xA, fmaxf(s[j][0], s[j][1])); xB = fmaxf(xB, fmaxf(s[j][2], s[j][3])); }
        xA = fmaxf(mA, quad_max(xA)); xB = fmaxf(mB, quad_max(xB));
        const float uA = xA > -INFINITY ? xA : 0.0f, uB = xB > -INFINITY ? xB : 0.0f;      // a row that has seen no key yet
        const float cA = ex2(mA - uA), cB = ex2(mB - uB);
        mA = xA; mB = xB;
        float pA = 0.0f, pB = 0.0f;
#pragma unroll
        for (int j = 0; j < NT; j++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                s[j][e] = ex2(s[j][e] - uA); s[j][2 + e] = ex2(s[j][2 + e] - uB);
                pA += s[j][e]; pB += s[j][2 + e];
            }
        lA = lA * cA + pA; lB = lB * cB + pB;
        if (__any_sync(0xffffffffu, cA != 1.0f || cB != 1.0f)) {
#pragma unroll
            for (int c = 0; c < VN; c++) { o[c][0] *= cA; o[c][1] *= cA; o[c][2] *= cB; o[c][3] *= cB; }
        }
        const uint32_t vAddr = smem_u32(shared ? K : K + S.kb * KEYS * 128);
#pragma unroll
        for (int kk = 0; kk < KEYS / 16; kk++) {
            uint32_t ph[4], pl[4];
            split_bf16(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]); split_bf16(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
            split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]); split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
            for (int c = 0; c < VN; c += 4) {
                if (c >= vt) break;
                uint32_t bv[2][4];
                ldm_x4_t(bv[0], vAddr + vOff[(c & 7) / 2] + (c >> 3) * (KEYS * 128) + kk * 16 * 128);
                ldm_x4_t(bv[1], vAddr + vOff[(c & 7) / 2 + 1] + (c >> 3) * (KEYS * 128) + kk * 16 * 128);
                mma_bf16(o[c], ph, bv[0][0], bv[0][1]); mma_bf16(o[c + 1], ph, bv[0][2], bv[0][3]);
                mma_bf16(o[c + 2], ph, bv[1][0], bv[1][1]); mma_bf16(o[c + 3], ph, bv[1][2], bv[1][3]);
                mma_bf16(o[c], pl, bv[0][0], bv[0][1]); mma_bf16(o[c + 1], pl, bv[0][2], bv[0][3]);
                mma_bf16(o[c + 2], pl, bv[1][0], bv[1][1]); mma_bf16(o[c + 3], pl, bv[1][2], bv[1][3]);
            }
        }
        release();
    }
    if (tid == 0 && s_abort)                                 // a wait ran out: let the copies in flight land before the block goes
        for (int t = max(0, issued - kGpStages); t < issued; t++)
            for (unsigned w = 0; w < (1u << 16) && !mbar_try_wait(full(t % kGpStages), (t / kGpStages) & 1); w++) {}
    lA = quad_sum(lA); lB = quad_sum(lB);
    auto finish = [&](int r, float m, float l, int e) {
        if (r >= rows) return;
        float f = 1.0f;
        if (a.sink) {
            const float u = fmaxf(m, 0.0f);
            f = ex2(m - u);
            l = l * f + ex2(-u);
        }
        f /= l;
        float* dst = a.out + (size_t)(b * a.T + r / rep) * a.ldo + (size_t)(g * rep + r % rep) * a.vdim;
#pragma unroll
        for (int c = 0; c < VN; c++) {
            const int i = c * 8 + 2 * t4;
            if (i < a.vdim) dst[i] = o[c][e] * f;
            if (i + 1 < a.vdim) dst[i + 1] = o[c][e + 1] * f;
        }
    };
    finish(ra, mA, lA, 0);
    finish(rb, mB, lB, 2);
}

constexpr size_t kSmemMax = 226 * 1024;       // beside the static part
template <typename K>
void raise(K kernel, bool& done) {
    if (!done) DJ_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    done = true;
}
bool cache_map(CUtensorMap* map, const void* base, int width, size_t rows, int keys) {
    EncodeTiledFn enc = encode_tiled_fn();
    if (enc == nullptr) return false;
    const cuuint64_t dims[2] = {(cuuint64_t)width, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)width * 2};
    const cuuint32_t box[2] = {64u, (cuuint32_t)keys};
    const cuuint32_t estr[2] = {1u, 1u};
    return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
               CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
GdParams params(const GroupedAttnArgs& a, int keys) {
    GdParams p = {};
    p.a = a; p.error = g_dev_error;
    const size_t rows = (size_t)a.B * a.G * a.maxSeq;
    if (!cache_map(&p.k, a.kcache, a.kw, rows, keys) || (a.vcache && !cache_map(&p.v, a.vcache, a.vw, rows, keys)))
        throw std::runtime_error("grouped attention: the cache cannot be described to the copy engine");
    return p;
}
// warps of a decode block: eight where two stages of their rings fit; blocks per SM as the registers of its form allow
int gd_warps(const GroupedAttnArgs& a) { return gd_smem(a, 8, 2) <= kSmemMax ? 8 : 4; }
int gd_blocks_per_sm(const GroupedAttnArgs& a) {
    const int vw = a.vcache ? a.vw : a.kw;
    return vw <= 64 && a.kw <= 128 && 2 * gd_smem(a, gd_warps(a), 3) <= kSmemMax ? 2 : 1;
}
int gd_stages(const GroupedAttnArgs& a) {
    const int warps = gd_warps(a);
    const size_t room = kSmemMax / gd_blocks_per_sm(a);
    int n = kGdMaxStages;
    while (n > 2 && gd_smem(a, warps, n) > room) n--;
    return n;
}
template <int VN, int NW>
void decode_with(const GroupedAttnArgs& a, cudaStream_t s) {
    static bool done = false;
    raise(k_grouped_decode<VN, NW>, done);
    GdParams p = params(a, kGdKeys);
    p.splits = grouped_mma_splits(a); p.stages = gd_stages(a);
    launch_k(k_grouped_decode<VN, NW>, dim3((unsigned)p.splits, (unsigned)((a.H / a.G + 7) / 8), (unsigned)(a.B * a.G)), dim3(32 * NW), gd_smem(a, NW, p.stages), s, true, p);
}
template <int VN>
void decode(const GroupedAttnArgs& a, cudaStream_t s) {
    if (gd_warps(a) == 8) decode_with<VN, 8>(a, s);
    else decode_with<VN, 4>(a, s);
}
template <int VN, int KEYS>
void prefill(const GroupedAttnArgs& a, const __nv_bfloat16* q, cudaStream_t s) {
    static bool done = false;
    raise(k_grouped_prefill<VN, KEYS>, done);
    const unsigned blocks = (unsigned)((a.T * (a.H / a.G) + kGpRows - 1) / kGpRows);
    launch_k(k_grouped_prefill<VN, KEYS>, dim3(blocks, (unsigned)(a.B * a.G)), dim3(kGpThreads), gp_smem(a, KEYS), s, true, params(a, KEYS), q);
}

}  // namespace

bool grouped_mma_fits(const GroupedAttnArgs& a) {
    return a.bf16 && (size_t)a.B * a.G * a.maxSeq < (1u << 31) && a.kw <= 256 && a.vw <= 256 && a.kw % 16 == 0 && a.vw % 16 == 0 && (a.vcache != nullptr || a.kpitch % 64 == 0);
}
int grouped_mma_splits(const GroupedAttnArgs& a) {
    const int blocks = a.B * a.G * ((a.H / a.G + 7) / 8), tiles = (a.maxSeq + kGdKeys - 1) / kGdKeys, warps = gd_warps(a);
    return std::max(1, std::min({gd_blocks_per_sm(a) * g_num_sms / blocks, (tiles + warps - 1) / warps, 512}));
}
void launch_grouped_decode(const GroupedAttnArgs& a, cudaStream_t s) {
    const int vw = a.vcache ? a.vw : a.kw;
    if (std::max(a.kw, vw) > 128) decode<32>(a, s);      // both head sizes bound the channels per lane
    else if (vw <= 64) decode<8>(a, s);
    else if (vw <= 128) decode<16>(a, s);
    else decode<32>(a, s);
}
void launch_grouped_prefill(const GroupedAttnArgs& a, const __nv_bfloat16* q, int qw, cudaStream_t s) {
    if (qw != a.kw) throw std::runtime_error("grouped attention: query rows do not match the cache");
    const int vw = a.vcache ? a.vw : a.kw;
    if (vw <= 64) prefill<8, 64>(a, q, s);
    else if (vw <= 128) prefill<16, 64>(a, q, s);
    else prefill<32, 32>(a, q, s);
}

}  // namespace dj
