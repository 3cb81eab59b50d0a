// Many-row projections with bf16 weights on the 5th-generation tensor cores: out[M × N] = A[M × K] · W[N × K]ᵀ.
//
// The activation rows are staged to bf16 in the workspace by k_stage_rows (norm and gate applied in fp32 there); both
// operands then travel as 64-column boxes with 128-byte swizzle through the tensor-memory accelerator.  Persistent CTAs,
// one per SM, walk 128 × BN output tiles (rows of tiles fastest: CTAs that run together share a weight tile in L2):
//   warp 4   one thread keeps a ring of (A, W) stages full; the first stages' weights are on their way before the
//            dependency wait
//   warp 5   one thread issues tcgen05.mma 128 × BN × 16 into one of two accumulators in tensor memory
//   warps 0-3  drain the other accumulator: tcgen05.ld, a shared-memory transpose, row-contiguous stores with residual,
//            soft cap or the gated pair
// Grouped form (table-routed experts): `tileExpert` gives each 128-row tile its expert (−1: no tile), whose weight rows
// start at expert · N; `rowMap` scatters output rows.  Every wait is bounded (codes 211-214 in the device error word).
#include "row_operand.cuh"
#include "tc_common.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr int kGM = 128, kGK = 64, kGThreads = 192;
constexpr int kABytes = kGM * kGK * 2;
constexpr int kEpiBytes = 4 * 32 * 33 * 4;

struct GemmTcParams {
    CUtensorMap a, w;
    int M, N, nK, mTiles, nTiles;
    const int* tileExpert; const int* rowMap;
    const float* lenPos; int lenT;               // rows = lenPos[0] + lenT, at most M (device-side length)
    const float* residual; int ldr;
    float* out; int ldo; __nv_bfloat16* outHalf; // outHalf: bf16 rows instead of fp32
    int gluRow; float limit; float* glu; int ldglu;
    float softcap; const float* bias; int pair;
    int* error;
};

// K-major, 128-byte swizzle: 8-row groups 1024 bytes apart, descriptor version 1, layout type 2
__device__ __forceinline__ uint64_t desc_sw128(uint32_t smem_addr) {
    return (uint64_t)((smem_addr >> 4) & 0x3fff) | ((uint64_t)1 << 16) | ((uint64_t)(1024 >> 4) << 32) | ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}

template <int BN> struct GemmShape {
    static constexpr int kStageBytes = kABytes + BN * kGK * 2;
    static constexpr int kStages = BN == 256 ? 4 : BN == 128 ? 6 : 8;
    static constexpr size_t kSmem = (size_t)kStages * kStageBytes + kEpiBytes + 1024;
    static constexpr int kTmem = 2 * BN < 32 ? 32 : 2 * BN;
    // bf16 × bf16 → fp32, both K-major
    static constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(kGM >> 4) << 24);
};

template <int BN>
__global__ void __launch_bounds__(kGThreads, 1) k_bf16_gemm_tc(const __grid_constant__ GemmTcParams p) {
    using S = GemmShape<BN>;
    extern __shared__ __align__(1024) unsigned char smem[];
    __shared__ __align__(8) unsigned long long s_bar[2 * S::kStages + 4];
    __shared__ uint32_t s_tmem;
    __shared__ volatile int s_abort;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const uint32_t raw = smem_u32(smem), base = (raw + 1023u) & ~1023u;
    float* const stg = reinterpret_cast<float*>(smem + (base - raw) + (size_t)S::kStages * S::kStageBytes) + warp * (32 * 33);
    auto full = [&](int s) { return smem_u32(&s_bar[s]); };
    auto empty = [&](int s) { return smem_u32(&s_bar[S::kStages + s]); };
    auto accFull = [&](int a) { return smem_u32(&s_bar[2 * S::kStages + a]); };
    auto accEmpty = [&](int a) { return smem_u32(&s_bar[2 * S::kStages + 2 + a]); };
    if (tid == 0) {
        for (int s = 0; s < S::kStages; s++) { mbar_init(full(s), 1); mbar_init(empty(s), 1); }
        for (int a = 0; a < 2; a++) { mbar_init(accFull(a), 1); mbar_init(accEmpty(a), 128); }
        s_abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 4) tmem_alloc(smem_u32(&s_tmem), S::kTmem);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = s_tmem;
    int rows = p.M, mTiles = p.mTiles, tiles = p.mTiles * p.nTiles;
    auto read_length = [&] {                         // after the dependency wait
        if (p.lenPos != nullptr) {
            rows = min(p.M, max((int)p.lenPos[0], 0) + p.lenT);
            mTiles = (rows + kGM - 1) / kGM;
            tiles = mTiles * p.nTiles;
        }
    };

    if (warp == 4) {
        if (lane == 0) {
            int early = 0;                                   // stages whose weights were requested before the wait
            if (p.tileExpert == nullptr && p.lenPos == nullptr && (int)blockIdx.x < tiles) {
                const int n0 = ((int)blockIdx.x / p.mTiles) * BN;
                for (; early < S::kStages && early < p.nK; early++) {
                    mbar_arrive_expect_tx(full(early), S::kStageBytes);
                    tma_box(base + early * S::kStageBytes + kABytes, &p.w, early * kGK, n0, full(early));
                }
            }
            pdl_wait();
            pdl_launch_dependents();
            read_length();
            unsigned it = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const int mt = t % mTiles;
                int wrow = (t / mTiles) * BN;
                if (p.tileExpert != nullptr) {
                    const int e = p.tileExpert[mt];
                    if (e < 0) continue;
                    wrow += e * p.N;
                }
                for (int kt = 0; kt < p.nK; kt++, it++) {
                    const int s = it % S::kStages;
                    const uint32_t dst = base + s * S::kStageBytes;
                    if ((int)it >= early) {
                        if (it >= (unsigned)S::kStages && !mbar_wait(empty(s), (it / S::kStages - 1) & 1, &s_abort, p.error, 211)) { ok = false; break; }
                        mbar_arrive_expect_tx(full(s), S::kStageBytes);
                        tma_box(dst + kABytes, &p.w, kt * kGK, wrow, full(s));
                    }
                    tma_box(dst, &p.a, kt * kGK, mt * kGM, full(s));
                }
            }
            if (!ok)                                         // a wait ran out: let the copies in flight land before the block goes
                for (unsigned back = 1; back <= (unsigned)S::kStages && back <= it; back++) {
                    const unsigned j = it - back;
                    for (unsigned w = 0; w < (1u << 16) && !mbar_try_wait(full(j % S::kStages), (j / S::kStages) & 1); w++) {}
                }
        }
        __syncwarp();
    } else if (warp == 5) {
        if (lane == 0) {
            pdl_wait();
            pdl_launch_dependents();
            read_length();
            unsigned it = 0, n = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                if (p.tileExpert != nullptr && p.tileExpert[t % mTiles] < 0) continue;
                const int a = n & 1;
                if (n >= 2 && !mbar_wait(accEmpty(a), (n / 2 - 1) & 1, &s_abort, p.error, 212)) break;
                tc_fence_after();
                for (int kt = 0; kt < p.nK; kt++, it++) {
                    const int s = it % S::kStages;
                    if (!mbar_wait(full(s), (it / S::kStages) & 1, &s_abort, p.error, 213)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t sa = base + s * S::kStageBytes, sw = sa + kABytes;
#pragma unroll
                    for (int k = 0; k < kGK / 16; k++)
                        umma_f16(tmem + (uint32_t)(a * BN), desc_sw128(sa + k * 32), desc_sw128(sw + k * 32), S::kIdesc, (kt | k) != 0);
                    umma_commit(empty(s));
                }
                if (ok) umma_commit(accFull(a));
                n++;
            }
        }
        __syncwarp();
    } else {
        pdl_wait();
        pdl_launch_dependents();
        read_length();
        unsigned n = 0;
        for (int t = blockIdx.x; t < tiles; t += gridDim.x) {
            const int mt = t % mTiles, n0 = (t / mTiles) * BN;
            if (p.tileExpert != nullptr && p.tileExpert[mt] < 0) continue;
            const int a = n & 1;
            if (!__all_sync(0xffffffffu, mbar_wait(accFull(a), (n / 2) & 1, &s_abort, p.error, 214))) break;
            tc_fence_after();
            const int mBase = mt * kGM + warp * 32;
            int myRow = mBase + lane < rows ? mBase + lane : -1;      // output row of tile row `lane`
            if (myRow >= 0 && p.rowMap != nullptr) myRow = p.rowMap[myRow];
#pragma unroll 1
            for (int c0 = 0; c0 < BN && n0 + c0 < p.N; c0 += 32) {
                uint32_t v[32];
                tmem_ld32(tmem + ((uint32_t)(warp * 32) << 16) + (uint32_t)(a * BN + c0), v);
#pragma unroll
                for (int j = 0; j < 32; j++) stg[lane * 33 + j] = __uint_as_float(v[j]);
                __syncwarp();
                const int nb = n0 + c0, nn = nb + lane;
                if (p.outHalf != nullptr) {
#pragma unroll 8
                    for (int i = 0; i < 32; i += 2) {
                        const int r = i + (lane >> 4), row = __shfl_sync(0xffffffffu, myRow, r), c = 2 * (lane & 15);
                        if (row >= 0 && nb + c < p.N)
                            *reinterpret_cast<__nv_bfloat162*>(p.outHalf + (size_t)row * p.ldo + nb + c) = __floats2bfloat162_rn(stg[r * 33 + c], stg[r * 33 + c + 1]);
                    }
                    __syncwarp();
                    continue;
                }
                if (nb < p.gluRow) {
                    const float myBias = p.bias != nullptr && nn < p.gluRow ? p.bias[nn] : 0.0f;
#pragma unroll 8
                    for (int i = 0; i < 32; i++) {
                        const int row = __shfl_sync(0xffffffffu, myRow, i);
                        if (row >= 0 && nn < p.gluRow) {
                            float val = stg[i * 33 + lane] + myBias;
                            if (p.residual) val += p.residual[(size_t)row * p.ldr + nn];
                            p.out[(size_t)row * p.ldo + nn] = softcap_f(val, p.softcap);
                        }
                    }
                }
                if (nb + 32 > p.gluRow && p.gluRow < p.N) {
                    const int pair = nb + 2 * (lane & 15);
#pragma unroll 4
                    for (int i = 0; i < 32; i += 2) {
                        const int r = i + (lane >> 4), row = __shfl_sync(0xffffffffu, myRow, r);
                        if (row >= 0 && pair >= p.gluRow && pair < p.N) {
                            const float g = stg[r * 33 + 2 * (lane & 15)], u = stg[r * 33 + 2 * (lane & 15) + 1];
                            p.glu[(size_t)row * p.ldglu + ((pair - p.gluRow) >> 1)] = pair_f(g, u, p.limit, p.pair);
                        }
                    }
                }
                __syncwarp();
            }
            tc_fence_before();
            mbar_arrive(accEmpty(a));
            n++;
        }
    }
    __syncthreads();
    if (warp == 4) { tc_fence_after(); tmem_dealloc(tmem, S::kTmem); }
}

bool encode_rows(CUtensorMap* map, const void* base, size_t K, size_t pitch, size_t rows, int boxRows) {
    EncodeTiledFn enc = encode_tiled_fn();
    if (!enc) return false;
    const cuuint64_t dims[2] = {(cuuint64_t)K, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)pitch * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kGK, (cuuint32_t)boxRows};
    const cuuint32_t estr[2] = {1u, 1u};
    return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
               CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int BN>
bool run(GemmTcParams& p, const void* a, int aK, int aPitch, size_t aRows, const Bf16View& w, cudaStream_t s) {
    using S = GemmShape<BN>;
    if (!encode_rows(&p.a, a, aK, aPitch, aRows, kGM) || !encode_rows(&p.w, w.w, w.Kp, w.Kp, w.N, BN)) return false;
    static bool attr = false;
    if (!attr) {
        DJ_CUDA_CHECK(cudaFuncSetAttribute(k_bf16_gemm_tc<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)S::kSmem));
        attr = true;
    }
    p.nTiles = (p.N + BN - 1) / BN;
    const int grid = std::min(p.mTiles * p.nTiles, g_num_sms);
    launch_k(k_bf16_gemm_tc<BN>, dim3((unsigned)grid), dim3(kGThreads), S::kSmem, s, true, p);
    return true;
}

// the tile width with the least work per SM, wider tiles first
int pick_width(int mTiles, int N) {
    int best = 256; double bestCost = 1e30;
    for (int bn : {256, 128, 64}) {
        const long tiles = (long)mTiles * ((N + bn - 1) / bn);
        const double cost = (double)((tiles + g_num_sms - 1) / g_num_sms) * (bn + 24);
        if (cost < bestCost) { bestCost = cost; best = bn; }
    }
    return best;
}
bool run_width(int bn, GemmTcParams& p, const void* a, int aK, int aPitch, size_t aRows, const Bf16View& w, cudaStream_t s) {
    return bn == 256 ? run<256>(p, a, aK, aPitch, aRows, w, s) : bn == 128 ? run<128>(p, a, aK, aPitch, aRows, w, s) : run<64>(p, a, aK, aPitch, aRows, w, s);
}

}  // namespace

// Plain form: stages a.M rows into a.ws, then multiplies.  Grouped form (tileExpert): the staged rows are in a.ws already,
// a.M of them in whole 128-row tiles, a.w holds every expert's a.nPer rows.  False when the shape does not qualify.
bool launch_bf16_gemm_tc(const Bf16LinearArgs& a, const GroupedRows* g, cudaStream_t s) {
    if (g_dev_error == nullptr || encode_tiled_fn() == nullptr || a.w.Kp % 8 != 0 || ((uintptr_t)a.ws & 15) != 0) return false;
    GemmTcParams p;
    p.M = a.M; p.N = g ? g->rowsPerExpert : a.w.N; p.nK = (a.w.Kp + kGK - 1) / kGK; p.mTiles = (a.M + kGM - 1) / kGM;
    p.tileExpert = g ? g->tileExpert : nullptr; p.rowMap = g ? g->rowMap : nullptr;
    p.residual = a.residual; p.ldr = a.ldr; p.out = a.out; p.ldo = a.ldo;
    p.gluRow = a.gluRow; p.limit = a.limit; p.glu = a.glu; p.ldglu = a.ldglu; p.softcap = a.softcap; p.bias = a.bias; p.pair = a.pair;
    p.error = g_dev_error;
    p.lenPos = nullptr; p.lenT = 0; p.outHalf = nullptr;
    if (!g) launch_stage_rows(a.a, a.b, a.w.Kp, a.M, nullptr, 1, a.ws, true, s);
    return run_width(pick_width(p.mTiles, p.N), p, a.ws, a.w.Kp, a.w.Kp, a.M, a.w, s);
}

void launch_bf16_gemm_rows(const __nv_bfloat16* rows, int lda, int K, const float* pos, int T, int maxRows, const Bf16View& w, __nv_bfloat16* out, int ldo,
                           cudaStream_t s) {
    GemmTcParams p = {};
    p.M = maxRows; p.N = w.N; p.nK = (K + kGK - 1) / kGK; p.mTiles = (maxRows + kGM - 1) / kGM;
    p.lenPos = pos; p.lenT = T; p.outHalf = out; p.ldo = ldo; p.gluRow = w.N; p.error = g_dev_error;
    if (lda % 8 != 0 || w.Kp % 8 != 0 || (w.N & 1) != 0 || g_dev_error == nullptr || !run_width(pick_width(p.mTiles, p.N), p, rows, K, lda, maxRows, w, s))
        throw std::runtime_error("bf16 product over cached rows: the shape does not qualify");
}

}  // namespace dj
