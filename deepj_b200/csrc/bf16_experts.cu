// Table-routed experts: a table row indexed by the token id names the `top` experts of the token, each of weight 1/top.
//
// Few rows, or models run in 32-bit: every (token, slot) entry is its own GEMV over its expert's weight rows
// (bf16_linear.cu).  Many rows: the entries are sorted by expert into 128-row tiles and the feed-forward runs as two
// grouped tensor-core products (bf16_gemm_tc.cu):
//   k_expert_plan     one block: entries per expert, tile → expert, padded position → entry
//   k_stage_rows      gathers the normed rows of the entries in that order
//   grouped product   gate and up pairs → gated values in the same order; staged again; down → one row per entry
//   k_expert_combine  out = residual + (1/top) Σ of the token's entry rows, in slot order
#include "row_operand.cuh"

#include <algorithm>

namespace dj {
namespace {

constexpr int kPlanThreads = 1024, kMaxExperts = 2048, kTileRows = 128;

__global__ void __launch_bounds__(kPlanThreads) k_expert_plan(const float* __restrict__ tok, const float* __restrict__ table, int entries, int top, int vocab,
                                                              int experts, int tiles, int* __restrict__ tileExpert, int* __restrict__ entryAt) {
    __shared__ int count[kMaxExperts], next[kMaxExperts];
    pdl_wait();
    pdl_launch_dependents();
    auto expert_of = [&](int e) {
        const int id = min(max((int)tok[e / top], 0), vocab - 1);
        return (int)table[(size_t)id * top + e % top];
    };
    for (int i = threadIdx.x; i < experts; i += kPlanThreads) count[i] = 0;
    for (int i = threadIdx.x; i < tiles * kTileRows; i += kPlanThreads) entryAt[i] = -1;
    for (int i = threadIdx.x; i < tiles; i += kPlanThreads) tileExpert[i] = -1;
    __syncthreads();
    for (int e = threadIdx.x; e < entries; e += kPlanThreads) atomicAdd(&count[expert_of(e)], 1);
    __syncthreads();
    if (threadIdx.x == 0) {
        int tile = 0;
        for (int i = 0; i < experts; i++) {
            next[i] = tile * kTileRows;
            for (int n = (count[i] + kTileRows - 1) / kTileRows; n > 0; n--) tileExpert[tile++] = i;
        }
    }
    __syncthreads();
    // where an entry lands inside its expert's rows does not matter: every row is computed on its own
    for (int e = threadIdx.x; e < entries; e += kPlanThreads) entryAt[atomicAdd(&next[expert_of(e)], 1)] = e;
}

__global__ void __launch_bounds__(256) k_expert_combine(const float* __restrict__ rows, int top, int d, const float* residual, int ldr, float* out, int ldo) {
    pdl_wait();
    pdl_launch_dependents();
    const int m = blockIdx.x;
    for (int n = threadIdx.x; n < d; n += 256) {
        float v = 0.0f;
        for (int s = 0; s < top; s++) v += rows[((size_t)m * top + s) * d + n];
        out[(size_t)m * ldo + n] = (residual ? residual[(size_t)m * ldr + n] : 0.0f) + v / (float)top;
    }
}

struct Layout { int tiles, rows; size_t stage, y, o, ints, total; };
Layout layout(const Bf16ExpertArgs& e) {
    Layout l;
    const int entries = e.M * e.top;
    l.tiles = std::min(entries, (entries + kTileRows - 1) / kTileRows + e.experts);      // a partly filled tile per expert at most
    l.rows = l.tiles * kTileRows;
    auto up64 = [](size_t n) { return (n + 63) / 64 * 64; };
    const size_t stageUp = up64((size_t)l.rows * e.up.Kp / 2 + 1), stageDown = up64((size_t)l.rows * e.down.Kp / 2 + 1);
    l.stage = 0;
    l.y = std::max(stageUp, stageDown);
    l.o = l.y + up64((size_t)l.rows * e.ff);
    l.ints = l.o + up64((size_t)entries * e.d);
    l.total = l.ints + up64((size_t)l.rows + l.tiles);
    return l;
}

constexpr int kGroupedMinEntries = 64;
bool grouped(const Bf16ExpertArgs& e) {
    return !e.exact && e.M > 16 && e.M * e.top >= kGroupedMinEntries && e.experts <= kMaxExperts;
}

}  // namespace

size_t bf16_experts_ws_floats(const Bf16ExpertArgs& e) {
    const size_t plain = (size_t)e.M * e.top * e.ff;
    return grouped(e) ? std::max(plain, layout(e).total) : plain;
}

void launch_bf16_experts(const Bf16ExpertArgs& e, cudaStream_t s) {
    if (e.M <= 0) return;
    if (!grouped(e)) {
        launch_bf16_expert_gemv(e, e.ws, s);
        return;
    }
    const Layout l = layout(e);
    int* entryAt = reinterpret_cast<int*>(e.ws + l.ints);
    int* tileExpert = entryAt + l.rows;
    launch_k(k_expert_plan, dim3(1), dim3(kPlanThreads), 0, s, true, e.tok, e.table, e.M * e.top, e.top, e.vocab, e.experts, l.tiles, tileExpert, entryAt);
    GroupedRows g = {tileExpert, nullptr, 2 * e.ff};
    launch_stage_rows(e.x, RowOperand(), e.up.Kp, l.rows, entryAt, e.top, e.ws + l.stage, true, s);
    Bf16LinearArgs up;
    up.w = e.up; up.M = l.rows; up.ws = e.ws + l.stage; up.gluRow = 0; up.limit = e.limit; up.glu = e.ws + l.y; up.ldglu = e.ff;
    bool ok = launch_bf16_gemm_tc(up, &g, s);
    RowOperand y;
    y.x = e.ws + l.y; y.ldx = e.ff; y.k = e.ff;
    if (ok) launch_stage_rows(y, RowOperand(), e.down.Kp, l.rows, nullptr, 1, e.ws + l.stage, true, s);
    Bf16LinearArgs down;
    down.w = e.down; down.M = l.rows; down.ws = e.ws + l.stage; down.gluRow = e.d; down.out = e.ws + l.o; down.ldo = e.d;
    g.rowMap = entryAt; g.rowsPerExpert = e.d;
    ok = ok && launch_bf16_gemm_tc(down, &g, s);
    if (!ok) { launch_bf16_expert_gemv(e, e.ws, s); return; }
    launch_k(k_expert_combine, dim3((unsigned)e.M), dim3(256), 0, s, true, (const float*)(e.ws + l.o), e.top, e.d, e.residual, e.ldr, e.out, e.ldo);
}

}  // namespace dj
