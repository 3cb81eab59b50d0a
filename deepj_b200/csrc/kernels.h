// Launcher declarations shared by the runtime (runtime.cu) and the kernel files.
// Every launcher enqueues on the given stream and never synchronises.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <cstdint>
#include <cstdlib>
#include <stdexcept>
#include <string>
#include <utility>
#include <vector>

#define DJ_CUDA_CHECK(expr)                                                                  \
    do {                                                                                     \
        cudaError_t _e = (expr);                                                             \
        if (_e != cudaSuccess)                                                               \
            throw std::runtime_error(std::string("CUDA error: ") + cudaGetErrorString(_e) + \
                                     " at " + __FILE__ + ":" + std::to_string(__LINE__));   \
    } while (0)

// Launchers of kernel files that a library built for one model family may leave out (build.py); the interpreter
// refuses their ops with a message when they are absent.
#define DJ_PART __attribute__((weak))

namespace dj {

// Counts kernel launches issued by this library (eager path and capture).
extern long long g_launches;
extern int g_num_sms;
// When true, launchers attach the programmatic-dependent-launch attribute so that
// a kernel's weight prefetch overlaps the tail of its predecessor.
extern bool g_use_pdl;
// Q8 GEMV kernel choice (environment DEEPJ_CUDA_GEMV = cpasync | fma to step down); shapes outside a
// kernel's domain fall through to the next one.
extern int g_gemv_mode;
extern int g_tc_terms;      // deepj_cuda_tc_configure
// Device int set non-zero when a bounded wait inside a kernel expired.
extern int* g_dev_error;
// Phase-trace ring (null unless tracing is on) and the number of traced launches so far.
constexpr int kTraceSlots = 4096;
extern unsigned long long* g_trace;
extern long long g_trace_launches;
unsigned long long* trace_slot();

// A Q8 weight as laid out in HBM: codes[N][Kp] int8 (Kp = K rounded up to 16, zero
// padded) followed by scales[N][nb] fp32, nb = ceil(K/32).
struct Q8View {
    const int8_t* codes;
    const float* scales;
    int K, N, Kp, nb;
};

// ── base ops (ComputeGraph op codes 1-42) ──
DJ_PART void launch_binary(int op, const float* a, const float* b, float* out, int n, cudaStream_t s);
DJ_PART void launch_unary(int op, const float* in, float* out, int n, cudaStream_t s);
DJ_PART void launch_scalar(int op, const float* in, float* out, float v, int n, cudaStream_t s);
DJ_PART void launch_clamp(const float* in, float* out, float lo, float hi, int n, cudaStream_t s);
DJ_PART void launch_matmul_f32(const float* a, const float* b, float* out, int m, int n, int k, cudaStream_t s);
DJ_PART void launch_transpose(const float* in, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_row_broadcast(int op, const float* a, const float* v, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_col_broadcast(int op, const float* a, const float* v, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_row_reduce(int op, const float* in, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_sum_rows(const float* in, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_sum_scalar(const float* in, float* out, long long n, cudaStream_t s);
DJ_PART void launch_softmax_rows(const float* in, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_softmax_backward(const float* g, const float* sm, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_layernorm_backward(const float* dxh, const float* xh, const float* sd, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_adamw(float* w, const float* g, float* mt, float* vt, float lr, float b1, float b2, float eps,
                  float wd, float bc1, float bc2, int n, cudaStream_t s);
DJ_PART void launch_scatter_add_rows(float* target, const float* idx, const float* grad, int tRows, int tCols, int nIdx, cudaStream_t s);
DJ_PART void launch_ce_loss(const float* logits, const float* targets, float* out, int rows, int cols, cudaStream_t s);
DJ_PART void launch_ce_grad(const float* logits, const float* targets, float* out, int rows, int cols, cudaStream_t s);

// ── Q8 ──
DJ_PART void launch_q8_quantize(const float* src, int src_ld, int K, int n_cols, int8_t* codes, float* scales,
                        int Kp, int nb, cudaStream_t s);
struct Q8LinearArgs {
    const float* x; int ldx;            // activations [M × K], row stride ldx
    const float* gamma; float eps;      // RMSNorm fused into the activation load when gamma != nullptr
    Q8View w;                           // plain linear / SwiGLU gate
    const float* bias;
    Q8View w2;                          // SwiGLU up projection (codes == nullptr → plain linear)
    const float* bias2;
    const float* residual; int ldr;
    float* out; int ldo;
    int M;
    float* ws = nullptr; int* tickets = nullptr;    // workspace (q8_batch_ws_floats) and counters for the batched kernel (M ≥ 3)
    // GPT blocks: beta != nullptr turns the fused norm into LayerNorm1D (mean and biased variance, γ and β);
    // act == 1 applies GELU after the bias.  The GEMV fuses both; the many-row kernels get them from a
    // normalising pass into ln_ws ([M × K] floats) before and an activation pass over `out` after.
    const float* beta = nullptr; int act = 0; float* ln_ws = nullptr;
};
DJ_PART void launch_q8_linear(const Q8LinearArgs& a, cudaStream_t s);
DJ_PART bool launch_q8_gemv_i8(const Q8LinearArgs& a, cudaStream_t s);
DJ_PART bool launch_q8_gemv_tma(const Q8LinearArgs& a, cudaStream_t s);     // K a multiple of 128; false = outside its domain
DJ_PART bool q8_gemv_i8_fuses_gpt(const Q8LinearArgs& a);     // true when launch_q8_gemv_i8 can take beta / act itself
DJ_PART void launch_layernorm_rows(const float* x, int ldx, const float* gamma, const float* beta, float eps, float* out, int K, int M, cudaStream_t s);
DJ_PART void launch_gelu_rows(float* buf, int ld, int N, int M, cudaStream_t s);
DJ_PART bool launch_q8_linear_batch(const Q8LinearArgs& a, int m0, int rows, float* ws, int* tickets, cudaStream_t s);
DJ_PART bool launch_q8_linear_batch_tma(const Q8LinearArgs& a, int m0, int rows, float* ws, int* tickets, cudaStream_t s);   // K a multiple of 128; same workspace
DJ_PART size_t q8_batch_ws_floats(int K, int N, bool swiglu);
DJ_PART bool launch_q8_linear_tc(const Q8LinearArgs& a, float* ws, cudaStream_t s);
DJ_PART size_t q8_tc_ws_floats(int M, int K, int N);     // activation tiles, row scales and, when the reduction is split, the partial outputs
DJ_PART double q8_tc_estimate_us(int M, int K, int N);
constexpr int kTcMinRows = 17;            // from this many activation rows on, a Q8 linear runs on the tcgen05 path

// ── decode attention ──
struct AttnDecodeArgs {
    float* qkv; int q_off, k_off, v_off, ld;   // current token's projections, one row per sequence
    void* kcache; void* vcache;                // this layer's planes [B][H][maxSeq][hd], fp32 or (kvHalf) fp16
    int maxSeq;
    const float* pos;                          // [B] floats holding the write position
    const float* cosT; const float* sinT;      // [maxSeq × hd/2]
    float* out; int ldo;                       // merged heads [B × H·hd]
    int B, H, hd;
    float scale;
    float* ws;                                 // split partials: [B][H][splits][hd + 2]
    int* tickets;                              // [B·H] zero-initialised, self-resetting counters
    int kvHalf = 0;                            // 1: the cache holds fp16 (keys rounded after the rotation, values rounded; fp32 arithmetic)
    int T = 1;                                 // tokens per sequence in this call: 1 = decode step, > 1 = prompt chunk (rows b·T + t)
    int splits;
};
constexpr int kAttnTickets = 1 << 16;
DJ_PART size_t attn_decode_ws_floats(int B, int H, int hd, int splits);
DJ_PART int attn_decode_splits(int B, int H, int maxSeq);
DJ_PART void launch_attn_decode(const AttnDecodeArgs& a, cudaStream_t s);
DJ_PART bool launch_attn_prefill_mma(const AttnDecodeArgs& a, cudaStream_t s);     // prompt chunks on the tensor cores (head dim 64 / 128)

// ── projections with bf16 weights (bf16_linear.cu, bf16_gemm_tc.cu) ──
// A bf16 weight as laid out in HBM: [N][Kp], Kp = K rounded up to 8, zero padded.
struct Bf16View { const __nv_bfloat16* w; int K, N, Kp; };
// One segment of an activation row: fp32 values, optionally RMS-normalised in groups and multiplied by sigmoid(gate).
struct RowOperand {
    const float* x = nullptr; int ldx = 0; int k = 0;                       // k == 0: no segment
    const float* gamma = nullptr; int groups = 0; float eps = 0.0f;         // groups == 0: no norm
    const float* gate = nullptr; int ldg = 0;
    // base != nullptr: the staged row is base + mult · norm(x), a sublayer's normed output added to the residual stream; the
    // sum is also written to `sum` (another buffer than base and x)
    const float* base = nullptr; int ldbase = 0; float mult = 0.0f; float* sum = nullptr; int ldsum = 0;
};
// What becomes of a (gate, up) pair of a gated feed-forward.
constexpr int kPairClamp = 0;     // g·sigmoid(1.702 g)·(u + 1) with g and u clamped
constexpr int kPairSilu = 1;      // g·sigmoid(g)·u
struct Bf16LinearArgs {
    RowOperand a, b;                           // b starts at weight column pad8(a.k)
    Bf16View w;
    const float* residual = nullptr; int ldr = 0;
    float* out = nullptr; int ldo = 0;         // weight rows [0, gluRow)
    int gluRow = 0; float limit = 0.0f;        // weight rows [gluRow, N) are (gate, up) pairs → glu, one value per pair
    float* glu = nullptr; int ldglu = 0;
    float softcap = 0.0f;                      // > 0: out = softcap · tanh(out / softcap)
    const float* bias = nullptr;               // [gluRow], added to the product
    int pair = kPairClamp;
    int M = 0;
    int exact = 0;                             // 1: fp32 products throughout
    float* ws = nullptr;                       // bf16_linear_ws_floats
};
DJ_PART void launch_bf16_store(const float* src, int rows, int cols, __nv_bfloat16* dst, long long dst_ld, cudaStream_t s);
DJ_PART const char* bf16_linear_check(const Bf16LinearArgs& a);      // nullptr, or why the shape is not supported
DJ_PART size_t bf16_linear_ws_floats(const Bf16LinearArgs& a);
DJ_PART void launch_bf16_linear(const Bf16LinearArgs& a, cudaStream_t s);
// Grouped rows of a tensor-core product: the expert of every 128-row tile (−1: none), where output rows go, rows per expert.
struct GroupedRows { const int* tileExpert; const int* rowMap; int rowsPerExpert; };
DJ_PART bool launch_bf16_gemm_tc(const Bf16LinearArgs& a, const GroupedRows* g, cudaStream_t s);
// out (bf16) = rows · Wᵀ for the first pos[0] + T bf16 rows (at most maxRows) of a row-major matrix with pitch lda.
DJ_PART void launch_bf16_gemm_rows(const __nv_bfloat16* rows, int lda, int K, const float* pos, int T, int maxRows, const Bf16View& w, __nv_bfloat16* out, int ldo,
                           cudaStream_t s);
DJ_PART void launch_stage_rows(const RowOperand& a, const RowOperand& b, int Kp, int rows, const int* map, int div, void* out, bool bf16, cudaStream_t s);
// out[m] = base[m] + mult · norm(x[m])·gamma, one group; out may be base
DJ_PART void launch_norm_add(const RowOperand& x, float* out, int ldo, int rows, cudaStream_t s);
DJ_PART void launch_bf16_block_linear(const float* x, int ldx, int xstr, const Bf16View& w, int heads, float* out, int ldo, int ostr, int M, cudaStream_t s);
// Table-routed experts: token id → `top` experts, each of weight 1/top.  up holds every expert's (gate, up) row pairs
// [experts·2ff][x.k], down [experts·d][ff].
struct Bf16ExpertArgs {
    RowOperand x;
    const float* tok; const float* table; int vocab, top, experts;
    Bf16View up, down; int ff, d; float limit;
    const float* residual; int ldr; float* out; int ldo;
    int M, exact;
    float* ws;                                 // bf16_experts_ws_floats
};
DJ_PART size_t bf16_experts_ws_floats(const Bf16ExpertArgs& e);
DJ_PART void launch_bf16_experts(const Bf16ExpertArgs& e, cudaStream_t s);
DJ_PART void launch_bf16_expert_gemv(const Bf16ExpertArgs& e, float* y, cudaStream_t s);

// ── generalized delta rule (delta_rule.cu) ──
struct DeltaRuleArgs {
    const float* proj; int ld, r_off, k_off, v_off, a_off, low_off;      // one row per token, heads side by side in every field
    const float* abias; Bf16View w2; const float* w0;                   // w2 [H·dim][rank]
    float* state;                              // this layer's [B][H][dim][dim]
    const float* pos;
    float* out; int ldo;                       // [rows][H·dim]
    int B, T, H, dim;
    bool early;                                // the state may be read before the dependency wait
    float* ws;                                 // delta_rule_ws_floats
};
DJ_PART bool delta_rule_fits(int dim, int rank);
DJ_PART size_t delta_rule_ws_floats(int B, int T, int H, int dim);
DJ_PART void launch_delta_rule(const DeltaRuleArgs& a, cudaStream_t s);

// ── latent attention (attn_latent.cu) ──
struct LatentAttnArgs {
    const float* q; int ldq;                   // [rows][H·(dim + rot)]
    const float* qc; int ldqc;                 // [rows][H·R]: the unrotated part taken into the latent space
    const float* kv; int ldkv;                 // [rows][R + rot]: the new latents (not normed) and key parts (not rotated)
    const float* gamma; float eps;
    void* cache; int bf16; int maxSeq;         // this layer's rows [B][maxSeq][R + rot]
    const float* pos; const float* cosT; const float* sinT;      // [maxSeq × rot/2]
    float* out; int ldo;                       // [rows][H·R]
    int B, T, H, dim, rot, R; float scale;
    bool early;                                // cached rows and positions may be read before the dependency wait
    int vdim; Bf16View uk, uv;                 // prompt chunks over expanded keys and values only: [H·dim][R], [H·vdim][R]
    float* ws;                                 // latent_attn_ws_floats / latent_prefill_ws_floats
};
DJ_PART bool latent_attn_fits(int R, int rot);
DJ_PART int latent_attn_splits(int rows, int H, int maxSeq);
DJ_PART size_t latent_attn_ws_floats(const LatentAttnArgs& a);
DJ_PART void launch_latent_attn(const LatentAttnArgs& a, cudaStream_t s);
DJ_PART void launch_latent_append(const LatentAttnArgs& a, cudaStream_t s);
// tensor-core forms (attn_latent_mma.cu)
DJ_PART bool latent_mma_fits(const LatentAttnArgs& a);
DJ_PART int latent_mma_splits(const LatentAttnArgs& a);
DJ_PART void launch_latent_mma(const LatentAttnArgs& a, cudaStream_t s);
DJ_PART bool latent_prefill_fits(const LatentAttnArgs& a);
DJ_PART size_t latent_prefill_ws_floats(const LatentAttnArgs& a);
DJ_PART void launch_latent_prefill(const LatentAttnArgs& a, cudaStream_t s);

// ── grouped attention over cached keys and values (attn_grouped.cu, attn_grouped_mma.cu) ──
struct GroupedAttnArgs {
    const float* proj; int ld, q_off, k_off, v_off;      // one row per token, heads side by side in every field; k_off < 0: nothing is appended
    const float* qgamma; const float* kgamma; float eps; // per head, over dim
    const float* qtab;                         // [maxSeq] factor of the queries by position, or null
    const float* rel; int relLen;              // [H][relLen] bias by distance (the last entry stands for everything beyond), or null
    void* kcache; void* vcache;                // [B·G][maxSeq][kw], [B·G][maxSeq][vw]; vcache null: the keys as projected are cached and are the values
    float* kscale; int kpitch;                 // … and their norms [B·G][kpitch]: 1 / root mean square of each key
    int kw, vw, bf16, maxSeq;
    const float* pos; float* out; int ldo;
    int B, T, H, G, dim, vdim; float scale; int sink;
    bool early;                                // cached rows and positions may be read before the dependency wait
    float* ws; int* tickets;
};
DJ_PART const char* grouped_attn_check(const GroupedAttnArgs& a);
DJ_PART size_t grouped_attn_ws_floats(const GroupedAttnArgs& a);
DJ_PART void launch_grouped_attn(const GroupedAttnArgs& a, cudaStream_t s);
DJ_PART bool grouped_mma_fits(const GroupedAttnArgs& a);
DJ_PART int grouped_mma_splits(const GroupedAttnArgs& a);
DJ_PART void launch_grouped_decode(const GroupedAttnArgs& a, cudaStream_t s);
DJ_PART void launch_grouped_prefill(const GroupedAttnArgs& a, const __nv_bfloat16* q, int qw, cudaStream_t s);

// ── matrix-memory recurrence with exponential gates (mlstm.cu) ──
struct MlstmArgs {
    const float* proj; int ld, q_off, k_off, v_off, i_off, f_off;
    float cap, qscale;
    float* state;                              // [B][H][vdim][dim]
    float* norm;                               // [2][B][H][dim + 1]: normaliser and running maximum, by parity of the position
    const float* pos; float* out; int ldo;
    int B, T, H, dim, vdim, exact;
    bool early;
    float* ws;
};
DJ_PART const char* mlstm_check(const MlstmArgs& a);
DJ_PART size_t mlstm_ws_floats(const MlstmArgs& a);
DJ_PART void launch_mlstm(const MlstmArgs& a, cudaStream_t s);

// ── misc ──
void launch_embed_gather(const float* table, const float* ids, float* out, int rows, int d, int vocab, cudaStream_t s);
// scratch: 2·16·rows ints of partial (key, index) pairs, tickets: rows zeroed self-resetting counters (rows ≤ kArgmaxRowsMax)
constexpr int kArgmaxRowsMax = 4096;
void launch_argmax_rows(const float* in, float* out, int rows, int cols, int* scratch, int* tickets, cudaStream_t s);
// topK = 0 means the whole row (the reference's convention); more than 1024 candidates sort the row in `ws`
// (sample_topk_ws_floats floats, 8-byte aligned).
void launch_sample_topk(const float* logits, const float* r, float* out, int rows, int cols, int topK, float temperature, float* ws,
                        cudaStream_t s);
size_t sample_topk_ws_floats(int rows, int cols, int topK);
void launch_add_scalar_inplace(float* buf, float v, int n, cudaStream_t s);
void launch_copy(const float* src, float* dst, long long n, cudaStream_t s);
void launch_synth_fill(float* out, unsigned long long seed, unsigned long long ordinal, float std_dev,
                       long long first, long long n, cudaStream_t s);

// ── tensor-parallel exchange over peer memory (tp.cu) ──
DJ_PART bool tp_ready();
DJ_PART int tp_world();
// mode 0: out = residual + bias + Σ_ranks in (all-reduce); mode 1: out[m][r·n_local + j] = in_r[m][j] (all-gather)
DJ_PART void launch_tp_exchange(const float* in, const float* bias, const float* residual, float* out, int M, int n_local, int mode,
                        cudaStream_t s);

// Read-only views of the runtime's buffer pool for entry points that live beside their kernels.
struct PoolF32 { float* ptr; size_t floats; };
struct PoolKV { void* ptr; int layers, B, H, maxSeq, hd, half; };
bool pool_f32(int id, PoolF32* out);
bool pool_kv(int id, PoolKV* out);
bool pool_q8(int id, Q8View* out);
// Serial number of a pool object (0 when the id does not exist); a released and re-created id gets a new serial.
unsigned long long pool_serial(int id);
// Registers device memory owned by a decode plan under `id` in the pool (released with the other objects).
void pool_add_plan(int id, void* dev_ptr, size_t bytes);

// ── whole-token decode kernel (decode_step.cu) ──
// Validates the plan object behind op 76 and appends the (id, serial) of everything it references to `refs`.
DJ_PART void decode_step_check(int plan_id, std::vector<std::pair<int, unsigned long long>>* refs);
DJ_PART void launch_decode_step(int plan_id, int feed_back, cudaStream_t s);
// The library's stream and device; the stream is null until the library has been initialised.
cudaStream_t runtime_stream();
int runtime_device();
// Drops every captured graph: called when addresses baked into kernel parameters (peer mappings, exchange
// buffers) stop being valid, so that the next flush of a cached stream is captured afresh.
void invalidate_graphs();
void set_last_error(const std::string& msg);

// Launch helper: plain <<<>>> or cudaLaunchKernelEx with the PDL attribute.
template <typename... KArgs, typename... Args>
inline void launch_k(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, bool pdl, Args... args) {
    g_launches++;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = s;
    cudaLaunchAttribute attr[1];
    if (pdl && g_use_pdl) {
        attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[0].val.programmaticStreamSerializationAllowed = 1;
        cfg.attrs = attr; cfg.numAttrs = 1;
    }
    DJ_CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...));
}

}  // namespace dj
