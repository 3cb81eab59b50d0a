// Table-routed experts: a table row indexed by the token id names the `top` experts of the token, each of weight 1/top.
//
// Few rows: every (token, slot) entry is its own GEMV over its expert's weight rows (bf16_linear.cu).
#include "row_operand.cuh"

namespace dj {

size_t bf16_experts_ws_floats(const Bf16ExpertArgs& e) { return (size_t)e.M * e.top * e.ff; }

void launch_bf16_experts(const Bf16ExpertArgs& e, cudaStream_t s) {
    if (e.M <= 0) return;
    launch_bf16_expert_gemv(e, e.ws, s);
}

}  // namespace dj
