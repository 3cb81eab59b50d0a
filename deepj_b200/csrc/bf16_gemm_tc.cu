// placeholder until the tensor-core form exists
#include "kernels.h"
namespace dj {
bool launch_bf16_gemm_tc(const Bf16LinearArgs&, const int*, const int*, cudaStream_t) { return false; }
}  // namespace dj
