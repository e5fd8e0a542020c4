// The windowed tensor-core attention (attention_window_mma.cuh): softmax with a distance bias that grows with the logarithm of the distance.
#include "attention_window_mma.cuh"

namespace cib {
int window_mma_log_bias(CIB_WM_ARGS_DECL) { return launch_window_mma_sizes<kWmLogBias>(CIB_WM_ARGS); }
}  // namespace cib
