// The windowed tensor-core attention (attention_window_mma.cuh): weights sigmoid(score + number per head), not normalised.
#include "attention_window_mma.cuh"

namespace cib {
int window_mma_sigmoid(CIB_WM_ARGS_DECL) { return launch_window_mma_sizes<kWmSigmoid>(CIB_WM_ARGS); }
}  // namespace cib
