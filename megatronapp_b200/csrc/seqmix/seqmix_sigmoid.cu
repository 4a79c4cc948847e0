// Paged grouped-query attention with logistic weights: the instances of seq_window.cuh's kernels for prompts of any head size and
// for decoding batches.
#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include "seq_window.cuh"

namespace b200seq {

bool sigmoid_attention_paged(const WindowAttnArgs& p, bool bf16, cudaStream_t s) { return run_window_attention<true>(p, bf16, s); }

}  // namespace b200seq
