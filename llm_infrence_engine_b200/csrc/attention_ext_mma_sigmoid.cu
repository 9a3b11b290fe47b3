// The tensor-core attention with extras, instances for: sigmoid weights.
#include "attention_ext_mma.cuh"

namespace attn_ext_mma {
int launch_sigmoid(const Params& P, dim3 grid, size_t smem, cudaStream_t s, int R, bool deep) { return launch_kind<attn_ext::SIGMOID>(P, grid, smem, s, R, deep); }
}  // namespace attn_ext_mma
