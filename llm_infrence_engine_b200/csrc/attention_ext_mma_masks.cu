// The tensor-core attention with extras, instances for: kept first tokens, chunks, a soft cap, a penalty by distance.
#include "attention_ext_mma.cuh"

namespace attn_ext_mma {
int launch_masks(const Params& P, dim3 grid, size_t smem, cudaStream_t s, int R, bool deep) { return launch_kind<attn_ext::MASKS>(P, grid, smem, s, R, deep); }
}  // namespace attn_ext_mma
