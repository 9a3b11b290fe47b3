// Linear attention with a fixed decay per head for DECODED tokens in bfloat16: every request of the step brings one row. S <- a S + k v^T,
// o = S^T q, with q, k, v passing silu as they are read. What bounds the step is the state, which is read and written once, so a block
// takes as many columns of a head's state as keep enough of them in flight: a column's D entries lie in one run of memory ([DV][D] per
// head), LPC lanes hold it in 16-byte pieces, a warp asks for UNROLL columns per group of lanes before it touches the first, and q and k
// are made once per block. Everything from the projections on is 32-bit.
#include "common.cuh"

namespace {

constexpr int THREADS = 256, UNROLL = 4;

__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.0f + __expf(-x)); }

template <int LPC, int NV>   // lanes per column, 16-byte pieces per lane: LPC * NV * 4 >= D
__global__ void __launch_bounds__(THREADS) linear_attention_step_kernel(const bf16* __restrict__ z, int z_stride, int q_col, int k_col, int v_col,
                                                                        const float* __restrict__ decay, float* __restrict__ state,
                                                                        const int* __restrict__ seq_starts, const int* __restrict__ seq_slots,
                                                                        float* __restrict__ out, int H, int D, int DV) {
    constexpr int CPW = 32 / LPC * UNROLL;               // columns per warp
    __shared__ __align__(16) float q_s[256], k_s[256];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, part = lane % LPC;
    const int h = blockIdx.y, r = blockIdx.z;
    const int c0 = (blockIdx.x * (THREADS / 32) + warp) * CPW + lane / LPC;   // my first column; the next ones 32 / LPC apart
    const float a = decay[h];
    pdl_trigger();
    pdl_wait();
    const int n = seq_starts[r];
    if (seq_starts[r + 1] <= n) return;
    float* st = state + ((size_t)seq_slots[r] * H + h) * DV * D;
    float4 S[UNROLL][NV];
#pragma unroll
    for (int u = 0; u < UNROLL; ++u)
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = c0 + u * (32 / LPC), d = (i * LPC + part) * 4;
            S[u][i] = (c < DV && d < D) ? *reinterpret_cast<const float4*>(st + (size_t)c * D + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    const bf16* row = z + (size_t)n * z_stride;
    float v[UNROLL];
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
        const int c = c0 + u * (32 / LPC);
        v[u] = c < DV ? to_f32(row[v_col + h * DV + c]) : 0.f;
    }
    for (int d = threadIdx.x; d < LPC * NV * 4; d += THREADS) {
        q_s[d] = d < D ? silu_fast(to_f32(row[q_col + h * D + d])) : 0.f;
        k_s[d] = d < D ? silu_fast(to_f32(row[k_col + h * D + d])) : 0.f;
    }
    __syncthreads();
    float4 q[NV], k[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        q[i] = *reinterpret_cast<const float4*>(q_s + (i * LPC + part) * 4);
        k[i] = *reinterpret_cast<const float4*>(k_s + (i * LPC + part) * 4);
    }
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
        const int c = c0 + u * (32 / LPC);
        const float vu = silu_fast(v[u]);
        float o = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int d = (i * LPC + part) * 4;
            float4 s = S[u][i];
            s.x = fmaf(a, s.x, k[i].x * vu); s.y = fmaf(a, s.y, k[i].y * vu); s.z = fmaf(a, s.z, k[i].z * vu); s.w = fmaf(a, s.w, k[i].w * vu);
            o = fmaf(s.x, q[i].x, o); o = fmaf(s.y, q[i].y, o); o = fmaf(s.z, q[i].z, o); o = fmaf(s.w, q[i].w, o);
            if (c < DV && d < D) *reinterpret_cast<float4*>(st + (size_t)c * D + d) = s;
        }
#pragma unroll
        for (int b = 1; b < LPC; b <<= 1) o += __shfl_xor_sync(0xffffffffu, o, b);
        if (part == 0 && c < DV) out[((size_t)n * H + h) * DV + c] = o;
    }
}

template <int LPC, int NV>
int launch(const bf16* z, int z_stride, int q_col, int k_col, int v_col, const float* decay, float* state, const int* seq_starts, const int* seq_slots,
           float* out, int H, int D, int DV, int R, cudaStream_t s) {
    constexpr int cols = THREADS / LPC * UNROLL;
    return launch_kernel(linear_attention_step_kernel<LPC, NV>, dim3((DV + cols - 1) / cols, H, R), dim3(THREADS), 0, s, z, z_stride, q_col, k_col, v_col,
                         decay, state, seq_starts, seq_slots, out, H, D, DV);
}

}  // namespace

// Every request's rows seq_starts[r] .. seq_starts[r + 1] - 1 are one row (or none). z: bfloat16 rows with q and k (H heads of D from q_col, k_col)
// and v (H heads of DV from v_col), before silu; D a multiple of 4, at most 256; state [slots][H][DV][D] float; out [N][H * DV] float.
LLMIE_API int llmie_linear_attention_step(const bf16* z, int z_stride, int q_col, int k_col, int v_col, const float* decay, float* state,
                                          const int* seq_starts, const int* seq_slots, float* out, int H, int D, int DV, int R, cudaStream_t s) {
    if (R <= 0) return 0;
    if (H <= 0 || D <= 0 || D > 256 || D % 4 || DV <= 0 || H > 65535 || R > 65535 || ((uintptr_t)state & 15)) return LLMIE_ERR_BAD_ARGUMENT;
#define LLMIE_STEP(LPC, NV) return launch<LPC, NV>(z, z_stride, q_col, k_col, v_col, decay, state, seq_starts, seq_slots, out, H, D, DV, R, s)
    if (D <= 32) LLMIE_STEP(8, 1);
    if (D <= 64) LLMIE_STEP(16, 1);
    if (D <= 128) LLMIE_STEP(32, 1);
    LLMIE_STEP(32, 2);
#undef LLMIE_STEP
}
