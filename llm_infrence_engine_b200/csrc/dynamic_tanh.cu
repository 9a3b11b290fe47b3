// Dynamic Tanh in place of a norm, for blocks that put it before a sublayer and on its result:
//   x <- x + tanh(a_post * y) * w_post + b_post;   h = tanh(a_pre * x) * w_pre + b_pre
// (a: one number, w and b: vectors over the row). It computes no mean or variance, so nothing is reduced: a thread keeps its
// columns' weights in registers and walks down the rows; one kernel does either half or both in a single pass over the stream.
// Everything is 32-bit up to the one rounding of h.
#include <math.h>

#include "common.cuh"

namespace {

// FAST: tanh(z) = 1 - 2 / (exp(2 z) + 1) with the fast exponential and division, an absolute error of about 1e-7: for h that is
// rounded to bfloat16, and for results that join a stream of magnitude 1 and more (whose own rounding is as large).
template <bool FAST>
__device__ __forceinline__ float tanh_of(float z) {
    if constexpr (FAST) return 1.0f - __fdividef(2.0f, __expf(2.0f * z) + 1.0f);
    return tanhf(z);
}

struct Affine {            // alpha, weight and bias of one of the two; weight == null: that half is not asked for
    const float* alpha;
    const float* w;
    const float* b;
};

// rows == nullptr: row r of x (stored back where y was added) -> row r of out; rows != nullptr: row rows[i] -> row i of out, and
// nothing of x or y is changed. With clear_y, y (a float buffer that the next sublayer adds into) is zero behind the read.
template <typename TY, typename TO, int VEC, bool FAST>
__global__ void __launch_bounds__(128) dynamic_tanh_kernel(float* __restrict__ x, TY* __restrict__ y, Affine post, int clear_y, Affine pre,
                                                           TO* __restrict__ out, const int* __restrict__ rows, int n_rows, int H) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    float a0 = 0.f, a1 = 0.f, w0[VEC], b0[VEC], w1[VEC], b1[VEC];
    pdl_trigger();
    const bool live = c < H;
    if (live) {   // weights of the model: fetched before the wait for the kernel before
        if (post.w) {
            a0 = *post.alpha;
            if constexpr (VEC == 4) { load4(post.w + c, w0); load4(post.b + c, b0); } else { w0[0] = post.w[c]; b0[0] = post.b[c]; }
        }
        if (pre.w) {
            a1 = *pre.alpha;
            if constexpr (VEC == 4) { load4(pre.w + c, w1); load4(pre.b + c, b1); } else { w1[0] = pre.w[c]; b1[0] = pre.b[c]; }
        }
    }
    pdl_wait();
    if (!live) return;
    for (int i = blockIdx.y; i < n_rows; i += gridDim.y) {
        const size_t at = (size_t)(rows ? rows[i] : i) * H + c;
        float v[VEC];
        if constexpr (VEC == 4) load4(x + at, v); else v[0] = x[at];
        if (y) {
            float u[VEC];
            if constexpr (VEC == 4) load4(y + at, u); else u[0] = to_f32(y[at]);
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] += fmaf(tanh_of<FAST>(a0 * u[j]), w0[j], b0[j]);
            if (!rows) {
                if constexpr (VEC == 4) store4(x + at, v); else x[at] = v[0];
                if (clear_y) {
                    const float zero[4] = {0.f, 0.f, 0.f, 0.f};
                    if constexpr (VEC == 4) store4(y + at, zero); else y[at] = from_f32<TY>(0.f);
                }
            }
        }
        if (pre.w) {
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] = fmaf(tanh_of<FAST>(a1 * v[j]), w1[j], b1[j]);
            TO* o = out + (size_t)i * H + c;
            if constexpr (VEC == 4) store4(o, v); else o[0] = from_f32<TO>(v[0]);
        }
    }
}

template <typename TY, typename TO, bool FAST>
int launch(float* x, void* y, const Affine& post, int clear_y, const Affine& pre, void* out, const int* rows, int n_rows, int H, int max_blocks,
           cudaStream_t s) {
    const void* ptrs[] = {x, y, post.w, post.b, pre.w, pre.b, out};
    bool vec = H % 4 == 0;
    for (const void* p : ptrs) vec = vec && (uintptr_t)p % 16 == 0;
    const int per = vec ? 4 : 1;
    const int cols = (H + per - 1) / per;
    const int threads = cols >= 128 ? 128 : ((cols + 31) / 32) * 32;
    const int gx = (cols + threads - 1) / threads;
    int gy = max_blocks / gx;
    gy = gy < 1 ? 1 : (gy > n_rows ? n_rows : gy);
    if (gy > 65535) gy = 65535;
    if (vec)
        return launch_kernel(dynamic_tanh_kernel<TY, TO, 4, FAST>, dim3(gx, gy), dim3(threads), 0, s, x, (TY*)y, post, clear_y, pre, (TO*)out, rows, n_rows, H);
    return launch_kernel(dynamic_tanh_kernel<TY, TO, 1, FAST>, dim3(gx, gy), dim3(threads), 0, s, x, (TY*)y, post, clear_y, pre, (TO*)out, rows, n_rows, H);
}

}  // namespace

// x [*, H] float32. y (or null) [*, H] in y_dtype with post_a / post_w / post_b; pre_a / pre_w / pre_b (or null) -> out [n_rows, H] in
// out_dtype. fast: the fast hyperbolic tangent. max_blocks: how many blocks of 128 threads the device holds at once.
LLMIE_API int llmie_dynamic_tanh(float* x, void* y, int y_dtype, const float* post_a, const float* post_w, const float* post_b, int clear_y,
                                 const float* pre_a, const float* pre_w, const float* pre_b, void* out, int out_dtype, const int* rows, int n_rows,
                                 int H, int fast, int max_blocks, cudaStream_t s) {
    if (n_rows <= 0) return 0;
    if (H <= 0 || (y && (!post_a || !post_w || !post_b)) || (pre_w && (!pre_a || !pre_b || !out)) || (!y && !pre_w) || max_blocks < 1 ||
        (clear_y && y_dtype != DT_F32))
        return LLMIE_ERR_BAD_ARGUMENT;
    const Affine post{post_a, y ? post_w : nullptr, post_b}, pre{pre_a, pre_w, pre_b};
#define LLMIE_DT(TY, TO)                                                                                                   \
    {                                                                                                                      \
        if (fast) return launch<TY, TO, true>(x, y, post, clear_y, pre, out, rows, n_rows, H, max_blocks, s);              \
        return launch<TY, TO, false>(x, y, post, clear_y, pre, out, rows, n_rows, H, max_blocks, s);                       \
    }
    if (y_dtype == DT_F32 && out_dtype == DT_F32) LLMIE_DT(float, float)
    if (y_dtype == DT_F32 && out_dtype == DT_BF16) LLMIE_DT(float, bf16)
    if (y_dtype == DT_BF16 && out_dtype == DT_BF16) LLMIE_DT(bf16, bf16)
    if (y_dtype == DT_BF16 && out_dtype == DT_F32) LLMIE_DT(bf16, float)
#undef LLMIE_DT
    return LLMIE_ERR_BAD_ARGUMENT;
}
