// The end of a sublayer whose RESULT is normed, and the beginning of the next one, in one kernel per row of the stream:
//   u = a, or coef (a / rms(a) wa + b / rms(b) wb)        (one result, or two side by side, each normed by itself)
//   x <- x + u / rms(u) w_post
//   out = x (rounded), or x / rms(x) w_pre, or nothing
// with rms(v) = sqrt(mean(v^2) + eps). Everything is 32-bit up to the rounding of `out`. One block per row; a thread keeps its
// elements in registers from one reduction to the next, and a reduction costs one barrier.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int MAX_WARPS = 16;

// Sum over the block; every thread gets it. `scratch`: MAX_WARPS floats that no other reduction of the kernel uses.
__device__ __forceinline__ float block_sum_once(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    v = warp_sum(v);
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    return warp_sum(lane < warps ? scratch[lane] : 0.f);
}

enum { OUT_NONE = 0, OUT_CAST = 1, OUT_NORM = 2 };

struct Args {
    float* x;
    void* a; void* b;               // b: null for one result
    const float* wa; const float* wb; float coef;
    const float* w_post;            // null: nothing is added
    const float* w_pre;
    void* out;
    const int* rows;                // null: row blockIdx.x and the stream is stored; else row rows[blockIdx.x] and nothing of it is
    int H; float eps; int clear_a, clear_b, mode;
};

template <typename TA, typename TB, typename TO, int VEC, int PER>
__global__ void __launch_bounds__(32 * MAX_WARPS) post_rms_kernel(const Args A) {
    __shared__ float scratch[4][MAX_WARPS];
    const int H = A.H, step = blockDim.x * VEC;
    pdl_trigger();
    float wp[PER][VEC];
    if (A.w_post) {   // a weight does not depend on the kernel before: asked for before the wait
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int i = p * step + threadIdx.x * VEC;
            if (i < H) { if constexpr (VEC == 4) load4(A.w_post + i, wp[p]); else wp[p][0] = A.w_post[i]; }
        }
    }
    pdl_wait();
    const int r = A.rows ? A.rows[blockIdx.x] : blockIdx.x;
    float* xr = A.x + (size_t)r * H;
    float x[PER][VEC], u[PER][VEC];
#pragma unroll
    for (int p = 0; p < PER; ++p) {
        const int i = p * step + threadIdx.x * VEC;
#pragma unroll
        for (int j = 0; j < VEC; ++j) x[p][j] = u[p][j] = 0.f;
        if (i < H) { if constexpr (VEC == 4) load4(xr + i, x[p]); else x[p][0] = xr[i]; }
    }
    if (A.w_post) {
        const float zero[4] = {0.f, 0.f, 0.f, 0.f};
        TA* ar = reinterpret_cast<TA*>(A.a) + (size_t)r * H;
        float sa = 0.f;
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int i = p * step + threadIdx.x * VEC;
            if (i < H) {
                if constexpr (VEC == 4) load4(ar + i, u[p]); else u[p][0] = to_f32(ar[i]);
                if (A.clear_a) { if constexpr (VEC == 4) store4(ar + i, zero); else ar[i] = from_f32<TA>(0.f); }
            }
#pragma unroll
            for (int j = 0; j < VEC; ++j) sa = fmaf(u[p][j], u[p][j], sa);
        }
        if (A.b) {
            TB* br = reinterpret_cast<TB*>(A.b) + (size_t)r * H;
            float v[PER][VEC], sb = 0.f;
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                const int i = p * step + threadIdx.x * VEC;
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[p][j] = 0.f;
                if (i < H) {
                    if constexpr (VEC == 4) load4(br + i, v[p]); else v[p][0] = to_f32(br[i]);
                    if (A.clear_b) { if constexpr (VEC == 4) store4(br + i, zero); else br[i] = from_f32<TB>(0.f); }
                }
#pragma unroll
                for (int j = 0; j < VEC; ++j) sb = fmaf(v[p][j], v[p][j], sb);
            }
            const float fa = A.coef / sqrtf(block_sum_once(sa, scratch[0]) / (float)H + A.eps);
            const float fb = A.coef / sqrtf(block_sum_once(sb, scratch[1]) / (float)H + A.eps);
            sa = 0.f;
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                const int i = p * step + threadIdx.x * VEC;
                if (i < H) {
                    float w1[VEC], w2[VEC];
                    if constexpr (VEC == 4) { load4(A.wa + i, w1); load4(A.wb + i, w2); } else { w1[0] = A.wa[i]; w2[0] = A.wb[i]; }
#pragma unroll
                    for (int j = 0; j < VEC; ++j) {
                        u[p][j] = u[p][j] * fa * w1[j] + v[p][j] * fb * w2[j];
                        sa = fmaf(u[p][j], u[p][j], sa);
                    }
                }
            }
        }
        const float f = 1.0f / sqrtf(block_sum_once(sa, scratch[2]) / (float)H + A.eps);
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int i = p * step + threadIdx.x * VEC;
            if (i < H) {
#pragma unroll
                for (int j = 0; j < VEC; ++j) x[p][j] = fmaf(u[p][j] * f, wp[p][j], x[p][j]);
                if (!A.rows) { if constexpr (VEC == 4) store4(xr + i, x[p]); else xr[i] = x[p][0]; }
            }
        }
    }
    if (A.mode == OUT_NONE) return;
    TO* o = reinterpret_cast<TO*>(A.out) + (size_t)blockIdx.x * H;
    float g = 1.f;
    if (A.mode == OUT_NORM) {
        float sx = 0.f;
#pragma unroll
        for (int p = 0; p < PER; ++p)
#pragma unroll
            for (int j = 0; j < VEC; ++j) sx = fmaf(x[p][j], x[p][j], sx);
        g = 1.0f / sqrtf(block_sum_once(sx, scratch[3]) / (float)H + A.eps);
    }
#pragma unroll
    for (int p = 0; p < PER; ++p) {
        const int i = p * step + threadIdx.x * VEC;
        if (i >= H) continue;
        if (A.mode == OUT_NORM) {
            float w[VEC];
            if constexpr (VEC == 4) load4(A.w_pre + i, w); else w[0] = A.w_pre[i];
#pragma unroll
            for (int j = 0; j < VEC; ++j) x[p][j] = x[p][j] * g * w[j];
        }
        if constexpr (VEC == 4) store4(o + i, x[p]); else o[i] = from_f32<TO>(x[p][0]);
    }
}

template <typename TA, typename TB, typename TO>
int launch(const Args& A, int n_out, cudaStream_t s) {
    auto aligned = [](const void* p) { return (uintptr_t)p % 16 == 0; };
    const bool vec = A.H % 4 == 0 && aligned(A.x) && aligned(A.a) && aligned(A.b) && aligned(A.wa) && aligned(A.wb) && aligned(A.w_post) &&
                     aligned(A.w_pre) && aligned(A.out);
    const int pieces = vec ? A.H / 4 : A.H;
    int threads = 32;
    while (threads < 512 && threads < pieces) threads *= 2;
    const int per = (pieces + threads - 1) / threads;
#define LLMIE_POST(V, P) return launch_kernel(post_rms_kernel<TA, TB, TO, V, P>, dim3(n_out), dim3(threads), 0, s, A)
    if (vec) {
        if (per <= 1) LLMIE_POST(4, 1);
        if (per <= 2) LLMIE_POST(4, 2);
        if (per <= 4) LLMIE_POST(4, 4);
        if (per <= 8) LLMIE_POST(4, 8);
    } else {
        if (per <= 4) LLMIE_POST(1, 4);
        if (per <= 24) LLMIE_POST(1, 24);
    }
#undef LLMIE_POST
    return LLMIE_ERR_BAD_ARGUMENT;   // rows of more than 16384 (or 12288) entries
}

}  // namespace

// mode 0: no output; 1: out = the row, rounded; 2: out = its RMS norm with w_pre. w_post null: nothing is added (a, b unused).
// A float32 output takes float32 results only.
LLMIE_API int llmie_post_rms(float* x, void* a, int a_dtype, int clear_a, void* b, int b_dtype, int clear_b, const float* wa, const float* wb,
                             float coef, const float* w_post, const float* w_pre, void* out, int out_dtype, int mode, const int* rows, int n_out,
                             int H, float eps, cudaStream_t s) {
    if (n_out <= 0) return 0;
    if (H <= 0 || mode < 0 || mode > 2 || (mode && !out) || (mode == 2 && !w_pre) || (w_post && !a) || (b && (!wa || !wb)) || (!w_post && !mode))
        return LLMIE_ERR_BAD_ARGUMENT;
    Args A{x, a, b, wa, wb, coef, w_post, w_pre, out, rows, H, eps, clear_a, clear_b, mode};
    if (!b) b_dtype = a_dtype;
    if (a_dtype == DT_F32 && b_dtype == DT_F32) return out_dtype == DT_F32 ? launch<float, float, float>(A, n_out, s) : launch<float, float, bf16>(A, n_out, s);
    if (mode && out_dtype == DT_F32) return LLMIE_ERR_BAD_ARGUMENT;
    if (a_dtype == DT_BF16 && b_dtype == DT_BF16) return launch<bf16, bf16, bf16>(A, n_out, s);
    if (a_dtype == DT_F32) return launch<float, bf16, bf16>(A, n_out, s);
    return launch<bf16, float, bf16>(A, n_out, s);
}
