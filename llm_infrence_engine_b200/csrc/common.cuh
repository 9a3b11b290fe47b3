// Shared by every kernel file: storage types, loads and stores through float, reductions, error codes.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define LLMIE_API extern "C" __attribute__((visibility("default")))

// Return codes of the exported functions (0 and CUDA's own codes are passed through unchanged).
#define LLMIE_ERR_BAD_ARGUMENT 100001

typedef __nv_bfloat16 bf16;

enum { DT_F32 = 0, DT_BF16 = 1 };

__device__ __forceinline__ float to_f32(float x) { return x; }
__device__ __forceinline__ float to_f32(bf16 x) { return __bfloat162float(x); }

template <typename T> __device__ __forceinline__ T from_f32(float x);
template <> __device__ __forceinline__ float from_f32<float>(float x) { return x; }
template <> __device__ __forceinline__ bf16 from_f32<bf16>(float x) { return __float2bfloat16_rn(x); }

// Round through the storage type and back: the value a later kernel would read.
template <typename T> __device__ __forceinline__ float round_through(float x) { return to_f32(from_f32<T>(x)); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result. `scratch` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    if (warp == 0) {
        float t = lane < nwarp ? scratch[lane] : 0.f;
        t = warp_sum(t);
        if (lane == 0) scratch[32] = t;
    }
    __syncthreads();
    return scratch[32];
}

// 16-byte vector of storage elements, read as floats.
template <typename T> struct Vec16;
template <> struct Vec16<float> {
    static constexpr int N = 4;
    __device__ __forceinline__ static void load(const float* p, float* out) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w;
    }
};
template <> struct Vec16<bf16> {
    static constexpr int N = 8;
    __device__ __forceinline__ static void load(const bf16* p, float* out) {
        const uint4 v = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            out[2 * i] = __uint_as_float(w[i] << 16);
            out[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
};

// Four consecutive storage elements through float (8- or 16-byte accesses; the address must be aligned to them).
__device__ __forceinline__ void load4(const float* p, float* v) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
__device__ __forceinline__ void load4(const bf16* p, float* v) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(t.x << 16); v[1] = __uint_as_float(t.x & 0xffff0000u);
    v[2] = __uint_as_float(t.y << 16); v[3] = __uint_as_float(t.y & 0xffff0000u);
}
__device__ __forceinline__ void store4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(bf16* p, const float* v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 t;
    t.x = *reinterpret_cast<const uint32_t*>(&a);
    t.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = t;
}

// 2^v and log2(v) by the hardware's approximation unit (errors of about 1e-7 of the result), denormals flushed.
__device__ __forceinline__ float hw_exp2(float v) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(v)); return y; }
__device__ __forceinline__ float hw_log2(float v) { float y; asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(v)); return y; }

// z times the normal distribution's share below z (the exact GELU) for results that are rounded to bfloat16: the share beyond |z| is
// t (a1 + t (a2 + ... + t a5)) e^(-z^2 / 2) / 2 with t = 1 / (1 + p |z| / sqrt 2), Abramowitz and Stegun, Handbook of Mathematical
// Functions, 7.1.26 (an error of at most 1.5e-7 in erf).
__device__ __forceinline__ float gelu_erf_fast(float z) {
    const float a = fabsf(z);
    const float t = __fdividef(1.0f, fmaf(0.3275911f * 0.7071067811865476f, a, 1.0f));
    float h = fmaf(t, 0.5f * 1.061405429f, 0.5f * -1.453152027f);
    h = fmaf(h, t, 0.5f * 1.421413741f);
    h = fmaf(h, t, 0.5f * -0.284496736f);
    h = fmaf(h, t, 0.5f * 0.254829592f);
    h = h * t * hw_exp2(-0.7213475204444817f * z * z);
    return fmaf(-a, h, fmaxf(z, 0.0f));
}
// The tanh form, 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))), likewise (tanh(t) = 1 - 2 / (exp(2 t) + 1)).
__device__ __forceinline__ float gelu_tanh_fast(float z) {
    const float t = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return z * (1.0f - __fdividef(1.0f, __expf(2.0f * t) + 1.0f));
}

// What a feed-forward's first product ends in; a compile-time choice, so that an epilogue's elements stand in one straight run of
// instructions (a branch per element, even a uniform one, would leave nothing to overlap their latencies with).
enum { UNIT_SILU = 0, UNIT_CLAMPED = 1, UNIT_GELU_TANH = 2, PLAIN_GELU_ERF = 3, PLAIN_GELU_TANH = 4, PLAIN_RELU2 = 5, PLAIN_SILU = 6 };
template <int UNIT>
__device__ __forceinline__ float plain_unit(float z) {
    if constexpr (UNIT == PLAIN_GELU_TANH) return gelu_tanh_fast(z);
    if constexpr (UNIT == PLAIN_SILU) return __fdividef(z, 1.0f + __expf(-z));
    if constexpr (UNIT == PLAIN_RELU2) { const float r = fmaxf(z, 0.f); return r * r; }
    return gelu_erf_fast(z);
}
template <int UNIT>
__device__ __forceinline__ float gated_unit(float g, float u, float limit, float alpha, float shift) {
    if constexpr (UNIT == UNIT_GELU_TANH) return gelu_tanh_fast(g) * u;
    if constexpr (UNIT == UNIT_CLAMPED) {   // min(g, limit) * sigmoid(alpha g) * (clamp(u) + shift)
        const float c = fminf(g, limit);
        return __fdividef(c, 1.0f + __expf(-alpha * c)) * (fminf(fmaxf(u, -limit), limit) + shift);
    }
    return __fdividef(g, 1.0f + __expf(-g)) * u;
}

static inline int launch_status() {
    return (int)cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------
// Programmatic dependent launch. A kernel launched through `launch_kernel` may start while the kernel
// before it on the stream is still running; it does whatever does not depend on that kernel (set-up,
// fetching weights), then calls pdl_wait(), which returns once the earlier kernel has finished and its
// writes are visible. Every kernel launched this way calls pdl_wait() exactly where its first access to
// anything an earlier kernel wrote (or still reads) would be, and ALWAYS calls it, so that completion
// stays ordered along the stream. pdl_trigger() lets the next kernel's blocks be scheduled from now on.
// Without the launch attribute both are no-ops.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;\n" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;\n" ::: "memory"); }

extern "C" int llmie_pdl_flag;  // 1: launch with the programmatic-serialization attribute (set by llmie_set_pdl)

// A kernel that runs long and wants the whole device launches alone (`alone` = true): blocks that move in while the kernel before
// still holds the multiprocessors go wherever room comes up first, several to one multiprocessor, and stay there.
template <typename... KArgs, typename... Args>
static inline int launch_kernel_on(bool alone, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = (llmie_pdl_flag && !alone) ? 1 : 0;
    return (int)cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

template <typename... KArgs, typename... Args>
static inline int launch_kernel(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = llmie_pdl_flag ? 1 : 0;
    return (int)cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
