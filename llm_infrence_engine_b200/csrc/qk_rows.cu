// Between the q/k(/v) projection and the attention, for mixers that norm the WHOLE query row and the whole key row of a token (not
// head by head): the normed queries leave in a row of their own with the columns of a gate behind them, the keys go to the token's
// cache slot. Two arrangements:
//   * values of their own: keys are stored normed, values as they are;
//   * values that are the keys before the norm (`key_scale` given): the keys are stored as they are, once, for both uses. The norm's
//     reciprocal root mean square, one number per token, goes to `key_scale`, and the norm's weight is multiplied into the queries:
//     q . (w k / rms) = (w q) . k / rms.
// Sums and scaling are 32-bit. The input is a product's rounded rows or its float32 sums (`clear`: set to zero behind the read, for
// the product that adds into them next). One block per token; no rotation.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int THREADS = 256;

struct Args {
    int z_stride, out_stride;       // elements per row
    const float* q_w; const float* k_w; float eps;
    const int* slots;
    float* key_scale;               // [pages][page_size], or null: values of their own
    int nq, nkv, dk, dv, page_size, gate_cols, write_kv, clear;
};

template <int VEC, typename TI> __device__ __forceinline__ void get(const TI* p, float* v) {
    if constexpr (VEC == 4) load4(p, v); else v[0] = to_f32(*p);
}
template <int VEC, typename T> __device__ __forceinline__ void put(T* p, const float* v) {
    if constexpr (VEC == 4) store4(p, v); else *p = from_f32<T>(v[0]);
}

template <typename TI, typename T, int VEC>
__global__ void __launch_bounds__(THREADS) qk_rows_norm_store_kernel(TI* __restrict__ z, T* __restrict__ q_out, T* __restrict__ k_pool,
                                                                     T* __restrict__ v_pool, const Args A) {
    __shared__ float scratch[2][THREADS / 32];
    pdl_trigger();
    pdl_wait();
    const int n = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int Q = A.nq * A.dk, KW = A.nkv * A.dk, rep = A.nq / A.nkv;
    TI* row = z + (size_t)n * A.z_stride;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x * VEC; i < Q + KW; i += THREADS * VEC) {   // (a vector never straddles: Q is a multiple of it)
        float v[VEC], s = 0.f;
        get<VEC>(row + i, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) s = fmaf(v[j], v[j], s);
        if (i < Q) sq += s; else sk += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) { scratch[0][warp] = sq; scratch[1][warp] = sk; }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) { sq += scratch[0][w]; sk += scratch[1][w]; }
    const float fq = 1.0f / sqrtf(sq / (float)Q + A.eps), fk = 1.0f / sqrtf(sk / (float)KW + A.eps);

    const float zero[4] = {0.f, 0.f, 0.f, 0.f};
    T* o = q_out + (size_t)n * A.out_stride;
    for (int i = threadIdx.x * VEC; i < Q; i += THREADS * VEC) {
        float v[VEC], w[VEC];
        get<VEC>(row + i, v);
        get<VEC>(A.q_w + i, w);
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[j] = v[j] * fq * w[j];
        if (A.key_scale) {
            const int h = i / A.dk;
            get<VEC>(A.k_w + (h / rep) * A.dk + (i - h * A.dk), w);
#pragma unroll
            for (int j = 0; j < VEC; ++j) v[j] *= w[j];
        }
        put<VEC>(o + i, v);
        if (A.clear) put<VEC>(row + i, reinterpret_cast<const float*>(zero));
    }
    int page = 0, off = 0;
    if (A.write_kv) {
        page = A.slots[n] / A.page_size;
        off = A.slots[n] - page * A.page_size;
        if (A.key_scale && threadIdx.x == 0) A.key_scale[A.slots[n]] = fk;
    }
    for (int i = threadIdx.x * VEC; i < KW; i += THREADS * VEC) {
        float v[VEC];
        get<VEC>(row + Q + i, v);
        if (A.write_kv) {
            const int g = i / A.dk;
            if (!A.key_scale) {
                float w[VEC];
                get<VEC>(A.k_w + i, w);
#pragma unroll
                for (int j = 0; j < VEC; ++j) v[j] = v[j] * fk * w[j];
            }
            put<VEC>(k_pool + (((size_t)page * A.nkv + g) * A.page_size + off) * A.dk + (i - g * A.dk), v);
        }
        if (A.clear) put<VEC>(row + Q + i, reinterpret_cast<const float*>(zero));
    }
    int at = Q + KW;
    if (!A.key_scale) {
        for (int i = threadIdx.x; i < A.nkv * A.dv; i += THREADS) {
            const int g = i / A.dv;
            if (A.write_kv) v_pool[(((size_t)page * A.nkv + g) * A.page_size + off) * A.dv + (i - g * A.dv)] = from_f32<T>(to_f32(row[at + i]));
            if (A.clear) row[at + i] = from_f32<TI>(0.f);
        }
        at += A.nkv * A.dv;
    }
    // the gate's columns as they are, then zeros up to the end of the row; whatever else the projection's row holds is padding
    for (int i = threadIdx.x; i < A.out_stride - Q; i += THREADS) o[Q + i] = from_f32<T>(i < A.gate_cols ? to_f32(row[at + i]) : 0.f);
    if (A.clear) {
        __syncthreads();
        for (int i = at + threadIdx.x; i < A.z_stride; i += THREADS) row[i] = from_f32<TI>(0.f);
    }
}

template <typename TI, typename T>
int launch(void* z, void* q_out, void* k_pool, void* v_pool, const Args& A, int N, cudaStream_t s) {
    auto aligned = [](const void* p) { return (uintptr_t)p % 16 == 0; };
    const bool vec = A.dk % 4 == 0 && A.z_stride % 4 == 0 && A.out_stride % 4 == 0 && aligned(z) && aligned(q_out) && aligned(k_pool) && aligned(A.q_w) && aligned(A.k_w);
    if (vec) return launch_kernel(qk_rows_norm_store_kernel<TI, T, 4>, dim3(N), dim3(THREADS), 0, s, (TI*)z, (T*)q_out, (T*)k_pool, (T*)v_pool, A);
    return launch_kernel(qk_rows_norm_store_kernel<TI, T, 1>, dim3(N), dim3(THREADS), 0, s, (TI*)z, (T*)q_out, (T*)k_pool, (T*)v_pool, A);
}

}  // namespace

// z [N] rows of z_stride: [nq heads of dk | nkv heads of dk | nkv heads of dv, unless key_scale is given | gate_cols | padding].
// q_out [N] rows of out_stride: [normed queries | gate columns | zeros]. clear needs a float32 input.
LLMIE_API int llmie_qk_rows_norm_store(void* z, int z_stride, void* q_out, int out_stride, const float* q_w, const float* k_w, float eps,
                                       const int* slots, void* k_pool, void* v_pool, float* key_scale, int N, int nq, int nkv, int dk, int dv,
                                       int page_size, int gate_cols, int write_kv, int clear, int in_dtype, int dtype, cudaStream_t s) {
    if (N <= 0) return 0;
    if (nq <= 0 || nkv <= 0 || nq % nkv || dk <= 0 || dv < 0 || page_size <= 0 || gate_cols < 0 || !q_w || !k_w || out_stride < nq * dk + gate_cols ||
        z_stride < (nq + nkv) * dk + (key_scale ? 0 : nkv * dv) + gate_cols || (write_kv && (!slots || !k_pool || (!key_scale && !v_pool))) ||
        (clear && in_dtype != DT_F32))
        return LLMIE_ERR_BAD_ARGUMENT;
    const Args A{z_stride, out_stride, q_w, k_w, eps, slots, key_scale, nq, nkv, dk, dv, page_size, gate_cols, write_kv, clear};
    if (in_dtype == DT_F32 && dtype == DT_F32) return launch<float, float>(z, q_out, k_pool, v_pool, A, N, s);
    if (in_dtype == DT_F32 && dtype == DT_BF16) return launch<float, bf16>(z, q_out, k_pool, v_pool, A, N, s);
    if (in_dtype == DT_BF16 && dtype == DT_BF16) return launch<bf16, bf16>(z, q_out, k_pool, v_pool, A, N, s);
    return LLMIE_ERR_BAD_ARGUMENT;
}
