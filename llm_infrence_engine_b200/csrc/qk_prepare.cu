// Between the q/k/v projection and the attention, for mixers whose heads are normed and only partly rotated: per head an
// optional root-mean-square norm with a weight, the rotation of the head's first `rot_dims` entries (pairs (i, i + rot_dims / 2)
// or neighbours (2 i, 2 i + 1)), then the query heads to a row of their own and the key and value heads into the token's
// cache slot. Value heads may turn too, over all their entries, by angles of their own (the cache then holds turned values).
// Keys and values may differ in size. Norm and rotation are 32-bit. The input is a product's rounded rows, or its float32 sums
// (`clear`: set to zero behind the read, for the product that adds into them next).
//
// Two forms: a warp per (token, head), for any size and with the norm; and, where no head is normed and sizes are multiples of
// 16, a thread per 16 entries of a head: the two runs of 8 that form pairs (or 16 neighbours), moved by 16-byte accesses.
#include <math.h>

#include "common.cuh"

namespace {

struct Turn {               // how one kind of head turns
    const float* cos_t;     // [N, dims / 2]
    const float* sin_t;
    int dims;               // 0: not at all
};

// z row: [nq heads of dk | nkv heads of dk | nkv heads of dv] from column 0. cos / sin: already multiplied by whatever factor the
// encoding puts on them.
template <typename TI, typename T>
__global__ void __launch_bounds__(128) qk_norm_rope_store_kernel(TI* __restrict__ z, int z_stride, T* __restrict__ q_out,
                                                                 const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                                                                 Turn qk, Turn vt, int interleaved, const int* __restrict__ slots,
                                                                 T* __restrict__ k_pool, T* __restrict__ v_pool, int N, int nq, int nkv,
                                                                 int dk, int dv, int page_size, int write_kv, int clear) {
    pdl_trigger();
    pdl_wait();
    const int heads = nq + 2 * nkv;
    const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (item >= N * heads) return;
    const int n = item / heads, j = item % heads;
    const bool value = j >= nq + nkv;
    const int D = value ? dv : dk;
    TI* src = z + (size_t)n * z_stride + (value ? (size_t)(nq + nkv) * dk + (size_t)(j - nq - nkv) * dv : (size_t)j * dk);
    if (j < nq || write_kv) {
        size_t dst_row = 0;
        if (j >= nq) {
            const int slot = slots[n];
            const int page = slot / page_size, off = slot % page_size;
            dst_row = ((size_t)page * nkv + (j - nq) % nkv) * page_size + off;
        }
        T* dst = j < nq ? q_out + ((size_t)n * nq + j) * dk : (value ? v_pool : k_pool) + dst_row * D;
        const float* w = value ? nullptr : (j < nq ? q_w : k_w);
        const Turn& t = value ? vt : qk;
        float f = 1.f;
        if (w) {
            float sq = 0.f;
            for (int i = lane; i < D; i += 32) { const float v = to_f32(src[i]); sq = fmaf(v, v, sq); }
            f = 1.0f / sqrtf(warp_sum(sq) / (float)D + eps);
        }
        const int half = t.dims / 2;
        for (int i = lane; i < half; i += 32) {
            const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
            float a = to_f32(src[ia]) * f, b = to_f32(src[ib]) * f;
            if (w) { a *= w[ia]; b *= w[ib]; }
            const float c = t.cos_t[(size_t)n * half + i], sn = t.sin_t[(size_t)n * half + i];
            dst[ia] = from_f32<T>(a * c - b * sn);
            dst[ib] = from_f32<T>(b * c + a * sn);
        }
        for (int i = t.dims + lane; i < D; i += 32) {
            float a = to_f32(src[i]) * f;
            if (w) a *= w[i];
            dst[i] = from_f32<T>(a);
        }
    }
    if (clear) {
        __syncwarp();
        for (int i = lane; i < D; i += 32) src[i] = from_f32<TI>(0.f);
    }
}

template <typename TI> __device__ __forceinline__ void load8(const TI* p, float* v);
template <> __device__ __forceinline__ void load8<bf16>(const bf16* p, float* v) { Vec16<bf16>::load(p, v); }
template <> __device__ __forceinline__ void load8<float>(const float* p, float* v) { load4(p, v); load4(p + 4, v + 4); }
__device__ __forceinline__ void store8(float* p, const float* v) { store4(p, v); store4(p + 4, v + 4); }
__device__ __forceinline__ void store8(bf16* p, const float* v) {
    uint4 packed;
    uint32_t* w = reinterpret_cast<uint32_t*>(&packed);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const __nv_bfloat162 t = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
        w[j] = *reinterpret_cast<const uint32_t*>(&t);
    }
    *reinterpret_cast<uint4*>(p) = packed;
}

// A thread per 16 entries of a head. Runs of the rotated part come first: run r of a head with `dims` turned entries holds entries
// 8 r .. 8 r + 7 and their partners dims / 2 further on (or, interleaved, entries 16 r .. 16 r + 15); the runs behind it pass.
template <typename TI, typename T>
__global__ void __launch_bounds__(128) qk_rope_store_vec_kernel(TI* __restrict__ z, int z_stride, T* __restrict__ q_out, Turn qk, Turn vt,
                                                                int interleaved, const int* __restrict__ slots, T* __restrict__ k_pool,
                                                                T* __restrict__ v_pool, int N, int nq, int nkv, int dk, int dv, int page_size,
                                                                int write_kv, int clear) {
    pdl_trigger();
    pdl_wait();
    const int kr = dk >> 4, vr = dv >> 4;
    const int qk_runs = (nq + nkv) * kr, per_token = qk_runs + nkv * vr;
    const long long item = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    const int n = (int)(item / per_token);
    if (n >= N) return;
    const int c = (int)(item - (long long)n * per_token);
    const bool value = c >= qk_runs;
    const int runs = value ? vr : kr;
    const int cc = value ? c - qk_runs : c;
    const int j = cc / runs, r = cc - j * runs;        // head (query and key heads counted through, or value head), run of it
    const Turn& t = value ? vt : qk;
    const int half = t.dims >> 1;
    const bool turned = r * 16 < t.dims;
    int ia = r * 16, ib = ia + 8;
    if (turned && !interleaved) { ia = r * 8; ib = ia + half; }
    const int D = value ? dv : dk;
    TI* src = z + (size_t)n * z_stride + (value ? (size_t)(nq + nkv) * dk : 0) + (size_t)j * D;
    float a[8], b[8];
    load8<TI>(src + ia, a);
    load8<TI>(src + ib, b);
    if (clear) {
        const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        store8(src + ia, zero);
        store8(src + ib, zero);
    }
    const bool key_side = value || j >= nq;
    if (key_side && !write_kv) return;
    if (turned) {
        float cs[8], sn[8];
        load8<float>(t.cos_t + (size_t)n * half + r * 8, cs);
        load8<float>(t.sin_t + (size_t)n * half + r * 8, sn);
        if (interleaved) {
            float y[16];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float u = i < 4 ? a[2 * i] : b[2 * i - 8], v = i < 4 ? a[2 * i + 1] : b[2 * i - 7];
                y[2 * i] = u * cs[i] - v * sn[i];
                y[2 * i + 1] = v * cs[i] + u * sn[i];
            }
#pragma unroll
            for (int i = 0; i < 8; ++i) { a[i] = y[i]; b[i] = y[8 + i]; }
        } else {
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const float u = a[i], v = b[i];
                a[i] = u * cs[i] - v * sn[i];
                b[i] = v * cs[i] + u * sn[i];
            }
        }
    }
    T* dst;
    if (!key_side) {
        dst = q_out + ((size_t)n * nq + j) * dk;
    } else {
        const int slot = slots[n];
        const int page = slot / page_size, off = slot - page * page_size;
        dst = (value ? v_pool : k_pool) + (((size_t)page * nkv + (value ? j : j - nq)) * page_size + off) * D;
    }
    store8(dst + ia, a);
    store8(dst + ib, b);
}

template <typename TI, typename T>
int launch(void* z, int z_stride, void* q_out, const float* q_w, const float* k_w, float eps, const Turn& qk, const Turn& vt, int interleaved,
           const int* slots, void* k_pool, void* v_pool, int N, int nq, int nkv, int dk, int dv, int page_size, int write_kv, int clear,
           cudaStream_t s) {
    const bool aligned = ((uintptr_t)z % 16 == 0) && ((uintptr_t)q_out % 16 == 0) && ((uintptr_t)k_pool % 16 == 0) && ((uintptr_t)v_pool % 16 == 0) &&
                         ((uintptr_t)qk.cos_t % 16 == 0) && ((uintptr_t)qk.sin_t % 16 == 0) && ((uintptr_t)vt.cos_t % 16 == 0) && ((uintptr_t)vt.sin_t % 16 == 0);
    if (!q_w && aligned && dk % 16 == 0 && dv % 16 == 0 && qk.dims % 16 == 0 && vt.dims % 16 == 0 && z_stride % 8 == 0) {
        const long long items = (long long)N * ((nq + nkv) * (dk / 16) + nkv * (dv / 16));
        return launch_kernel(qk_rope_store_vec_kernel<TI, T>, dim3((unsigned)((items + 127) / 128)), dim3(128), 0, s, (TI*)z, z_stride, (T*)q_out, qk,
                             vt, interleaved, slots, (T*)k_pool, (T*)v_pool, N, nq, nkv, dk, dv, page_size, write_kv, clear);
    }
    const long long items = (long long)N * (nq + 2 * nkv);
    return launch_kernel(qk_norm_rope_store_kernel<TI, T>, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, s, (TI*)z, z_stride, (T*)q_out, q_w, k_w,
                         eps, qk, vt, interleaved, slots, (T*)k_pool, (T*)v_pool, N, nq, nkv, dk, dv, page_size, write_kv, clear);
}

}  // namespace

// v_cos / v_sin: [N, dv / 2], or null when values do not turn. clear needs a float32 input.
LLMIE_API int llmie_qk_norm_rope_store(void* z, int z_stride, void* q_out, const float* q_w, const float* k_w, float eps,
                                       const float* cos_t, const float* sin_t, int rot_dims, int interleaved, const float* v_cos,
                                       const float* v_sin, const int* slots, void* k_pool, void* v_pool, int N, int nq, int nkv, int dk, int dv,
                                       int page_size, int write_kv, int clear, int in_dtype, int dtype, cudaStream_t s) {
    if (N <= 0) return 0;
    if (nq <= 0 || nkv <= 0 || dk <= 0 || dv <= 0 || rot_dims < 0 || rot_dims % 2 || rot_dims > dk || page_size <= 0 ||
        (rot_dims && (!cos_t || !sin_t)) || (write_kv && (!slots || !k_pool || !v_pool)) || ((q_w == nullptr) != (k_w == nullptr)) ||
        ((v_cos == nullptr) != (v_sin == nullptr)) || (v_cos && dv % 2) || (clear && in_dtype != DT_F32))
        return LLMIE_ERR_BAD_ARGUMENT;
    const Turn qk{cos_t, sin_t, rot_dims}, vt{v_cos, v_sin, v_cos ? dv : 0};
#define LLMIE_QKP(TI, T) return launch<TI, T>(z, z_stride, q_out, q_w, k_w, eps, qk, vt, interleaved, slots, k_pool, v_pool, N, nq, nkv, dk, dv, \
                                              page_size, write_kv, clear, s)
    if (in_dtype == DT_F32 && dtype == DT_F32) LLMIE_QKP(float, float);
    if (in_dtype == DT_F32 && dtype == DT_BF16) LLMIE_QKP(float, bf16);
    if (in_dtype == DT_BF16 && dtype == DT_BF16) LLMIE_QKP(bf16, bf16);
#undef LLMIE_QKP
    return LLMIE_ERR_BAD_ARGUMENT;
}
