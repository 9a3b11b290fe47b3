// Linear attention with a fixed decay per head for PROMPT PORTIONS, on the tensor cores: S <- a S + k v^T; o = S^T q, taken a chunk of
// CHUNK tokens at a time. With S the state before a chunk and i, j counting the chunk's tokens from 0 (n of them):
//
//   o_i = a^(i+1) S^T q_i + sum_(j <= i) a^(i-j) (q_i . k_j) v_j;      S <- a^n S + sum_j a^(n-1-j) k_j v_j^T
//
// q, k, v are the ACTIVATED projections in bfloat16; everything else is 32-bit: the state and all sums are float accumulators, the
// powers of a are floats from a table. Where a 32-bit number has to enter a product as an operand (the state in S^T q, the weights
// a^(i-j) (q_i . k_j), the scaled values a^(n-1-j) v_j) it does so as the sum of two bfloat16 numbers, in two products, which keeps 16
// of its bits; the other operand is exact.
//
// A block owns one request, one head and COLS columns of its values: S [D, COLS] lives in the accumulators of its eight warps (a warp
// to 16 rows of D, or to two such runs) from the first token of the portion to the last. Warp (m, half) makes the outputs of tokens
// 16 m .. 16 m + 15: `half` takes every second run of 16 keys j and every second run of 16 entries of D, and the two halves' sums meet
// in shared memory. Chunks come by cp.async, two stages.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int CHUNK = 64, COLS = 16, THREADS = 256, VS = COLS + 8;

__device__ __forceinline__ void ldsm_x4(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src, int src_bytes) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(src), "r"(src_bytes));
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

// (x, y) as two bfloat16 pairs whose sums are x and y to 16 bits
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// KD: runs of 16 entries of D (padded with zeros)
template <int KD>
__global__ void __launch_bounds__(THREADS) linear_attention_mma_kernel(const bf16* __restrict__ z, int z_stride, int q_col, int k_col, int v_col,
                                                                       const float* __restrict__ decay, float* __restrict__ state,
                                                                       const int* __restrict__ seq_starts, const int* __restrict__ seq_slots,
                                                                       float* __restrict__ out, int H, int D, int DV) {
    constexpr int QS = 16 * KD + 8;          // row stride of queries and keys: + 16 bytes keeps ldmatrix off bank conflicts
    constexpr int MT = (KD + 7) / 8;         // runs of 16 rows of S per warp
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);        // [2][CHUNK][QS]
    bf16* Ks = Qs + 2 * CHUNK * QS;                      // [2][CHUNK][QS]
    bf16* Vs = Ks + 2 * CHUNK * QS;                      // [2][CHUNK][VS]
    bf16* Wh = Vs + 2 * CHUNK * VS;                      // [CHUNK][VS]: the scaled values, upper and lower part
    bf16* Wl = Wh + CHUNK * VS;
    bf16* Sh = Wl + CHUNK * VS;                          // [16 KD][VS]: the state, upper and lower part
    bf16* Sl = Sh + 16 * KD * VS;
    float* part = reinterpret_cast<float*>(Sl + 16 * KD * VS);   // [CHUNK][COLS]: the second halves' sums
    float* pw = part + CHUNK * COLS;                     // [CHUNK + 1]: powers of the decay

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gid = lane >> 2, tig = lane & 3;
    const int m = warp >> 1, half = warp & 1;
    const int c0 = blockIdx.x * COLS, h = blockIdx.y, r = blockIdx.z;

    if (tid <= CHUNK) {   // a^tid by repeated squaring
        float b = decay[h], y = 1.f;
        for (int e = tid; e > 0; e >>= 1) {
            if (e & 1) y *= b;
            b *= b;
        }
        pw[tid] = y;
    }
    pdl_wait();
    const int s0 = seq_starts[r], L = seq_starts[r + 1] - s0;
    const int nchunks = (L + CHUNK - 1) / CHUNK;

    auto load_chunk = [&](int c, int stage) {
        const int base = s0 + c * CHUNK, count = min(CHUNK, L - c * CHUNK);
        constexpr int segs = 2 * KD;
        for (int i = tid; i < CHUNK * segs; i += THREADS) {
            const int t = i / segs, d = (i % segs) * 8;
            const bool ok = t < count && d < D;
            const bf16* row = z + (size_t)(base + (ok ? t : 0)) * z_stride + (ok ? h * D + d : 0);
            cp_async16(Qs + (stage * CHUNK + t) * QS + d, row + q_col, ok ? 16 : 0);
            cp_async16(Ks + (stage * CHUNK + t) * QS + d, row + k_col, ok ? 16 : 0);
        }
        if (tid < CHUNK * (COLS / 8)) {
            const int t = tid / (COLS / 8), d = (tid % (COLS / 8)) * 8;
            const bool ok = t < count && c0 + d < DV;
            cp_async16(Vs + (stage * CHUNK + t) * VS + d, z + (size_t)(base + (ok ? t : 0)) * z_stride + v_col + (ok ? h * DV + c0 + d : 0), ok ? 16 : 0);
        }
    };
    if (nchunks > 0) load_chunk(0, 0);
    cp_commit();

    // my rows of the state: rows mt * 16 + gid (+ 8), columns nt * 8 + 2 tig (+ 1)
    float* st = state + ((size_t)seq_slots[r] * H + h) * DV * D;
    float S[MT][2][4];
#pragma unroll
    for (int k = 0; k < MT; ++k)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = (warp + 8 * k) * 16 + gid + 8 * (e >> 1), c = c0 + nt * 8 + 2 * tig + (e & 1);
                S[k][nt][e] = (d < D && c < DV) ? st[(size_t)c * D + d] : 0.f;
            }

    for (int c = 0; c < nchunks; ++c) {
        const int stage = c & 1;
        const int n = min(CHUNK, L - c * CHUNK);
        const bf16* Q = Qs + stage * CHUNK * QS;
        const bf16* Kc = Ks + stage * CHUNK * QS;
        const bf16* V = Vs + stage * CHUNK * VS;
        cp_wait<0>();
        __syncthreads();                      // this chunk is in shared memory; everyone is done with the other stage, S and W
        if (c + 1 < nchunks) load_chunk(c + 1, stage ^ 1);
        cp_commit();

        // the state and the scaled values as two-part operands
#pragma unroll
        for (int k = 0; k < MT; ++k) {
            const int mt = warp + 8 * k;
            if (mt >= KD) continue;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    uint32_t hi, lo;
                    split2(S[k][nt][2 * i], S[k][nt][2 * i + 1], hi, lo);
                    const int at = (mt * 16 + gid + 8 * i) * VS + nt * 8 + 2 * tig;
                    *reinterpret_cast<uint32_t*>(Sh + at) = hi;
                    *reinterpret_cast<uint32_t*>(Sl + at) = lo;
                }
        }
        for (int i = tid; i < CHUNK * COLS / 2; i += THREADS) {
            const int t = i / (COLS / 2), d = (i % (COLS / 2)) * 2;
            const float f = t < n ? pw[n - 1 - t] : 0.f;
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(V + t * VS + d);
            uint32_t hi, lo;
            split2(__low2float(v) * f, __high2float(v) * f, hi, lo);
            *reinterpret_cast<uint32_t*>(Wh + t * VS + d) = hi;
            *reinterpret_cast<uint32_t*>(Wl + t * VS + d) = lo;
        }

        // my tokens' products with my keys: runs j16 = half, half + 2 up to my own
        float A[2][2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) A[u][nt][0] = A[u][nt][1] = A[u][nt][2] = A[u][nt][3] = 0.f;
        const int runs = m >= half ? (m - half) / 2 + 1 : 0;
        const bf16* qa = Q + (m * 16 + (lane & 15)) * QS + (lane >> 4) * 8;
        const bf16* kb = Kc + ((lane & 7) + ((lane >> 4) << 3)) * QS + ((lane >> 3) & 1) * 8;
        uint32_t qf[KD][4];
#pragma unroll
        for (int k = 0; k < KD; ++k) ldsm_x4(qf[k], qa + k * 16);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            if (u >= runs) break;
            const bf16* kr = kb + (half + 2 * u) * 16 * QS;
#pragma unroll
            for (int k = 0; k < KD; ++k) {
                uint32_t b[4];
                ldsm_x4(b, kr + k * 16);
                mma_bf16(A[u][0], qf[k], b[0], b[1]);
                mma_bf16(A[u][1], qf[k], b[2], b[3]);
            }
        }
        uint32_t ah[2][4], al[2][4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            if (u >= runs) break;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int row = m * 16 + gid + 8 * i, j = (half + 2 * u) * 16 + nt * 8 + 2 * tig;
                    const float f0 = row >= j ? pw[row - j] : 0.f, f1 = row >= j + 1 ? pw[row - j - 1] : 0.f;
                    split2(A[u][nt][2 * i] * f0, A[u][nt][2 * i + 1] * f1, ah[u][nt * 2 + i], al[u][nt * 2 + i]);
                }
        }
        __syncthreads();                      // the state and the scaled values are there

        // outputs: the state's share (my half of D), then my keys' share
        float O[2][4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) O[nt][0] = O[nt][1] = O[nt][2] = O[nt][3] = 0.f;
#pragma unroll
        for (int k = 0; k < KD; ++k) {
            if ((k & 1) != half) continue;
            uint32_t b[4];
            const int at = (k * 16 + (lane & 15)) * VS + (lane >> 4) * 8;
            ldsm_x4_t(b, Sh + at);
            mma_bf16(O[0], qf[k], b[0], b[1]);
            mma_bf16(O[1], qf[k], b[2], b[3]);
            ldsm_x4_t(b, Sl + at);
            mma_bf16(O[0], qf[k], b[0], b[1]);
            mma_bf16(O[1], qf[k], b[2], b[3]);
        }
        {
            const float f0 = pw[m * 16 + gid + 1], f1 = pw[m * 16 + gid + 9];
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) { O[nt][0] *= f0; O[nt][1] *= f0; O[nt][2] *= f1; O[nt][3] *= f1; }
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            if (u >= runs) break;
            uint32_t b[4];
            ldsm_x4_t(b, V + ((half + 2 * u) * 16 + (lane & 15)) * VS + (lane >> 4) * 8);
            mma_bf16(O[0], ah[u], b[0], b[1]);
            mma_bf16(O[1], ah[u], b[2], b[3]);
            mma_bf16(O[0], al[u], b[0], b[1]);
            mma_bf16(O[1], al[u], b[2], b[3]);
        }
        if (half) {
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int i = 0; i < 2; ++i)
                    *reinterpret_cast<float2*>(part + (m * 16 + gid + 8 * i) * COLS + nt * 8 + 2 * tig) = make_float2(O[nt][2 * i], O[nt][2 * i + 1]);
        }
        // the state: my rows of K^T times the scaled values
        const float fn = pw[n];
#pragma unroll
        for (int k = 0; k < MT; ++k) {
            const int mt = warp + 8 * k;
            if (mt >= KD) continue;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[k][nt][e] *= fn;
            const bf16* ka = Kc + ((lane & 7) + ((lane >> 4) & 1) * 8) * QS + mt * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int t = 0; t < CHUNK / 16; ++t) {
                uint32_t a[4], b[4];
                ldsm_x4_t(a, ka + t * 16 * QS);
                const int at = (t * 16 + (lane & 15)) * VS + (lane >> 4) * 8;
                ldsm_x4_t(b, Wh + at);
                mma_bf16(S[k][0], a, b[0], b[1]);
                mma_bf16(S[k][1], a, b[2], b[3]);
                ldsm_x4_t(b, Wl + at);
                mma_bf16(S[k][0], a, b[0], b[1]);
                mma_bf16(S[k][1], a, b[2], b[3]);
            }
        }
        __syncthreads();                      // the second halves' sums are there
        if (!half) {
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int row = m * 16 + gid + 8 * i, col = nt * 8 + 2 * tig;
                    if (row >= n || c0 + col >= DV) continue;
                    const float2 p = *reinterpret_cast<const float2*>(part + row * COLS + col);
                    *reinterpret_cast<float2*>(out + ((size_t)(s0 + c * CHUNK + row) * H + h) * DV + c0 + col) =
                        make_float2(O[nt][2 * i] + p.x, O[nt][2 * i + 1] + p.y);
                }
        }
    }
    cp_wait<0>();
    pdl_trigger();
#pragma unroll
    for (int k = 0; k < MT; ++k)
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int d = (warp + 8 * k) * 16 + gid + 8 * (e >> 1), c = c0 + nt * 8 + 2 * tig + (e & 1);
                if (d < D && c < DV) st[(size_t)c * D + d] = S[k][nt][e];
            }
}

template <int KD>
int launch(const bf16* z, int z_stride, int q_col, int k_col, int v_col, const float* decay, float* state, const int* seq_starts, const int* seq_slots,
           float* out, int H, int D, int DV, int R, cudaStream_t s) {
    constexpr size_t smem = 2 * ((size_t)4 * CHUNK * (16 * KD + 8) + 4 * CHUNK * VS + 2 * 16 * KD * VS) + sizeof(float) * (CHUNK * COLS + CHUNK + 8);
    static bool set = false;
    if (!set) {
        cudaError_t e = cudaFuncSetAttribute(linear_attention_mma_kernel<KD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        set = true;
    }
    return launch_kernel_on(true, linear_attention_mma_kernel<KD>, dim3((DV + COLS - 1) / COLS, H, R), dim3(THREADS), smem, s, z, z_stride, q_col, k_col, v_col,
                            decay, state, seq_starts, seq_slots, out, H, D, DV);
}

}  // namespace

// 1 if the kernel takes these sizes: rows of heads that start on 16-byte boundaries, keys of up to 256 entries.
LLMIE_API int llmie_linear_attention_mma_fits(int D, int DV) { return D % 8 == 0 && DV % 8 == 0 && D >= 8 && D <= 256 && DV >= 8; }

// z: bfloat16 rows with ACTIVATED q and k (H heads of D from q_col, k_col) and v (H heads of DV from v_col), columns and stride multiples of
// 8; decay [H]; state [slots][H][DV][D] float; out [N][H * DV] float.
LLMIE_API int llmie_linear_attention_mma(const bf16* z, int z_stride, int q_col, int k_col, int v_col, const float* decay, float* state,
                                         const int* seq_starts, const int* seq_slots, float* out, int H, int D, int DV, int R, cudaStream_t s) {
    if (R <= 0) return 0;
    if (H <= 0 || H > 65535 || R > 65535 || !llmie_linear_attention_mma_fits(D, DV) || z_stride % 8 || q_col % 8 || k_col % 8 || v_col % 8 ||
        ((uintptr_t)z % 16) || ((uintptr_t)out % 8))
        return LLMIE_ERR_BAD_ARGUMENT;
#define LLMIE_LA(KD) return launch<KD>(z, z_stride, q_col, k_col, v_col, decay, state, seq_starts, seq_slots, out, H, D, DV, R, s)
    if (D <= 32) LLMIE_LA(2);
    if (D <= 64) LLMIE_LA(4);
    if (D <= 96) LLMIE_LA(6);
    if (D <= 128) LLMIE_LA(8);
    if (D <= 192) LLMIE_LA(12);
    LLMIE_LA(16);
#undef LLMIE_LA
}
