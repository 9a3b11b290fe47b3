// The exported functions of the tensor-core attention with extras (see attention_ext_mma.cuh).
#include "attention_ext_mma.cuh"

using namespace attn_ext_mma;

// the most row blocks per warp that registers allow for value rows of 32 * nt entries
static int max_r(int nt) { return nt <= 2 ? 4 : (nt <= 8 ? 2 : 1); }


// 0 if the kernel does not take these sizes (bfloat16 only): dk a multiple of 16, dv one of 32 * {1, 2, 3, 4, 6, 8, 12, 16}, and
// shared memory for two stages of keys. Otherwise the most rows a tile may have: 32, 64 or 128.
LLMIE_API int llmie_attention_ext_mma_fits(int dk, int dv, int own_values) {
    const int nt = dv / 32;
    const bool nt_ok = dv % 32 == 0 && (nt == 1 || nt == 2 || nt == 3 || nt == 4 || nt == 6 || nt == 8 || nt == 12 || nt == 16);
    if (!(dk % 16 == 0 && dk >= 16 && nt_ok && (own_values || dv <= dk))) return 0;
    for (int r = max_r(nt); r >= 1; r >>= 1)
        if (smem_bytes(dk, dv, own_values != 0, r) <= 227 * 1024) return ROWS * r;
    return 0;
}

// tile_info: [tiles][2] = (first token, tokens) with at most tile_rows / gh tokens of one request per tile, or null: one token per
// tile. tile_rows: 32, 64 or 128 (at most what llmie_attention_ext_mma_fits says); gh = min(group, 32) heads per token in a tile;
// scratch (num_splits > 1): N * nq * num_splits * (dv + 2) floats.
LLMIE_API int llmie_paged_attention_ext_mma(const bf16* q, int q_stride, const bf16* k_pool, const bf16* v_pool, const int* block_table,
                                            int max_blocks, const int* token_seq, const int* positions, const int* tile_info, int tiles,
                                            int tile_rows, bf16* out, float* scratch, int N, int nq, int nkv, int dk, int dv, int page_size,
                                            float scale, int window, int num_splits, float temp_coef, int temp_every, const float* rel,
                                            const int* rows_of, int n_rows_of, int rel_rows, const float* sink, const bf16* gate,
                                            int gate_stride, int gate_mode, int keep_first, int chunk, float softcap, const float* sig_bias, const float* log_r1,
                                            const float* log_r2, const float* turn_cos, const float* turn_sin, int turn_neighbours, const float* key_scale, cudaStream_t s) {
    if (N <= 0 || tiles <= 0) return 0;
    const int fits = llmie_attention_ext_mma_fits(dk, dv, v_pool != nullptr);
    if (nkv <= 0 || nq % nkv || !fits || tile_rows > fits || (tile_rows != 32 && tile_rows != 64 && tile_rows != 128) || page_size <= 0 ||
        num_splits < 1 || (num_splits > 1 && !scratch) || q_stride % 8 || ((uintptr_t)q % 16) || ((uintptr_t)k_pool % 16) ||
        ((uintptr_t)v_pool % 16) || (rel && (!rows_of || rel_rows < 1)) || (gate_mode && !gate))
        return LLMIE_ERR_BAD_ARGUMENT;
    Params P;
    P.q = q; P.q_stride = q_stride; P.k_pool = k_pool; P.v_pool = v_pool; P.block_table = block_table; P.max_blocks = max_blocks;
    P.token_seq = token_seq; P.positions = positions; P.tile_info = tile_info; P.out = out;
    P.part_acc = scratch; P.part_ml = scratch ? scratch + (size_t)N * nq * num_splits * dv : nullptr;
    P.nq = nq; P.nkv = nkv; P.dk = dk; P.dv = dv; P.page_size = page_size; P.scale = scale; P.window = window; P.num_splits = num_splits;
    const int G = nq / nkv;
    P.gh = G < ROWS ? G : ROWS;
    P.head_chunks = (G + P.gh - 1) / P.gh;
    P.ex.temp_coef = temp_coef; P.ex.temp_every = temp_every; P.ex.rel = rel; P.ex.rows_of = rows_of; P.ex.n_rows_of = n_rows_of;
    P.ex.rel_rows = rel_rows; P.ex.sink = sink; P.ex.gate = gate; P.ex.gate_stride = gate_stride; P.ex.gate_mode = gate_mode;
    P.ex.keep_first = keep_first; P.ex.chunk = chunk; P.ex.softcap = softcap;
    P.ex.sig_bias = sig_bias; P.ex.log_r1 = log_r1; P.ex.log_r2 = log_r2;
    P.ex.turn_cos = turn_cos; P.ex.turn_sin = turn_sin; P.ex.turn_neighbours = turn_neighbours;
    P.ex.key_scale = key_scale;
    if (attn_ext::bad_extras(P.ex, dv) || (sig_bias && (rel || keep_first || chunk || softcap != 0.f || key_scale))) return LLMIE_ERR_BAD_ARGUMENT;
    if ((long long)nkv * P.head_chunks > 65535 || num_splits > 65535) return LLMIE_ERR_BAD_ARGUMENT;
    const dim3 grid(tiles, nkv * P.head_chunks, num_splits);
    const int R = tile_rows / ROWS;
    // decoded tokens alone (no tiles of several tokens): a deeper ring where two blocks still fit on a multiprocessor with it
    // (measured at heads of 128, where it costs the second block: batch 64 at 4,096 keys 162 -> 225 us; heads of 64 gain 2 %)
    const size_t table_bytes = rel ? bias_bytes(rel_rows, G < ROWS ? G : ROWS, n_rows_of) : 0;
    const bool deep = !tile_info && R == 1 &&
                      2 * (smem_bytes(dk, dv, v_pool != nullptr, 1, DEEP) + (table_bytes <= 32 * 1024 ? table_bytes : 0) + 1024) <= 227 * 1024;
    size_t smem = smem_bytes(dk, dv, v_pool != nullptr, R, deep ? DEEP : 2);
    if (turn_cos) {   // the sums of all rows pass through shared memory at the end
        const size_t need = sizeof(float) * (size_t)tile_rows * dv;
        if (smem < need) smem = need;
    }
    P.bias_in_smem = 0;
    if (rel && rel_rows <= 65535 && bias_bytes(rel_rows, P.gh, n_rows_of) <= 32 * 1024 && smem + bias_bytes(rel_rows, P.gh, n_rows_of) <= 227 * 1024) {
        P.bias_in_smem = 1;
        smem += bias_bytes(rel_rows, P.gh, n_rows_of);
    }
    P.key_scale_at = 0;
    if (key_scale) {
        P.key_scale_at = (unsigned)smem;   // (a multiple of 8: whole rows of 16 bytes, floats, an even number of 16-bit row numbers)
        if (P.key_scale_at % 8) P.key_scale_at += 8 - P.key_scale_at % 8;
        smem = P.key_scale_at + sizeof(float) * KEYS * (deep ? DEEP : 2);
        if (smem > 227 * 1024) return LLMIE_ERR_BAD_ARGUMENT;
    }
    const int kind = attn_ext::kind_of(P.ex);
    int rc = kind == attn_ext::SIGMOID ? launch_sigmoid(P, grid, smem, s, R, deep)
           : kind == attn_ext::MASKS ? launch_masks(P, grid, smem, s, R, deep) : launch_plain(P, grid, smem, s, R, deep);
    if (rc) return rc;
    if (num_splits > 1) {
        attn_ext::attn_ext_combine_kernel<bf16><<<N * nq, 128, 0, s>>>(P.part_acc, P.part_ml, out, nq, dv, num_splits, P.ex);
        rc = launch_status();
    }
    return rc;
}
