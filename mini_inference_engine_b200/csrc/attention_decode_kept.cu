// Decode attention under a window (or block of positions) that keeps the first `keep` keys of the sequence in sight: the kernel of
// attention_decode.cu with the kept keys' tiles walked in front of the window's (the table entries of the pages between the two
// are never followed).  A library of its own, so that models without such a window do not compile these instances.
#include "attention_decode.cuh"

// Parameters as mie_decode_attention (attention_decode.cu), without the rotation inside the kernel; keep > 0, window != 0.
extern "C" int mie_decode_attention_kept(const void* q, int64_t q_stride, const void* k_cache, const void* v_cache,
                                         const int* block_tables, int table_stride, const int* row_q_start,
                                         const int* row_q_len, const int* row_ctx_len, int num_rows, void* out,
                                         int num_heads, int num_kv_heads, int head_dim, int page_size, float scale,
                                         int window, int keep, int splits, float* part_o, float* part_lse, int* counters,
                                         int stages, int64_t num_pages, int64_t check_pages, int min_part_tiles, int out_f32,
                                         float softcap, const float* sink, const float* dist_bias, int dist_len, const float* slope, cudaStream_t stream) {
    if (window == 0 || keep <= 0) return MIE_ERR_BAD_ARG;
    const ScoreMods mods{softcap, sink, dist_bias, dist_len, slope};
    return decode_attention_launch<true>(q, q_stride, k_cache, v_cache, block_tables, table_stride, row_q_start, row_q_len,
                                         row_ctx_len, num_rows, out, num_heads, num_kv_heads, head_dim, page_size, scale,
                                         window, splits, part_o, part_lse, counters, stream, stages, num_pages, check_pages,
                                         g_range_report, min_part_tiles, nullptr, nullptr, 0, out_f32 != 0, &mods, keep);
}

// Non-zero when a block of any launch so far gave up a bounded wait (TMA copies that did not arrive).
extern "C" int mie_decode_attention_kept_error(void) { return g_error_host ? *g_error_host : 0; }
extern "C" void mie_decode_attention_kept_clear_error(void) { if (g_error_host) *g_error_host = 0; }
