// Entry points of the windowed tensor-core attention (attention_window_mma.cuh) and its softmax form.
#include "attention_window_mma.cuh"

using namespace cib;

extern "C" int cib_window_attention_mma_supports(int dim, int vdim, int nq, int nkv) {
    return (dim == 64 || dim == 128) && (vdim == 32 || vdim == 64 || vdim == 128) && nkv > 0 && nq % nkv == 0;
}

// num_tiles: the sum over requests of ceil(tokens_r * (nq / nkv) / 64), or any upper bound of it (CTAs that find no
// tile leave).  num_splits > 1: every row tile's key tiles are shared out to so many CTAs, which leave float32 partial
// results in `partial` ([tokens * nq][num_splits][vdim + 2]: output, running maximum, sum) for a second kernel to merge.
// chunked: the window is a chunk (keys from floor(i / window) * window on); slopes, sinks: float32 [nq] or null.
// sigmoid_bias: float32 [nq], weights sigmoid(score + bias) without normalisation; r1, r2: float32 [nq], the bias
// -r1 ln(1 + r2 (i - j)); gate: gate logits [tokens][nq * vdim] or, with gate_per_head, [tokens][nq] (rows gate_stride apart).
// few_rows: no request has more than 16 rows (tokens * nq / nkv) in this launch, e.g. a decode step: the form whose
// warps share out a tile's keys instead of its rows runs (any tile with more rows still takes the row-parallel path).
extern "C" int cib_window_attention_mma(const void* q, int q_stride, void* out, int out_stride, const void* cache,
                                        int num_pages, int page_size, const int* block_table, int table_stride,
                                        const int* query_start_loc, const int* seq_lens, int num_requests, int num_tiles,
                                        int nq, int nkv, int dim, int vdim, float scale, float cap, int window,
                                        int keep_first, int num_splits, float* partial, int num_tokens, int chunked,
                                        int few_rows, const float* slopes, const float* sinks, const float* sigmoid_bias,
                                        const float* r1, const float* r2, const void* gate, int gate_stride, int gate_per_head,
                                        cudaStream_t stream) {
    CIB_REQUIRE(cib_window_attention_mma_supports(dim, vdim, nq, nkv), "window_attention_mma: sizes %d / %d are not taken by this kernel", dim, vdim);
    CIB_REQUIRE(num_requests >= 0 && num_tiles >= 0 && nkv <= 65535, "window_attention_mma: bad sizes");
    CIB_REQUIRE(num_splits >= 1 && num_splits <= 64 && (num_splits == 1 || partial), "window_attention_mma: %d splits need room for their partial results", num_splits);
    CIB_REQUIRE(page_size > 0 && num_pages > 0 && table_stride > 0 && window >= 0 && keep_first >= 0, "window_attention_mma: bad cache geometry");
    CIB_REQUIRE(q_stride % 8 == 0 && ((uintptr_t)q % 16) == 0 && out_stride % 2 == 0 && ((uintptr_t)out % 4) == 0 && ((uintptr_t)cache % 16) == 0,
                "window_attention_mma: q and cache rows must be 16-byte aligned and out rows 4-byte aligned");
    CIB_REQUIRE((r1 == nullptr) == (r2 == nullptr) && !(r1 && sigmoid_bias) && !(slopes && (r1 || sigmoid_bias)) && !(sinks && sigmoid_bias),
                "window_attention_mma: one distance bias at a time; weights that are not normalised have neither bias nor sink");
    if (num_requests == 0 || num_tiles == 0) return 0;
    const WindowExtras ex{sigmoid_bias, r1, r2, (const __nv_bfloat16*)gate, gate_stride, gate_per_head};
    const bool few = few_rows != 0;
    if (sigmoid_bias)
        return window_mma_sigmoid(q, q_stride, out, out_stride, cache, num_pages, page_size, block_table, table_stride, query_start_loc,
                                  seq_lens, num_requests, num_tiles, nq, nkv, dim, vdim, scale, cap, window, keep_first, num_splits,
                                  partial, num_tokens, chunked, few, slopes, sinks, ex, stream);
    if (r1)
        return window_mma_log_bias(q, q_stride, out, out_stride, cache, num_pages, page_size, block_table, table_stride, query_start_loc,
                                   seq_lens, num_requests, num_tiles, nq, nkv, dim, vdim, scale, cap, window, keep_first, num_splits,
                                   partial, num_tokens, chunked, few, slopes, sinks, ex, stream);
    return launch_window_mma_sizes<kWmSoftmax>(q, q_stride, out, out_stride, cache, num_pages, page_size, block_table, table_stride,
                                               query_start_loc, seq_lens, num_requests, num_tiles, nq, nkv, dim, vdim, scale, cap,
                                               window, keep_first, num_splits, partial, num_tokens, chunked, few, slopes, sinks, ex, stream);
}
