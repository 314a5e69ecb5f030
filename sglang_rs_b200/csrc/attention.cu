// Entry point of the generic paged attention; the kernels are in attention_kernels.cuh.
#include "attention_kernels.cuh"

SRB_DEFINE_LAST_ERROR()

// Scratch (only when split_size > 0): part_acc holds rows * n_q * max_splits * head_dim
// floats and part_ml rows * n_q * max_splits * 2 floats.
extern "C" int srb_paged_attention(const void* q, const void* k_pool, const void* v_pool, void* out,
                                   float* part_acc, float* part_ml, const int* positions,
                                   const int* row_request, const int* block_table, int table_stride, int rows,
                                   int n_q, int n_kv, int head_dim, int page_size, int num_pages, int window,
                                   int split_size, int max_splits, float scale, int* error_word, int dtype,
                                   void* stream) {
  return paged_attention_dispatch(q, k_pool, v_pool, out, part_acc, part_ml, positions, row_request, block_table,
                                  table_stride, rows, n_q, n_kv, head_dim, page_size, num_pages, window, split_size,
                                  max_splits, scale, error_word, dtype, stream);
}

// The same with the two optional terms: `sinks` (one float per query head, or null), values of `value_dim`
// entries (0: as wide as the keys), and, with v_pool null, values that are the head of the key rows.
extern "C" int srb_paged_attention_ex(const void* q, const void* k_pool, const void* v_pool, void* out,
                                      float* part_acc, float* part_ml, const int* positions,
                                      const int* row_request, const int* block_table, int table_stride, int rows,
                                      int n_q, int n_kv, int head_dim, int page_size, int num_pages, int window,
                                      int split_size, int max_splits, float scale, int* error_word, int dtype,
                                      const float* sinks, int value_dim, void* stream) {
  return paged_attention_dispatch_ex(q, k_pool, v_pool, out, part_acc, part_ml, positions, row_request, block_table,
                                     table_stride, rows, n_q, n_kv, head_dim, page_size, num_pages, window, split_size,
                                     max_splits, scale, error_word, dtype, sinks, value_dim, stream);
}

// The same with a mask by chunks of positions: with `chunk` > 0 a row sees, of the keys up to its own, only those of
// its own chunk (positions floor(pos / chunk) * chunk .. pos), whatever portion of a prompt brought it.
extern "C" int srb_paged_attention_masked(const void* q, const void* k_pool, const void* v_pool, void* out,
                                          float* part_acc, float* part_ml, const int* positions,
                                          const int* row_request, const int* block_table, int table_stride, int rows,
                                          int n_q, int n_kv, int head_dim, int page_size, int num_pages, int window,
                                          int chunk, int split_size, int max_splits, float scale, int* error_word,
                                          int dtype, const float* sinks, int value_dim, void* stream) {
  return paged_attention_dispatch_masked(q, k_pool, v_pool, out, part_acc, part_ml, positions, row_request, block_table,
                                         table_stride, rows, n_q, n_kv, head_dim, page_size, num_pages, window, chunk,
                                         split_size, max_splits, scale, error_word, dtype, sinks, value_dim, stream);
}

// The same with a gate per (row, query head): `gates` (float [rows, n_q], or null) multiplies each head's result,
// `out_scale` every result; `out_pitch` elements lie between rows of the output (0: dense).
extern "C" int srb_paged_attention_gated(const void* q, const void* k_pool, const void* v_pool, void* out,
                                         float* part_acc, float* part_ml, const int* positions,
                                         const int* row_request, const int* block_table, int table_stride, int rows,
                                         int n_q, int n_kv, int head_dim, int page_size, int num_pages, int window,
                                         int chunk, int split_size, int max_splits, float scale, int* error_word,
                                         int dtype, const float* sinks, int value_dim, const float* gates, long long out_pitch,
                                         float out_scale, void* stream) {
  return paged_attention_dispatch_masked(q, k_pool, v_pool, out, part_acc, part_ml, positions, row_request, block_table,
                                         table_stride, rows, n_q, n_kv, head_dim, page_size, num_pages, window, chunk,
                                         split_size, max_splits, scale, error_word, dtype, sinks, value_dim, stream, gates,
                                         out_pitch, out_scale);
}
