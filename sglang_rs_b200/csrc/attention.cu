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
// `out_scale` every result; `out_pitch` elements lie between rows of the output (0: dense).  `terms` (or null): kept first
// tokens, a cap on the scores, two maps per head (AttnTerms); with two maps n_q counts the maps and `out` is float.
extern "C" int srb_paged_attention_terms(const void* q, const void* k_pool, const void* v_pool, void* out,
                                         float* part_acc, float* part_ml, const int* positions,
                                         const int* row_request, const int* block_table, int table_stride, int rows,
                                         int n_q, int n_kv, int head_dim, int page_size, int num_pages, int window,
                                         int chunk, int split_size, int max_splits, float scale, int* error_word,
                                         int dtype, const float* sinks, int value_dim, const float* gates, long long out_pitch,
                                         float out_scale, const AttnTerms* terms, void* stream) {
  return paged_attention_dispatch_masked(q, k_pool, v_pool, out, part_acc, part_ml, positions, row_request, block_table,
                                         table_stride, rows, n_q, n_kv, head_dim, page_size, num_pages, window, chunk,
                                         split_size, max_splits, scale, error_word, dtype, sinks, value_dim, stream, gates,
                                         out_pitch, out_scale, terms);
}

extern "C" int srb_paged_attention_gated(const void* q, const void* k_pool, const void* v_pool, void* out,
                                         float* part_acc, float* part_ml, const int* positions,
                                         const int* row_request, const int* block_table, int table_stride, int rows,
                                         int n_q, int n_kv, int head_dim, int page_size, int num_pages, int window,
                                         int chunk, int split_size, int max_splits, float scale, int* error_word,
                                         int dtype, const float* sinks, int value_dim, const float* gates, long long out_pitch,
                                         float out_scale, void* stream) {
  return srb_paged_attention_terms(q, k_pool, v_pool, out, part_acc, part_ml, positions, row_request, block_table, table_stride,
                                   rows, n_q, n_kv, head_dim, page_size, num_pages, window, chunk, split_size, max_splits,
                                   scale, error_word, dtype, sinks, value_dim, gates, out_pitch, out_scale, nullptr, stream);
}

// ---- two maps per head: the join -----------------------------------------------------------------------------------
// a: float [rows, 2 heads, width], map t of head h at 2 h + t.  out[row, h] = scale * o / sqrt(mean(o^2) + eps) with
// o = a_1 - lambda a_2, all in 32-bit; a warp per head.
template <typename T>
__global__ void map_combine_kernel(const float* __restrict__ a, T* __restrict__ out, int rows, int heads, int width,
                                   size_t out_pitch, float lambda, float scale, float eps) {
  const int lane = threadIdx.x & 31;
  const long long number = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (number >= (long long)rows * heads) return;
  const size_t row = number / heads, head = number % heads;
  const float* first = a + (size_t)number * 2 * width;
  float squares = 0.f;
  for (int e = lane; e < width; e += 32) {
    const float o = first[e] - lambda * first[width + e];
    squares += o * o;
  }
  const float factor = scale / sqrtf(srb_warp_sum(squares) / (float)width + eps);
  for (int e = lane; e < width; e += 32)
    out[row * out_pitch + head * width + e] = srb_from_float<T>((first[e] - lambda * first[width + e]) * factor);
}

extern "C" int srb_map_combine(const float* a, void* out, int rows, int heads, int width, long long out_pitch, float lambda,
                               float scale, float eps, int dtype, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (heads <= 0 || width <= 0 || out_pitch < (long long)heads * width) SRB_FAIL("map_combine: %d heads of %d entries do not fit the rows of the output", heads, width);
  const unsigned blocks = (unsigned)(((long long)rows * heads + 3) / 4);
  if (dtype == SRB_DTYPE_F32)
    map_combine_kernel<float><<<blocks, 128, 0, (cudaStream_t)stream>>>(a, (float*)out, rows, heads, width, (size_t)out_pitch, lambda, scale, eps);
  else if (dtype == SRB_DTYPE_BF16)
    map_combine_kernel<__nv_bfloat16><<<blocks, 128, 0, (cudaStream_t)stream>>>(a, (__nv_bfloat16*)out, rows, heads, width, (size_t)out_pitch, lambda, scale, eps);
  else
    SRB_FAIL("map_combine: unknown dtype %d", dtype);
  SRB_LAUNCH_CHECK("map_combine");
  return SRB_OK;
}
