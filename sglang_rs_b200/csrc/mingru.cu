// minGRU: a recurrence per channel whose gate and candidate read the current token only, over a state of `width` 32-bit
// floats per request.  A row of the projection holds (at three column offsets) z, x and g, `width` entries each:
//
//   z_t = sigmoid(z + z_bias)     u = x + x_bias     c_t = u + 1/2 where u >= 0, sigmoid(u) where u < 0
//   S_t = (1 - z_t) S_(t-1) + z_t c_t                out_t = S_t silu(g)
//
// Every channel runs by itself, so a step is bound by reading the projection.  Steps in which every request brings one row
// (decoded tokens) are one pass.  Other steps cut each request's rows into chunks of 32: (1) per (chunk, channel) the chunk as
// an affine map S -> A S + B, (2) per (request, channel) the states before every chunk, in order, the slot receiving the last
// one, (3) per (chunk, channel) the rows again from the state before the chunk.  Everything between the projection and the
// result is 32-bit in both dtypes.  A request whose first row of the step is at position 0 starts from zero whatever its slot
// holds; rows at negative positions pad a captured step and are skipped.
#include "common.cuh"
#include <math.h>

SRB_DEFINE_LAST_ERROR()
SRB_DEFINE_PDL_SWITCH()

#define GRU_CHUNK 32
#define GRU_THREADS 128
#define GRU_BATCH 8              // rows whose loads are in flight together

struct GruArgs {
  const void* proj;
  long long pitch;
  int z_at, x_at, g_at, width;
  const float* z_bias;
  const float* x_bias;
  const int* positions;
  const int* cu_rows;
  const int* state_slots;
  float* state;                  // [slots, width]
  float* maps;                   // [chunks][2][width]: A and B of a chunk; A is replaced by the state before the chunk
  void* out;
  long long out_pitch;
  int requests, write_state;
  float scale;                   // a factor on every result
};

// (1 - z, z c) of a row: S <- keep S + add
__device__ __forceinline__ float2 gru_row(float z, float x) {
  const float gate = __fdividef(1.0f, 1.0f + expf(-z));   // (a quotient to 2 units in the last place)
  const float candidate = x >= 0.f ? x + 0.5f : __fdividef(1.0f, 1.0f + expf(-x));
  return make_float2(1.0f - gate, gate * candidate);
}
__device__ __forceinline__ float gru_silu(float g) { return __fdividef(g, 1.0f + expf(-g)); }

template <typename T>
__global__ void __launch_bounds__(GRU_THREADS) gru_single_kernel(GruArgs a) {
  srb_launch_dependents();
  const int c = blockIdx.x * GRU_THREADS + threadIdx.x, request = blockIdx.y;
  const float zb = c < a.width ? a.z_bias[c] : 0.f, xb = c < a.width ? a.x_bias[c] : 0.f;
  srb_grid_dependency_wait();
  if (c >= a.width) return;
  const int row = a.cu_rows[request];
  if (a.cu_rows[request + 1] != row + 1) return;           // (the launcher is only used for steps of single rows)
  const int pos = a.positions[row];
  if (pos < 0) return;
  const T* p = reinterpret_cast<const T*>(a.proj) + (size_t)row * a.pitch + c;
  float* state = a.state + (size_t)a.state_slots[request] * a.width + c;
  const float z = srb_to_float(p[a.z_at]), x = srb_to_float(p[a.x_at]), g = srb_to_float(p[a.g_at]);
  const float before = pos == 0 ? 0.f : *state;
  const float2 m = gru_row(z + zb, x + xb);
  const float s = fmaf(m.x, before, m.y);
  reinterpret_cast<T*>(a.out)[(size_t)row * a.out_pitch + c] = srb_from_float<T>(s * gru_silu(g) * a.scale);
  if (a.write_state) *state = s;
}

// the request and the chunk of it that block `index` works on; false: there is no such chunk
__device__ __forceinline__ bool gru_find(const GruArgs& a, int index, int& request, int& row0, int& n) {
  int first = 0;
  for (request = 0; request < a.requests; ++request) {
    const int begin = a.cu_rows[request], rows = a.cu_rows[request + 1] - begin;
    const int chunks = (rows + GRU_CHUNK - 1) / GRU_CHUNK;
    if (index < first + chunks) {
      row0 = begin + (index - first) * GRU_CHUNK;
      n = min(GRU_CHUNK, begin + rows - row0);
      return true;
    }
    first += chunks;
  }
  return false;
}

// V neighbouring channels of a row: one load, or (two bfloat16) four bytes
template <typename T, int V> struct GruPiece { T v[V]; };
template <typename T, int V> __device__ __forceinline__ GruPiece<T, V> gru_load(const T* p) {
  GruPiece<T, V> r;
  if constexpr (sizeof(T) * V == 4) *reinterpret_cast<unsigned*>(r.v) = *reinterpret_cast<const unsigned*>(p);
  else r.v[0] = *p;
  return r;
}
template <typename T, int V> __device__ __forceinline__ void gru_store(T* p, const GruPiece<T, V>& r) {
  if constexpr (sizeof(T) * V == 4) *reinterpret_cast<unsigned*>(p) = *reinterpret_cast<const unsigned*>(r.v);
  else *p = r.v[0];
}

// OUTPUT false: the chunk's map; true: the rows from the state before the chunk.  A thread takes V channels.
template <typename T, int V, bool OUTPUT>
__global__ void __launch_bounds__(GRU_THREADS) gru_chunk_kernel(GruArgs a) {
  srb_launch_dependents();
  const int c = (blockIdx.x * GRU_THREADS + threadIdx.x) * V;
  float zb[V], xb[V];
#pragma unroll
  for (int k = 0; k < V; ++k) {
    zb[k] = c < a.width ? a.z_bias[c + k] : 0.f;
    xb[k] = c < a.width ? a.x_bias[c + k] : 0.f;
  }
  srb_grid_dependency_wait();
  int request, row0, n;
  if (!gru_find(a, blockIdx.y, request, row0, n) || c >= a.width) return;
  const T* p = reinterpret_cast<const T*>(a.proj) + (size_t)row0 * a.pitch + c;
  T* out = reinterpret_cast<T*>(a.out) + (size_t)row0 * a.out_pitch + c;
  float* map = a.maps + (size_t)blockIdx.y * 2 * a.width + c;
  float keep[V], s[V];
#pragma unroll
  for (int k = 0; k < V; ++k) { keep[k] = 1.f; s[k] = OUTPUT ? map[k] : 0.f; }
#pragma unroll 1
  for (int t0 = 0; t0 < n; t0 += GRU_BATCH) {
    GruPiece<T, V> z[GRU_BATCH], x[GRU_BATCH], g[GRU_BATCH];
#pragma unroll
    for (int j = 0; j < GRU_BATCH; ++j)
      if (t0 + j < n) {
        const T* row = p + (size_t)(t0 + j) * a.pitch;
        z[j] = gru_load<T, V>(row + a.z_at);
        x[j] = gru_load<T, V>(row + a.x_at);
        if (OUTPUT) g[j] = gru_load<T, V>(row + a.g_at);
      }
#pragma unroll
    for (int j = 0; j < GRU_BATCH; ++j)
      if (t0 + j < n) {
        GruPiece<T, V> y;
#pragma unroll
        for (int k = 0; k < V; ++k) {
          const float2 m = gru_row(srb_to_float(z[j].v[k]) + zb[k], srb_to_float(x[j].v[k]) + xb[k]);
          s[k] = fmaf(m.x, s[k], m.y);
          if (OUTPUT) y.v[k] = srb_from_float<T>(s[k] * gru_silu(srb_to_float(g[j].v[k])) * a.scale);
          else keep[k] *= m.x;
        }
        if (OUTPUT) gru_store<T, V>(out + (size_t)(t0 + j) * a.out_pitch, y);
      }
  }
  if (!OUTPUT) {
#pragma unroll
    for (int k = 0; k < V; ++k) {
      map[k] = keep[k];
      map[a.width + k] = s[k];
    }
  }
}

__global__ void __launch_bounds__(GRU_THREADS) gru_prefix_kernel(GruArgs a) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int c = blockIdx.x * GRU_THREADS + threadIdx.x, request = blockIdx.y;
  if (c >= a.width) return;
  int first = 0;
  for (int r = 0; r < request; ++r) first += (a.cu_rows[r + 1] - a.cu_rows[r] + GRU_CHUNK - 1) / GRU_CHUNK;
  const int begin = a.cu_rows[request], rows = a.cu_rows[request + 1] - begin;
  if (rows <= 0) return;
  const int start = a.positions[begin];
  if (start < 0) return;
  float* state = a.state + (size_t)a.state_slots[request] * a.width + c;
  float s = start == 0 ? 0.f : *state;
  const int chunks = (rows + GRU_CHUNK - 1) / GRU_CHUNK;
  float* map = a.maps + (size_t)first * 2 * a.width + c;
  for (int c0 = 0; c0 < chunks; c0 += GRU_BATCH) {
    float keep[GRU_BATCH], add[GRU_BATCH];
#pragma unroll
    for (int k = 0; k < GRU_BATCH; ++k)
      if (c0 + k < chunks) {
        keep[k] = map[(size_t)(c0 + k) * 2 * a.width];
        add[k] = map[(size_t)(c0 + k) * 2 * a.width + a.width];
      }
#pragma unroll
    for (int k = 0; k < GRU_BATCH; ++k)
      if (c0 + k < chunks) {
        map[(size_t)(c0 + k) * 2 * a.width] = s;
        s = fmaf(keep[k], s, add[k]);
      }
  }
  if (a.write_state) *state = s;
}

template <typename T>
static int launch_gru(const GruArgs& a, int single_rows, int chunks, cudaStream_t s) {
  const int blocks = (a.width + GRU_THREADS - 1) / GRU_THREADS;
  if (blocks > 65535) SRB_FAIL("mingru: %d channels exceed one launch", a.width);
  if (single_rows) {
    SRB_CUDA_CALL(srb_launch(gru_single_kernel<T>, dim3(blocks, a.requests), dim3(GRU_THREADS), 0, s, a));
    SRB_LAUNCH_CHECK("mingru_single");
    return SRB_OK;
  }
  if (chunks > 65535) SRB_FAIL("mingru: %d chunks exceed one launch", chunks);
  constexpr int PAIR = sizeof(T) == 2 ? 2 : 1;
  const bool pair = PAIR == 2 && ((a.width | a.z_at | a.x_at | a.g_at | a.pitch | a.out_pitch) & 1) == 0 &&
                    (((uintptr_t)a.proj | (uintptr_t)a.out) & 3) == 0;
  const int v = pair ? 2 : 1;
  const dim3 grid((a.width / v + GRU_THREADS - 1) / GRU_THREADS, chunks);
  SRB_CUDA_CALL(srb_launch(pair ? gru_chunk_kernel<T, PAIR, false> : gru_chunk_kernel<T, 1, false>, grid, dim3(GRU_THREADS), 0, s, a));
  SRB_CUDA_CALL(srb_launch(gru_prefix_kernel, dim3(blocks, a.requests), dim3(GRU_THREADS), 0, s, a));
  SRB_CUDA_CALL(srb_launch(pair ? gru_chunk_kernel<T, PAIR, true> : gru_chunk_kernel<T, 1, true>, grid, dim3(GRU_THREADS), 0, s, a));
  SRB_LAUNCH_CHECK("mingru");
  return SRB_OK;
}

extern "C" int srb_mingru_chunk_tokens() { return GRU_CHUNK; }

// `single_rows`: every request of the step brings exactly one row (`maps` and `chunks` are then unused).  Otherwise `chunks`:
// the number of chunks of the step, sum over the requests of ceil(rows / srb_mingru_chunk_tokens()), or more; `maps`: chunks *
// 2 * width floats of scratch.  `scale`: a factor on every result.  out: rows `out_pitch` elements apart, of the projection's type.
extern "C" int srb_mingru(const void* proj, long long pitch, int z_at, int x_at, int g_at, int width, const float* z_bias,
                          const float* x_bias, const int* positions, const int* cu_rows, const int* state_slots, float* state,
                          float* maps, void* out, long long out_pitch, int rows, int requests, int chunks, int single_rows,
                          int write_state, float scale, int dtype, void* stream) {
  if (rows <= 0 || requests <= 0) return SRB_OK;
  if (width <= 0) SRB_FAIL("mingru: %d channels", width);
  if (requests > 65535) SRB_FAIL("mingru: %d requests exceed one launch", requests);
  if (z_at < 0 || x_at < 0 || g_at < 0 || (long long)z_at + width > pitch || (long long)x_at + width > pitch || (long long)g_at + width > pitch)
    SRB_FAIL("mingru: rows of the projection are too short");
  if (!single_rows && (chunks <= 0 || !maps)) SRB_FAIL("mingru: the chunks' maps need scratch memory");
  if (out_pitch < width) SRB_FAIL("mingru: rows of the output overlap");
  GruArgs a;
  a.proj = proj; a.pitch = pitch; a.z_at = z_at; a.x_at = x_at; a.g_at = g_at; a.width = width; a.z_bias = z_bias; a.x_bias = x_bias;
  a.positions = positions; a.cu_rows = cu_rows; a.state_slots = state_slots; a.state = state; a.maps = maps; a.out = out;
  a.out_pitch = out_pitch; a.requests = requests; a.write_state = write_state; a.scale = scale;
  if (dtype == SRB_DTYPE_F32) return launch_gru<float>(a, single_rows, chunks, (cudaStream_t)stream);
  if (dtype == SRB_DTYPE_BF16) return launch_gru<__nv_bfloat16>(a, single_rows, chunks, (cudaStream_t)stream);
  SRB_FAIL("mingru: unknown dtype %d", dtype);
}
