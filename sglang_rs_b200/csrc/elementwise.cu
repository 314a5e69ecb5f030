// Row-wise kernels of the decoder: embedding gather, fused residual-add + RMSNorm,
// SiLU(gate)*up, bias add.  All arithmetic is 32-bit; T is the storage type of
// activations and weights (float or bfloat16).  The residual stream is 32-bit in both.
//
// Reference formulas: RMSNorm y = x / sqrt(mean(x^2) + eps) * w
// (crates/sglang-kernel/src/cpu.rs:26-34), SiLU*mul g / (1 + exp(-g)) * u (cpu.rs:119-123),
// embedding row copy with out-of-range ids flagged (cuda_bf16_kernels.rs:14-37).
#include "common.cuh"
#include "activations.cuh"

SRB_DEFINE_LAST_ERROR()
SRB_DEFINE_PDL_SWITCH()

// residual[row, :] = float(table[ids[row], :]) * scale; a bad id writes zeros and flags.
template <typename T>
__global__ void embedding_kernel(const int* __restrict__ ids, const T* __restrict__ table,
                                 float* __restrict__ residual, int width, int vocab, int* error_word, float scale) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int row = blockIdx.x;
  const int id = ids[row];
  const bool bad = id < 0 || id >= vocab;
  if (bad && threadIdx.x == 0) atomicOr(error_word, SRB_FLAG_BAD_TOKEN);
  const T* src = table + (size_t)(bad ? 0 : id) * width;
  float* dst = residual + (size_t)row * width;
  if (sizeof(T) == 2 && width % 8 == 0 && (((uintptr_t)table | (uintptr_t)residual) & 15) == 0) {
    for (int i = threadIdx.x * 8; i < width; i += blockDim.x * 8) {
      const uint4 raw = *reinterpret_cast<const uint4*>(src + i);
      const __nv_bfloat162* pair = reinterpret_cast<const __nv_bfloat162*>(&raw);
      float4 lo, hi;
      const float2 a = __bfloat1622float2(pair[0]), b = __bfloat1622float2(pair[1]);
      const float2 c = __bfloat1622float2(pair[2]), d = __bfloat1622float2(pair[3]);
      lo = bad ? make_float4(0.f, 0.f, 0.f, 0.f) : make_float4(a.x * scale, a.y * scale, b.x * scale, b.y * scale);
      hi = bad ? make_float4(0.f, 0.f, 0.f, 0.f) : make_float4(c.x * scale, c.y * scale, d.x * scale, d.y * scale);
      *reinterpret_cast<float4*>(dst + i) = lo;
      *reinterpret_cast<float4*>(dst + i + 4) = hi;
    }
    return;
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = bad ? 0.f : srb_to_float(src[i]) * scale;
}

// x = residual[src] (+ delta[src]); optionally residual[src] = x; out[row] = T(x * rsqrt * w).
// `row_index` (optional) picks the source rows, so the final norm touches only the rows
// whose logits are wanted.  The row is staged in shared memory between the two passes.
// The pending sum may also arrive as `num_parts` float partial sums (a matrix product cut
// along K), `part_stride` elements apart; they are added in part order.
template <typename T>
__global__ void add_rmsnorm_kernel(float* __restrict__ residual, const T* __restrict__ delta,
                                   const float* __restrict__ delta_parts, int num_parts, size_t part_stride,
                                   const float* __restrict__ weight, T* __restrict__ out,
                                   const int* __restrict__ row_index, int width, float eps,
                                   int write_residual) {
  extern __shared__ float staged[];          // width floats, then 33 floats of scratch
  float* scratch = staged + width;
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int row = blockIdx.x;
  const size_t src = (size_t)(row_index ? row_index[row] : row) * width;
  float partial = 0.f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float x = residual[src + i];
    if (delta) x += srb_to_float(delta[src + i]);
    for (int part = 0; part < num_parts; ++part) x += delta_parts[part * part_stride + src + i];
    if (write_residual) residual[src + i] = x;
    staged[i] = x;
    partial += x * x;
  }
  const float total = srb_block_sum(partial, scratch);
  const float inv = 1.0f / sqrtf(total / (float)width + eps);
  T* dst = out + (size_t)row * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x)
    dst[i] = srb_from_float<T>(staged[i] * inv * weight[i]);
}


// four consecutive values in one access (the address is a multiple of 4 elements)
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  uint2 raw;
  *reinterpret_cast<__nv_bfloat162*>(&raw.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&raw.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = raw;
}

// The same for widths that are a multiple of 4 and fit 4 * ITER values per thread: the row
// stays in registers, every load of a thread is issued before the first use (the row is
// small and the kernel is bound by latency, not by bandwidth), and the additions keep the
// order residual, delta, part 0, part 1, ...
template <typename T, int ITER>
__global__ void __launch_bounds__(1024)
add_rmsnorm_vec_kernel(float* __restrict__ residual, const T* __restrict__ delta,
                       const float* __restrict__ delta_parts, int num_parts, size_t part_stride,
                       const float* __restrict__ weight, T* __restrict__ out, const int* __restrict__ row_index,
                       int width, float eps, int write_residual) {
  // the partial sums of a thread's four columns are asked for eight at a time, so that a row of a decode step
  // costs one or two trips to L2, not one per few parts (measured at Qwen3-8B sizes: 3 % at batch 1, 7 % at 16)
  constexpr int PART_BATCH = ITER == 1 ? 8 : 4;
  __shared__ float scratch[33];
  srb_mark(SRB_MARK_NORM, 0);
  srb_launch_dependents();
  srb_grid_dependency_wait();
  srb_mark(SRB_MARK_NORM, 1);
  // the norm's weight travels with the row's loads, not after the sum of squares
  float4 w[ITER];
#pragma unroll
  for (int it = 0; it < ITER; ++it) {
    const int i = (it * blockDim.x + threadIdx.x) * 4;
    w[it] = i < width ? *reinterpret_cast<const float4*>(weight + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int row = blockIdx.x;
  const size_t src = (size_t)(row_index ? row_index[row] : row) * width;
  float4 x[ITER];
  float partial = 0.f;
#pragma unroll
  for (int it = 0; it < ITER; ++it) {
    const int i = (it * blockDim.x + threadIdx.x) * 4;
    x[it] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < width) {
      x[it] = *reinterpret_cast<const float4*>(residual + src + i);
      float4 whole = make_float4(0.f, 0.f, 0.f, 0.f);
      if (delta) whole = load4(delta + src + i);
      for (int first = 0; first < num_parts || first == 0; first += PART_BATCH) {
        float4 d[PART_BATCH];
#pragma unroll
        for (int j = 0; j < PART_BATCH; ++j)
          if (first + j < num_parts) d[j] = *reinterpret_cast<const float4*>(delta_parts + (first + j) * part_stride + src + i);
        if (first == 0 && delta) {
          x[it].x += whole.x; x[it].y += whole.y; x[it].z += whole.z; x[it].w += whole.w;
        }
#pragma unroll
        for (int j = 0; j < PART_BATCH; ++j) {
          if (first + j < num_parts) {
            x[it].x += d[j].x; x[it].y += d[j].y; x[it].z += d[j].z; x[it].w += d[j].w;
          }
        }
      }
      if (write_residual) *reinterpret_cast<float4*>(residual + src + i) = x[it];
      partial += x[it].x * x[it].x + x[it].y * x[it].y + x[it].z * x[it].z + x[it].w * x[it].w;
    }
  }
  const float total = srb_block_sum(partial, scratch);
  const float inv = 1.0f / sqrtf(total / (float)width + eps);
  T* dst = out + (size_t)row * width;
#pragma unroll
  for (int it = 0; it < ITER; ++it) {
    const int i = (it * blockDim.x + threadIdx.x) * 4;
    if (i < width)
      store4(dst + i, make_float4(x[it].x * inv * w[it].x, x[it].y * inv * w[it].y, x[it].z * inv * w[it].z, x[it].w * inv * w[it].w));
  }
  srb_mark(SRB_MARK_NORM, 2);
}

// out[row, j] = act(gate_up[row, j]) * gate_up[row, inner + j], act being SRB_ACT_* `activation`
template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int rows, int inner, int activation,
                                float act_param) {
  const size_t total = (size_t)rows * inner;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (size_t)gridDim.x * blockDim.x) {
    const size_t row = idx / inner, col = idx % inner;
    const float g = srb_to_float(gate_up[row * 2 * inner + col]);
    const float u = srb_to_float(gate_up[row * 2 * inner + inner + col]);
    out[idx] = srb_from_float<T>(srb_gated<true>(activation, g, u, act_param));
  }
}

// The same with eight bfloat16 values (16 bytes) per thread and access; `inner` a multiple of 8.
__global__ void silu_mul_bf16x8_kernel(const __nv_bfloat16* __restrict__ gate_up, __nv_bfloat16* __restrict__ out,
                                       int rows, int inner, int activation, float act_param) {
  const int per_row = inner / 8;
  const size_t total = (size_t)rows * per_row;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (size_t)gridDim.x * blockDim.x) {
    const size_t row = idx / per_row, col = (idx % per_row) * 8;
    const uint4 g4 = *reinterpret_cast<const uint4*>(gate_up + row * 2 * inner + col);
    const uint4 u4 = *reinterpret_cast<const uint4*>(gate_up + row * 2 * inner + inner + col);
    const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&g4);
    const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&u4);
    uint4 o4;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o4);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 g = __bfloat1622float2(g2[j]), u = __bfloat1622float2(u2[j]);
      // the result is rounded to bfloat16 (8 bits): the hardware's exponential and division are exact enough
      o2[j] = __floats2bfloat162_rn(srb_gated<false>(activation, g.x, u.x, act_param), srb_gated<false>(activation, g.y, u.y, act_param));
    }
    *reinterpret_cast<uint4*>(out + row * inner + col) = o4;
  }
}

template <typename T>
__global__ void add_bias_kernel(T* __restrict__ values, const float* __restrict__ bias, int rows, int width) {
  const size_t total = (size_t)rows * width;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total;
       idx += (size_t)gridDim.x * blockDim.x)
    values[idx] = srb_from_float<T>(srb_to_float(values[idx]) + bias[idx % width]);
}

static int elementwise_grid(size_t total, int block) {
  size_t blocks = (total + block - 1) / block;
  const size_t cap = (size_t)srb_sm_count() * 16;
  return (int)(blocks < 1 ? 1 : (blocks > cap ? cap : blocks));
}

// `scale` multiplies every value of the row in 32-bit (1 leaves the table's values as they are).
extern "C" int srb_embedding_scaled(const int* ids, const void* table, float* residual, int rows, int width,
                                    int vocab, int* error_word, int dtype, float scale, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (width <= 0 || vocab <= 0) SRB_FAIL("embedding: width %d and vocabulary %d must be positive", width, vocab);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == SRB_DTYPE_F32)
    SRB_CUDA_CALL(srb_launch(embedding_kernel<float>, dim3(rows), dim3(256), 0, s, ids, (const float*)table, residual,
                             width, vocab, error_word, scale));
  else if (dtype == SRB_DTYPE_BF16)
    SRB_CUDA_CALL(srb_launch(embedding_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, s, ids,
                             (const __nv_bfloat16*)table, residual, width, vocab, error_word, scale));
  else
    SRB_FAIL("embedding: unknown dtype %d", dtype);
  SRB_LAUNCH_CHECK("embedding");
  return SRB_OK;
}

extern "C" int srb_embedding(const int* ids, const void* table, float* residual, int rows, int width,
                             int vocab, int* error_word, int dtype, void* stream) {
  return srb_embedding_scaled(ids, table, residual, rows, width, vocab, error_word, dtype, 1.0f, stream);
}

template <typename T>
static int launch_add_rmsnorm(float* residual, const void* delta, const float* delta_parts, int num_parts,
                              size_t part_stride, const float* weight, void* out, const int* row_index, int rows,
                              int width, float eps, int write_residual, cudaStream_t s) {
  // widths that are a multiple of 4 (so float4 accesses stay aligned) and fit the registers
  const bool aligned = width % 4 == 0 && (((uintptr_t)residual | (uintptr_t)delta_parts | (uintptr_t)weight) & 15) == 0 &&
                       (((uintptr_t)delta | (uintptr_t)out) & (4 * sizeof(T) - 1)) == 0 && part_stride % 4 == 0;
  if (aligned && width <= 4 * 1024 * 2) {
    int threads = ((width / 4 + 31) / 32) * 32;
    if (threads > 1024) threads = 1024;
    if (width <= 4 * threads)
      SRB_CUDA_CALL(srb_launch(add_rmsnorm_vec_kernel<T, 1>, dim3(rows), dim3(threads), 0, s, residual, (const T*)delta,
                               delta_parts, num_parts, part_stride, weight, (T*)out, row_index, width, eps,
                               write_residual));
    else
      SRB_CUDA_CALL(srb_launch(add_rmsnorm_vec_kernel<T, 2>, dim3(rows), dim3(threads), 0, s, residual, (const T*)delta,
                               delta_parts, num_parts, part_stride, weight, (T*)out, row_index, width, eps,
                               write_residual));
    SRB_LAUNCH_CHECK("add_rmsnorm");
    return SRB_OK;
  }
  const size_t smem = (size_t)(width + 33) * sizeof(float);
  if (smem > 227 * 1024) SRB_FAIL("add_rmsnorm: width %d needs %zu bytes of shared memory (limit 232448)", width, smem);
  if (smem > 48 * 1024)
    SRB_CUDA_CALL(cudaFuncSetAttribute(add_rmsnorm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const int block = width >= 2048 ? 512 : (width >= 512 ? 256 : 128);
  SRB_CUDA_CALL(srb_launch(add_rmsnorm_kernel<T>, dim3(rows), dim3(block), smem, s, residual, (const T*)delta,
                           delta_parts, num_parts, part_stride, weight, (T*)out, row_index, width, eps,
                           write_residual));
  SRB_LAUNCH_CHECK("add_rmsnorm");
  return SRB_OK;
}

// delta: [rows_of_residual, width] of the output's type, or null; delta_parts: `num_parts` float
// tensors of that shape, `part_stride` elements apart, or null.
extern "C" int srb_add_rmsnorm(float* residual, const void* delta, const float* delta_parts, int num_parts,
                               long long part_stride, const float* weight, void* out, const int* row_index,
                               int rows, int width, float eps, int write_residual, int dtype, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (width <= 0) SRB_FAIL("add_rmsnorm: width %d must be positive", width);
  if (!(eps >= 0.f)) SRB_FAIL("add_rmsnorm: eps must be finite and non-negative");
  if (num_parts < 0 || (num_parts > 0 && !delta_parts)) SRB_FAIL("add_rmsnorm: partial sums are missing");
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == SRB_DTYPE_F32)
    return launch_add_rmsnorm<float>(residual, delta, delta_parts, num_parts, (size_t)part_stride, weight, out,
                                     row_index, rows, width, eps, write_residual, s);
  if (dtype == SRB_DTYPE_BF16)
    return launch_add_rmsnorm<__nv_bfloat16>(residual, delta, delta_parts, num_parts, (size_t)part_stride, weight,
                                             out, row_index, rows, width, eps, write_residual, s);
  SRB_FAIL("add_rmsnorm: unknown dtype %d", dtype);
}

// ---- a norm of the pending term, the residual sum, and the norm that follows, in one kernel ----------
// x = residual[src] + inner(delta[src]); residual[src] = x if asked; out[row] = outer(x), rounded to T.
// inner and outer are each one of
//   SRB_NORM_NONE   v                                          (no weights)
//   SRB_NORM_RMS    v / sqrt(mean(v^2) + eps) * w
//   SRB_NORM_LAYER  (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps) * w + b
// with eps inside the root; every mean, the sum and the scaling are 32-bit.  The pending term arrives
// in T (`delta`) or in float (`delta_f32`); with neither, x is the residual.  `extra` (optional, float,
// [rows of residual, width]) is written, rounded, behind the row in `out` (columns width .. 2 width - 1):
// the input of a product that reads the stream beside another one.  `out_pitch`: elements between rows of out.
#define SRB_NORM_NONE 0
#define SRB_NORM_RMS 1
#define SRB_NORM_LAYER 2

struct NormSpec {
  int kind;
  const float* weight;
  const float* bias;
  float eps;
  int groups;      // SRB_NORM_RMS only: the row is cut into this many equal consecutive parts, each divided by its own root mean square
  float scale;     // multiplies the normalised values (1: as they are)
};

// normalises `v` (width floats in shared memory) in place; every thread of the block calls it
__device__ __forceinline__ void norm_in_place(float* v, int width, const NormSpec& n, float* scratch) {
  if (n.kind == SRB_NORM_NONE) return;
  if (n.kind == SRB_NORM_RMS && n.groups > 1) {
    const int part = width / n.groups;
    for (int g = 0; g < n.groups; ++g) {
      float* u = v + g * part;
      const float* w = n.weight + g * part;
      float partial = 0.f;
      for (int i = threadIdx.x; i < part; i += blockDim.x) partial += u[i] * u[i];
      const float inv = 1.0f / sqrtf(srb_block_sum(partial, scratch) / (float)part + n.eps);
      for (int i = threadIdx.x; i < part; i += blockDim.x) u[i] = u[i] * inv * w[i] * n.scale;
    }
    __syncthreads();
    return;
  }
  float mean = 0.f;
  if (n.kind == SRB_NORM_LAYER) {
    float partial = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) partial += v[i];
    mean = srb_block_sum(partial, scratch) / (float)width;
  }
  float partial = 0.f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float c = v[i] - mean;
    partial += c * c;
  }
  const float inv = 1.0f / sqrtf(srb_block_sum(partial, scratch) / (float)width + n.eps);
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float y = (v[i] - mean) * inv * n.weight[i];
    if (n.kind == SRB_NORM_LAYER && n.bias) y += n.bias[i];
    v[i] = y * n.scale;
  }
  __syncthreads();
}

template <typename T>
__global__ void norm_add_norm_kernel(float* __restrict__ residual, const T* __restrict__ delta,
                                     const float* __restrict__ delta_f32, NormSpec inner, NormSpec outer,
                                     T* __restrict__ out, size_t out_pitch, const float* __restrict__ extra,
                                     const int* __restrict__ row_index, int width, int write_residual,
                                     const float* __restrict__ addend, size_t addend_pitch, int num_parts, size_t part_stride) {
  extern __shared__ float staged[];          // width floats, then 33 floats of scratch
  float* scratch = staged + width;
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int row = blockIdx.x;
  const size_t src_row = row_index ? row_index[row] : row, src = src_row * width;
  const bool pending = delta || delta_f32;
  if (pending) {
    if (num_parts > 0) {
      // partial sums of a product cut along K, added in part order
      for (int i = threadIdx.x; i < width; i += blockDim.x) {
        float sum = 0.f;
        for (int first = 0; first < num_parts; first += 4) {       // four loads in flight
          float d[4];
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (first + j < num_parts) d[j] = delta_f32[(first + j) * part_stride + src + i];
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (first + j < num_parts) sum += d[j];
        }
        staged[i] = sum;
      }
    } else {
      for (int i = threadIdx.x; i < width; i += blockDim.x)
        staged[i] = delta ? srb_to_float(delta[src + i]) : delta_f32[src + i];
    }
    __syncthreads();
    norm_in_place(staged, width, inner, scratch);
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float x = residual[src + i];
    if (pending) x += staged[i];
    if (addend) x += addend[src_row * addend_pitch + i];
    if (write_residual && (pending || addend)) residual[src + i] = x;
    staged[i] = x;
  }
  if (!out) return;
  __syncthreads();
  norm_in_place(staged, width, outer, scratch);
  T* dst = out + (size_t)row * out_pitch;
  for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = srb_from_float<T>(staged[i]);
  if (extra)
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[width + i] = srb_from_float<T>(extra[src + i]);
}

// The same for RMS norms over the whole row (or none), with the row in registers: four consecutive entries per thread and item,
// ITEMS of them, all loads of a thread in flight together.  Widths that are multiples of four, rows on 16-byte borders (of
// floats), no `extra`.
template <typename T, int ITEMS, bool PARTS>
__global__ void __launch_bounds__(ITEMS == 1 ? 1024 : 256, ITEMS == 1 ? 1 : (ITEMS == 2 ? 4 : 1))
norm_add_norm_vec_kernel(float* __restrict__ residual, const T* __restrict__ delta, const float* __restrict__ delta_f32,
                         NormSpec inner, NormSpec outer, T* __restrict__ out, size_t out_pitch, const int* __restrict__ row_index,
                         int width, int write_residual, const float* __restrict__ addend, size_t addend_pitch, int num_parts,
                         size_t part_stride) {
  __shared__ float scratch[33];
  srb_launch_dependents();
  const int step = blockDim.x * 4;
  float4 wi[ITEMS], wo[ITEMS];
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {                     // the weights are constants: ahead of the wait
    const int i = threadIdx.x * 4 + it * step;
    wi[it] = wo[it] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < width && inner.kind != SRB_NORM_NONE) wi[it] = *reinterpret_cast<const float4*>(inner.weight + i);
    if (i < width && out && outer.kind != SRB_NORM_NONE) wo[it] = *reinterpret_cast<const float4*>(outer.weight + i);
  }
  srb_grid_dependency_wait();
  const size_t src_row = row_index ? row_index[blockIdx.x] : blockIdx.x, src = src_row * width;
  const bool pending = delta || delta_f32;
  float4 x[ITEMS], d[ITEMS];
  float squares = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int i = threadIdx.x * 4 + it * step;
    x[it] = d[it] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < width) {
      x[it] = *reinterpret_cast<const float4*>(residual + src + i);
      if (delta) d[it] = load4(delta + src + i);
      else if (!PARTS && delta_f32) d[it] = load4(delta_f32 + src + i);
    }
  }
  if (PARTS) {
    // partial sums of a product cut along K, added in part order, the loads of several parts in flight
    constexpr int AHEAD = ITEMS == 1 ? 8 : 4;
    for (int first = 0; first < num_parts; first += AHEAD) {
#pragma unroll
      for (int it = 0; it < ITEMS; ++it) {
        const int i = threadIdx.x * 4 + it * step;
        if (i >= width) break;
        float4 p[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
          if (first + j < num_parts) p[j] = load4(delta_f32 + (first + j) * part_stride + src + i);
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
          if (first + j < num_parts) { d[it].x += p[j].x; d[it].y += p[j].y; d[it].z += p[j].z; d[it].w += p[j].w; }
      }
    }
  }
  if (pending) {
    float factor = 1.f;
    if (inner.kind != SRB_NORM_NONE) {
#pragma unroll
      for (int it = 0; it < ITEMS; ++it) squares += d[it].x * d[it].x + d[it].y * d[it].y + d[it].z * d[it].z + d[it].w * d[it].w;
      factor = 1.0f / sqrtf(srb_block_sum(squares, scratch) / (float)width + inner.eps);
    }
#pragma unroll
    for (int it = 0; it < ITEMS; ++it) {
      if (inner.kind != SRB_NORM_NONE) {
        d[it].x = d[it].x * factor * wi[it].x * inner.scale; d[it].y = d[it].y * factor * wi[it].y * inner.scale;
        d[it].z = d[it].z * factor * wi[it].z * inner.scale; d[it].w = d[it].w * factor * wi[it].w * inner.scale;
      }
      x[it].x += d[it].x; x[it].y += d[it].y; x[it].z += d[it].z; x[it].w += d[it].w;
    }
  }
  squares = 0.f;
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int i = threadIdx.x * 4 + it * step;
    if (i >= width) break;
    if (addend) {
      const float4 a = load4(addend + src_row * addend_pitch + i);
      x[it].x += a.x; x[it].y += a.y; x[it].z += a.z; x[it].w += a.w;
    }
    if (write_residual && (pending || addend)) *reinterpret_cast<float4*>(residual + src + i) = x[it];
    squares += x[it].x * x[it].x + x[it].y * x[it].y + x[it].z * x[it].z + x[it].w * x[it].w;
  }
  if (!out) return;
  float factor = 1.f;
  if (outer.kind != SRB_NORM_NONE) factor = 1.0f / sqrtf(srb_block_sum(squares, scratch) / (float)width + outer.eps);
#pragma unroll
  for (int it = 0; it < ITEMS; ++it) {
    const int i = threadIdx.x * 4 + it * step;
    if (i >= width) break;
    if (outer.kind != SRB_NORM_NONE) {
      x[it].x = x[it].x * factor * wo[it].x * outer.scale; x[it].y = x[it].y * factor * wo[it].y * outer.scale;
      x[it].z = x[it].z * factor * wo[it].z * outer.scale; x[it].w = x[it].w * factor * wo[it].w * outer.scale;
    }
    store4(out + (size_t)blockIdx.x * out_pitch + i, x[it]);
  }
}

template <typename T>
static int launch_norm_add_norm_vec(float* residual, const void* delta, const float* delta_f32, const NormSpec& inner, const NormSpec& outer,
                                    void* out, long long out_pitch, const int* row_index, int rows, int width, int write_residual,
                                    const float* addend, long long addend_pitch, int num_parts, long long part_stride, cudaStream_t s) {
  const int quads = width / 4;
  // few rows: as many threads as the row has pieces; many: two pieces a thread
  const int items = quads <= 1024 && rows <= 64 ? 1 : (quads <= 512 ? 2 : (quads <= 1024 ? 4 : 8));
  const int threads = ((quads + items - 1) / items + 31) / 32 * 32;
#define SRB_NORM_VEC(ITEMS)                                                                                                    \
  SRB_CUDA_CALL(srb_launch(num_parts > 0 ? norm_add_norm_vec_kernel<T, ITEMS, true> : norm_add_norm_vec_kernel<T, ITEMS, false>, dim3(rows), dim3(threads), 0, s, residual, (const T*)delta,    \
                           delta_f32, inner, outer, (T*)out, (size_t)out_pitch, row_index, width, write_residual, addend,     \
                           (size_t)addend_pitch, num_parts, (size_t)part_stride))
  if (items == 1) SRB_NORM_VEC(1);
  else if (items == 2) SRB_NORM_VEC(2);
  else if (items == 4) SRB_NORM_VEC(4);
  else SRB_NORM_VEC(8);
#undef SRB_NORM_VEC
  SRB_LAUNCH_CHECK("norm_add_norm");
  return SRB_OK;
}

// `*_groups` (RMS norms only; 1: the whole row) and `*_scale` (1: none) as NormSpec says.  `addend` (optional, float,
// rows `addend_pitch` floats apart; 0: one row for all): a second term of the sum, added after the pending one: x = residual +
// inner(delta) + addend.
// `num_parts` > 0: `delta_f32` holds that many partial sums of the pending term, `part_stride` floats apart, which are
// added in part order before the inner norm.
extern "C" int srb_norm_add_norm_parts(float* residual, const void* delta, const float* delta_f32, int inner_kind,
                                    const float* inner_weight, const float* inner_bias, float inner_eps, int inner_groups,
                                    float inner_scale, int outer_kind, const float* outer_weight, const float* outer_bias,
                                    float outer_eps, int outer_groups, float outer_scale, void* out, long long out_pitch,
                                    const float* extra, const int* row_index, int rows, int width, int write_residual,
                                    int dtype, const float* addend, long long addend_pitch, int num_parts, long long part_stride,
                                    void* stream) {
  if (rows <= 0) return SRB_OK;
  if (num_parts < 0 || (num_parts > 0 && (!delta_f32 || delta))) SRB_FAIL("norm_add_norm: partial sums come as float and alone");
  for (int groups : {inner_groups, outer_groups})
    if (groups < 1 || width % groups) SRB_FAIL("norm_add_norm: a row of %d entries does not split into %d equal parts", width, groups);
  if ((inner_groups > 1 && inner_kind != SRB_NORM_RMS) || (outer_groups > 1 && outer_kind != SRB_NORM_RMS))
    SRB_FAIL("norm_add_norm: only an RMS norm is taken in parts");
  if (width <= 0) SRB_FAIL("norm_add_norm: width %d must be positive", width);
  for (int kind : {inner_kind, outer_kind})
    if (kind < SRB_NORM_NONE || kind > SRB_NORM_LAYER) SRB_FAIL("norm_add_norm: unknown kind of norm %d", kind);
  if ((inner_kind != SRB_NORM_NONE && !inner_weight) || (out && outer_kind != SRB_NORM_NONE && !outer_weight))
    SRB_FAIL("norm_add_norm: a norm without its weight");
  if (!(inner_eps >= 0.f) || !(outer_eps >= 0.f)) SRB_FAIL("norm_add_norm: eps must be finite and non-negative");
  if (out && out_pitch < (long long)width * (extra ? 2 : 1)) SRB_FAIL("norm_add_norm: rows of the output overlap");
  const size_t smem = (size_t)(width + 33) * sizeof(float);
  if (smem > 227 * 1024) SRB_FAIL("norm_add_norm: width %d needs %zu bytes of shared memory (limit 232448)", width, smem);
  const NormSpec inner{inner_kind, inner_weight, inner_bias, inner_eps, inner_groups, inner_scale};
  const NormSpec outer{outer_kind, outer_weight, outer_bias, outer_eps, outer_groups, outer_scale};
  const int block = width >= 2048 ? 512 : (width >= 512 ? 256 : 128);
  cudaStream_t s = (cudaStream_t)stream;
  const size_t element = dtype == SRB_DTYPE_BF16 ? 2 : 4;
  const bool plain = inner_kind != SRB_NORM_LAYER && outer_kind != SRB_NORM_LAYER && inner_groups == 1 && outer_groups == 1 && !extra &&
                     width % 4 == 0 && width <= 8192 && out_pitch % 4 == 0 && part_stride % 4 == 0 && addend_pitch % 4 == 0 &&
                     (((uintptr_t)residual | (uintptr_t)delta_f32 | (uintptr_t)addend | (uintptr_t)inner_weight | (uintptr_t)outer_weight) & 15) == 0 &&
                     (((uintptr_t)delta | (uintptr_t)out) & (4 * element - 1)) == 0;
  if (plain && dtype == SRB_DTYPE_F32)
    return launch_norm_add_norm_vec<float>(residual, delta, delta_f32, inner, outer, out, out_pitch, row_index, rows, width, write_residual,
                                           addend, addend_pitch, num_parts, part_stride, s);
  if (plain && dtype == SRB_DTYPE_BF16)
    return launch_norm_add_norm_vec<__nv_bfloat16>(residual, delta, delta_f32, inner, outer, out, out_pitch, row_index, rows, width,
                                                   write_residual, addend, addend_pitch, num_parts, part_stride, s);
  if (dtype == SRB_DTYPE_F32) {
    if (smem > 48 * 1024)
      SRB_CUDA_CALL(cudaFuncSetAttribute(norm_add_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    SRB_CUDA_CALL(srb_launch(norm_add_norm_kernel<float>, dim3(rows), dim3(block), smem, s, residual, (const float*)delta,
                             delta_f32, inner, outer, (float*)out, (size_t)out_pitch, extra, row_index, width,
                             write_residual, addend, (size_t)addend_pitch, num_parts, (size_t)part_stride));
  } else if (dtype == SRB_DTYPE_BF16) {
    if (smem > 48 * 1024)
      SRB_CUDA_CALL(cudaFuncSetAttribute(norm_add_norm_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem));
    SRB_CUDA_CALL(srb_launch(norm_add_norm_kernel<__nv_bfloat16>, dim3(rows), dim3(block), smem, s, residual,
                             (const __nv_bfloat16*)delta, delta_f32, inner, outer, (__nv_bfloat16*)out, (size_t)out_pitch,
                             extra, row_index, width, write_residual, addend, (size_t)addend_pitch, num_parts, (size_t)part_stride));
  } else {
    SRB_FAIL("norm_add_norm: unknown dtype %d", dtype);
  }
  SRB_LAUNCH_CHECK("norm_add_norm");
  return SRB_OK;
}

extern "C" int srb_norm_add_norm_ex(float* residual, const void* delta, const float* delta_f32, int inner_kind,
                                    const float* inner_weight, const float* inner_bias, float inner_eps, int inner_groups,
                                    float inner_scale, int outer_kind, const float* outer_weight, const float* outer_bias,
                                    float outer_eps, int outer_groups, float outer_scale, void* out, long long out_pitch,
                                    const float* extra, const int* row_index, int rows, int width, int write_residual,
                                    int dtype, void* stream) {
  return srb_norm_add_norm_parts(residual, delta, delta_f32, inner_kind, inner_weight, inner_bias, inner_eps, inner_groups,
                                 inner_scale, outer_kind, outer_weight, outer_bias, outer_eps, outer_groups, outer_scale, out,
                                 out_pitch, extra, row_index, rows, width, write_residual, dtype, nullptr, 0, 0, 0, stream);
}

extern "C" int srb_norm_add_norm(float* residual, const void* delta, const float* delta_f32, int inner_kind,
                                 const float* inner_weight, const float* inner_bias, float inner_eps, int outer_kind,
                                 const float* outer_weight, const float* outer_bias, float outer_eps, void* out,
                                 long long out_pitch, const float* extra, const int* row_index, int rows, int width,
                                 int write_residual, int dtype, void* stream) {
  return srb_norm_add_norm_ex(residual, delta, delta_f32, inner_kind, inner_weight, inner_bias, inner_eps, 1, 1.0f, outer_kind,
                              outer_weight, outer_bias, outer_eps, 1, 1.0f, out, out_pitch, extra, row_index, rows, width,
                              write_residual, dtype, stream);
}

// ---- two sublayers that read one norm: the residual sum of both, scaled ------------------------------
// residual += mult * (a + b), in 32-bit.  a: T [rows, width] (`a`), float (`a_f32`, `a_parts` tensors `a_part_stride`
// floats apart, added in order: partial sums of a product cut along K), or neither; b: float [rows, width] or null.
// `rounded` (optional, T [rows, width]) receives the new residual rounded: the input of a product that reads the stream.
template <typename T>
__global__ void scaled_sum_kernel(float* __restrict__ residual, const T* __restrict__ a, const float* __restrict__ a_f32,
                                  int a_parts, size_t a_part_stride, const float* __restrict__ b, float mult,
                                  T* __restrict__ rounded, size_t total) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
    float y = 0.f;
    if (a) y = srb_to_float(a[idx]);
    for (int part = 0; part < a_parts; ++part) y += a_f32[part * a_part_stride + idx];
    if (b) y += b[idx];
    const float x = fmaf(mult, y, residual[idx]);
    residual[idx] = x;
    if (rounded) rounded[idx] = srb_from_float<T>(x);
  }
}

extern "C" int srb_scaled_sum(float* residual, const void* a, const float* a_f32, int a_parts, long long a_part_stride,
                              const float* b, float mult, void* rounded, int rows, int width, int dtype, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (width <= 0) SRB_FAIL("scaled_sum: width %d must be positive", width);
  if (a_parts < 0 || (a_parts > 0 && !a_f32)) SRB_FAIL("scaled_sum: partial sums are missing");
  const size_t total = (size_t)rows * width;
  cudaStream_t s = (cudaStream_t)stream;
  const int grid = elementwise_grid(total, 256);
  if (dtype == SRB_DTYPE_F32)
    SRB_CUDA_CALL(srb_launch(scaled_sum_kernel<float>, dim3(grid), dim3(256), 0, s, residual, (const float*)a, a_f32, a_parts,
                             (size_t)a_part_stride, b, mult, (float*)rounded, total));
  else if (dtype == SRB_DTYPE_BF16)
    SRB_CUDA_CALL(srb_launch(scaled_sum_kernel<__nv_bfloat16>, dim3(grid), dim3(256), 0, s, residual, (const __nv_bfloat16*)a,
                             a_f32, a_parts, (size_t)a_part_stride, b, mult, (__nv_bfloat16*)rounded, total));
  else
    SRB_FAIL("scaled_sum: unknown dtype %d", dtype);
  SRB_LAUNCH_CHECK("scaled_sum");
  return SRB_OK;
}

// ---- a gate that a table's row, chosen by the token, multiplies --------------------------------------
// out[r, j] = act(gate[r, j]) * table[ids[r], offset + j], j < dim; table rows are `table_pitch` entries long.
template <typename T>
__global__ void token_gate_kernel(const T* __restrict__ gate, const int* __restrict__ ids, const T* __restrict__ table,
                                  size_t table_pitch, int offset, int vocab, int dim, int activation, T* __restrict__ out,
                                  int* __restrict__ error_word) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int row = blockIdx.x;
  const int id = ids[row];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) atomicOr(error_word, SRB_FLAG_BAD_TOKEN);
    for (int j = threadIdx.x; j < dim; j += blockDim.x) out[(size_t)row * dim + j] = srb_from_float<T>(0.f);
    return;
  }
  const T* e = table + (size_t)id * table_pitch + offset;
  for (int j = threadIdx.x; j < dim; j += blockDim.x)
    out[(size_t)row * dim + j] = srb_from_float<T>(srb_gated<true>(activation, srb_to_float(gate[(size_t)row * dim + j]), srb_to_float(e[j])));
}

extern "C" int srb_token_gate(const void* gate, const int* ids, const void* table, long long table_pitch, int offset, int vocab,
                              int rows, int dim, int activation, void* out, int* error_word, int dtype, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (dim <= 0 || offset < 0 || offset + dim > table_pitch || vocab <= 0) SRB_FAIL("token_gate: %d entries from %d do not fit rows of %lld", dim, offset, table_pitch);
  if (activation < 0 || activation >= SRB_ACT_COUNT || activation == SRB_ACT_SWIGLU_CLAMP) SRB_FAIL("token_gate: activation %d is not taken", activation);
  cudaStream_t s = (cudaStream_t)stream;
  const int block = dim >= 256 ? 256 : (dim >= 64 ? 64 : 32);
  if (dtype == SRB_DTYPE_F32)
    SRB_CUDA_CALL(srb_launch(token_gate_kernel<float>, dim3(rows), dim3(block), 0, s, (const float*)gate, ids, (const float*)table,
                             (size_t)table_pitch, offset, vocab, dim, activation, (float*)out, error_word));
  else if (dtype == SRB_DTYPE_BF16)
    SRB_CUDA_CALL(srb_launch(token_gate_kernel<__nv_bfloat16>, dim3(rows), dim3(block), 0, s, (const __nv_bfloat16*)gate, ids,
                             (const __nv_bfloat16*)table, (size_t)table_pitch, offset, vocab, dim, activation,
                             (__nv_bfloat16*)out, error_word));
  else
    SRB_FAIL("token_gate: unknown dtype %d", dtype);
  SRB_LAUNCH_CHECK("token_gate");
  return SRB_OK;
}

// values *= factor (32-bit, in place): a model's constant on its logits
__global__ void scale_values_kernel(float* __restrict__ values, float factor, size_t total) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x)
    values[idx] *= factor;
}

extern "C" int srb_scale_values(float* values, long long total, float factor, void* stream) {
  if (total <= 0) return SRB_OK;
  SRB_CUDA_CALL(srb_launch(scale_values_kernel, dim3(elementwise_grid((size_t)total, 256)), dim3(256), 0, (cudaStream_t)stream,
                           values, factor, (size_t)total));
  SRB_LAUNCH_CHECK("scale_values");
  return SRB_OK;
}

// `act_param`: the parameter of an activation that has one
extern "C" int srb_gated_mul_param(const void* gate_up, void* out, int rows, int inner, int activation, float act_param,
                                   int dtype, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (inner <= 0) SRB_FAIL("gated_mul: inner width %d must be positive", inner);
  if (activation < 0 || activation >= SRB_ACT_COUNT) SRB_FAIL("gated_mul: unknown activation %d", activation);
  cudaStream_t s = (cudaStream_t)stream;
  const int grid = elementwise_grid((size_t)rows * inner, 256);
  if (dtype == SRB_DTYPE_F32)
    silu_mul_kernel<float><<<grid, 256, 0, s>>>((const float*)gate_up, (float*)out, rows, inner, activation, act_param);
  else if (dtype == SRB_DTYPE_BF16 && inner % 8 == 0 && (((uintptr_t)gate_up | (uintptr_t)out) & 15) == 0) {
    size_t blocks = ((size_t)rows * (inner / 8) + 255) / 256;
    if (blocks > srb_sm_count() * 64) blocks = srb_sm_count() * 64;
    silu_mul_bf16x8_kernel<<<(int)blocks, 256, 0, s>>>((const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, rows, inner, activation, act_param);
  } else if (dtype == SRB_DTYPE_BF16)
    silu_mul_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>((const __nv_bfloat16*)gate_up, (__nv_bfloat16*)out, rows,
                                                        inner, activation, act_param);
  else
    SRB_FAIL("gated_mul: unknown dtype %d", dtype);
  SRB_LAUNCH_CHECK("gated_mul");
  return SRB_OK;
}

extern "C" int srb_gated_mul(const void* gate_up, void* out, int rows, int inner, int activation, int dtype,
                             void* stream) {
  if (activation == SRB_ACT_SWIGLU_CLAMP) SRB_FAIL("gated_mul: an activation with a parameter comes with its parameter");
  return srb_gated_mul_param(gate_up, out, rows, inner, activation, 0.f, dtype, stream);
}

extern "C" int srb_add_bias(void* values, const float* bias, int rows, int width, int dtype, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (width <= 0) SRB_FAIL("add_bias: width %d must be positive", width);
  cudaStream_t s = (cudaStream_t)stream;
  const int grid = elementwise_grid((size_t)rows * width, 256);
  if (dtype == SRB_DTYPE_F32)
    add_bias_kernel<float><<<grid, 256, 0, s>>>((float*)values, bias, rows, width);
  else if (dtype == SRB_DTYPE_BF16)
    add_bias_kernel<__nv_bfloat16><<<grid, 256, 0, s>>>((__nv_bfloat16*)values, bias, rows, width);
  else
    SRB_FAIL("add_bias: unknown dtype %d", dtype);
  SRB_LAUNCH_CHECK("add_bias");
  return SRB_OK;
}

// tokens[i] = source[index[i]] where index[i] >= 0: rows whose token was chosen on the device by
// the step before and has not been to the host yet.  An index outside the source flags a bad token.
__global__ void take_tokens_kernel(int* __restrict__ tokens, const int* __restrict__ source,
                                   const int* __restrict__ index, int rows, int source_rows, int* error_word) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= rows) return;
  const int from = index[i];
  if (from < 0) return;
  if (from >= source_rows) {
    atomicOr(error_word, SRB_FLAG_BAD_TOKEN);
    return;
  }
  tokens[i] = source[from];
}

extern "C" int srb_take_tokens(int* tokens, const int* source, const int* index, int rows, int source_rows,
                               int* error_word, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (source_rows <= 0) SRB_FAIL("take_tokens: the source has no rows");
  take_tokens_kernel<<<(rows + 127) / 128, 128, 0, (cudaStream_t)stream>>>(tokens, source, index, rows, source_rows,
                                                                          error_word);
  SRB_LAUNCH_CHECK("take_tokens");
  return SRB_OK;
}
