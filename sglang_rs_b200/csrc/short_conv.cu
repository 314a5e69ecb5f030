// A short causal convolution over time per channel, then SiLU, for mixers that keep state per request (the state-space
// mixer, the gated delta rule):
//
//   y[t, c] = silu(bias[c] + sum_j weight[c, j] u[t - (taps - 1) + j, c])      zeros before the sequence starts
//
// The inputs u are `channels` columns of a projection's rows (`proj` points at the first of them).  A request's slot of
// state begins, in 32-bit floats, with the convolution's last taps - 1 inputs [taps - 1][channels] (oldest first);
// whatever else the mixer keeps follows.  Kernels:
//
//   short_conv_kernel        every row of the step (32-bit result, or rounded to bfloat16 for kernels that feed tensor cores),
//                            reading earlier rows of the same request from the step and, before the step's first row,
//                            from the slot
//   short_conv_keep_kernel   the slot's inputs are replaced by the last taps - 1 of the sequence (a second launch: rows
//                            read the old ones)
//   short_conv_single_kernel both in one launch, for steps in which every request brings one row (decoded tokens): the
//                            thread that reads a channel's inputs is the one that replaces them
//
// The sum is 32-bit.  Rows at negative positions pad a captured step and give zeros.
#include "common.cuh"
#include <math.h>

SRB_DEFINE_LAST_ERROR()
SRB_DEFINE_PDL_SWITCH()

#define CONV_MAX_TAPS 16
#define CONV_ROWS 8              // rows of the step that one thread takes in steps of many rows

struct ConvShape {
  int channels, taps;
  long long proj_pitch;           // elements between rows of the projection
  long long slot_floats;          // floats of state per request
};

// SiLU of the convolution's sum as the result's type: a bfloat16 result keeps 8 bits of mantissa, so the quick exponential
// and quotient (about 22 bits) round to the same number but for ties
template <typename O> __device__ __forceinline__ O conv_result(float acc);
template <> __device__ __forceinline__ float conv_result<float>(float acc) { return acc / (1.0f + expf(-acc)); }
template <> __device__ __forceinline__ __nv_bfloat16 conv_result<__nv_bfloat16>(float acc) {
  return __float2bfloat16_rn(__fdividef(acc, 1.0f + __expf(-acc)));
}

// grid (channel blocks, ceil(rows / ROWS)), so that blocks that run together read neighbouring pieces of the same rows:
// a thread takes one channel of ROWS consecutive rows (CONV_ROWS in steps
// of many rows, so that the filter is read once and the rows' loads are in flight together; 1 in steps of few rows).
// TAPS: the filter's length, or 0 for any.
template <typename T, typename O, int TAPS, int ROWS>
__global__ void short_conv_kernel(const T* __restrict__ proj, const float* __restrict__ weight, const float* __restrict__ bias,
                                  const int* __restrict__ positions, const int* __restrict__ row_request,
                                  const int* __restrict__ cu_rows, const int* __restrict__ state_slots,
                                  const float* __restrict__ state, O* __restrict__ out, int rows, ConvShape s) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= s.channels) return;
  const int taps = TAPS > 0 ? TAPS : s.taps;
  constexpr int HELD = TAPS > 0 ? TAPS : 1;
  float w[HELD];
  if (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < HELD; ++j) w[j] = weight[(size_t)c * TAPS + j];
  }
  const float b = bias ? bias[c] : 0.f;
  const int row0 = blockIdx.y * ROWS;
  // what the rows need to know, all loads in flight together: position, rows of the request before it, the slot
  int pos[ROWS], ahead[ROWS], slot[ROWS];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const bool live = row0 + r < rows;
    pos[r] = live ? positions[row0 + r] : -1;
    ahead[r] = live ? row_request[row0 + r] : 0;
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int request = ahead[r];
    ahead[r] = row0 + r - cu_rows[request];
    slot[r] = state_slots[request];
  }
  if constexpr (TAPS > 0) {
    // the inputs of rows row0 - (TAPS - 1) .. row0 + ROWS - 1 of the step, whichever request they belong to
    float u[ROWS + HELD - 1];
#pragma unroll
    for (int k = 0; k < ROWS + HELD - 1; ++k) {
      const int row = row0 + k - (HELD - 1);
      u[k] = (row >= 0 && row < rows) ? srb_to_float(proj[(size_t)row * s.proj_pitch + c]) : 0.f;
    }
    // rows in the middle of a request's rows of the step: every input is one of the step's
    bool inside = row0 + ROWS <= rows;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) inside = inside && pos[r] >= HELD - 1 && ahead[r] >= HELD - 1;
    if (inside) {
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        float acc = b;
#pragma unroll
        for (int j = 0; j < HELD; ++j) acc = fmaf(w[j], u[r + j], acc);
        out[(size_t)(row0 + r) * s.channels + c] = conv_result<O>(acc);
      }
      return;
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      if (row0 + r >= rows) break;
      O* dst = out + (size_t)(row0 + r) * s.channels + c;
      if (pos[r] < 0) { *dst = srb_from_float<O>(0.f); continue; }
      const float* kept = state + (size_t)slot[r] * s.slot_floats;
      float acc = b;
#pragma unroll
      for (int j = 0; j < HELD; ++j) {
        const int back = HELD - 1 - j;
        if (pos[r] - back < 0) continue;                   // zeros before the start of the sequence
        const float v = back <= ahead[r] ? u[r + j] : kept[(size_t)(HELD - 1 - (back - ahead[r])) * s.channels + c];
        acc = fmaf(w[j], v, acc);
      }
      *dst = conv_result<O>(acc);
    }
  } else {
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int row = row0 + r;
    if (row >= rows) break;
    O* dst = out + (size_t)row * s.channels + c;
    if (pos[r] < 0) { *dst = srb_from_float<O>(0.f); continue; }
    const float* kept = state + (size_t)slot[r] * s.slot_floats;
    float acc = b;
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j;
      if (pos[r] - back < 0) continue;                     // zeros before the start of the sequence
      float v;
      if (back <= ahead[r])
        v = srb_to_float(proj[(size_t)(row - back) * s.proj_pitch + c]);
      else
        v = kept[(size_t)(taps - 1 - (back - ahead[r])) * s.channels + c];
      acc = fmaf(weight[(size_t)c * taps + j], v, acc);
    }
    *dst = conv_result<O>(acc);
  }
  }
}

// One thread per (request, channel): the slot's inputs become the last taps - 1 of the sequence after this step.
template <typename T>
__global__ void short_conv_keep_kernel(const T* __restrict__ proj, const int* __restrict__ positions,
                                       const int* __restrict__ cu_rows, const int* __restrict__ state_slots,
                                       float* __restrict__ state, ConvShape s) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int request = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= s.channels) return;
  const int first = cu_rows[request], count = cu_rows[request + 1] - first;
  if (count <= 0) return;
  const int start = positions[first];
  if (start < 0) return;
  float* kept = state + (size_t)state_slots[request] * s.slot_floats;
  const int keep = s.taps - 1;
  float fresh[CONV_MAX_TAPS];
#pragma unroll
  for (int k = 0; k < CONV_MAX_TAPS; ++k) {
    if (k >= keep) break;
    const int at = start + count - keep + k;           // position in the sequence of the k-th kept input
    float v = 0.f;
    if (at >= start) v = srb_to_float(proj[(size_t)(first + at - start) * s.proj_pitch + c]);
    else if (at >= 0) v = kept[(size_t)(at - start + keep) * s.channels + c];
    fresh[k] = v;
  }
#pragma unroll
  for (int k = 0; k < CONV_MAX_TAPS; ++k) {
    if (k >= keep) break;
    kept[(size_t)k * s.channels + c] = fresh[k];
  }
}

// One thread per (request, channel), every request with one row: the convolution of the row, then the slot's inputs move up
// by one.  TAPS: the filter's length, or 0 for any.
template <typename T, typename O, int TAPS>
__global__ void short_conv_single_kernel(const T* __restrict__ proj, const float* __restrict__ weight, const float* __restrict__ bias,
                                         const int* __restrict__ positions, const int* __restrict__ cu_rows,
                                         const int* __restrict__ state_slots, float* __restrict__ state, O* __restrict__ out,
                                         int write_state, ConvShape s) {
  srb_launch_dependents();
  const int request = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int taps = TAPS > 0 ? TAPS : s.taps;
  constexpr int HELD = TAPS > 0 ? TAPS : CONV_MAX_TAPS;
  float w[HELD];
  if (c < s.channels) {                                    // the filter is a constant: ahead of the wait
#pragma unroll
    for (int j = 0; j < HELD; ++j) w[j] = j < taps ? weight[(size_t)c * taps + j] : 0.f;
  }
  srb_grid_dependency_wait();
  if (c >= s.channels) return;
  const int row = cu_rows[request];
  if (cu_rows[request + 1] != row + 1) return;             // (the launcher is only used for steps of single rows)
  O* dst = out + (size_t)row * s.channels + c;
  const int pos = positions[row];
  if (pos < 0) { *dst = srb_from_float<O>(0.f); return; }
  float* kept = state + (size_t)state_slots[request] * s.slot_floats + c;
  float u[HELD];
#pragma unroll
  for (int j = 0; j < HELD; ++j) {
    u[j] = 0.f;
    if (j < taps - 1) { if (pos - (taps - 1 - j) >= 0) u[j] = kept[(size_t)j * s.channels]; }
    else if (j == taps - 1) u[j] = srb_to_float(proj[(size_t)row * s.proj_pitch + c]);
  }
  float acc = bias ? bias[c] : 0.f;
#pragma unroll
  for (int j = 0; j < HELD; ++j)
    if (j < taps) acc = fmaf(w[j], u[j], acc);
  *dst = conv_result<O>(acc);
  if (!write_state) return;
#pragma unroll
  for (int j = 0; j + 1 < HELD; ++j)
    if (j < taps - 1) kept[(size_t)j * s.channels] = u[j + 1];
}

// bfloat16 to bfloat16 in steps of many rows: a thread takes two neighbouring channels of CONV_ROWS rows, 4 bytes a load.
template <int TAPS>
__global__ void __launch_bounds__(128)
short_conv_pair_kernel(const __nv_bfloat16* __restrict__ proj, const float* __restrict__ weight, const float* __restrict__ bias,
                       const int* __restrict__ positions, const int* __restrict__ row_request, const int* __restrict__ cu_rows,
                       const int* __restrict__ state_slots, const float* __restrict__ state, __nv_bfloat16* __restrict__ out, int rows,
                       ConvShape s) {
  constexpr int ROWS = CONV_ROWS;
  srb_launch_dependents();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 2;
  float w0[TAPS], w1[TAPS], b0 = 0.f, b1 = 0.f;
  if (c < s.channels) {                                    // constants: ahead of the wait
#pragma unroll
    for (int j = 0; j < TAPS; ++j) { w0[j] = weight[(size_t)c * TAPS + j]; w1[j] = weight[(size_t)(c + 1) * TAPS + j]; }
    if (bias) { b0 = bias[c]; b1 = bias[c + 1]; }
  }
  srb_grid_dependency_wait();
  if (c >= s.channels) return;
  const int row0 = blockIdx.y * ROWS;
  __nv_bfloat162 u[ROWS + TAPS - 1];                        // the inputs of rows row0 - (TAPS - 1) .. row0 + ROWS - 1
#pragma unroll
  for (int k = 0; k < ROWS + TAPS - 1; ++k) {
    const int row = row0 + k - (TAPS - 1);
    u[k] = (row >= 0 && row < rows) ? *reinterpret_cast<const __nv_bfloat162*>(proj + (size_t)row * s.proj_pitch + c)
                                    : __floats2bfloat162_rn(0.f, 0.f);
  }
  int pos[ROWS], request[ROWS];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const bool live = row0 + r < rows;
    pos[r] = live ? positions[row0 + r] : -1;
    request[r] = live ? row_request[row0 + r] : 0;
  }
  // rows in the middle of a request's rows of the step: every input is one of the step's
  const bool inside = row0 + ROWS <= rows && pos[0] >= TAPS - 1 && request[0] == request[ROWS - 1] &&
                      row0 - cu_rows[request[0]] >= TAPS - 1;
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    if (row0 + r >= rows) break;
    float y0 = b0, y1 = b1;
    if (inside) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const float2 v = __bfloat1622float2(u[r + j]);
        y0 = fmaf(w0[j], v.x, y0);
        y1 = fmaf(w1[j], v.y, y1);
      }
    } else if (pos[r] >= 0) {
      const int ahead = row0 + r - cu_rows[request[r]];
      const float* kept = state + (size_t)state_slots[request[r]] * s.slot_floats + c;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int back = TAPS - 1 - j;
        if (pos[r] - back < 0) continue;                   // zeros before the start of the sequence
        float2 v = __bfloat1622float2(u[r + j]);
        if (back > ahead) {
          const float* at = kept + (size_t)(TAPS - 1 - (back - ahead)) * s.channels;
          v = make_float2(at[0], at[1]);
        }
        y0 = fmaf(w0[j], v.x, y0);
        y1 = fmaf(w1[j], v.y, y1);
      }
    } else {
      y0 = y1 = 0.f;
    }
    __nv_bfloat162 y;
    y.x = conv_result<__nv_bfloat16>(y0);
    y.y = conv_result<__nv_bfloat16>(y1);
    *reinterpret_cast<__nv_bfloat162*>(out + (size_t)(row0 + r) * s.channels + c) = y;
  }
}

template <typename T, typename O>
static int launch_short_conv(const void* proj, const float* weight, const float* bias, const int* positions,
                             const int* row_request, const int* cu_rows, const int* state_slots, float* state, void* out,
                             int rows, int requests, int write_state, int single_rows, const ConvShape& s, cudaStream_t st) {
  const int block = 128;
  const dim3 request_grid((s.channels + block - 1) / block, requests);
  if (single_rows) {
#define CONV_SINGLE(TAPS)                                                                                                    \
  SRB_CUDA_CALL(srb_launch(short_conv_single_kernel<T, O, TAPS>, request_grid, dim3(block), 0, st, (const T*)proj, weight,   \
                           bias, positions, cu_rows, state_slots, state, (O*)out, write_state, s))
    if (s.taps == 4) CONV_SINGLE(4);
    else if (s.taps == 3) CONV_SINGLE(3);
    else if (s.taps == 2) CONV_SINGLE(2);
    else CONV_SINGLE(0);
#undef CONV_SINGLE
    SRB_LAUNCH_CHECK("short_conv_single");
    return SRB_OK;
  }
  const bool many = rows >= 64 * CONV_ROWS;
  const int per = many ? CONV_ROWS : 1;
  const dim3 grid((s.channels + block - 1) / block, (rows + per - 1) / per);
  if (grid.y > 65535) SRB_FAIL("short_conv: %d rows exceed one launch", rows);
#define CONV_LAUNCH(TAPS, ROWS)                                                                                              \
  SRB_CUDA_CALL(srb_launch(short_conv_kernel<T, O, TAPS, ROWS>, grid, dim3(block), 0, st, (const T*)proj, weight, bias,     \
                           positions, row_request, cu_rows, state_slots, (const float*)state, (O*)out, rows, s))
  bool pairs = false;
  if constexpr (sizeof(T) == 2 && sizeof(O) == 2) {
    pairs = many && s.taps >= 2 && s.taps <= 4 && s.channels % 2 == 0 && s.proj_pitch % 2 == 0 && (((uintptr_t)proj | (uintptr_t)out) & 3) == 0;
    if (pairs) {
      auto kernel = s.taps == 4 ? short_conv_pair_kernel<4> : (s.taps == 3 ? short_conv_pair_kernel<3> : short_conv_pair_kernel<2>);
      SRB_CUDA_CALL(srb_launch(kernel, dim3((s.channels / 2 + block - 1) / block, grid.y), dim3(block), 0, st, (const __nv_bfloat16*)proj,
                               weight, bias, positions, row_request, cu_rows, state_slots, (const float*)state, (__nv_bfloat16*)out, rows, s));
    }
  }
  if (pairs) {}
  else if (s.taps == 4 && many) CONV_LAUNCH(4, CONV_ROWS);
  else if (s.taps == 4) CONV_LAUNCH(4, 1);
  else if (s.taps == 3 && many) CONV_LAUNCH(3, CONV_ROWS);
  else if (s.taps == 2 && many) CONV_LAUNCH(2, CONV_ROWS);
  else if (many) CONV_LAUNCH(0, CONV_ROWS);
  else CONV_LAUNCH(0, 1);
#undef CONV_LAUNCH
  if (write_state && s.taps > 1)
    SRB_CUDA_CALL(srb_launch(short_conv_keep_kernel<T>, request_grid, dim3(block), 0, st, (const T*)proj, positions, cu_rows,
                             state_slots, state, s));
  SRB_LAUNCH_CHECK("short_conv");
  return SRB_OK;
}

// proj: the first of the `channels` columns of the projection's first row, rows `proj_pitch` elements apart; weight
// [channels, taps], bias [channels] or null (float); out: [rows, channels] of `out_dtype` (float, or bfloat16 beside a
// bfloat16 projection).  `single_rows`: every request of the step brings exactly one row (the caller knows it from the
// step's shape, so nothing is decided from device memory).
extern "C" int srb_short_conv(const void* proj, long long proj_pitch, const float* weight, const float* bias,
                              const int* positions, const int* row_request, const int* cu_rows, const int* state_slots,
                              float* state, long long slot_floats, void* out, int rows, int requests, int channels, int taps,
                              int write_state, int single_rows, int dtype, int out_dtype, void* stream) {
  if (rows <= 0 || requests <= 0) return SRB_OK;
  if (channels <= 0) SRB_FAIL("short_conv: %d channels", channels);
  if (taps < 1 || taps > CONV_MAX_TAPS) SRB_FAIL("short_conv: a convolution over %d tokens is outside 1 .. %d", taps, CONV_MAX_TAPS);
  if (proj_pitch < channels) SRB_FAIL("short_conv: rows of the projection are too short");
  if (slot_floats < (long long)(taps - 1) * channels) SRB_FAIL("short_conv: a slot of %lld floats is too small", slot_floats);
  if (requests > 65535) SRB_FAIL("short_conv: %d requests exceed one launch", requests);
  ConvShape s;
  s.channels = channels; s.taps = taps; s.proj_pitch = proj_pitch; s.slot_floats = slot_floats;
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == SRB_DTYPE_F32 && out_dtype == SRB_DTYPE_F32)
    return launch_short_conv<float, float>(proj, weight, bias, positions, row_request, cu_rows, state_slots, state, out, rows,
                                           requests, write_state, single_rows, s, st);
  if (dtype == SRB_DTYPE_BF16 && out_dtype == SRB_DTYPE_F32)
    return launch_short_conv<__nv_bfloat16, float>(proj, weight, bias, positions, row_request, cu_rows, state_slots, state, out,
                                                   rows, requests, write_state, single_rows, s, st);
  if (dtype == SRB_DTYPE_BF16 && out_dtype == SRB_DTYPE_BF16)
    return launch_short_conv<__nv_bfloat16, __nv_bfloat16>(proj, weight, bias, positions, row_request, cu_rows, state_slots, state,
                                                           out, rows, requests, write_state, single_rows, s, st);
  SRB_FAIL("short_conv: a projection of dtype %d with a result of dtype %d is not taken", dtype, out_dtype);
}
