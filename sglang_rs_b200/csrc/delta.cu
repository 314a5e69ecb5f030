// The gated delta rule: linear attention whose state forgets by a decay and corrects itself by what it already holds for
// a key, over a state of fixed size per request.
//
// Per head with q_t, k_t (dim entries) and v_t (vdim entries), all three behind a short convolution and SiLU
// (short_conv.cu), S being [dim, vdim] and zero before the sequence's first token:
//
//   k' = k / sqrt(sum k^2 + 1e-6)           q' = q / sqrt(sum q^2 + 1e-6) * dim^-1/2            beta = sigmoid(b)
//   S <- diag(g) S       u = beta (v - S^T k')       S <- S + k' u^T       o = S^T q'
//
// Value head h uses q/k head h / (heads / kv_heads).  The decay g is one number per head and token,
// g = exp(-exp(A_log) softplus(a + dt_bias)), or (`channel_decay`) one per head, token and row of S, g_d =
// exp(-exp(A_log) softplus(a_d + dt_bias_d)).
//
// A request's slot of state holds, in 32-bit floats, the convolution's last taps - 1 inputs (padded to a multiple of four
// floats), then S as [heads][vdim][dim] (a value column's dim entries together).
//
//   srb_delta_scan       the recurrence, token by token: a block owns some value columns of a head in registers (a column's
//                        entries cut over the lanes beside it), stages 16 tokens' q, k, v, decays in shared memory and walks
//                        them; decoded tokens, float32 and odd sizes
//   srb_delta_chunks     the same recurrence for prompt portions in bfloat16, in chunks of 64 tokens on the tensor cores
//                        (described above those kernels)
//   srb_delta_gate_norm  per head o / sqrt(mean(o^2) + eps) * weight * gate(g), rounded
//
// Unit vectors, step sizes, decays and their logarithms, the state and all sums are 32-bit in both dtypes.  A request whose
// first row of the step is at position 0 starts from zero whatever its slot holds; rows at negative positions pad a captured
// step and are skipped.
#include "common.cuh"
#include <math.h>

SRB_DEFINE_LAST_ERROR()
SRB_DEFINE_PDL_SWITCH()

#define DELTA_TOKENS 16          // tokens staged in shared memory at a time
#define DELTA_THREADS 256

struct DeltaArgs {
  const void* x;                 // [rows, channels]: q (kv_heads * dim) | k (kv_heads * dim) | v (heads * vdim), convolved
  const void* beta;              // logits of beta: `heads` columns of a projection
  const void* decay;             // a: `heads` columns, or with channel_decay heads * dim
  long long beta_pitch, decay_pitch;
  const float* a_log;            // [heads]
  const float* dt_bias;          // [heads], or with channel_decay [heads * dim]
  const int* positions;
  const int* cu_rows;
  const int* state_slots;
  float* state;
  float* out;                    // [rows, heads * vdim]
  long long slot_floats;
  int conv_floats;               // where S starts in a slot
  int heads, kv_heads, dim, vdim, channels;
  int channel_decay, write_state, requests;
  float unit_eps, q_scale;
};

__device__ __forceinline__ float delta_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float delta_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }

// grid (heads * column blocks, requests); NS lanes share a column of the state, each with NR of its entries (groups of four
// consecutive ones, the groups dealt out over the lanes)
template <typename T, typename X, int NS, int NR, bool CHANNEL>
__global__ void __launch_bounds__(DELTA_THREADS) delta_scan_kernel(DeltaArgs a) {
  constexpr int PB = DELTA_THREADS / NS, DP = NS * NR, WARPS = DELTA_THREADS / 32;
  extern __shared__ __align__(16) float delta_smem[];
  float* q_s = delta_smem;                               // [DELTA_TOKENS][DP]
  float* k_s = q_s + DELTA_TOKENS * DP;
  float* g_s = k_s + DELTA_TOKENS * DP;                  // [DELTA_TOKENS][DP] with CHANNEL, else [DELTA_TOKENS]
  float* v_s = g_s + DELTA_TOKENS * (CHANNEL ? DP : 1);  // [DELTA_TOKENS][PB]
  float* b_s = v_s + DELTA_TOKENS * PB;                  // [DELTA_TOKENS]
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int dim = a.dim, vdim = a.vdim;
  const int column_blocks = (vdim + PB - 1) / PB;
  const int head = blockIdx.x / column_blocks, c0 = (blockIdx.x % column_blocks) * PB;
  const int request = blockIdx.y;
  const int first = a.cu_rows[request], count = a.cu_rows[request + 1] - first;
  if (count <= 0) return;
  const int start = a.positions[first];
  if (start < 0) return;
  const int tid = threadIdx.x, ns = tid % NS, cl = tid / NS, c = c0 + cl;
  const int warp = tid >> 5, lane = tid & 31;
  const bool active = c < vdim;
  float* mine = a.state + (size_t)a.state_slots[request] * a.slot_floats + a.conv_floats + ((size_t)head * vdim + c) * dim;
  float4 st[NR / 4];
  const bool vector = dim % 4 == 0;                      // (slots and S start on 16-byte borders)
#pragma unroll
  for (int i = 0; i < NR / 4; ++i) {
    const int d = (i * NS + ns) * 4;
    st[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active && start > 0) {
      if (vector) {
        if (d < dim) st[i] = *reinterpret_cast<const float4*>(mine + d);
      } else {
        if (d < dim) st[i].x = mine[d];
        if (d + 1 < dim) st[i].y = mine[d + 1];
        if (d + 2 < dim) st[i].z = mine[d + 2];
        if (d + 3 < dim) st[i].w = mine[d + 3];
      }
    }
  }
  const int qk_head = head / (a.heads / a.kv_heads);
  const float rate = expf(a.a_log[head]);
  const X* x = reinterpret_cast<const X*>(a.x);
  const T* beta = reinterpret_cast<const T*>(a.beta);
  const T* decay = reinterpret_cast<const T*>(a.decay);
  const int k_at = a.kv_heads * dim, v_at = 2 * a.kv_heads * dim;
  for (int t0 = 0; t0 < count; t0 += DELTA_TOKENS) {
    const int tc = min(DELTA_TOKENS, count - t0);
    if (t0) __syncthreads();                             // the tokens before are done with
    // a warp per unit vector: the sum of squares and the scaled entries
    for (int item = warp; item < 2 * tc; item += WARPS) {
      const int t = item >> 1, is_k = item & 1;
      const X* src = x + (size_t)(first + t0 + t) * a.channels + (is_k ? k_at : 0) + qk_head * dim;
      float* dst = (is_k ? k_s : q_s) + t * DP;
      float squares = 0.f;
      for (int d = lane; d < DP; d += 32) {
        const float v = d < dim ? srb_to_float(src[d]) : 0.f;
        dst[d] = v;
        squares = fmaf(v, v, squares);
      }
      const float scale = (is_k ? 1.0f : a.q_scale) / sqrtf(srb_warp_sum(squares) + a.unit_eps);
      for (int d = lane; d < DP; d += 32) dst[d] *= scale;      // each lane its own entries
    }
    for (int i = tid; i < tc * PB; i += DELTA_THREADS) {
      const int t = i / PB, p = i - t * PB;
      v_s[i] = c0 + p < vdim ? srb_to_float(x[(size_t)(first + t0 + t) * a.channels + v_at + head * vdim + c0 + p]) : 0.f;
    }
    if (CHANNEL) {
      for (int i = tid; i < tc * DP; i += DELTA_THREADS) {
        const int t = i / DP, d = i - t * DP;
        float g = 1.f;
        if (d < dim)
          g = expf(-rate * delta_softplus(srb_to_float(decay[(size_t)(first + t0 + t) * a.decay_pitch + head * dim + d]) +
                                          a.dt_bias[head * dim + d]));
        g_s[i] = g;
      }
    } else if (tid < tc) {
      g_s[tid] = expf(-rate * delta_softplus(srb_to_float(decay[(size_t)(first + t0 + tid) * a.decay_pitch + head]) + a.dt_bias[head]));
    }
    if (tid >= 32 && tid - 32 < tc)
      b_s[tid - 32] = delta_sigmoid(srb_to_float(beta[(size_t)(first + t0 + tid - 32) * a.beta_pitch + head]));
    __syncthreads();
    for (int t = 0; t < tc; ++t) {
      const float4* k4 = reinterpret_cast<const float4*>(k_s + t * DP);
      const float4* q4 = reinterpret_cast<const float4*>(q_s + t * DP);
      const float4* g4 = reinterpret_cast<const float4*>(g_s + t * DP);      // (CHANNEL only)
      const float whole = CHANNEL ? 1.f : g_s[t];
      float4 k[NR / 4];
      float held = 0.f;
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        k[i] = k4[i * NS + ns];
        float4 g = make_float4(whole, whole, whole, whole);
        if (CHANNEL) g = g4[i * NS + ns];
        st[i].x *= g.x; st[i].y *= g.y; st[i].z *= g.z; st[i].w *= g.w;
        held = fmaf(st[i].x, k[i].x, held);
        held = fmaf(st[i].y, k[i].y, held);
        held = fmaf(st[i].z, k[i].z, held);
        held = fmaf(st[i].w, k[i].w, held);
      }
#pragma unroll
      for (int offset = NS / 2; offset > 0; offset >>= 1) held += __shfl_xor_sync(0xffffffffu, held, offset);
      const float u = b_s[t] * (v_s[t * PB + cl] - held);
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const float4 q = q4[i * NS + ns];
        st[i].x = fmaf(k[i].x, u, st[i].x);
        st[i].y = fmaf(k[i].y, u, st[i].y);
        st[i].z = fmaf(k[i].z, u, st[i].z);
        st[i].w = fmaf(k[i].w, u, st[i].w);
        o = fmaf(st[i].x, q.x, o);
        o = fmaf(st[i].y, q.y, o);
        o = fmaf(st[i].z, q.z, o);
        o = fmaf(st[i].w, q.w, o);
      }
#pragma unroll
      for (int offset = NS / 2; offset > 0; offset >>= 1) o += __shfl_xor_sync(0xffffffffu, o, offset);
      if (ns == 0 && active) a.out[(size_t)(first + t0 + t) * a.heads * vdim + (size_t)head * vdim + c] = o;
    }
  }
  if (!a.write_state || !active) return;
#pragma unroll
  for (int i = 0; i < NR / 4; ++i) {
    const int d = (i * NS + ns) * 4;
    if (vector) {
      if (d < dim) *reinterpret_cast<float4*>(mine + d) = st[i];
    } else {
      if (d < dim) mine[d] = st[i].x;
      if (d + 1 < dim) mine[d + 1] = st[i].y;
      if (d + 2 < dim) mine[d + 2] = st[i].z;
      if (d + 3 < dim) mine[d + 3] = st[i].w;
    }
  }
}

extern "C" long long srb_delta_slot_floats(int heads, int kv_heads, int dim, int vdim, int taps) {
  const long long conv = (long long)(taps - 1) * (2LL * kv_heads * dim + (long long)heads * vdim);
  return ((conv + 3) / 4 * 4 + (long long)heads * dim * vdim + 3) / 4 * 4;
}

static int delta_args(DeltaArgs& a, const void* x, const void* beta, long long beta_pitch, const void* decay, long long decay_pitch,
                      const float* a_log, const float* dt_bias, const int* positions, const int* cu_rows, const int* state_slots,
                      float* state, long long slot_floats, float* out, int requests, int heads, int kv_heads, int dim, int vdim,
                      int taps, int channel_decay, float unit_eps, int write_state) {
  if (heads <= 0 || kv_heads <= 0 || dim <= 0 || vdim <= 0 || heads % kv_heads)
    SRB_FAIL("delta: %d heads on %d q/k heads of %d x %d entries do not fit", heads, kv_heads, dim, vdim);
  if (taps < 1) SRB_FAIL("delta: a convolution over %d tokens", taps);
  if (slot_floats < srb_delta_slot_floats(heads, kv_heads, dim, vdim, taps) || slot_floats % 4 || ((uintptr_t)state & 15))
    SRB_FAIL("delta: slots of %lld floats are too small or start off 16-byte borders", slot_floats);
  if (requests > 65535) SRB_FAIL("delta: %d requests exceed one launch", requests);
  a.x = x; a.beta = beta; a.beta_pitch = beta_pitch; a.decay = decay; a.decay_pitch = decay_pitch; a.a_log = a_log; a.dt_bias = dt_bias;
  a.positions = positions; a.cu_rows = cu_rows; a.state_slots = state_slots; a.state = state; a.slot_floats = slot_floats; a.out = out;
  a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.vdim = vdim; a.channels = 2 * kv_heads * dim + heads * vdim;
  a.conv_floats = (int)(((long long)(taps - 1) * a.channels + 3) / 4 * 4);
  a.channel_decay = channel_decay; a.write_state = write_state; a.requests = requests;
  a.unit_eps = unit_eps; a.q_scale = 1.0f / sqrtf((float)dim);
  return SRB_OK;
}

template <typename T, typename X, int NS, int NR, bool CHANNEL>
static int launch_delta_scan(const DeltaArgs& a, cudaStream_t s) {
  constexpr int PB = DELTA_THREADS / NS, DP = NS * NR;
  const dim3 grid(a.heads * ((a.vdim + PB - 1) / PB), a.requests);
  const size_t smem = (size_t)DELTA_TOKENS * (2 * DP + (CHANNEL ? DP : 1) + PB + 1) * sizeof(float);
  auto kernel = delta_scan_kernel<T, X, NS, NR, CHANNEL>;
  if (smem > 48 * 1024) SRB_CUDA_CALL(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  SRB_CUDA_CALL(srb_launch(kernel, grid, dim3(DELTA_THREADS), smem, s, a));
  SRB_LAUNCH_CHECK("delta_scan");
  return SRB_OK;
}

template <typename T, typename X>
static int dispatch_delta_scan(const DeltaArgs& a, cudaStream_t s) {
  if (a.dim > 512) SRB_FAIL("delta_scan: heads of %d entries exceed 512", a.dim);
  if (a.dim > 256) return a.channel_decay ? launch_delta_scan<T, X, 32, 16, true>(a, s) : launch_delta_scan<T, X, 32, 16, false>(a, s);
  if (a.dim > 128) return a.channel_decay ? launch_delta_scan<T, X, 16, 16, true>(a, s) : launch_delta_scan<T, X, 16, 16, false>(a, s);
  if (a.dim > 64) return a.channel_decay ? launch_delta_scan<T, X, 8, 16, true>(a, s) : launch_delta_scan<T, X, 8, 16, false>(a, s);
  return a.channel_decay ? launch_delta_scan<T, X, 8, 8, true>(a, s) : launch_delta_scan<T, X, 8, 8, false>(a, s);
}

// x: float [rows, channels] (what srb_short_conv wrote); beta, decay: columns of projections of `dtype`; out: float [rows,
// heads * vdim]
extern "C" int srb_delta_scan(const float* x, const void* beta, long long beta_pitch, const void* decay, long long decay_pitch,
                              const float* a_log, const float* dt_bias, const int* positions, const int* cu_rows,
                              const int* state_slots, float* state, long long slot_floats, float* out, int rows, int requests,
                              int heads, int kv_heads, int dim, int vdim, int taps, int channel_decay, float unit_eps,
                              int write_state, int dtype, void* stream) {
  if (rows <= 0 || requests <= 0) return SRB_OK;
  DeltaArgs a;
  if (delta_args(a, x, beta, beta_pitch, decay, decay_pitch, a_log, dt_bias, positions, cu_rows, state_slots, state, slot_floats, out,
                 requests, heads, kv_heads, dim, vdim, taps, channel_decay, unit_eps, write_state) != SRB_OK)
    return SRB_ERR_INVALID;
  if (dtype == SRB_DTYPE_F32) return dispatch_delta_scan<float, float>(a, (cudaStream_t)stream);
  if (dtype == SRB_DTYPE_BF16) return dispatch_delta_scan<__nv_bfloat16, float>(a, (cudaStream_t)stream);
  SRB_FAIL("delta_scan: unknown dtype %d", dtype);
}

// ---- norm, weight and gate per head ------------------------------------------------------------------------------------
// A warp per (row, head): out[row, head, i] = o / sqrt(mean(o^2) + eps) * weight[i] * scale * gate, the gate being
// sigmoid(g) or silu(g).
template <typename T>
__global__ void delta_gate_norm_kernel(const float* __restrict__ o, const T* __restrict__ g, long long g_pitch,
                                       const float* __restrict__ weight, float eps, float scale, int silu, int rows, int heads,
                                       int vdim, T* __restrict__ out, long long out_pitch) {
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)rows * heads) return;
  const int row = (int)(item / heads), head = (int)(item - (long long)row * heads);
  const float* src = o + ((size_t)row * heads + head) * vdim;
  const T* gate = g + (size_t)row * g_pitch + (size_t)head * vdim;
  T* dst = out + (size_t)row * out_pitch + (size_t)head * vdim;
  constexpr int HELD = 4;                                  // entries of a lane that stay in registers (vdim up to 128)
  float v[HELD], z[HELD];
  float squares = 0.f;
#pragma unroll
  for (int j = 0; j < HELD; ++j) {
    const int i = lane + 32 * j;
    v[j] = i < vdim ? src[i] : 0.f;
    z[j] = i < vdim ? srb_to_float(gate[i]) : 0.f;
    squares = fmaf(v[j], v[j], squares);
  }
  for (int i = lane + 32 * HELD; i < vdim; i += 32) squares = fmaf(src[i], src[i], squares);
  const float inv = scale / sqrtf(srb_warp_sum(squares) / (float)vdim + eps);
#pragma unroll
  for (int j = 0; j < HELD; ++j) {
    const int i = lane + 32 * j;
    if (i < vdim) dst[i] = srb_from_float<T>(v[j] * inv * weight[i] * (silu ? z[j] * delta_sigmoid(z[j]) : delta_sigmoid(z[j])));
  }
  for (int i = lane + 32 * HELD; i < vdim; i += 32) {
    const float y = srb_to_float(gate[i]);
    dst[i] = srb_from_float<T>(src[i] * inv * weight[i] * (silu ? y * delta_sigmoid(y) : delta_sigmoid(y)));
  }
}

// o: float [rows, heads * vdim]; g: heads * vdim columns of a projection; weight float [vdim]; out: rows `out_pitch` apart;
// silu 0: the gate is sigmoid(g), 1: silu(g); `scale`: a factor on everything
extern "C" int srb_delta_gate_norm(const float* o, const void* g, long long g_pitch, const float* weight, float eps, float scale,
                                   int silu, int rows, int heads, int vdim, void* out, long long out_pitch, int dtype, void* stream) {
  if (rows <= 0) return SRB_OK;
  if (heads <= 0 || vdim <= 0) SRB_FAIL("delta_gate_norm: %d heads of %d entries", heads, vdim);
  if (!(eps >= 0.f)) SRB_FAIL("delta_gate_norm: eps must be finite and non-negative");
  if (out_pitch < (long long)heads * vdim) SRB_FAIL("delta_gate_norm: rows of the output overlap");
  const long long items = (long long)rows * heads;
  const int warps = 4;
  const dim3 grid((unsigned)((items + warps - 1) / warps));
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == SRB_DTYPE_F32)
    SRB_CUDA_CALL(srb_launch(delta_gate_norm_kernel<float>, grid, dim3(warps * 32), 0, s, o, (const float*)g, g_pitch, weight, eps,
                             scale, silu, rows, heads, vdim, (float*)out, out_pitch));
  else if (dtype == SRB_DTYPE_BF16)
    SRB_CUDA_CALL(srb_launch(delta_gate_norm_kernel<__nv_bfloat16>, grid, dim3(warps * 32), 0, s, o, (const __nv_bfloat16*)g, g_pitch,
                             weight, eps, scale, silu, rows, heads, vdim, (__nv_bfloat16*)out, out_pitch));
  else
    SRB_FAIL("delta_gate_norm: unknown dtype %d", dtype);
  SRB_LAUNCH_CHECK("delta_gate_norm");
  return SRB_OK;
}
