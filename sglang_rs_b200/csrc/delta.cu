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
template <typename T, typename X, int NS, int NR, bool CHANNEL, int THREADS>
__global__ void __launch_bounds__(THREADS) delta_scan_kernel(DeltaArgs a) {
  constexpr int PB = THREADS / NS, DP = NS * NR, WARPS = THREADS / 32;
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
    for (int i = tid; i < tc * PB; i += THREADS) {
      const int t = i / PB, p = i - t * PB;
      v_s[i] = c0 + p < vdim ? srb_to_float(x[(size_t)(first + t0 + t) * a.channels + v_at + head * vdim + c0 + p]) : 0.f;
    }
    if (CHANNEL) {
      for (int i = tid; i < tc * DP; i += THREADS) {
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

template <typename T, typename X, int NS, int NR, bool CHANNEL, int THREADS>
static int launch_delta_scan(const DeltaArgs& a, cudaStream_t s) {
  constexpr int PB = THREADS / NS, DP = NS * NR;
  const dim3 grid(a.heads * ((a.vdim + PB - 1) / PB), a.requests);
  const size_t smem = (size_t)DELTA_TOKENS * (2 * DP + (CHANNEL ? DP : 1) + PB + 1) * sizeof(float);
  auto kernel = delta_scan_kernel<T, X, NS, NR, CHANNEL, THREADS>;
  if (smem > 48 * 1024) SRB_CUDA_CALL(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  SRB_CUDA_CALL(srb_launch(kernel, grid, dim3(THREADS), smem, s, a));
  SRB_LAUNCH_CHECK("delta_scan");
  return SRB_OK;
}

// `single_rows`: steps of decoded tokens read and write each state once, so more and smaller blocks, which all fit the chip
// together at small batches, are quicker
template <typename T, typename X>
static int dispatch_delta_scan(const DeltaArgs& a, int single_rows, cudaStream_t s) {
  if (a.dim > 512) SRB_FAIL("delta_scan: heads of %d entries exceed 512", a.dim);
#define DELTA_SCAN(NS, NR)                                                                                                  \
  (a.channel_decay ? (single_rows ? launch_delta_scan<T, X, NS, NR, true, 128>(a, s) : launch_delta_scan<T, X, NS, NR, true, DELTA_THREADS>(a, s)) \
                   : (single_rows ? launch_delta_scan<T, X, NS, NR, false, 128>(a, s) : launch_delta_scan<T, X, NS, NR, false, DELTA_THREADS>(a, s)))
  if (a.dim > 256) return DELTA_SCAN(32, 16);
  if (a.dim > 128) return DELTA_SCAN(16, 16);
  if (a.dim > 64) return DELTA_SCAN(8, 16);
  return DELTA_SCAN(8, 8);
#undef DELTA_SCAN
}

// x: float [rows, channels] (what srb_short_conv wrote); beta, decay: columns of projections of `dtype`; out: float [rows,
// heads * vdim]; `single_rows`: every request of the step brings one row (a hint; the results are the same)
extern "C" int srb_delta_scan(const float* x, const void* beta, long long beta_pitch, const void* decay, long long decay_pitch,
                              const float* a_log, const float* dt_bias, const int* positions, const int* cu_rows,
                              const int* state_slots, float* state, long long slot_floats, float* out, int rows, int requests,
                              int heads, int kv_heads, int dim, int vdim, int taps, int channel_decay, float unit_eps,
                              int write_state, int single_rows, int dtype, void* stream) {
  if (rows <= 0 || requests <= 0) return SRB_OK;
  DeltaArgs a;
  if (delta_args(a, x, beta, beta_pitch, decay, decay_pitch, a_log, dt_bias, positions, cu_rows, state_slots, state, slot_floats, out,
                 requests, heads, kv_heads, dim, vdim, taps, channel_decay, unit_eps, write_state) != SRB_OK)
    return SRB_ERR_INVALID;
  if (dtype == SRB_DTYPE_F32) return dispatch_delta_scan<float, float>(a, single_rows, (cudaStream_t)stream);
  if (dtype == SRB_DTYPE_BF16) return dispatch_delta_scan<__nv_bfloat16, float>(a, single_rows, (cudaStream_t)stream);
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

// The same in bfloat16 with four consecutive entries a lane: LANES lanes take a head of 4 LANES entries (32, 64 or 128), so a warp
// takes 32 / LANES heads; rows and columns on 8-byte borders.
template <int LANES>
__global__ void __launch_bounds__(128)
delta_gate_norm_quad_kernel(const float* __restrict__ o, const __nv_bfloat16* __restrict__ g, long long g_pitch,
                            const float* __restrict__ weight, float eps, float scale, int silu, int rows, int heads,
                            __nv_bfloat16* __restrict__ out, long long out_pitch) {
  srb_launch_dependents();
  const int lane = threadIdx.x % LANES;
  const float4 w = *reinterpret_cast<const float4*>(weight + lane * 4);
  srb_grid_dependency_wait();
  const long long item = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / LANES;
  const bool live = item < (long long)rows * heads;
  const int row = live ? (int)(item / heads) : 0, head = live ? (int)(item - (long long)row * heads) : 0;
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  uint2 raw = make_uint2(0u, 0u);
  if (live) {
    v = *reinterpret_cast<const float4*>(o + (size_t)item * (4 * LANES) + lane * 4);
    raw = *reinterpret_cast<const uint2*>(g + (size_t)row * g_pitch + (size_t)head * (4 * LANES) + lane * 4);
  }
  float squares = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
#pragma unroll
  for (int offset = LANES / 2; offset > 0; offset >>= 1) squares += __shfl_xor_sync(0xffffffffu, squares, offset);
  if (!live) return;
  const float inv = scale / sqrtf(squares / (float)(4 * LANES) + eps);
  const float2 za = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 zb = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  auto gate = [&](float z) { return silu ? z * delta_sigmoid(z) : delta_sigmoid(z); };
  const __nv_bfloat162 ya = __floats2bfloat162_rn(v.x * inv * w.x * gate(za.x), v.y * inv * w.y * gate(za.y));
  const __nv_bfloat162 yb = __floats2bfloat162_rn(v.z * inv * w.z * gate(zb.x), v.w * inv * w.w * gate(zb.y));
  raw.x = *reinterpret_cast<const unsigned*>(&ya);
  raw.y = *reinterpret_cast<const unsigned*>(&yb);
  *reinterpret_cast<uint2*>(out + (size_t)row * out_pitch + (size_t)head * (4 * LANES) + lane * 4) = raw;
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
  if (dtype == SRB_DTYPE_BF16 && (vdim == 32 || vdim == 64 || vdim == 128) && g_pitch % 4 == 0 && out_pitch % 4 == 0 &&
      (((uintptr_t)o | (uintptr_t)weight) & 15) == 0 && (((uintptr_t)g | (uintptr_t)out) & 7) == 0) {
    auto kernel = vdim == 128 ? delta_gate_norm_quad_kernel<32> : (vdim == 64 ? delta_gate_norm_quad_kernel<16> : delta_gate_norm_quad_kernel<8>);
    SRB_CUDA_CALL(srb_launch(kernel, dim3((unsigned)((items * (vdim / 4) + 127) / 128)), dim3(128), 0, s, o, (const __nv_bfloat16*)g, g_pitch,
                             weight, eps, scale, silu, rows, heads, (__nv_bfloat16*)out, out_pitch));
    SRB_LAUNCH_CHECK("delta_gate_norm");
    return SRB_OK;
  }
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

// ---- prompt portions in bfloat16: chunks of tokens on the tensor cores ---------------------------------------------------
// The rows of every request are cut into chunks of DC_TOKENS (64) tokens (from the request's first row of the step).  Inside a
// chunk that starts from state S and holds tokens 0 .. n-1, with c_t the sum of the logarithms of the decays up to t (a number,
// or one per row of S; never positive, and never rising), k' and q' the unit vectors, and (k e^c) meaning entry by entry:
//     L[t, j] = beta_t sum_d k'_t k'_j e^(c_t - c_j)   for j < t           A[t, j] = sum_d q'_t k'_j e^(c_t - c_j)   for j <= t
//     (1 + L) U = beta (V - (K' e^c) S)                                    o_t = (q'_t e^(c_t)) S + sum_j A[t, j] u_j
//     S <- e^(c_(n-1)) S + sum_j (k'_j e^(c_(n-1) - c_j)) u_j^T
// so U = T beta V - W S with T = (1 + L)^-1 and W = T beta (K' e^c).  Every exponential is of a number that is not positive.
// With a decay per row of S the sums behind L and A do not factor into e^(c_t) and e^(-c_j), which could overflow: they are taken
// block by block of 16 tokens with both factors relative to c just before the row block: left of the diagonal both exponents are
// then not positive; a diagonal block whose c falls by more than 2^100 in some row of S is taken pair by pair.  Two kernels:
//   1. delta_chunk_prepare: per (chunk, head), in parallel: A, T, W, T beta V and the scaled q' and k'
//   2. delta_chunk_walk: per (request, head, VS value columns) the chunks in order, S in registers: U, the results, the next S
// x goes in as bfloat16 (what the convolution wrote); whatever is 32-bit by the design and has to be an operand of a product
// goes in as the sum of two bfloat16 numbers, its rounding and the rounding of the rest (16 bits of mantissa), in two products,
// or three where both operands are such sums; accumulation is 32-bit (mma.sync m16n8k16).
// Heads of up to 128 entries (padded to 64 or 128 with zeros), widths that are multiples of eight.
#include "mma_helpers.cuh"

#define DC_TOKENS 64
#define DC_PREPARE_THREADS 256
#define DC_PAD 8
#define DC_LOG2E 1.4426950408889634f
#define DC_FASTEST -40.0f        // log2 of the smallest decay: below 2^-40 of a state nothing is left beside a 32-bit sum, and the
                                 // sums of logarithms down a chunk, whose differences are taken, keep their last bits

__device__ __forceinline__ unsigned dc_word(const __nv_bfloat16* p) { return *reinterpret_cast<const unsigned*>(p); }
// (a, b) as two packed pairs: the roundings and the roundings of what they left
__device__ __forceinline__ void dc_split2(float a, float b, unsigned& hi, unsigned& lo) {
  hi = pack_bf16(a, b);
  const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&hi);
  const float2 f = __bfloat1622float2(h);
  lo = pack_bf16(a - f.x, b - f.y);
}
// 2^x for the factors of a chunk: the hardware's exponential (2 units in the last place), results below 2^-126 are zero
__device__ __forceinline__ float dc_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float2 dc_pair(const __nv_bfloat16* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}

// What kernel 1 hands to kernel 2, per (chunk, head); all pieces start on 16-byte borders.
template <int DP, bool CHANNEL>
struct DeltaChunkLayout {
  static constexpr int ROWS = DC_TOKENS * DP * 2;                          // bytes of a [64][DP] operand
  static constexpr int W = 0;                                              // -W: roundings, then the rest
  static constexpr int Q = 2 * ROWS;                                       // CHANNEL: q' e^c, k' e^(c_last - c), each in two
  static constexpr int K = Q + (CHANNEL ? 2 * ROWS : 0);
  static constexpr int A = K + (CHANNEL ? 2 * ROWS : 0);                   // [64][64] in two
  static constexpr int F = A + 2 * DC_TOKENS * DC_TOKENS * 2;              // floats: CHANNEL e^(c_last) [DP]; else q's and k's
  static constexpr int FLOATS = CHANNEL ? DP : 2 * DC_TOKENS + 4;          // factors per token and e^(c_last)
  static constexpr int V = F + FLOATS * 4;                                 // T beta V, transposed: float [vp][64]
  static __host__ __device__ long long bytes(int vp) { return V + (long long)vp * DC_TOKENS * 4; }
};

// the request and the chunk of it that block `index` works on; false: there is no such chunk
__device__ __forceinline__ bool dc_find(const DeltaArgs& a, int index, int& request, int& row0, int& n) {
  int first = 0;
  for (request = 0; request < a.requests; ++request) {
    const int begin = a.cu_rows[request], rows = a.cu_rows[request + 1] - begin;
    const int chunks = (rows + DC_TOKENS - 1) / DC_TOKENS;
    if (index < first + chunks) {
      row0 = begin + (index - first) * DC_TOKENS;
      n = min(DC_TOKENS, begin + rows - row0);
      return true;
    }
    first += chunks;
  }
  return false;
}

template <int DP, bool CHANNEL>
struct DeltaPrepareSmem {
  static constexpr int XP = DP + DC_PAD, CP = DP + 2, TP = DC_TOKENS + DC_PAD, LP = DC_TOKENS + 4;
  static constexpr int K = 0;                                              // bfloat16 [64][XP]
  static constexpr int Q = K + DC_TOKENS * XP * 2;                         // bfloat16 [64][XP]; later T scaled, in two [64][TP]
  static constexpr int T_BYTES = 2 * DC_TOKENS * TP * 2;
  static constexpr int QB = DC_TOKENS * XP * 2 > T_BYTES ? DC_TOKENS * XP * 2 : T_BYTES;
  static constexpr int LT = Q + QB;                                        // L and T, float [64][LP] each; later k' e^c in two
  static constexpr int LT_BYTES_A = 2 * DC_TOKENS * LP * 4, LT_BYTES_B = CHANNEL ? 2 * DC_TOKENS * XP * 2 : T_BYTES;
  static constexpr int LT_BYTES = LT_BYTES_A > LT_BYTES_B ? LT_BYTES_A : LT_BYTES_B;
  static constexpr int C = LT + LT_BYTES;                                  // CHANNEL: c, float [64][CP]; later v
  static constexpr int C_BYTES = CHANNEL ? DC_TOKENS * CP * 4 : 0;
  static constexpr int small(int vp) {
    const int v = DC_TOKENS * (vp + DC_PAD) * 2;
    return C + (C_BYTES > v ? C_BYTES : v);
  }
  static constexpr int SMALL_FLOATS = 4 * DC_TOKENS + 4 * DP + 16;          // per token: beta, 1/|k|, scale/|q|, c; totals
  static constexpr int bytes(int vp) { return small(vp) + SMALL_FLOATS * 4; }
};

template <int DP, bool CHANNEL>
__global__ void __launch_bounds__(DC_PREPARE_THREADS, 2) delta_chunk_prepare_kernel(DeltaArgs a, unsigned char* scratch, int vp) {
  using M = DeltaPrepareSmem<DP, CHANNEL>;
  using P = DeltaChunkLayout<DP, CHANNEL>;
  constexpr int XP = M::XP, CP = M::CP, TP = M::TP, LP = M::LP, NTH = DC_PREPARE_THREADS;
  extern __shared__ __align__(16) unsigned char dp_smem[];
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(dp_smem + M::K);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(dp_smem + M::Q);
  float* ls = reinterpret_cast<float*>(dp_smem + M::LT);                   // [64][LP]
  float* ts = ls + DC_TOKENS * LP;                                         // [64][LP]: A first, then T
  float* cs = reinterpret_cast<float*>(dp_smem + M::C);                    // [64][CP], in units of log2 (CHANNEL)
  float* beta_s = reinterpret_cast<float*>(dp_smem + M::small(vp));
  float* ik_s = beta_s + DC_TOKENS;
  float* iq_s = ik_s + DC_TOKENS;
  float* cum_s = iq_s + DC_TOKENS;                                         // one decay per head: c, in units of log2
  float* part_s = cum_s + DC_TOKENS;                                       // [4][DP]; then the first DP floats are zeros
  const float* zero_s = part_s;
  int* mild_s = reinterpret_cast<int*>(part_s + 4 * DP);                   // [4]
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int head = blockIdx.y, dim = a.dim, vdim = a.vdim;
  int request, row0, n;
  if (!dc_find(a, blockIdx.x, request, row0, n)) return;
  const int qk_head = head / (a.heads / a.kv_heads);
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x) + (size_t)row0 * a.channels;
  const __nv_bfloat16* beta = reinterpret_cast<const __nv_bfloat16*>(a.beta);
  const __nv_bfloat16* decay = reinterpret_cast<const __nv_bfloat16*>(a.decay);
  unsigned char* place = scratch + ((size_t)blockIdx.x * a.heads + head) * P::bytes(vp);

  // q and k as they lie, zeros beyond the chunk's tokens and the head's entries
  for (int i = tid; i < DC_TOKENS * DP / 8; i += NTH) {
    const int t = i / (DP / 8), d = i % (DP / 8) * 8;
    const bool live = t < n && d < dim;
    const __nv_bfloat16* from = x + (size_t)(live ? t : 0) * a.channels + qk_head * dim + (live ? d : 0);
    cp_async_16(qs + t * XP + d, from, live ? 16 : 0);
    cp_async_16(ks + t * XP + d, from + a.kv_heads * dim, live ? 16 : 0);
  }
  cp_async_commit();
  const float rate = expf(a.a_log[head]) * DC_LOG2E;
  if (tid < DC_TOKENS) beta_s[tid] = tid < n ? delta_sigmoid(__bfloat162float(beta[(size_t)(row0 + tid) * a.beta_pitch + head])) : 0.f;
  if (CHANNEL) {
    // running sums down the tokens: a thread takes one row of the state for a part of the tokens, then adds the parts before
    constexpr int PARTS = NTH / DP, PER = DC_TOKENS / PARTS;
    const int d = tid % DP, part = tid / DP;
    float sum = 0.f;
    if (d < dim) {
      const float bias = a.dt_bias[head * dim + d];
      const __nv_bfloat16* from = decay + (size_t)row0 * a.decay_pitch + head * dim + d;
      for (int t0 = part * PER; t0 < (part + 1) * PER; t0 += 8) {
        float v[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = t0 + j < n ? __bfloat162float(from[(size_t)(t0 + j) * a.decay_pitch]) : 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          if (t0 + j < n) sum += fmaxf(-rate * delta_softplus(v[j] + bias), DC_FASTEST);
          cs[(t0 + j) * CP + d] = sum;
        }
      }
    } else {
      for (int t = part * PER; t < (part + 1) * PER; ++t) cs[t * CP + d] = 0.f;
    }
    part_s[part * DP + d] = sum;
    __syncthreads();
    float before = 0.f;
    for (int p = 0; p < part; ++p) before += part_s[p * DP + d];
    if (part)
      for (int t = part * PER; t < (part + 1) * PER; ++t) cs[t * CP + d] += before;
  } else if (warp == 0) {
    float v0 = 0.f, v1 = 0.f;                              // a lane takes tokens 2 lane and 2 lane + 1
    const float bias = a.dt_bias[head];
    const int t = 2 * lane;
    if (t < n) v0 = fmaxf(-rate * delta_softplus(__bfloat162float(decay[(size_t)(row0 + t) * a.decay_pitch + head]) + bias), DC_FASTEST);
    if (t + 1 < n) v1 = fmaxf(-rate * delta_softplus(__bfloat162float(decay[(size_t)(row0 + t + 1) * a.decay_pitch + head]) + bias), DC_FASTEST);
    float total = v0 + v1;
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
      const float other = __shfl_up_sync(0xffffffffu, total, offset);
      if (lane >= offset) total += other;
    }
    cum_s[t + 1] = total;
    cum_s[t] = total - v1;
  }
  cp_async_wait<0>();
  __syncthreads();
  if (CHANNEL)
    for (int d = tid; d < DP; d += NTH) part_s[d] = 0.f;   // (every thread has taken its parts' totals)
  // lengths: a warp takes eight tokens
  for (int t = warp * 8; t < warp * 8 + 8; ++t) {
    float kk = 0.f, qq = 0.f;
    for (int d = lane * 2; d < DP; d += 64) {
      const float2 k = dc_pair(ks + t * XP + d), q = dc_pair(qs + t * XP + d);
      kk = fmaf(k.x, k.x, fmaf(k.y, k.y, kk));
      qq = fmaf(q.x, q.x, fmaf(q.y, q.y, qq));
    }
    kk = srb_warp_sum(kk);
    qq = srb_warp_sum(qq);
    if (lane == 0) {
      ik_s[t] = 1.0f / sqrtf(kk + a.unit_eps);
      iq_s[t] = a.q_scale / sqrtf(qq + a.unit_eps);
    }
  }
  __syncthreads();

  // ---- L and A.  Warps 0-3 take the rows of K, 4-7 those of Q, a block of 16 rows each
  // (the second four count their blocks backwards, so that the long rows are spread over the SM's quarters)
  const int kind = warp >> 2, rb = kind ? 3 - (warp & 3) : warp & 3;
  const int r0 = rb * 16 + g, r1 = r0 + 8;
  const __nv_bfloat16* rows_s = kind ? qs : ks;
  float* into = kind ? ts : ls;
  if (!CHANNEL) {
    float acc[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DP / 16; ++kk) {
      const int col = kk * 16 + 2 * t4;
      unsigned ra[4] = {dc_word(rows_s + r0 * XP + col), dc_word(rows_s + r1 * XP + col), dc_word(rows_s + r0 * XP + col + 8),
                        dc_word(rows_s + r1 * XP + col + 8)};
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
        if (nt < 2 * rb + 2) {
          const __nv_bfloat16* b = ks + (nt * 8 + g) * XP + col;
          mma_bf16(acc[nt], ra, dc_word(b), dc_word(b + 8));
        }
    }
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
      if (nt < 2 * rb + 2) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = e < 2 ? r0 : r1, j = nt * 8 + 2 * t4 + (e & 1);
          float v = 0.f;
          if (j < t || (kind && j == t))
            v = acc[nt][e] * (kind ? iq_s[t] : beta_s[t] * ik_s[t]) * ik_s[j] * dc_exp2(cum_s[t] - cum_s[j]);
          into[t * LP + j] = v;
        }
      }
  } else {
    // c falls by what inside the row block?  Up to 2^100 both factors of a diagonal block can be taken relative to c just
    // before it, too (what the mask discards stays finite)
    const float* ref = rb ? cs + (rb * 16 - 1) * CP : zero_s;
    float fall = 0.f;
    for (int d = lane; d < DP; d += 32) fall = fmaxf(fall, ref[d] - cs[(rb * 16 + 15) * CP + d]);
    const bool mild = srb_warp_max(fall) <= 100.f;
    if (lane == 0 && kind == 0) mild_s[rb] = mild;
    const int tiles = mild ? 2 * rb + 2 : 2 * rb;
    // the two warps of a row block take every second tile of eight columns, for the rows of K and of Q together
    float acc_k[4][4], acc_q[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc_k[i][e] = acc_q[i][e] = 0.f;
    const float k0 = beta_s[r0] * ik_s[r0], k1 = beta_s[r1] * ik_s[r1], q0 = iq_s[r0], q1 = iq_s[r1];
    if (kind < tiles) {
#pragma unroll 1
      for (int kk = 0; kk < DP / 16; ++kk) {
        unsigned kh[4], kl[4], qh[4], ql[4];
        float2 from[2];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int d = kk * 16 + 2 * t4 + 8 * half;
          from[half] = *reinterpret_cast<const float2*>(ref + d);
          const float2 c0 = *reinterpret_cast<const float2*>(cs + r0 * CP + d), c1 = *reinterpret_cast<const float2*>(cs + r1 * CP + d);
          const float2 e0 = make_float2(dc_exp2(c0.x - from[half].x), dc_exp2(c0.y - from[half].y));
          const float2 e1 = make_float2(dc_exp2(c1.x - from[half].x), dc_exp2(c1.y - from[half].y));
          float2 v = dc_pair(ks + r0 * XP + d);
          dc_split2(v.x * k0 * e0.x, v.y * k0 * e0.y, kh[2 * half], kl[2 * half]);
          v = dc_pair(ks + r1 * XP + d);
          dc_split2(v.x * k1 * e1.x, v.y * k1 * e1.y, kh[2 * half + 1], kl[2 * half + 1]);
          v = dc_pair(qs + r0 * XP + d);
          dc_split2(v.x * q0 * e0.x, v.y * q0 * e0.y, qh[2 * half], ql[2 * half]);
          v = dc_pair(qs + r1 * XP + d);
          dc_split2(v.x * q1 * e1.x, v.y * q1 * e1.y, qh[2 * half + 1], ql[2 * half + 1]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int nt = 2 * i + kind;
          if (nt < tiles) {
            const int j = nt * 8 + g;
            const float scale = ik_s[j];
            unsigned bh[2], bl[2];
#pragma unroll
            for (int half = 0; half < 2; ++half) {
              const int d = kk * 16 + 2 * t4 + 8 * half;
              const float2 v = dc_pair(ks + j * XP + d), c = *reinterpret_cast<const float2*>(cs + j * CP + d);
              dc_split2(v.x * scale * dc_exp2(from[half].x - c.x), v.y * scale * dc_exp2(from[half].y - c.y), bh[half], bl[half]);
            }
            mma_bf16(acc_k[i], kh, bh[0], bh[1]);
            mma_bf16(acc_q[i], qh, bh[0], bh[1]);
            mma_bf16(acc_k[i], kh, bl[0], bl[1]);
            mma_bf16(acc_q[i], qh, bl[0], bl[1]);
            mma_bf16(acc_k[i], kl, bh[0], bh[1]);
            mma_bf16(acc_q[i], ql, bh[0], bh[1]);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int nt = 2 * i + kind;
        if (nt < tiles) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int t = e < 2 ? r0 : r1, j = nt * 8 + 2 * t4 + (e & 1);
            ls[t * LP + j] = j < t ? acc_k[i][e] : 0.f;
            ts[t * LP + j] = j <= t ? acc_q[i][e] : 0.f;
          }
        }
      }
    }
    __syncthreads();
    // diagonal blocks in which some decay falls faster, pair by pair (t >= j): 136 pairs each
    for (int item = tid; item < 4 * 136; item += NTH) {
      const int block = item / 136, pair = item - block * 136;
      if (mild_s[block]) continue;
      int t = (int)((sqrtf(8.0f * pair + 1.0f) - 1.0f) * 0.5f);
      while ((t + 1) * (t + 2) / 2 <= pair) ++t;           // (the root may be off by one)
      while (t * (t + 1) / 2 > pair) --t;
      const int j = block * 16 + pair - t * (t + 1) / 2;
      t += block * 16;
      float kk = 0.f, qk = 0.f;
      for (int d = 0; d < DP; d += 2) {
        const float2 ct = *reinterpret_cast<const float2*>(cs + t * CP + d), cj = *reinterpret_cast<const float2*>(cs + j * CP + d);
        const float2 kj = dc_pair(ks + j * XP + d), kt = dc_pair(ks + t * XP + d), qt = dc_pair(qs + t * XP + d);
        const float e0 = kj.x * dc_exp2(ct.x - cj.x), e1 = kj.y * dc_exp2(ct.y - cj.y);
        kk = fmaf(kt.x, e0, fmaf(kt.y, e1, kk));
        qk = fmaf(qt.x, e0, fmaf(qt.y, e1, qk));
      }
      ls[t * LP + j] = j < t ? kk * beta_s[t] * ik_s[t] * ik_s[j] : 0.f;
      ts[t * LP + j] = qk * iq_s[t] * ik_s[j];
    }
  }
  __syncthreads();

  // ---- A leaves in two; so do the scaled q' and k' (CHANNEL) or their factors
  {
    __nv_bfloat16* ah = reinterpret_cast<__nv_bfloat16*>(place + P::A);
    __nv_bfloat16* al = ah + DC_TOKENS * DC_TOKENS;
    for (int i = tid; i < DC_TOKENS * DC_TOKENS / 2; i += NTH) {
      const int t = i / (DC_TOKENS / 2), j = i % (DC_TOKENS / 2) * 2;
      unsigned hi, lo;
      dc_split2(j <= t ? ts[t * LP + j] : 0.f, j + 1 <= t ? ts[t * LP + j + 1] : 0.f, hi, lo);
      *reinterpret_cast<unsigned*>(ah + t * DC_TOKENS + j) = hi;
      *reinterpret_cast<unsigned*>(al + t * DC_TOKENS + j) = lo;
    }
  }
  float* factors = reinterpret_cast<float*>(place + P::F);
  if (CHANNEL) {
    __nv_bfloat16* qh = reinterpret_cast<__nv_bfloat16*>(place + P::Q);
    __nv_bfloat16* kh = reinterpret_cast<__nv_bfloat16*>(place + P::K);
    const float* last = cs + (DC_TOKENS - 1) * CP;
    for (int i = tid; i < DC_TOKENS * DP / 2; i += NTH) {
      const int t = i / (DP / 2), d = i % (DP / 2) * 2;
      const float2 c = *reinterpret_cast<const float2*>(cs + t * CP + d), end = *reinterpret_cast<const float2*>(last + d);
      const float2 q = dc_pair(qs + t * XP + d), k = dc_pair(ks + t * XP + d);
      unsigned hi, lo;
      dc_split2(q.x * iq_s[t] * dc_exp2(c.x), q.y * iq_s[t] * dc_exp2(c.y), hi, lo);
      *reinterpret_cast<unsigned*>(qh + t * DP + d) = hi;
      *reinterpret_cast<unsigned*>(qh + DC_TOKENS * DP + t * DP + d) = lo;
      dc_split2(k.x * ik_s[t] * dc_exp2(end.x - c.x), k.y * ik_s[t] * dc_exp2(end.y - c.y), hi, lo);
      *reinterpret_cast<unsigned*>(kh + t * DP + d) = hi;
      *reinterpret_cast<unsigned*>(kh + DC_TOKENS * DP + t * DP + d) = lo;
    }
    for (int d = tid; d < DP; d += NTH) factors[d] = dc_exp2(last[d]);
  } else if (tid < DC_TOKENS) {
    factors[tid] = iq_s[tid] * dc_exp2(cum_s[tid]);
    factors[DC_TOKENS + tid] = ik_s[tid] * dc_exp2(cum_s[DC_TOKENS - 1] - cum_s[tid]);
    if (tid == 0) factors[2 * DC_TOKENS] = dc_exp2(cum_s[DC_TOKENS - 1]);
  }
  __syncthreads();

  // ---- T = (1 + L)^-1: two diagonal blocks of 32 by forward substitution (a lane takes a column), then the block below them,
  // T_10 = -T_11 L_10 T_00
  if (warp < 2) {
    const int b = warp * 32;
    float col[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      const float4* row = reinterpret_cast<const float4*>(ls + (b + i) * LP + b);
      float v[4] = {i == lane ? 1.f : 0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int m = 0; m < i; m += 4) {
        const float4 l = row[m / 4];
        v[0] = fmaf(-l.x, col[m], v[0]);
        if (m + 1 < i) v[1] = fmaf(-l.y, col[m + 1], v[1]);
        if (m + 2 < i) v[2] = fmaf(-l.z, col[m + 2], v[2]);
        if (m + 3 < i) v[3] = fmaf(-l.w, col[m + 3], v[3]);
      }
      col[i] = (v[0] + v[1]) + (v[2] + v[3]);
    }
#pragma unroll
    for (int i = 0; i < 32; ++i) ts[(b + i) * LP + b + lane] = col[i];
  }
  __syncthreads();
  {
    const int i = tid >> 3, j = (tid & 7) * 4;             // four entries of a row of a 32 x 32 block
    const float4* left[2] = {reinterpret_cast<const float4*>(ls + (32 + i) * LP), reinterpret_cast<const float4*>(ts + (32 + i) * LP + 32)};
    float* mine = ts + (32 + i) * LP + j;
#pragma unroll
    for (int pass = 0; pass < 2; ++pass) {                 // L_10 T_00, kept where the result goes; then -T_11 times that
      const float* right = ts + (pass ? 32 * LP : 0) + j;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int m = 0; m < 32; m += 4) {
        const float4 l = left[pass][m / 4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float4 r = *reinterpret_cast<const float4*>(right + (m + k) * LP);
          const float f = k == 0 ? l.x : (k == 1 ? l.y : (k == 2 ? l.z : l.w));
          v.x = fmaf(f, r.x, v.x); v.y = fmaf(f, r.y, v.y); v.z = fmaf(f, r.z, v.z); v.w = fmaf(f, r.w, v.w);
        }
      }
      if (pass) {
        __syncthreads();                                   // every thread has read the product before
        v = make_float4(-v.x, -v.y, -v.z, -v.w);
      }
      *reinterpret_cast<float4*>(mine) = v;
      __syncthreads();
    }
  }
  // ---- T with its columns scaled, in two: times beta (for V), and without channels times beta |k|^-1 e^c (for K as it lies)
  __nv_bfloat16* th = qs;                                  // [64][TP], then the rest
  __nv_bfloat16* tl = th + DC_TOKENS * TP;
  for (int i = tid; i < DC_TOKENS * DC_TOKENS / 2; i += NTH) {
    const int t = i / (DC_TOKENS / 2), j = i % (DC_TOKENS / 2) * 2;
    unsigned hi, lo;
    dc_split2(j <= t ? ts[t * LP + j] * beta_s[j] : 0.f, j + 1 <= t ? ts[t * LP + j + 1] * beta_s[j + 1] : 0.f, hi, lo);
    *reinterpret_cast<unsigned*>(th + t * TP + j) = hi;
    *reinterpret_cast<unsigned*>(tl + t * TP + j) = lo;
  }
  __syncthreads();
  __nv_bfloat16* second = reinterpret_cast<__nv_bfloat16*>(dp_smem + M::LT);
  if (CHANNEL) {
    // k' e^c in two, over L and T
    for (int i = tid; i < DC_TOKENS * DP / 2; i += NTH) {
      const int t = i / (DP / 2), d = i % (DP / 2) * 2;
      const float2 c = *reinterpret_cast<const float2*>(cs + t * CP + d), k = dc_pair(ks + t * XP + d);
      unsigned hi, lo;
      dc_split2(k.x * ik_s[t] * dc_exp2(c.x), k.y * ik_s[t] * dc_exp2(c.y), hi, lo);
      *reinterpret_cast<unsigned*>(second + t * XP + d) = hi;
      *reinterpret_cast<unsigned*>(second + DC_TOKENS * XP + t * XP + d) = lo;
    }
  } else {
    // T once more, its columns scaled for K (from the scaled copy: T itself lies where this goes)
    for (int i = tid; i < DC_TOKENS * DC_TOKENS / 2; i += NTH) {
      const int t = i / (DC_TOKENS / 2), j = i % (DC_TOKENS / 2) * 2;
      const float2 h = dc_pair(th + t * TP + j), l = dc_pair(tl + t * TP + j);
      unsigned hi, lo;
      dc_split2((h.x + l.x) * ik_s[j] * dc_exp2(cum_s[j]), (h.y + l.y) * ik_s[j + 1] * dc_exp2(cum_s[j + 1]), hi, lo);
      *reinterpret_cast<unsigned*>(second + t * TP + j) = hi;
      *reinterpret_cast<unsigned*>(second + DC_TOKENS * TP + t * TP + j) = lo;
    }
  }
  __syncthreads();
  // ---- v over c
  const int VP = vp + DC_PAD;
  __nv_bfloat16* vs = reinterpret_cast<__nv_bfloat16*>(cs);
  for (int i = tid; i < DC_TOKENS * vp / 8; i += NTH) {
    const int t = i / (vp / 8), c = i % (vp / 8) * 8;
    const bool live = t < n && c < vdim;
    cp_async_16(vs + t * VP + c, x + (size_t)(live ? t : 0) * a.channels + 2 * a.kv_heads * dim + head * vdim + (live ? c : 0), live ? 16 : 0);
  }
  cp_async_commit();

  // ---- -W [64][DP]: warps take 16 tokens and half of the columns
  {
    constexpr int NT = DP / 16;
    float acc[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
    const __nv_bfloat16* lh = CHANNEL ? th : second;
    const __nv_bfloat16* ll = CHANNEL ? tl : second + DC_TOKENS * TP;
    const int matrix = lane >> 3, inner = lane & 7;
#pragma unroll
    for (int kk = 0; kk < DC_TOKENS / 16; ++kk) {
      if (kk > rb) break;                                  // T is zero above the diagonal
      unsigned hi[4], lo[4];
      const int at = (rb * 16 + (matrix & 1) * 8 + inner) * TP + kk * 16 + (matrix >> 1) * 8;
      ldmatrix_x4(hi[0], hi[1], hi[2], hi[3], lh + at);
      ldmatrix_x4(lo[0], lo[1], lo[2], lo[3], ll + at);
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) {
        const int d = kind * (DP / 2) + nt * 8;
        if (CHANNEL) {
          unsigned b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, second + (matrix >> 1) * DC_TOKENS * XP + (kk * 16 + (matrix & 1) * 8 + inner) * XP + d);
          mma_bf16(acc[nt], hi, b0, b1);
          mma_bf16(acc[nt], hi, b2, b3);
          mma_bf16(acc[nt], lo, b0, b1);
        } else {
          if (nt & 1) continue;                            // two tiles of eight columns at a time
          unsigned b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, ks + (kk * 16 + (matrix & 1) * 8 + inner) * XP + d + (matrix >> 1) * 8);
          mma_bf16(acc[nt], hi, b0, b1);
          mma_bf16(acc[nt], lo, b0, b1);
          mma_bf16(acc[nt + 1], hi, b2, b3);
          mma_bf16(acc[nt + 1], lo, b2, b3);
        }
      }
    }
    __nv_bfloat16* wh = reinterpret_cast<__nv_bfloat16*>(place + P::W);
    __nv_bfloat16* wl = wh + DC_TOKENS * DP;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int d = kind * (DP / 2) + nt * 8 + 2 * t4;
      unsigned hi, lo;
      dc_split2(-acc[nt][0], -acc[nt][1], hi, lo);
      *reinterpret_cast<unsigned*>(wh + r0 * DP + d) = hi;
      *reinterpret_cast<unsigned*>(wl + r0 * DP + d) = lo;
      dc_split2(-acc[nt][2], -acc[nt][3], hi, lo);
      *reinterpret_cast<unsigned*>(wh + r1 * DP + d) = hi;
      *reinterpret_cast<unsigned*>(wl + r1 * DP + d) = lo;
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  // ---- (T beta V)^T [vp][64]: a warp takes 16 value columns at a time; the left operand is V read across its rows
  {
    float* vt = reinterpret_cast<float*>(place + P::V);
    const int matrix = lane >> 3, inner = lane & 7;
    for (int c0 = warp * 16; c0 < vp; c0 += 8 * 16) {
      float acc[8][4];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DC_TOKENS / 16; ++kk) {
        unsigned va[4];                                    // rows: value columns, inner index: tokens
        ldmatrix_x4_trans(va[0], va[1], va[2], va[3], vs + (kk * 16 + (matrix >> 1) * 8 + inner) * VP + c0 + (matrix & 1) * 8);
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          if (nt < 2 * kk) continue;                       // tokens before these give nothing
          unsigned b0, b1, b2, b3;
          ldmatrix_x4(b0, b1, b2, b3, th + (matrix >> 1) * DC_TOKENS * TP + (nt * 8 + inner) * TP + kk * 16 + (matrix & 1) * 8);
          mma_bf16(acc[nt], va, b0, b1);
          mma_bf16(acc[nt], va, b2, b3);
        }
      }
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        *reinterpret_cast<float2*>(vt + (c0 + g) * DC_TOKENS + nt * 8 + 2 * t4) = make_float2(acc[nt][0], acc[nt][1]);
        *reinterpret_cast<float2*>(vt + (c0 + g + 8) * DC_TOKENS + nt * 8 + 2 * t4) = make_float2(acc[nt][2], acc[nt][3]);
      }
    }
  }
}

// MT: tiles of 16 value columns per block; four warps per tile share the tokens (U, results) and the rows of S (next S).
template <int DP, bool CHANNEL, int MT>
struct DeltaWalkSmem {
  static constexpr int XP = DP + DC_PAD, TP = DC_TOKENS + DC_PAD, VS = 16 * MT, QK = CHANNEL ? 2 : 1;
  static constexpr int ROWS = DC_TOKENS * XP * 2;
  static constexpr int W = 0, Q = W + 2 * ROWS, K = Q + QK * ROWS, A = K + QK * ROWS, A_HALF = DC_TOKENS * TP * 2;
  static constexpr int S = A + 2 * A_HALF, S_HALF = VS * XP * 2;
  static constexpr int U = S + 2 * S_HALF, U_HALF = VS * TP * 2;           // U in two; without channels also U times k's factors
  static constexpr int F = U + (CHANNEL ? 2 : 4) * U_HALF;
  static constexpr int BYTES = F + (CHANNEL ? DP : 2 * DC_TOKENS + 4) * 4;
};

template <int DP, bool CHANNEL, int MT>
__global__ void __launch_bounds__(128 * MT) delta_chunk_walk_kernel(DeltaArgs a, const unsigned char* scratch, int vp) {
  using M = DeltaWalkSmem<DP, CHANNEL, MT>;
  using P = DeltaChunkLayout<DP, CHANNEL>;
  constexpr int XP = M::XP, TP = M::TP, NTH = 128 * MT, DT = DP / 32;      // DT: tiles of eight rows of S that a warp owns
  extern __shared__ __align__(16) unsigned char dw_smem[];
  __nv_bfloat16* ws = reinterpret_cast<__nv_bfloat16*>(dw_smem + M::W);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(dw_smem + M::Q);
  __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(dw_smem + M::K);
  __nv_bfloat16* as = reinterpret_cast<__nv_bfloat16*>(dw_smem + M::A);
  __nv_bfloat16* ss = reinterpret_cast<__nv_bfloat16*>(dw_smem + M::S);
  __nv_bfloat16* us = reinterpret_cast<__nv_bfloat16*>(dw_smem + M::U);
  float* fs = reinterpret_cast<float*>(dw_smem + M::F);
  srb_launch_dependents();
  srb_grid_dependency_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int tile = warp >> 2, part = warp & 3, matrix = lane >> 3, inner = lane & 7;
  const int head = blockIdx.y, request = blockIdx.z, dim = a.dim, vdim = a.vdim;
  const int begin = a.cu_rows[request], rows = a.cu_rows[request + 1] - begin;
  if (rows <= 0) return;
  const int start = a.positions[begin];
  if (start < 0) return;
  int first = 0;
  for (int r = 0; r < request; ++r) first += (a.cu_rows[r + 1] - a.cu_rows[r] + DC_TOKENS - 1) / DC_TOKENS;
  const int chunks = (rows + DC_TOKENS - 1) / DC_TOKENS;
  const int c_tile = blockIdx.x * M::VS + tile * 16;                       // the warp's value columns: c_tile + g, c_tile + g + 8
  const int c_lo = c_tile + g, c_hi = c_lo + 8;
  const int qk_head = head / (a.heads / a.kv_heads);
  const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(a.x);
  float* state = a.state + (size_t)a.state_slots[request] * a.slot_floats + a.conv_floats + (size_t)head * vdim * dim;

  // the warp's part of S^T: columns c_lo, c_hi, rows d = part * DP / 4 + nt * 8 + 2 t4, + 1
  float s[DT][4];
#pragma unroll
  for (int nt = 0; nt < DT; ++nt) {
    const int d = part * (DP / 4) + nt * 8 + 2 * t4;
    s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
    if (start > 0 && d < dim) {                            // (dim is even)
      if (c_lo < vdim) { const float2 v = *reinterpret_cast<const float2*>(state + (size_t)c_lo * dim + d); s[nt][0] = v.x; s[nt][1] = v.y; }
      if (c_hi < vdim) { const float2 v = *reinterpret_cast<const float2*>(state + (size_t)c_hi * dim + d); s[nt][2] = v.x; s[nt][3] = v.y; }
    }
  }
  auto place_of = [&](int chunk) { return scratch + ((size_t)(first + chunk) * a.heads + head) * P::bytes(vp); };
  auto keep_state = [&]() {
#pragma unroll
    for (int nt = 0; nt < DT; ++nt) {
      const int d = part * (DP / 4) + nt * 8 + 2 * t4;
      unsigned hi, lo;
      dc_split2(s[nt][0], s[nt][1], hi, lo);
      __nv_bfloat16* at = ss + (tile * 16 + g) * XP + d;
      *reinterpret_cast<unsigned*>(at) = hi;
      *reinterpret_cast<unsigned*>(at + M::S_HALF / 2) = lo;
      dc_split2(s[nt][2], s[nt][3], hi, lo);
      *reinterpret_cast<unsigned*>(at + 8 * XP) = hi;
      *reinterpret_cast<unsigned*>(at + 8 * XP + M::S_HALF / 2) = lo;
    }
  };
  auto fetch_rows = [&](__nv_bfloat16* to, const unsigned char* from, int halves) {      // operands in two: [halves * 64][DP]
    for (int i = tid; i < halves * DC_TOKENS * DP / 8; i += NTH) {
      const int t = i / (DP / 8), d = i % (DP / 8) * 8;
      cp_async_16(to + t * XP + d, from + (size_t)i * 16, 16);
    }
  };
  auto fetch_x = [&](__nv_bfloat16* to, int column, int chunk) {                         // q or k as they lie
    for (int i = tid; i < DC_TOKENS * DP / 8; i += NTH) {
      const int t = i / (DP / 8), d = i % (DP / 8) * 8;
      const bool live = chunk * DC_TOKENS + t < rows && d < dim;
      cp_async_16(to + t * XP + d, x + (size_t)(begin + (live ? chunk * DC_TOKENS + t : 0)) * a.channels + column + (live ? d : 0), live ? 16 : 0);
    }
  };
  auto fetch_wq = [&](int chunk) {
    const unsigned char* place = place_of(chunk);
    fetch_rows(ws, place + P::W, 2);
    if (CHANNEL) fetch_rows(qs, place + P::Q, 2); else fetch_x(qs, qk_head * dim, chunk);
    cp_async_commit();
  };
  auto fetch_ak = [&](int chunk) {
    const unsigned char* place = place_of(chunk);
    for (int i = tid; i < 2 * DC_TOKENS * DC_TOKENS / 8; i += NTH) {
      const int t = i / (DC_TOKENS / 8), j = i % (DC_TOKENS / 8) * 8;
      cp_async_16(as + t * TP + j, place + P::A + (size_t)i * 16, 16);
    }
    if (CHANNEL) fetch_rows(ks, place + P::K, 2); else fetch_x(ks, (a.kv_heads + qk_head) * dim, chunk);
    for (int i = tid; i < P::FLOATS / 4; i += NTH) cp_async_16(fs + i * 4, place + P::F + (size_t)i * 16, 16);
    cp_async_commit();
  };
  float uv[2][4];                                          // the warp's 16 tokens of T beta V, for the chunk to come
  auto fetch_v = [&](int chunk) {
    const float* vt = reinterpret_cast<const float*>(place_of(chunk) + P::V);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int t = part * 16 + nt * 8 + 2 * t4;
      float2 lo = make_float2(0.f, 0.f), hi = lo;
      if (c_lo < vp) lo = *reinterpret_cast<const float2*>(vt + (size_t)c_lo * DC_TOKENS + t);
      if (c_hi < vp) hi = *reinterpret_cast<const float2*>(vt + (size_t)c_hi * DC_TOKENS + t);
      uv[nt][0] = lo.x; uv[nt][1] = lo.y; uv[nt][2] = hi.x; uv[nt][3] = hi.y;
    }
  };
  fetch_wq(0);
  fetch_v(0);
  keep_state();
  for (int chunk = 0; chunk < chunks; ++chunk) {
    cp_async_wait<0>();
    __syncthreads();                                       // W, q and the state are there; A, k and U are no longer read
    fetch_ak(chunk);
    // U = T beta V - W S and (q e^c) S for the warp's 16 tokens; the products of the roundings and of the rests go into sums of
    // their own, so that consecutive products do not wait for each other
    float u[2][4], o[2][4], u_rest[2][2][4], o_rest[2][2][4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        u[nt][e] = uv[nt][e];
        o[nt][e] = u_rest[0][nt][e] = u_rest[1][nt][e] = o_rest[0][nt][e] = o_rest[1][nt][e] = 0.f;
      }
#pragma unroll 4
    for (int kk = 0; kk < DP / 16; ++kk) {
      unsigned sh[4], sl[4], w[2][4], q[2][4];
      const __nv_bfloat16* at = ss + (tile * 16 + (matrix & 1) * 8 + inner) * XP + kk * 16 + (matrix >> 1) * 8;
      ldmatrix_x4(sh[0], sh[1], sh[2], sh[3], at);
      ldmatrix_x4(sl[0], sl[1], sl[2], sl[3], at + M::S_HALF / 2);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        const int row = part * 16 + nt * 8 + inner, column = kk * 16 + (matrix & 1) * 8;
        ldmatrix_x4(w[nt][0], w[nt][1], w[nt][2], w[nt][3], ws + (matrix >> 1) * DC_TOKENS * XP + row * XP + column);
        if (CHANNEL) ldmatrix_x4(q[nt][0], q[nt][1], q[nt][2], q[nt][3], qs + (matrix >> 1) * DC_TOKENS * XP + row * XP + column);
      }
      if (!CHANNEL)                                        // both tiles of eight tokens at once
        ldmatrix_x4(q[0][0], q[0][1], q[1][0], q[1][1], qs + (part * 16 + (matrix >> 1) * 8 + inner) * XP + kk * 16 + (matrix & 1) * 8);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) mma_bf16(u[nt], sh, w[nt][0], w[nt][1]);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) mma_bf16(o[nt], sh, q[nt][0], q[nt][1]);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) mma_bf16(u_rest[0][nt], sh, w[nt][2], w[nt][3]);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) mma_bf16(u_rest[1][nt], sl, w[nt][0], w[nt][1]);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) mma_bf16(o_rest[1][nt], sl, q[nt][0], q[nt][1]);
      if (CHANNEL) {
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) mma_bf16(o_rest[0][nt], sh, q[nt][2], q[nt][3]);
      }
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        u[nt][e] += u_rest[0][nt][e] + u_rest[1][nt][e];
        o[nt][e] += o_rest[0][nt][e] + o_rest[1][nt][e];
        o_rest[0][nt][e] = o_rest[1][nt][e] = 0.f;
      }
    cp_async_wait<0>();                                    // A, k and the factors (each thread its own copies; the barrier below joins them)
    if (!CHANNEL) __syncthreads();                         // the factors are read below by every thread
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int t = part * 16 + nt * 8 + 2 * t4;
      unsigned hi, lo;
      __nv_bfloat16* at = us + (tile * 16 + g) * TP + t;
      dc_split2(u[nt][0], u[nt][1], hi, lo);
      *reinterpret_cast<unsigned*>(at) = hi;
      *reinterpret_cast<unsigned*>(at + M::U_HALF / 2) = lo;
      dc_split2(u[nt][2], u[nt][3], hi, lo);
      *reinterpret_cast<unsigned*>(at + 8 * TP) = hi;
      *reinterpret_cast<unsigned*>(at + 8 * TP + M::U_HALF / 2) = lo;
      if (!CHANNEL) {
        const float k0 = fs[DC_TOKENS + t], k1 = fs[DC_TOKENS + t + 1];
        at += M::U_HALF;                                   // U times k's factors, behind the two halves of U
        dc_split2(u[nt][0] * k0, u[nt][1] * k1, hi, lo);
        *reinterpret_cast<unsigned*>(at) = hi;
        *reinterpret_cast<unsigned*>(at + M::U_HALF / 2) = lo;
        dc_split2(u[nt][2] * k0, u[nt][3] * k1, hi, lo);
        *reinterpret_cast<unsigned*>(at + 8 * TP) = hi;
        *reinterpret_cast<unsigned*>(at + 8 * TP + M::U_HALF / 2) = lo;
        const float q0 = fs[t], q1 = fs[t + 1];
        o[nt][0] *= q0; o[nt][1] *= q1; o[nt][2] *= q0; o[nt][3] *= q1;
      }
    }
    __syncthreads();                                       // U, A, k are there; W, q and the state before are no longer read
    if (chunk + 1 < chunks) {
      fetch_wq(chunk + 1);
      fetch_v(chunk + 1);
    }
    // the next S: the decay, then U^T k over the chunk's tokens
    const float whole = CHANNEL ? 1.f : fs[2 * DC_TOKENS];
#pragma unroll
    for (int nt = 0; nt < DT; ++nt) {
      float e0 = whole, e1 = whole;
      if (CHANNEL) { const int d = part * (DP / 4) + nt * 8 + 2 * t4; e0 = fs[d]; e1 = fs[d + 1]; }
      s[nt][0] *= e0; s[nt][1] *= e1; s[nt][2] *= e0; s[nt][3] *= e1;
    }
#pragma unroll
    for (int kk = 0; kk < DC_TOKENS / 16; ++kk) {
      const __nv_bfloat16* at = us + (tile * 16 + (matrix & 1) * 8 + inner) * TP + kk * 16 + (matrix >> 1) * 8;
      unsigned uh[4], ul[4], k[DT][4];
      ldmatrix_x4(uh[0], uh[1], uh[2], uh[3], at);
      ldmatrix_x4(ul[0], ul[1], ul[2], ul[3], at + M::U_HALF / 2);
      if (CHANNEL) {
#pragma unroll
        for (int nt = 0; nt < DT; ++nt)
          ldmatrix_x4_trans(k[nt][0], k[nt][1], k[nt][2], k[nt][3], ks + (matrix >> 1) * DC_TOKENS * XP +
                            (kk * 16 + (matrix & 1) * 8 + inner) * XP + part * (DP / 4) + nt * 8);
      } else {
#pragma unroll
        for (int nt = 0; nt < DT; nt += 2)                 // two tiles of eight rows of S at once
          ldmatrix_x4_trans(k[nt][0], k[nt][1], k[nt + 1][0], k[nt + 1][1], ks + (kk * 16 + (matrix & 1) * 8 + inner) * XP +
                            part * (DP / 4) + nt * 8 + (matrix >> 1) * 8);
      }
      if (kk <= part) {                                    // A is zero above the diagonal
        unsigned b[2][4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
          ldmatrix_x4(b[nt][0], b[nt][1], b[nt][2], b[nt][3], as + (matrix >> 1) * DC_TOKENS * TP +
                      (part * 16 + nt * 8 + inner) * TP + kk * 16 + (matrix & 1) * 8);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) mma_bf16(o[nt], uh, b[nt][0], b[nt][1]);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) mma_bf16(o_rest[0][nt], uh, b[nt][2], b[nt][3]);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) mma_bf16(o_rest[1][nt], ul, b[nt][0], b[nt][1]);
      }
      if (!CHANNEL) {
        ldmatrix_x4(uh[0], uh[1], uh[2], uh[3], at + M::U_HALF);
        ldmatrix_x4(ul[0], ul[1], ul[2], ul[3], at + M::U_HALF + M::U_HALF / 2);
      }
#pragma unroll
      for (int nt = 0; nt < DT; ++nt) mma_bf16(s[nt], uh, k[nt][0], k[nt][1]);
      if (CHANNEL) {
#pragma unroll
        for (int nt = 0; nt < DT; ++nt) mma_bf16(s[nt], uh, k[nt][2], k[nt][3]);
      }
#pragma unroll
      for (int nt = 0; nt < DT; ++nt) mma_bf16(s[nt], ul, k[nt][0], k[nt][1]);
    }
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[nt][e] += o_rest[0][nt][e] + o_rest[1][nt][e];
    if (chunk + 1 < chunks) keep_state();
    const int left = rows - chunk * DC_TOKENS;
    float* out = a.out + (size_t)(begin + chunk * DC_TOKENS) * a.heads * vdim + (size_t)head * vdim;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int t = part * 16 + nt * 8 + 2 * t4;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int token = t + (e & 1), c = e < 2 ? c_lo : c_hi;
        if (token < left && c < vdim) out[(size_t)token * a.heads * vdim + c] = o[nt][e];
      }
    }
  }
  if (!a.write_state) return;
#pragma unroll
  for (int nt = 0; nt < DT; ++nt) {
    const int d = part * (DP / 4) + nt * 8 + 2 * t4;
    if (d >= dim) continue;
    if (c_lo < vdim) *reinterpret_cast<float2*>(state + (size_t)c_lo * dim + d) = make_float2(s[nt][0], s[nt][1]);
    if (c_hi < vdim) *reinterpret_cast<float2*>(state + (size_t)c_hi * dim + d) = make_float2(s[nt][2], s[nt][3]);
  }
}

static int delta_padded_columns(int vdim) { return (vdim + 15) / 16 * 16; }

template <int DP, bool CHANNEL>
static int launch_delta_chunks(const DeltaArgs& a, unsigned char* scratch, int chunks, cudaStream_t s) {
  const int vp = delta_padded_columns(a.vdim);
  const int smem1 = DeltaPrepareSmem<DP, CHANNEL>::bytes(vp);
  if (smem1 > 227 * 1024) SRB_FAIL("delta_chunks: %d bytes of shared memory exceed 232448", smem1);
  SRB_CUDA_CALL(cudaFuncSetAttribute(delta_chunk_prepare_kernel<DP, CHANNEL>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem1));
  SRB_CUDA_CALL(srb_launch(delta_chunk_prepare_kernel<DP, CHANNEL>, dim3(chunks, a.heads), dim3(DC_PREPARE_THREADS), smem1, s, a, scratch, vp));
  SRB_LAUNCH_CHECK("delta_chunk_prepare");
  // two tiles of value columns per block share the fetched operands; with a decay per row of S (more to fetch and to multiply per
  // column) one tile per block is quicker while that fills no more SMs than there are
  const int mt = (vp % 32 != 0 || (CHANNEL && (long long)vp / 16 * a.heads * a.requests <= srb_sm_count())) ? 1 : 2;
  if (mt == 2) {
    const int smem2 = DeltaWalkSmem<DP, CHANNEL, 2>::BYTES;
    SRB_CUDA_CALL(cudaFuncSetAttribute(delta_chunk_walk_kernel<DP, CHANNEL, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem2));
    SRB_CUDA_CALL(srb_launch(delta_chunk_walk_kernel<DP, CHANNEL, 2>, dim3(vp / 32, a.heads, a.requests), dim3(256), smem2, s, a,
                             (const unsigned char*)scratch, vp));
  } else {
    const int smem2 = DeltaWalkSmem<DP, CHANNEL, 1>::BYTES;
    SRB_CUDA_CALL(cudaFuncSetAttribute(delta_chunk_walk_kernel<DP, CHANNEL, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem2));
    SRB_CUDA_CALL(srb_launch(delta_chunk_walk_kernel<DP, CHANNEL, 1>, dim3(vp / 16, a.heads, a.requests), dim3(128), smem2, s, a,
                             (const unsigned char*)scratch, vp));
  }
  SRB_LAUNCH_CHECK("delta_chunk_walk");
  return SRB_OK;
}

// Tokens of a chunk, whether these sizes are taken, and the scratch a chunk needs per head.
extern "C" int srb_delta_chunk_tokens() { return DC_TOKENS; }
extern "C" int srb_delta_chunks_supports(int dim, int vdim, int dtype) {
  return dtype == SRB_DTYPE_BF16 && dim >= 8 && dim <= 128 && dim % 8 == 0 && vdim >= 8 && vdim <= 256 && vdim % 8 == 0;
}
extern "C" long long srb_delta_chunk_bytes(int dim, int vdim, int channel_decay) {
  const int vp = delta_padded_columns(vdim);
  if (dim <= 64) return channel_decay ? DeltaChunkLayout<64, true>::bytes(vp) : DeltaChunkLayout<64, false>::bytes(vp);
  return channel_decay ? DeltaChunkLayout<128, true>::bytes(vp) : DeltaChunkLayout<128, false>::bytes(vp);
}

// What srb_delta_scan computes, for prompt portions in bfloat16.  x: bfloat16 [rows, channels] (srb_short_conv with a bfloat16
// result); `chunks`: at least the number of chunks of the step, sum over the requests of ceil(rows / srb_delta_chunk_tokens());
// `scratch`: chunks * heads * srb_delta_chunk_bytes() bytes on a 16-byte border.
extern "C" int srb_delta_chunks(const void* x, const void* beta, long long beta_pitch, const void* decay, long long decay_pitch,
                                const float* a_log, const float* dt_bias, const int* positions, const int* cu_rows,
                                const int* state_slots, float* state, long long slot_floats, void* scratch, float* out, int rows,
                                int requests, int chunks, int heads, int kv_heads, int dim, int vdim, int taps, int channel_decay,
                                float unit_eps, int write_state, void* stream) {
  if (rows <= 0 || requests <= 0 || chunks <= 0) return SRB_OK;
  if (!srb_delta_chunks_supports(dim, vdim, SRB_DTYPE_BF16)) SRB_FAIL("delta_chunks: heads of %d x %d entries are not taken", dim, vdim);
  if (heads > 65535) SRB_FAIL("delta_chunks: %d heads exceed one launch", heads);
  DeltaArgs a;
  if (delta_args(a, x, beta, beta_pitch, decay, decay_pitch, a_log, dt_bias, positions, cu_rows, state_slots, state, slot_floats, out,
                 requests, heads, kv_heads, dim, vdim, taps, channel_decay, unit_eps, write_state) != SRB_OK)
    return SRB_ERR_INVALID;
  if (((uintptr_t)x & 15) || ((uintptr_t)scratch & 15)) SRB_FAIL("delta_chunks: the convolved inputs and the scratch must start on 16-byte borders");
  cudaStream_t s = (cudaStream_t)stream;
  if (dim <= 64)
    return channel_decay ? launch_delta_chunks<64, true>(a, (unsigned char*)scratch, chunks, s) : launch_delta_chunks<64, false>(a, (unsigned char*)scratch, chunks, s);
  return channel_decay ? launch_delta_chunks<128, true>(a, (unsigned char*)scratch, chunks, s) : launch_delta_chunks<128, false>(a, (unsigned char*)scratch, chunks, s);
}
