// The gated delta rule with a decay per key channel, behind short causal convolutions, for prompts, portions of prompts and
// single decoded tokens alike.
//
// (1) delta_prepare.  A row of the input product holds q | k | v | beta | bottlenecks, float32.  Every channel of q, k and v
// passes a causal convolution over its request's tokens (zeros before the start; the taps - 1 inputs before a portion come
// from the request's state slot, which then takes the portion's last ones) and silu; q and k heads become unit vectors,
// x / sqrt(sum x^2 + unit_eps), q also times dim^(-1/2); beta passes a sigmoid; the bottlenecks are copied in the products'
// dtype.  A warp does a few neighbouring tokens of one head.  The warp of a request's first token of the step also does the
// other tokens that read the slot, and writes the slot when it has: the only reader and the only writer of a slot's
// channels in a step are that one warp.
//
// (2) delta_rule.  Per request and head a float32 state S [dim][vdim] lives in the request's slot.  For each token, in order,
// with a decay g[i] per row:
//     S[i][c] = g[i] S[i][c];  u[c] = beta (v[c] - sum_i S[i][c] k[i]);  S[i][c] += k[i] u[c];  o[c] = sum_i S[i][c] q[i]
// g = exp(-rate_h softplus(raw + bias)).  Then out[c] = o[c] / sqrt(mean_c(o^2) + eps) * norm_w[c] * sigmoid(gate[c]).
//
// Short portions walk the tokens: a block per (request, head), the rows of a column over RS neighbouring threads with RPT
// entries each in registers.
//
// Long portions are cut into chunks of DR_C tokens.  With L_t the running sums of log g inside a chunk and S the state before
// it, the u_t of a chunk solve a triangular system:
//     u_t + sum_(s<t) A[t][s] u_s = beta_t (v_t - (exp(L_t) k_t)^T S),   A[t][s] = beta_t sum_d k_t k_s exp(L_t - L_s)
// so with T = (I + A)^-1 diag(beta), W = T (exp(L) k) and U = T V they are u = U - W S, and
//     o_t = (exp(L_t) q_t)^T S + sum_(s<=t) P[t][s] u_s,   P[t][s] = sum_d q_t k_s exp(L_t - L_s)
//     S'  = exp(L_C) S + sum_s (exp(L_C - L_s) k_s) u_s^T.
// Every exponent is a sum of logarithms of decays, at most 0: nothing overflows however fast the decays are.  Launch A forms
// W, U, P and the scaled q and k of every chunk and head side by side; launch B walks each request's chunks, a block per
// (request, head, slab of columns), the state in registers and the next chunk's operands on their way by asynchronous
// copies; a third launch finishes the heads.  The result differs from the token walk by rounding only.
#include "common.cuh"
#include <math.h>

constexpr int DR_C = 16;            // tokens of a chunk
constexpr int DR_GROUP = 16;        // tokens that the walk stages at a time
constexpr int DR_TOK = 8;           // neighbouring tokens that a warp of delta_prepare does in a large step (one in a small one)
constexpr float DR_LOG2E = 1.4426950408889634f;
// A decay is at least 2^-32: what is left of the state is then below the rounding of anything that is added to it, and the
// running sums of logarithms stay short enough for their differences to be exact to float32.
constexpr float DR_LOG2_MIN = -32.f;

// ------------------------------------------------------------------------------------------ (1) delta_prepare
struct DeltaPrepareArgs {
  const float* proj; long long ld;
  const float* taps_w;               // [channels][taps]
  int taps;
  float unit_eps, q_scale;
  float* state;                      // [slots][max(taps - 1, 1)][channels]
  const int *state_slots, *cu_q, *seq_lens, *req_index;
  float* qkv;                        // [tokens][channels]
  float* beta;                       // [tokens][heads]
  void* low; int low_dtype, low_width, low_cols;
  int tokens, kv_heads, heads, dim, vdim, channels, tok;
};

// The conv output (before silu) of channel c for token t, the i-th of its request's tokens of this step.
__device__ __forceinline__ float dp_conv(const DeltaPrepareArgs& a, int t, int i, int c, const float* slot) {
  const float* w = a.taps_w + (size_t)c * a.taps;
  float y = 0.f;
  for (int j = 0; j < a.taps; ++j) {
    const int s = i - a.taps + 1 + j;
    const float x = s >= 0 ? a.proj[(size_t)(t - (a.taps - 1 - j)) * a.ld + c] : slot[(size_t)(a.taps - 1 + s) * a.channels + c];
    y = fmaf(w[j], x, y);
  }
  return y;
}

__device__ __forceinline__ void dp_token(const DeltaPrepareArgs& a, int t, int i, int c0, int width, bool unit, float gain,
                                         const float* slot, int lane) {
  float* dst = a.qkv + (size_t)t * a.channels + c0;
  if (width <= 256) {
    float y[8];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int e = j * 32 + lane;
      y[j] = 0.f;
      if (e < width) {
        const float v = dp_conv(a, t, i, c0 + e, slot);
        y[j] = v / (1.f + expf(-v));
        ss = fmaf(y[j], y[j], ss);
      }
    }
    const float f = unit ? gain / sqrtf(warp_sum(ss) + a.unit_eps) : 1.f;
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (j * 32 + lane < width) dst[j * 32 + lane] = y[j] * f;
    return;
  }
  float ss = 0.f;
  for (int e = lane; e < width; e += 32) {
    const float v = dp_conv(a, t, i, c0 + e, slot);
    const float y = v / (1.f + expf(-v));
    dst[e] = y;
    ss = fmaf(y, y, ss);
  }
  if (!unit) return;
  const float f = gain / sqrtf(warp_sum(ss) + a.unit_eps);
  for (int e = lane; e < width; e += 32) dst[e] *= f;               // each lane its own elements
}

// The slot's inputs of `width` channels from c0 on after a portion of len tokens that starts at row t.
__device__ __forceinline__ void dp_keep(const DeltaPrepareArgs& a, float* slot, int t, int len, int c0, int width, int lane) {
  const int past = a.taps - 1;
  for (int e = lane; e < width; e += 32) {               // rows in ascending order: a row reads a later one or the portion
    const int c = c0 + e;
    for (int p = 0; p < past; ++p)
      slot[(size_t)p * a.channels + c] = len + p < past ? slot[(size_t)(len + p) * a.channels + c]
                                                        : a.proj[(size_t)(t + len + p - past) * a.ld + c];
  }
}

template <typename T>
__device__ __forceinline__ void dp_rest(const DeltaPrepareArgs& a, int t, int lane) {       // beta and the bottlenecks
  const float* row = a.proj + (size_t)t * a.ld + a.channels;
  for (int e = lane; e < a.heads; e += 32) a.beta[(size_t)t * a.heads + e] = 1.f / (1.f + expf(-row[e]));
  T* dst = (T*)a.low + (size_t)t * a.low_cols;
  for (int e = lane; e < a.low_cols; e += 32) dst[e] = from_f32<T>(e < a.low_width ? row[a.heads + e] : 0.f);
}

template <typename T>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(DeltaPrepareArgs a) {
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int G = a.kv_heads, units = 2 * G + a.heads;
  if (unit > units) return;
  const int ta = blockIdx.y * a.tok, tb = min(ta + a.tok, a.tokens);
  if (unit == units) {
    for (int t = ta; t < tb; ++t) dp_rest<T>(a, t, lane);
    return;
  }
  const bool is_v = unit >= 2 * G;
  const int width = is_v ? a.vdim : a.dim;
  const int c0 = is_v ? 2 * G * a.dim + (unit - 2 * G) * a.vdim : unit * a.dim;
  const float gain = unit < G ? a.q_scale : 1.f;
  const int past = a.taps - 1;
  for (int t = ta; t < tb; ++t) {
    const int r = a.req_index[t];
    if (a.seq_lens[r] <= 0) continue;
    const int i = t - a.cu_q[r], len = a.cu_q[r + 1] - a.cu_q[r];
    float* slot = a.state + (size_t)a.state_slots[r] * max(past, 1) * a.channels;
    if (i > 0) {
      if (i >= past) dp_token(a, t, i, c0, width, !is_v, gain, slot, lane);       // reads no state
      continue;
    }
    const int first = min(len, max(past, 1));
    for (int j = 0; j < first; ++j) dp_token(a, t + j, j, c0, width, !is_v, gain, slot, lane);
    dp_keep(a, slot, t, len, c0, width, lane);
  }
}

// The same for heads of up to 128 channels, multiples of 4, and two to four taps: a lane has four neighbouring channels, their
// taps and their last inputs in registers, so that a token costs one 16-byte load.
template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
delta_prepare_rolling_kernel(DeltaPrepareArgs a) {
  ifb_pdl_wait();
  ifb_pdl_trigger();
  constexpr int PAST = TAPS - 1;
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int G = a.kv_heads, units = 2 * G + a.heads;
  if (unit > units) return;
  const int ta = blockIdx.y * a.tok, tb = min(ta + a.tok, a.tokens);
  if (unit == units) {
    for (int t = ta; t < tb; ++t) dp_rest<T>(a, t, lane);
    return;
  }
  const bool is_v = unit >= 2 * G;
  const int width = is_v ? a.vdim : a.dim;
  const int c = (is_v ? 2 * G * a.dim + (unit - 2 * G) * a.vdim : unit * a.dim) + lane * 4;
  const float gain = unit < G ? a.q_scale : 1.f;
  const bool on = lane * 4 < width;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float w[4][TAPS];
#pragma unroll
  for (int x = 0; x < 4; ++x)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[x][j] = on ? a.taps_w[(size_t)(c + x) * TAPS + j] : 0.f;
  auto input = [&](int t) { return on ? *reinterpret_cast<const float4*>(a.proj + (size_t)t * a.ld + c) : zero; };
  auto emit = [&](int t, const float4* last, const float4 now) {       // last[PAST - 1]: the input before this one
    float4 y = make_float4(now.x * w[0][PAST], now.y * w[1][PAST], now.z * w[2][PAST], now.w * w[3][PAST]);
#pragma unroll
    for (int j = 0; j < PAST; ++j) {
      y.x = fmaf(last[j].x, w[0][j], y.x); y.y = fmaf(last[j].y, w[1][j], y.y);
      y.z = fmaf(last[j].z, w[2][j], y.z); y.w = fmaf(last[j].w, w[3][j], y.w);
    }
    y.x = y.x / (1.f + expf(-y.x)); y.y = y.y / (1.f + expf(-y.y)); y.z = y.z / (1.f + expf(-y.z)); y.w = y.w / (1.f + expf(-y.w));
    if (!is_v) {
      const float f = gain / sqrtf(warp_sum(y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w) + a.unit_eps);
      y.x *= f; y.y *= f; y.z *= f; y.w *= f;
    }
    if (on) *reinterpret_cast<float4*>(a.qkv + (size_t)t * a.channels + c) = y;
  };
  float4 last[PAST];
  int have = -1;                                         // `last` holds the inputs before this token
  for (int t = ta; t < tb; ++t) {
    const int r = a.req_index[t];
    if (a.seq_lens[r] <= 0) continue;
    const int i = t - a.cu_q[r], len = a.cu_q[r + 1] - a.cu_q[r];
    if (i > 0 && i < PAST) continue;                     // done by the warp of the request's first token
    if (i > 0) {
      if (have != t) {
#pragma unroll
        for (int j = 0; j < PAST; ++j) last[j] = input(t - PAST + j);
      }
      const float4 now = input(t);
      emit(t, last, now);
#pragma unroll
      for (int j = 0; j + 1 < PAST; ++j) last[j] = last[j + 1];
      last[PAST - 1] = now;
      have = t + 1;
      continue;
    }
    float* slot = a.state + (size_t)a.state_slots[r] * PAST * a.channels + c;
    float4 held[PAST];
#pragma unroll
    for (int j = 0; j < PAST; ++j) held[j] = last[j] = on ? *reinterpret_cast<const float4*>(slot + (size_t)j * a.channels) : zero;
#pragma unroll
    for (int k = 0; k < PAST; ++k) {                     // the tokens that read the slot
      if (k >= len) break;
      const float4 now = input(t + k);
      emit(t + k, last, now);
#pragma unroll
      for (int j = 0; j + 1 < PAST; ++j) last[j] = last[j + 1];
      last[PAST - 1] = now;
    }
    if (on) {
#pragma unroll
      for (int p = 0; p < PAST; ++p) {                   // entry len + p of [held inputs | portion]
        float4 v = zero;
        if (len + p >= PAST) v = input(t + len + p - PAST);
#pragma unroll
        for (int j = 0; j < PAST; ++j)
          if (len + p == j) v = held[j];
        *reinterpret_cast<float4*>(slot + (size_t)p * a.channels) = v;
      }
    }
    have = t + PAST;
  }
}

template <typename T>
static int dp_launch(DeltaPrepareArgs a, cudaStream_t stream) {
  a.tok = a.tokens <= 512 ? 1 : DR_TOK;
  const int chunks = (a.tokens + a.tok - 1) / a.tok;
  if (chunks > 65535) return IFB_ERR_SIZE;
  dim3 grid((2 * a.kv_heads + a.heads + 1 + 7) / 8, chunks);
  const bool rolling = a.dim <= 128 && a.vdim <= 128 && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld % 4 == 0 &&
                       (((uintptr_t)a.proj | (uintptr_t)a.qkv | (uintptr_t)a.state) & 15) == 0;
  if (rolling && a.taps == 2) return ifb_launch(delta_prepare_rolling_kernel<T, 2>, grid, dim3(256), 0, stream, a);
  if (rolling && a.taps == 3) return ifb_launch(delta_prepare_rolling_kernel<T, 3>, grid, dim3(256), 0, stream, a);
  if (rolling && a.taps == 4) return ifb_launch(delta_prepare_rolling_kernel<T, 4>, grid, dim3(256), 0, stream, a);
  return ifb_launch(delta_prepare_kernel<T>, grid, dim3(256), 0, stream, a);
}

IFB_EXPORT int ifb_delta_prepare(const float* proj, long long ld, const float* taps_w, int taps, float unit_eps, float q_scale,
                                 float* state, const int* state_slots, const int* cu_q, const int* seq_lens, const int* req_index,
                                 float* qkv, float* beta, void* low, int low_dtype, int low_width, int low_cols, int tokens,
                                 int kv_heads, int heads, int dim, int vdim, cudaStream_t stream) {
  if (tokens <= 0) return IFB_OK;
  if (kv_heads < 1 || heads < 1 || dim < 1 || vdim < 1 || taps < 1 || low_cols < low_width) return IFB_ERR_SIZE;
  const int channels = 2 * kv_heads * dim + heads * vdim;
  DeltaPrepareArgs a{proj, ld, taps_w, taps, unit_eps, q_scale, state, state_slots, cu_q, seq_lens, req_index, qkv, beta, low, low_dtype,
                     low_width, low_cols, tokens, kv_heads, heads, dim, vdim, channels, 1};
  if (low_dtype == IFB_BF16) return dp_launch<__nv_bfloat16>(a, stream);
  if (low_dtype != IFB_F32) return IFB_ERR_DTYPE;
  return dp_launch<float>(a, stream);
}

// ------------------------------------------------------------------------------------------ (2) delta_rule
struct DeltaRuleArgs {
  const float* qkv; int ldc;           // rows q | k | v
  const float* up; int ldu;            // rows raw decays [heads * dim] | gates [heads * vdim]
  const float* beta;                   // [tokens][heads]
  const float *rate, *bias, *norm_w;   // [heads], [heads * dim], [vdim]
  float eps;
  float* state;                        // [slots][heads][dim][vdim]
  const int *state_slots, *cu_q, *seq_lens;
  void* out;                           // [tokens][heads * vdim], T
  float* raw;                          // [tokens][heads * vdim]: outputs before the finish, where a head is done in slabs
  float* chunks;                       // scratch of the chunked form
  int kv_heads, heads, dim, vdim, slabs, requests;
};

// log2 of the decay
__device__ __forceinline__ float dr_log2_decay(float x, float rate) {
  const float sp = x > 20.f ? x : log1pf(expf(x));
  return fmaxf(-rate * sp * DR_LOG2E, DR_LOG2_MIN);
}

// out = o / rms(o) * norm_w * sigmoid(gate) for one (token, head), by one warp
template <typename T>
__device__ __forceinline__ void dr_finish(const DeltaRuleArgs& a, const float* o, int t, int h, int lane) {
  const int vdim = a.vdim;
  float ss = 0.f;
  for (int e = lane; e < vdim; e += 32) ss = fmaf(o[e], o[e], ss);
  const float rn = 1.f / sqrtf(warp_sum(ss) / (float)vdim + a.eps);
  T* dst = (T*)a.out + ((size_t)t * a.heads + h) * vdim;
  const float* gate = a.up + (size_t)t * a.ldu + a.heads * a.dim + h * vdim;
  for (int e = lane; e < vdim; e += 32) dst[e] = from_f32<T>(o[e] * rn * a.norm_w[e] / (1.f + expf(-gate[e])));
}

template <typename T>
__global__ void __launch_bounds__(128)
delta_finish_kernel(DeltaRuleArgs a, long long items) {
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= items) return;
  dr_finish<T>(a, a.raw + item * a.vdim, (int)(item / a.heads), (int)(item % a.heads), threadIdx.x & 31);
}

template <typename T, int RS, int RPT>
__global__ void __launch_bounds__(512, 1)
delta_walk_kernel(DeltaRuleArgs a) {
  constexpr int DMAX = RS * RPT, PITCH = RPT + 4, ROW = RS * PITCH;       // parts start in different banks
  extern __shared__ float sm[];
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const int cols = blockDim.x / RS, part = threadIdx.x % RS, cl = threadIdx.x / RS;
  const int h = blockIdx.x / a.slabs, c0 = (blockIdx.x % a.slabs) * cols, c = c0 + cl, r = blockIdx.y;
  if (a.seq_lens[r] <= 0) return;
  const int dim = a.dim, vdim = a.vdim, hk = h / (a.heads / a.kv_heads);
  const int width = min(cols, vdim - c0);
  float* qs = sm;                              // [GROUP][ROW]
  float* ks = qs + DR_GROUP * ROW;
  float* gs = ks + DR_GROUP * ROW;
  float* vs = gs + DR_GROUP * ROW;             // [GROUP][cols]
  float* os = vs + DR_GROUP * cols;            // [GROUP][cols]
  float* bs = os + DR_GROUP * cols;            // [GROUP]
  const bool col = c < vdim;
  const int r0 = part * RPT;
  float* sp = a.state + (((size_t)a.state_slots[r] * a.heads + h) * dim) * vdim + c;
  float S[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) S[i] = (col && r0 + i < dim) ? sp[(size_t)(r0 + i) * vdim] : 0.f;
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float rate = a.rate[h];
  const int t1 = a.cu_q[r + 1];
  for (int g0 = a.cu_q[r]; g0 < t1; g0 += DR_GROUP) {
    const int cnt = min(DR_GROUP, t1 - g0);
    for (int idx = threadIdx.x; idx < cnt * DMAX; idx += blockDim.x) {
      const int t = idx / DMAX, i = idx % DMAX;
      float qv = 0.f, kv = 0.f, gv = 1.f;
      if (i < dim) {
        const float* row = a.qkv + (size_t)(g0 + t) * a.ldc;
        qv = row[hk * dim + i];
        kv = row[(a.kv_heads + hk) * dim + i];
        gv = exp2f(dr_log2_decay(a.up[(size_t)(g0 + t) * a.ldu + h * dim + i] + a.bias[h * dim + i], rate));
      }
      const int at = t * ROW + (i / RPT) * PITCH + i % RPT;
      qs[at] = qv; ks[at] = kv; gs[at] = gv;
    }
    for (int idx = threadIdx.x; idx < cnt * width; idx += blockDim.x) {
      const int t = idx / width, e = idx % width;
      vs[t * cols + e] = a.qkv[(size_t)(g0 + t) * a.ldc + 2 * a.kv_heads * dim + h * vdim + c0 + e];
    }
    if (threadIdx.x < cnt) bs[threadIdx.x] = a.beta[(size_t)(g0 + threadIdx.x) * a.heads + h];
    __syncthreads();
    for (int t = 0; t < cnt; ++t) {            // whole warps walk together: the parts of a column meet by shuffles
      const float4* q4 = reinterpret_cast<const float4*>(qs + t * ROW + part * PITCH);
      const float4* k4 = reinterpret_cast<const float4*>(ks + t * ROW + part * PITCH);
      const float4* g4 = reinterpret_cast<const float4*>(gs + t * ROW + part * PITCH);
      float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll
      for (int i = 0; i < RPT / 4; ++i) {
        const float4 g = g4[i], k = k4[i];
        S[4 * i] *= g.x; S[4 * i + 1] *= g.y; S[4 * i + 2] *= g.z; S[4 * i + 3] *= g.w;
        d0 = fmaf(S[4 * i], k.x, d0); d1 = fmaf(S[4 * i + 1], k.y, d1);
        d2 = fmaf(S[4 * i + 2], k.z, d2); d3 = fmaf(S[4 * i + 3], k.w, d3);
      }
      float d = (d0 + d1) + (d2 + d3);
#pragma unroll
      for (int m = 1; m < RS; m <<= 1) d += __shfl_xor_sync(0xffffffffu, d, m);
      const float u = bs[t] * (vs[t * cols + cl] - d);
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
      for (int i = 0; i < RPT / 4; ++i) {
        const float4 k = k4[i], q = q4[i];
        S[4 * i] = fmaf(k.x, u, S[4 * i]); S[4 * i + 1] = fmaf(k.y, u, S[4 * i + 1]);
        S[4 * i + 2] = fmaf(k.z, u, S[4 * i + 2]); S[4 * i + 3] = fmaf(k.w, u, S[4 * i + 3]);
        o0 = fmaf(S[4 * i], q.x, o0); o1 = fmaf(S[4 * i + 1], q.y, o1);
        o2 = fmaf(S[4 * i + 2], q.z, o2); o3 = fmaf(S[4 * i + 3], q.w, o3);
      }
      float o = (o0 + o1) + (o2 + o3);
#pragma unroll
      for (int m = 1; m < RS; m <<= 1) o += __shfl_xor_sync(0xffffffffu, o, m);
      if (part == 0) os[t * cols + cl] = o;
    }
    __syncthreads();
    for (int t = warp; t < cnt; t += warps) {
      const float* o = os + t * cols;
      if (a.raw) {                             // the head has other slabs: the second kernel finishes it
        float* dst = a.raw + ((size_t)(g0 + t) * a.heads + h) * vdim + c0;
        for (int e = lane; e < width; e += 32) dst[e] = o[e];
      } else {
        dr_finish<T>(a, o, g0 + t, h, lane);
      }
    }
    __syncthreads();
  }
  if (col) {
#pragma unroll
    for (int i = 0; i < RPT; ++i)
      if (r0 + i < dim) sp[(size_t)(r0 + i) * vdim] = S[i];
  }
}

// Heads with more than 256 rows: the state stays in device memory.  A block per (request, head), its threads over the
// columns.  Slow (the state crosses the memory bus twice for every token) and exact.
template <typename T>
__global__ void __launch_bounds__(256)
delta_wide_kernel(DeltaRuleArgs a) {
  extern __shared__ float sm[];
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const int r = blockIdx.y, h = blockIdx.x, dim = a.dim, vdim = a.vdim, hk = h / (a.heads / a.kv_heads);
  if (a.seq_lens[r] <= 0) return;
  float *qs = sm, *ks = qs + dim, *gs = ks + dim, *os = gs + dim;      // [dim] x 3, [vdim]
  float* S = a.state + ((size_t)a.state_slots[r] * a.heads + h) * dim * vdim;
  for (int t = a.cu_q[r]; t < a.cu_q[r + 1]; ++t) {
    const float* row = a.qkv + (size_t)t * a.ldc;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
      qs[i] = row[hk * dim + i];
      ks[i] = row[(a.kv_heads + hk) * dim + i];
      gs[i] = exp2f(dr_log2_decay(a.up[(size_t)t * a.ldu + h * dim + i] + a.bias[h * dim + i], a.rate[h]));
    }
    __syncthreads();
    const float beta = a.beta[(size_t)t * a.heads + h];
    for (int c = threadIdx.x; c < vdim; c += blockDim.x) {
      float d = 0.f, o = 0.f;
      for (int i = 0; i < dim; ++i) d = fmaf(gs[i] * S[(size_t)i * vdim + c], ks[i], d);
      const float u = beta * (row[2 * a.kv_heads * dim + h * vdim + c] - d);
      for (int i = 0; i < dim; ++i) {
        const float s = fmaf(ks[i], u, gs[i] * S[(size_t)i * vdim + c]);
        S[(size_t)i * vdim + c] = s;
        o = fmaf(s, qs[i], o);
      }
      os[c] = o;
    }
    __syncthreads();
    if (threadIdx.x < 32) dr_finish<T>(a, os, t, h, threadIdx.x & 31);
    __syncthreads();
  }
}

// ---- the chunked form
constexpr int DR_PP = DR_C + 4;     // pitch of a row of P, so that neighbouring rows start in different banks
// One (chunk, head) of the scratch: W, Q, K [DR_C][dp] each, P [DR_C][DR_PP], decay [dp], U [DR_C][vp]
__host__ __device__ __forceinline__ int dr_dp(int dim) { return dim <= 32 ? 32 : dim <= 64 ? 64 : dim <= 128 ? 128 : 256; }
__host__ __device__ __forceinline__ int dr_vp(int vdim) { return (vdim + 31) / 32 * 32; }
__host__ __device__ __forceinline__ size_t dr_chunk_floats(int dim, int vdim) {
  return (size_t)3 * DR_C * dr_dp(dim) + DR_C * DR_PP + dr_dp(dim) + (size_t)DR_C * dr_vp(vdim);
}

// The chunk that row `row` of the grid is; false: beyond the last
__device__ __forceinline__ bool dr_find_chunk(const DeltaRuleArgs& a, int row, int& t0, int& cnt) {
  for (int i = 0; i < a.requests; ++i) {
    const int ql = a.seq_lens[i] > 0 ? a.cu_q[i + 1] - a.cu_q[i] : 0;
    const int n = (ql + DR_C - 1) / DR_C;
    if (row < n) {
      t0 = a.cu_q[i] + row * DR_C;
      cnt = min(DR_C, a.cu_q[i + 1] - t0);
      return true;
    }
    row -= n;
  }
  return false;
}

// 2^x for x at most 0 (what underflows is 0)
__device__ __forceinline__ float dr_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

constexpr int DA_THREADS = 320;                        // 8 threads for each of the 40 (t, four neighbouring s <= t) items

template <int DP>
__global__ void __launch_bounds__(DA_THREADS)
delta_chunk_kernel(DeltaRuleArgs a) {
  extern __shared__ float sm[];
  ifb_pdl_wait();
  ifb_pdl_trigger();
  constexpr int PITCH = DP + 1;
  int t0, cnt;
  if (!dr_find_chunk(a, blockIdx.y, t0, cnt)) return;
  const int h = blockIdx.x, dim = a.dim, vdim = a.vdim, vp = dr_vp(vdim);
  const int hk = h / (a.heads / a.kv_heads), tid = threadIdx.x;
  float* qs = sm;                                      // [DR_C][PITCH]
  float* ks = qs + DR_C * PITCH;
  float* ls = ks + DR_C * PITCH;                       // log2 of the decays, then their running sums
  float* As = ls + DR_C * PITCH;                       // [DR_C][DR_C + 1]
  float* Ts = As + DR_C * (DR_C + 1);                  // [DR_C][DR_C + 1]
  float* bs = Ts + DR_C * (DR_C + 1);                  // [DR_C]
  float* base = a.chunks + ((size_t)blockIdx.y * a.heads + h) * dr_chunk_floats(dim, vdim);
  float *gW = base, *gQ = gW + DR_C * DP, *gK = gQ + DR_C * DP, *gP = gK + DR_C * DP, *gG = gP + DR_C * DR_PP, *gU = gG + DP;
  const float rate = a.rate[h];
  for (int idx = tid; idx < DR_C * DP; idx += DA_THREADS) {
    const int t = idx / DP, i = idx % DP;
    float qv = 0.f, kv = 0.f, lv = 0.f;
    if (t < cnt && i < dim) {
      const float* row = a.qkv + (size_t)(t0 + t) * a.ldc;
      qv = row[hk * dim + i];
      kv = row[(a.kv_heads + hk) * dim + i];
      lv = dr_log2_decay(a.up[(size_t)(t0 + t) * a.ldu + h * dim + i] + a.bias[h * dim + i], rate);
    }
    qs[t * PITCH + i] = qv; ks[t * PITCH + i] = kv; ls[t * PITCH + i] = lv;
  }
  if (tid < DR_C) bs[tid] = tid < cnt ? a.beta[(size_t)(t0 + tid) * a.heads + h] : 0.f;
  __syncthreads();
  if (tid < DP) {
    float s = 0.f;
#pragma unroll
    for (int t = 0; t < DR_C; ++t) { s += ls[t * PITCH + tid]; ls[t * PITCH + tid] = s; }
  }
  __syncthreads();
  {
    // item (t, g): the pairs of t with s = 4 g .. 4 g + 3 (those beyond t count for nothing); its 8 neighbouring threads share
    // the channels
    const int item = tid >> 3, lane8 = tid & 7;
    const int band = item < 4 ? 0 : item < 12 ? 1 : item < 24 ? 2 : 3;             // t / 4: bands of 4, 8, 12 and 16 items
    const int in = item - 2 * band * (band + 1), t = 4 * band + in / (band + 1), s0 = 4 * (in % (band + 1));
    float ak[4] = {0.f, 0.f, 0.f, 0.f}, aq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int i = lane8; i < DP; i += 8) {
      const float kt = ks[t * PITCH + i], qt = qs[t * PITCH + i], lt = ls[t * PITCH + i];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float ke = ks[(s0 + x) * PITCH + i] * dr_exp2(fminf(lt - ls[(s0 + x) * PITCH + i], 0.f));
        ak[x] = fmaf(kt, ke, ak[x]);
        aq[x] = fmaf(qt, ke, aq[x]);
      }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int m = 1; m < 8; m <<= 1) {
        ak[x] += __shfl_xor_sync(0xffffffffu, ak[x], m);
        aq[x] += __shfl_xor_sync(0xffffffffu, aq[x], m);
      }
    if (lane8 == 0)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int s = s0 + x;
        if (s > t) continue;
        As[t * (DR_C + 1) + s] = s < t ? bs[t] * ak[x] : 0.f;
        gP[t * DR_PP + s] = aq[x];
        if (s < t) gP[s * DR_PP + t] = 0.f;
      }
  }
  __syncthreads();
  if (tid < 32) {
    if (tid < DR_C) {                                  // column tid of (I + A)^-1, forward substitution
      float x[DR_C];
#pragma unroll
      for (int t = 0; t < DR_C; ++t) {
        float v0 = t == tid ? 1.f : 0.f, v1 = 0.f;
#pragma unroll
        for (int s = 0; s < t; ++s) {
          if (s & 1) v1 = fmaf(-As[t * (DR_C + 1) + s], x[s], v1);
          else v0 = fmaf(-As[t * (DR_C + 1) + s], x[s], v0);
        }
        x[t] = v0 + v1;
      }
#pragma unroll
      for (int t = 0; t < DR_C; ++t) Ts[t * (DR_C + 1) + tid] = x[t] * bs[tid];
    }
  } else {
    for (int idx = tid - 32; idx < DR_C * DP; idx += DA_THREADS - 32) {
      const int t = idx / DP, i = idx % DP;
      const float l = ls[t * PITCH + i], end = ls[(DR_C - 1) * PITCH + i];
      gQ[idx] = qs[t * PITCH + i] * dr_exp2(l);
      gK[idx] = ks[t * PITCH + i] * dr_exp2(end - l);
      if (t == 0) gG[i] = dr_exp2(end);
    }
  }
  __syncthreads();
  for (int j = tid; j < DP + vp; j += DA_THREADS) {    // W: a thread per channel; U: a thread per column
    float x[DR_C];
    float* dst;
    int step;
    if (j < DP) {
#pragma unroll
      for (int t = 0; t < DR_C; ++t) x[t] = ks[t * PITCH + j] * dr_exp2(ls[t * PITCH + j]);
      dst = gW + j; step = DP;
    } else {
      const int c = j - DP;
#pragma unroll
      for (int t = 0; t < DR_C; ++t)
        x[t] = (t < cnt && c < vdim) ? a.qkv[(size_t)(t0 + t) * a.ldc + 2 * a.kv_heads * dim + h * vdim + c] : 0.f;
      dst = gU + c; step = vp;
    }
#pragma unroll
    for (int t = 0; t < DR_C; ++t) {
      float v = 0.f;
#pragma unroll
      for (int s = 0; s <= t; ++s) v = fmaf(Ts[t * (DR_C + 1) + s], x[s], v);
      dst[(size_t)t * step] = v;
    }
  }
}

__device__ __forceinline__ void dr_copy16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// Each of LP neighbouring lanes holds 16 numbers; lane i is left with the sums over the lanes of numbers i TK .. i TK + TK - 1,
// TK = 16 / LP, in x[0 .. TK - 1].
template <int LP>
__device__ __forceinline__ void dr_reduce16(float* x, int i) {
#pragma unroll
  for (int half = 8; half >= 16 / LP; half >>= 1) {
    const int mask = half * LP / 16;
    const bool up = i & mask;
#pragma unroll
    for (int j = 0; j < half; ++j) {
      const float send = up ? x[j] : x[j + half], keep = up ? x[j + half] : x[j];
      x[j] = keep + __shfl_xor_sync(0xffffffffu, send, mask);
    }
  }
}

// A block per (head, slab of columns) and request: thread (column, part), LP parts of a column in neighbouring lanes, part p
// with rows b 4 LP + 4 p + i, b = 0 .. DP / (4 LP) - 1, i = 0 .. 3, of CPT columns.
constexpr int DC_THREADS = 128;
template <int DP, int LP, int CPT>
__global__ void __launch_bounds__(DC_THREADS)
delta_carry_kernel(DeltaRuleArgs a) {
  constexpr int CB = DC_THREADS / LP, NC = CB * CPT;                  // columns side by side, columns of the block
  constexpr int NB = DP / (4 * LP), TK = 16 / LP;
  constexpr int OPER = 3 * DR_C * DP + DR_C * DR_PP + DP;             // W, Q, K, P, decay: contiguous in the scratch
  constexpr int STAGE = OPER + DR_C * NC;
  extern __shared__ __align__(16) float sm[];
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const int r = blockIdx.y, h = blockIdx.x / a.slabs, c0 = (blockIdx.x % a.slabs) * NC;
  if (a.seq_lens[r] <= 0) return;
  const int dim = a.dim, vdim = a.vdim, vp = dr_vp(vdim), tid = threadIdx.x, p = tid % LP, cl = tid / LP;
  int first = 0;                                        // the request's first chunk among all
  for (int i = 0; i < r; ++i) first += a.seq_lens[i] > 0 ? (a.cu_q[i + 1] - a.cu_q[i] + DR_C - 1) / DR_C : 0;
  const int ta = a.cu_q[r], tb = a.cu_q[r + 1], n = (tb - ta + DR_C - 1) / DR_C;
  const size_t per = dr_chunk_floats(dim, vdim);
  const float* src = a.chunks + ((size_t)first * a.heads + h) * per;
  float* us = sm + 2 * STAGE;                           // [NC][DR_C + 4]: u of a column, read as float4
  float* os = us + NC * (DR_C + 4);                     // [2][DR_C][NC]
  float* sp = a.state + (((size_t)a.state_slots[r] * a.heads + h) * dim) * vdim;
  float S[CPT][NB * 4];
#pragma unroll
  for (int x = 0; x < CPT; ++x) {
    const int c = c0 + x * CB + cl;
#pragma unroll
    for (int i = 0; i < NB * 4; ++i) {
      const int row = (i >> 2) * 4 * LP + p * 4 + (i & 3);
      S[x][i] = (c < vdim && row < dim) ? sp[(size_t)row * vdim + c] : 0.f;
    }
  }
  auto ask = [&](int j) {
    const float* g = src + (size_t)j * a.heads * per;
    float* s = sm + (j & 1) * STAGE;
    for (int i = tid * 4; i < OPER; i += DC_THREADS * 4) dr_copy16(s + i, g + i);
    for (int i = tid * 4; i < DR_C * NC; i += DC_THREADS * 4) dr_copy16(s + OPER + i, g + OPER + (size_t)(i / NC) * vp + c0 + i % NC);
    asm volatile("cp.async.commit_group;\n" ::);
  };
  auto give = [&](int j) {                              // outputs of chunk j from shared memory, whole row segments
    const float* o = os + (j & 1) * DR_C * NC;
    for (int i = tid; i < DR_C * NC; i += DC_THREADS) {
      const int t = ta + j * DR_C + i / NC, c = c0 + i % NC;
      if (t < tb && c < vdim) a.raw[((size_t)t * a.heads + h) * vdim + c] = o[i];
    }
  };
  // acc[x][t] = this part's share of sum_rows M[t][row] S[x][row]; eight tokens' chains side by side
  auto times_state = [&](const float* M, float (&acc)[CPT][DR_C]) {
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int t = 0; t < DR_C; ++t) acc[x][t] = 0.f;
#pragma unroll
    for (int b = 0; b < NB; ++b)
#pragma unroll
      for (int tg = 0; tg < DR_C; tg += 8) {
        float4 m[8];
#pragma unroll
        for (int t = 0; t < 8; ++t) m[t] = *reinterpret_cast<const float4*>(M + (tg + t) * DP + b * 4 * LP + p * 4);
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
#pragma unroll
          for (int t = 0; t < 8; ++t) acc[x][tg + t] = fmaf(m[t].x, S[x][4 * b], acc[x][tg + t]);
#pragma unroll
          for (int t = 0; t < 8; ++t) acc[x][tg + t] = fmaf(m[t].y, S[x][4 * b + 1], acc[x][tg + t]);
#pragma unroll
          for (int t = 0; t < 8; ++t) acc[x][tg + t] = fmaf(m[t].z, S[x][4 * b + 2], acc[x][tg + t]);
#pragma unroll
          for (int t = 0; t < 8; ++t) acc[x][tg + t] = fmaf(m[t].w, S[x][4 * b + 3], acc[x][tg + t]);
        }
      }
  };
  ask(0);
  for (int j = 0; j < n; ++j) {
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();                                    // chunk j is here, and everybody is done with chunk j - 1
    if (j + 1 < n) ask(j + 1);
    if (j > 0) give(j - 1);
    const float* s = sm + (j & 1) * STAGE;
    const float *Ws = s, *Qs = Ws + DR_C * DP, *Ks = Qs + DR_C * DP, *Ps = Ks + DR_C * DP, *Gs = Ps + DR_C * DR_PP, *Us = Gs + DP;
    float acc[CPT][DR_C];
    times_state(Ws, acc);
#pragma unroll
    for (int x = 0; x < CPT; ++x) {
      dr_reduce16<LP>(acc[x], p);
#pragma unroll
      for (int m = 0; m < TK; ++m)
        us[(x * CB + cl) * (DR_C + 4) + TK * p + m] = Us[(TK * p + m) * NC + x * CB + cl] - acc[x][m];
    }
    __syncwarp();                                       // the lanes of a column are in one warp
    times_state(Qs, acc);                               // what the state before the chunk gives to the outputs
#pragma unroll
    for (int x = 0; x < CPT; ++x) dr_reduce16<LP>(acc[x], p);
    float u[CPT][DR_C];
#pragma unroll
    for (int x = 0; x < CPT; ++x)
#pragma unroll
      for (int t = 0; t < DR_C; t += 4)
        *reinterpret_cast<float4*>(&u[x][t]) = *reinterpret_cast<const float4*>(us + (x * CB + cl) * (DR_C + 4) + t);
#pragma unroll
    for (int b = 0; b < NB; ++b) {
      const float4 gv = *reinterpret_cast<const float4*>(Gs + b * 4 * LP + p * 4);
#pragma unroll
      for (int x = 0; x < CPT; ++x) { S[x][4 * b] *= gv.x; S[x][4 * b + 1] *= gv.y; S[x][4 * b + 2] *= gv.z; S[x][4 * b + 3] *= gv.w; }
    }
#pragma unroll
    for (int t = 0; t < DR_C; ++t)
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        const float4 kv = *reinterpret_cast<const float4*>(Ks + t * DP + b * 4 * LP + p * 4);
#pragma unroll
        for (int x = 0; x < CPT; ++x) {
          S[x][4 * b] = fmaf(kv.x, u[x][t], S[x][4 * b]); S[x][4 * b + 1] = fmaf(kv.y, u[x][t], S[x][4 * b + 1]);
          S[x][4 * b + 2] = fmaf(kv.z, u[x][t], S[x][4 * b + 2]); S[x][4 * b + 3] = fmaf(kv.w, u[x][t], S[x][4 * b + 3]);
        }
      }
#pragma unroll
    for (int m = 0; m < TK; ++m) {
      float4 pv[4];
#pragma unroll
      for (int t = 0; t < 4; ++t) pv[t] = *reinterpret_cast<const float4*>(Ps + (TK * p + m) * DR_PP + 4 * t);
#pragma unroll
      for (int x = 0; x < CPT; ++x) {
        float y[4];
#pragma unroll
        for (int t = 0; t < 4; ++t)
          y[t] = fmaf(pv[t].w, u[x][4 * t + 3], fmaf(pv[t].z, u[x][4 * t + 2], fmaf(pv[t].y, u[x][4 * t + 1], pv[t].x * u[x][4 * t])));
        os[(j & 1) * DR_C * NC + (TK * p + m) * NC + x * CB + cl] = acc[x][m] + ((y[0] + y[1]) + (y[2] + y[3]));
      }
    }
    __syncwarp();                                       // u was read by all its lanes before the next chunk writes it
  }
  __syncthreads();
  give(n - 1);
#pragma unroll
  for (int x = 0; x < CPT; ++x) {
    const int c = c0 + x * CB + cl;
#pragma unroll
    for (int i = 0; i < NB * 4; ++i) {
      const int row = (i >> 2) * 4 * LP + p * 4 + (i & 3);
      if (c < vdim && row < dim) sp[(size_t)row * vdim + c] = S[x][i];
    }
  }
}

static int dr_walk_parts(int dim) { return dim <= 128 ? 4 : 8; }
static int dr_walk_cols(int dim, int vdim) {
  const int rs = dr_walk_parts(dim), per_warp = 32 / rs;
  return min(512 / rs, (vdim + per_warp - 1) / per_warp * per_warp);
}

template <typename T, int RS, int RPT>
static int dr_walk(DeltaRuleArgs a, cudaStream_t s) {
  const int cols = dr_walk_cols(a.dim, a.vdim);
  const size_t smem = ((size_t)DR_GROUP * (3 * RS * (RPT + 4) + 2 * cols) + DR_GROUP) * sizeof(float);
  IFB_ALLOW_SMEM((delta_walk_kernel<T, RS, RPT>), smem);
  return ifb_launch(delta_walk_kernel<T, RS, RPT>, dim3(a.heads * a.slabs, a.requests), dim3(cols * RS), smem, s, a);
}

template <int DP, int LP, int CPT>
static int dr_carry(DeltaRuleArgs a, cudaStream_t s) {
  constexpr int NC = DC_THREADS / LP * CPT, STAGE = 3 * DR_C * DP + DR_C * DR_PP + DP + DR_C * NC;
  const size_t smem = (size_t)(2 * STAGE + NC * (DR_C + 4) + 2 * DR_C * NC) * sizeof(float);
  a.slabs = (a.vdim + NC - 1) / NC;
  IFB_ALLOW_SMEM((delta_carry_kernel<DP, LP, CPT>), smem);
  // not early: blocks placed while the chunks' launch still fills the device crowd on the SMs that are free first
  return ifb_launch_opt(false, delta_carry_kernel<DP, LP, CPT>, dim3(a.heads * a.slabs, a.requests), dim3(DC_THREADS), smem, s, a);
}

template <int DP>
static int dr_chunked(DeltaRuleArgs a, int rows, int columns, cudaStream_t s) {
  const size_t smem = (size_t)(3 * DR_C * (DP + 1) + 2 * DR_C * (DR_C + 1) + DR_C) * sizeof(float);
  IFB_ALLOW_SMEM(delta_chunk_kernel<DP>, smem);
  const int st = ifb_launch(delta_chunk_kernel<DP>, dim3(a.heads, rows), dim3(DA_THREADS), smem, s, a);
  if (st != IFB_OK) return st;
  // columns per block: 8 (16 lanes a column), 16 (8 lanes), 32 (8 lanes, two columns each)
  if constexpr (DP >= 64)
    if (columns == 8) return dr_carry<DP, 16, 1>(a, s);
  if constexpr (DP <= 128)
    if (columns == 32) return dr_carry<DP, 8, 2>(a, s);
  return dr_carry<DP, 8, 1>(a, s);
}

template <typename T>
static int dr_run(DeltaRuleArgs a, int tokens, int columns, cudaStream_t s) {
  if (a.dim > 256) {
    const size_t smem = (size_t)(3 * a.dim + a.vdim) * sizeof(float);
    if (smem > 200 * 1024) return IFB_ERR_SIZE;
    IFB_ALLOW_SMEM(delta_wide_kernel<T>, smem);
    return ifb_launch(delta_wide_kernel<T>, dim3(a.heads, a.requests), dim3(256), smem, s, a);
  }
  int st;
  if (a.chunks) {
    const long long rows = (tokens + DR_C - 1) / DR_C + a.requests;
    if (rows > 65535 || !a.raw) return IFB_ERR_SIZE;
    switch (dr_dp(a.dim)) {
      case 32: st = dr_chunked<32>(a, (int)rows, columns, s); break;
      case 64: st = dr_chunked<64>(a, (int)rows, columns, s); break;
      case 128: st = dr_chunked<128>(a, (int)rows, columns, s); break;
      default: st = dr_chunked<256>(a, (int)rows, columns, s);
    }
  } else {
    const int cols = dr_walk_cols(a.dim, a.vdim);
    a.slabs = (a.vdim + cols - 1) / cols;
    if (a.slabs > 1 && !a.raw) return IFB_ERR_ARG;
    if (a.slabs == 1) a.raw = nullptr;
    st = a.dim <= 32 ? dr_walk<T, 4, 8>(a, s) : a.dim <= 64 ? dr_walk<T, 4, 16>(a, s)
       : a.dim <= 128 ? dr_walk<T, 4, 32>(a, s) : dr_walk<T, 8, 32>(a, s);
    if (a.slabs == 1) return st;
  }
  if (st != IFB_OK) return st;
  const long long items = (long long)tokens * a.heads;
  return ifb_launch(delta_finish_kernel<T>, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, s, a, items);
}

// Slabs of columns that the walk splits a head of these sizes into; with more than one the caller gives `raw`.
IFB_EXPORT int ifb_delta_rule_slabs(int dim, int vdim) {
  if (dim > 256) return 1;
  const int cols = dr_walk_cols(dim, vdim);
  return (vdim + cols - 1) / cols;
}

// Floats of scratch of the chunked form for a step of these sizes.
IFB_EXPORT long long ifb_delta_rule_scratch_floats(int tokens, int requests, int heads, int dim, int vdim) {
  return ((long long)(tokens + DR_C - 1) / DR_C + requests) * heads * (long long)dr_chunk_floats(dim, vdim);
}

// chunks: null for the token walk, else ifb_delta_rule_scratch_floats(...) floats, 16-byte aligned, for the chunked form (heads of
// up to 256 rows), which needs `raw` too.  columns: 8, 16 or 32, the columns of a block of the chunked form: few for a
// small grid, many where the blocks cover the device anyway (fewer reads of shared memory per product).
IFB_EXPORT int ifb_delta_rule(const float* qkv, int ldc, const float* up, int ldu, const float* beta, const float* rate,
                              const float* bias, const float* norm_w, float eps, float* state, const int* state_slots,
                              const int* cu_q, const int* seq_lens, void* out, int out_dtype, float* raw, float* chunks, int columns,
                              int requests, int tokens, int kv_heads, int heads, int dim, int vdim, cudaStream_t stream) {
  if (requests <= 0 || tokens <= 0) return IFB_OK;
  if (kv_heads < 1 || heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || requests > 65535) return IFB_ERR_SIZE;
  if (chunks && (((uintptr_t)chunks & 15) || (columns != 8 && columns != 16 && columns != 32))) return IFB_ERR_ARG;
  DeltaRuleArgs a{qkv, ldc, up, ldu, beta, rate, bias, norm_w, eps, state, state_slots, cu_q, seq_lens, out, raw, chunks, kv_heads, heads,
                  dim, vdim, 1, requests};
  if (out_dtype == IFB_F32) return dr_run<float>(a, tokens, columns, stream);
  if (out_dtype == IFB_BF16) return dr_run<__nv_bfloat16>(a, tokens, columns, stream);
  return IFB_ERR_DTYPE;
}
