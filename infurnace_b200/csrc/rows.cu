// Row kernels: the embedding with a pair table, and the norm, gate and factor between a mixer's core and its output product.
#include "common.cuh"
#include <math.h>

// ------------------------------------------------------------------------------------------
// out[t] = table[ids[t]] + pairs[row], row = (prev * mul_prev + ids[t] * mul_cur) mod buckets with prev the token before t in
// its sequence, or row `buckets` at position 0.  For a request's first token of the step prev is the number in its state
// slot; the block of that token then writes the request's last token of the step there: the only reader and the only writer
// of a slot in a step are that one block.  A block per token.  An id outside the vocabulary reads no memory: the row is
// zeros and IFB_DEV_ERR_TOKEN_ID is recorded (prev, which is such an id only where that was recorded, counts as 0 then).
// ------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
embed_bigram_kernel(const void* __restrict__ table, const void* __restrict__ pairs, int dtype, const int* __restrict__ ids,
                    const int* __restrict__ positions, const int* __restrict__ req_index, const int* __restrict__ cu_q,
                    const int* __restrict__ seq_lens, const int* __restrict__ state_slots, float* __restrict__ state, int buckets,
                    long long mul_prev, long long mul_cur, float* __restrict__ out, int hidden, int vocab, int* __restrict__ err) {
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const int t = blockIdx.x, r = req_index[t], id = ids[t];
  const bool live = seq_lens[r] > 0, first = live && t == cu_q[r];
  int prev = 0;
  if (first) prev = (int)state[state_slots[r]];
  else if (live) prev = ids[t - 1];
  if (prev < 0 || prev >= vocab) prev = 0;
  if (first) {
    __syncthreads();                                   // everybody has read the slot
    if (threadIdx.x == 0) state[state_slots[r]] = (float)ids[cu_q[r + 1] - 1];
  }
  if (id < 0 || id >= vocab) {
    for (int e = threadIdx.x; e < hidden; e += blockDim.x) out[(size_t)t * hidden + e] = 0.f;
    if (threadIdx.x == 0) atomicCAS(err, 0, IFB_DEV_ERR_TOKEN_ID);
    return;
  }
  const long long row = positions[t] == 0 ? buckets : (prev * mul_prev + id * mul_cur) % buckets;
  for (int e = threadIdx.x; e < hidden; e += blockDim.x)
    out[(size_t)t * hidden + e] = load_as_f32(table, dtype, (size_t)id * hidden + e) + load_as_f32(pairs, dtype, (size_t)row * hidden + e);
}

// mul_prev and mul_cur: reduced modulo buckets by the caller; buckets below 2^31, ids below 2^24 (a float32 holds them).
IFB_EXPORT int ifb_embed_bigram(const void* table, const void* pairs, int dtype, const int* ids, const int* positions, const int* req_index,
                                const int* cu_q, const int* seq_lens, const int* state_slots, float* state, int buckets,
                                long long mul_prev, long long mul_cur, float* out, int n, int hidden, int vocab, int* err,
                                cudaStream_t stream) {
  if (n <= 0) return IFB_OK;
  if (buckets < 1 || vocab < 1 || vocab > (1 << 24) || mul_prev < 0 || mul_cur < 0 || mul_prev >= buckets || mul_cur >= buckets || !err)
    return IFB_ERR_ARG;
  if (dtype != IFB_F32 && dtype != IFB_BF16) return IFB_ERR_DTYPE;
  const int threads = hidden >= 256 ? 256 : ((hidden + 31) / 32) * 32;
  return ifb_launch(embed_bigram_kernel, dim3(n), dim3(threads), 0, stream, table, pairs, dtype, ids, positions, req_index, cu_q, seq_lens,
                    state_slots, state, buckets, mul_prev, mul_cur, out, hidden, vocab, err);
}

// ------------------------------------------------------------------------------------------
// out[n][:] = scale * norm(x[n][:]) * act(gate[n][:]).  The norm (optional) divides each of `groups` equal parts of a row by its
// own root mean square and multiplies by a weight of the row's length or, shared by the parts, of a part's.  act: sigmoid or
// silu; gate may be null.  Rows of x, gate and out may be slices of wider rows.  A warp per part of up to 256 elements, else
// a block.
// ------------------------------------------------------------------------------------------
struct NormGateArgs {
  const void* x; long long ldx;
  const float* weight; int shared_weight;      // null: none
  int norm; float eps;
  const float* gate; long long ldg; int silu;
  float scale;
  void* out; long long ldo;
  int groups, part;
  long long items;
};

template <typename TO>
__device__ __forceinline__ void ng_store(const NormGateArgs& a, long long n, int g, int e, float x, float f) {
  float y = x * f;
  const int c = g * a.part + e;
  if (a.weight) y *= a.weight[a.shared_weight ? e : c];
  if (a.gate) {
    const float z = a.gate[n * a.ldg + c];
    const float s = 1.f / (1.f + expf(-z));
    y *= a.silu ? z * s : s;
  }
  ((TO*)a.out)[n * a.ldo + c] = from_f32<TO>(y);
}

template <typename TX, typename TO>
__global__ void __launch_bounds__(256)
norm_gate_warp_kernel(NormGateArgs a) {
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= a.items) return;
  const int lane = threadIdx.x & 31, g = (int)(item % a.groups);
  const long long n = item / a.groups;
  const TX* x = (const TX*)a.x + n * a.ldx + (long long)g * a.part;
  float v[8];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int e = j * 32 + lane;
    v[j] = e < a.part ? to_f32<TX>(x[e]) : 0.f;
    ss = fmaf(v[j], v[j], ss);
  }
  const float f = a.norm ? a.scale / sqrtf(warp_sum(ss) / (float)a.part + a.eps) : a.scale;
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (j * 32 + lane < a.part) ng_store<TO>(a, n, g, j * 32 + lane, v[j], f);
}

template <typename TX, typename TO>
__global__ void __launch_bounds__(256)
norm_gate_block_kernel(NormGateArgs a) {
  __shared__ float scratch[33];
  ifb_pdl_wait();
  ifb_pdl_trigger();
  const int g = (int)(blockIdx.x % a.groups);
  const long long n = blockIdx.x / a.groups;
  const TX* x = (const TX*)a.x + n * a.ldx + (long long)g * a.part;
  float v[8];                                            // the first 2,048 elements stay in registers
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int e = j * 256 + threadIdx.x;
    v[j] = e < a.part ? to_f32<TX>(x[e]) : 0.f;
    ss = fmaf(v[j], v[j], ss);
  }
  float f = a.scale;
  if (a.norm) {
    for (int e = 2048 + threadIdx.x; e < a.part; e += 256) { const float y = to_f32<TX>(x[e]); ss = fmaf(y, y, ss); }
    f = a.scale / sqrtf(block_sum(ss, scratch) / (float)a.part + a.eps);
  }
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (j * 256 + threadIdx.x < a.part) ng_store<TO>(a, n, g, j * 256 + threadIdx.x, v[j], f);
  for (int e = 2048 + threadIdx.x; e < a.part; e += 256) ng_store<TO>(a, n, g, e, to_f32<TX>(x[e]), f);
}

template <typename TX, typename TO>
static int ng_launch(const NormGateArgs& a, cudaStream_t s) {
  if (a.part <= 256)
    return ifb_launch(norm_gate_warp_kernel<TX, TO>, dim3((unsigned)((a.items + 7) / 8)), dim3(256), 0, s, a);
  return ifb_launch(norm_gate_block_kernel<TX, TO>, dim3((unsigned)a.items), dim3(256), 0, s, a);
}

IFB_EXPORT int ifb_norm_gate_rows(const void* x, int x_dtype, long long ldx, const float* weight, int shared_weight, int norm, float eps,
                                  const float* gate, long long ldg, int silu, float scale, void* out, int out_dtype, long long ldo,
                                  int n, int width, int groups, cudaStream_t stream) {
  if (n <= 0 || width <= 0) return IFB_OK;
  if (groups < 1 || width % groups) return IFB_ERR_SIZE;
  const long long items = (long long)n * groups;
  if (items > 0x7fffffffll) return IFB_ERR_SIZE;
  NormGateArgs a{x, ldx, weight, shared_weight, norm, eps, gate, ldg, silu, scale, out, ldo, groups, width / groups, items};
  const bool xb = x_dtype == IFB_BF16, ob = out_dtype == IFB_BF16;
  if ((!xb && x_dtype != IFB_F32) || (!ob && out_dtype != IFB_F32)) return IFB_ERR_DTYPE;
  if (xb) return ob ? ng_launch<__nv_bfloat16, __nv_bfloat16>(a, stream) : ng_launch<__nv_bfloat16, float>(a, stream);
  return ob ? ng_launch<float, __nv_bfloat16>(a, stream) : ng_launch<float, float>(a, stream);
}
