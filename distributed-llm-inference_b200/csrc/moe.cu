// A routed mixture of small feed-forwards: the router (float32 throughout), and the experts' products one (token, chosen expert) pair at a
// time on the CUDA cores, for float32 models and for sizes that the tensor-core products (moe_few.cu, the grouped form in dense_gemm.cu) do
// not take.
#include <math_constants.h>

#include "common.cuh"
#include "expert_act.cuh"

using namespace dli;

namespace {

constexpr int ROUTE_THREADS = 512;  // at most: sixteen warps, an expert's row each, for a step of few tokens (a handful of blocks); four warps for more
constexpr int ROUTE_MANY_TOKENS = 256;  // from here on a block takes several tokens
constexpr int MAX_TOP = 32;
enum { ROUTE_SIGMOID = 0, ROUTE_SOFTMAX_CHOSEN = 1, ROUTE_SOFTMAX_ALL = 2 };

// sum_i w[i] * xs[i] over a warp (xs: the token's row as floats in shared memory); 16-byte loads when `vec`
template <typename T>
__device__ __forceinline__ float warp_dot(const T* __restrict__ w, const float* __restrict__ xs, int len, int lane, bool vec) {
  float acc = 0.f;
  if (vec) {
    for (int i = lane * 8; i < len; i += 256) {
      float v[8];
      load8(w + i, v);
#pragma unroll
      for (int k = 0; k < 8; ++k) acc = fmaf(v[k], xs[i + k], acc);
    }
  } else {
    for (int i = lane; i < len; i += 32) acc = fmaf(to_float(w[i]), xs[i], acc);
  }
  return warp_sum(acc);
}

// What a token chooses.  z = W_r x (float32 sums of float32 products); s = sigmoid(z); choice = s + correction.
// Groups: `groups` equal runs of neighbouring experts; a group's mark is the sum of its two largest choice scores (its
// one score if it has one expert); only the `keep` groups with the largest marks stay eligible.  The `top` eligible experts
// with the largest choice scores are chosen (ties: the lower index), in that order; weights = s[chosen] / (sum + 1e-20) * scale.
// mode ROUTE_SOFTMAX_CHOSEN: choice = z + correction instead, and weights = softmax over the chosen experts' choices * scale.
// mode ROUTE_SOFTMAX_ALL: s = softmax(z) over all experts, choice = s + correction, and weights = s[chosen] * scale as they are.
// Done by one warp, from the token's scores (ROUTE_SOFTMAX_ALL: its logits) and choice scores in shared memory.
__device__ __forceinline__ void choose_experts(int* __restrict__ ids, float* __restrict__ weights, float* score, float* choice, float* mark, int* picked,
                                               const float* __restrict__ correction, int E, int top, int groups, int keep, float scale, int mode, int lane) {
  if (mode == ROUTE_SOFTMAX_ALL) {  // the logits become their softmax
    float high = -CUDART_INF_F, sum = 0.f;
    for (int e = lane; e < E; e += 32) high = fmaxf(high, score[e]);
    high = warp_max(high);
    for (int e = lane; e < E; e += 32) sum += expf(score[e] - high);
    sum = warp_sum(sum);
    for (int e = lane; e < E; e += 32) {
      const float s = expf(score[e] - high) / sum;
      score[e] = s;
      choice[e] = s + correction[e];
    }
    __syncwarp();
  }
  if (groups > 1) {
    const int per = E / groups;
    for (int g = lane; g < groups; g += 32) {
      float a = -CUDART_INF_F, b = -CUDART_INF_F;  // the two largest
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float c = choice[e];
        if (c > a) { b = a; a = c; }
        else if (c > b) b = c;
      }
      mark[g] = per > 1 ? a + b : a;
    }
    __syncwarp();
    // the `keep` best groups: the others' experts cannot be chosen
    for (int round = 0; round < groups - keep; ++round) {  // drop the worst remaining group (ties: the higher index goes first)
      float worst = CUDART_INF_F;
      int at = -1;
      for (int g = lane; g < groups; g += 32) {
        const float m = mark[g];
        if (m != CUDART_INF_F && (m < worst || (m == worst && g > at))) { worst = m; at = g; }
      }
      for (int off = 16; off > 0; off >>= 1) {
        const float ow = __shfl_xor_sync(0xffffffffu, worst, off);
        const int oa = __shfl_xor_sync(0xffffffffu, at, off);
        if (oa >= 0 && (at < 0 || ow < worst || (ow == worst && oa > at))) { worst = ow; at = oa; }
      }
      if (lane == 0) mark[at] = CUDART_INF_F;  // +inf marks a dropped group
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (mark[e / per] == CUDART_INF_F) choice[e] = -CUDART_INF_F;
    __syncwarp();
  }
  float total = 0.f, largest = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -CUDART_INF_F;
    int at = -1;
    for (int e = lane; e < E; e += 32) {
      const float c = choice[e];
      if (at < 0 || c > best) {
        if (c > best || at < 0) { best = c; at = e; }
      }
    }
    for (int off = 16; off > 0; off >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, off);
      const int oa = __shfl_xor_sync(0xffffffffu, at, off);
      if (oa >= 0 && (at < 0 || ob > best || (ob == best && oa < at))) { best = ob; at = oa; }
    }
    if (lane == 0) {
      picked[k] = at;
      choice[at] = -CUDART_INF_F;
    }
    if (mode == ROUTE_SOFTMAX_CHOSEN) {  // the first one chosen has the largest logit
      if (k == 0) largest = score[at];
      total += expf(score[at] - largest);
    } else {
      total += score[at];
    }
    __syncwarp();
  }
  const float f = mode == ROUTE_SOFTMAX_ALL ? scale : scale / (mode == ROUTE_SOFTMAX_CHOSEN ? total : total + 1e-20f);
  for (int k = lane; k < top; k += 32) {
    ids[k] = picked[k];
    weights[k] = (mode == ROUTE_SOFTMAX_CHOSEN ? expf(score[picked[k]] - largest) : score[picked[k]]) * f;
  }
}

__device__ __forceinline__ void put_score(float* score, float* choice, int e, float z, const float* __restrict__ correction, int mode) {
  const float s = mode == ROUTE_SIGMOID ? 1.f / (1.f + expf(-z)) : mode == ROUTE_SOFTMAX_CHOSEN ? z + correction[e] : z;
  score[e] = s;
  choice[e] = mode == ROUTE_SIGMOID ? s + correction[e] : s;
}

// A step of few tokens: a block per token, a warp per expert's row in turn.
template <typename T>
__global__ void __launch_bounds__(ROUTE_THREADS) moe_route_kernel(int* __restrict__ ids, float* __restrict__ weights, const T* __restrict__ x,
                                                                  const float* __restrict__ router, const float* __restrict__ correction,
                                                                  int W, int E, int top, int groups, int keep, float scale, int mode) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];  // x [W] | score [E] | choice [E] | mark [groups]
  float* xs = sm;
  float* score = xs + W;
  float* choice = score + E;
  float* mark = choice + E;
  __shared__ int picked[MAX_TOP];
  const size_t t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int i = threadIdx.x; i < W; i += blockDim.x) xs[i] = to_float(x[t * W + i]);
  __syncthreads();
  const bool vec = (W % 8) == 0 && (((uintptr_t)router) & 15) == 0;
  for (int e = warp; e < E; e += blockDim.x >> 5) {
    const float z = warp_dot<float>(router + (size_t)e * W, xs, W, lane, vec);
    if (lane == 0) put_score(score, choice, e, z, correction, mode);
  }
  __syncthreads();
  if (warp == 0) choose_experts(ids + t * top, weights + t * top, score, choice, mark, picked, correction, E, top, groups, keep, scale, mode, lane);
}

// A portion of many tokens: a block takes four of them and a warp four experts' rows at a time, so that a number of either, once read,
// serves four products.  Every sum is added up in the order of the kernel above.  W a multiple of 8, 16-byte aligned rows.
constexpr int ROUTE_TOKENS = 4, ROUTE_ROWS = 4;
template <typename T>
__global__ void __launch_bounds__(ROUTE_TOKENS * 32) moe_route_many_kernel(int* __restrict__ ids, float* __restrict__ weights, const T* __restrict__ x,
                                                                           const float* __restrict__ router, const float* __restrict__ correction, int n,
                                                                           int W, int E, int top, int groups, int keep, float scale, int mode) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];  // per token: score [E] | choice [E] | mark [groups]
  __shared__ int picked[ROUTE_TOKENS][MAX_TOP];
  const int per_token = 2 * E + groups;
  const size_t t0 = (size_t)blockIdx.x * ROUTE_TOKENS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const T* rows[ROUTE_TOKENS];
#pragma unroll
  for (int j = 0; j < ROUTE_TOKENS; ++j) rows[j] = x + (t0 + j < (size_t)n ? t0 + j : (size_t)n - 1) * W;
  for (int e0 = warp * ROUTE_ROWS; e0 < E; e0 += ROUTE_TOKENS * ROUTE_ROWS) {
    float acc[ROUTE_ROWS][ROUTE_TOKENS];
#pragma unroll
    for (int r = 0; r < ROUTE_ROWS; ++r)
#pragma unroll
      for (int j = 0; j < ROUTE_TOKENS; ++j) acc[r][j] = 0.f;
    const float* w[ROUTE_ROWS];
#pragma unroll
    for (int r = 0; r < ROUTE_ROWS; ++r) w[r] = router + (size_t)min(e0 + r, E - 1) * W;
    for (int i = lane * 8; i < W; i += 256) {
      float xv[ROUTE_TOKENS][8];
#pragma unroll
      for (int j = 0; j < ROUTE_TOKENS; ++j) load8(rows[j] + i, xv[j]);
#pragma unroll
      for (int r = 0; r < ROUTE_ROWS; ++r) {
        float wv[8];
        load8(w[r] + i, wv);
#pragma unroll
        for (int j = 0; j < ROUTE_TOKENS; ++j)
#pragma unroll
          for (int k = 0; k < 8; ++k) acc[r][j] = fmaf(wv[k], xv[j][k], acc[r][j]);
      }
    }
#pragma unroll
    for (int r = 0; r < ROUTE_ROWS; ++r)
#pragma unroll
      for (int j = 0; j < ROUTE_TOKENS; ++j) {
        const float z = warp_sum(acc[r][j]);
        if (lane == 0 && e0 + r < E) put_score(sm + j * per_token, sm + j * per_token + E, e0 + r, z, correction, mode);
      }
  }
  __syncthreads();
  const size_t t = t0 + warp;  // a warp chooses for one token
  if (t < (size_t)n) {
    float* score = sm + warp * per_token;
    choose_experts(ids + t * top, weights + t * top, score, score + E, score + 2 * E, picked[warp], correction, E, top, groups, keep, scale, mode, lane);
  }
}

constexpr int PAIR_THREADS = 128;
constexpr int PAIR_ROWS = 16;  // rows of the intermediate size a block computes

// GLU: hidden[pair][j] = act(gate_e[j] . x) * (up_e[j] . x), e = ids[pair], x the pair's token; w [E][2 ff][W]: gate rows, then up rows.
// Else: hidden[pair][j] = act(up_e[j] . x); w [E][ff][W].  A pair whose expert is E or above (an identity) has no hidden row.
// The sums are rounded to the activation dtype before the activation, as a product that stored them would have.
template <typename T, bool GLU>
__global__ void __launch_bounds__(PAIR_THREADS) moe_pair_up_kernel(T* __restrict__ hidden, const T* __restrict__ x, const int* __restrict__ ids,
                                                                        const T* __restrict__ w, int W, int ff, int E, int top, int act) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float xs[];
  const size_t pair = blockIdx.y;
  const size_t t = pair / top;
  const int e = ids[pair];
  if (e >= E) return;  // the whole block
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int i = threadIdx.x; i < W; i += PAIR_THREADS) xs[i] = to_float(x[t * W + i]);
  __syncthreads();
  const T* we = w + (size_t)e * (GLU ? 2 : 1) * ff * W;
  const bool vec = (W % 8) == 0 && (((uintptr_t)w) & 15) == 0;
  const int j0 = blockIdx.x * PAIR_ROWS;
  for (int j = j0 + warp; j < min(j0 + PAIR_ROWS, ff); j += PAIR_THREADS / 32) {
    const float g = warp_dot<T>(we + (size_t)j * W, xs, W, lane, vec);
    if constexpr (GLU) {
      const float u = warp_dot<T>(we + (size_t)(ff + j) * W, xs, W, lane, vec);
      if (lane == 0) hidden[pair * ff + j] = from_float<T>(glu_act(to_float(from_float<T>(g)), act) * to_float(from_float<T>(u)));
    } else {
      if (lane == 0) hidden[pair * ff + j] = from_float<T>(plain_act(to_float(from_float<T>(g)), act));
    }
  }
}

// out[t][c] = sum_k weights[t][k] * y_k (+ shared[t][c]), y_k = down_e(k)[c] . hidden[t top + k], or x[t][c] for an identity (e >= E);
// added in the order of the choice, float32, one rounding.  w [E][W][ff]; shared may be null.
template <typename T>
__global__ void __launch_bounds__(PAIR_THREADS) moe_pair_down_kernel(T* __restrict__ out, const T* __restrict__ hidden, const int* __restrict__ ids,
                                                                     const float* __restrict__ weights, const T* __restrict__ w,
                                                                     const T* __restrict__ x, const T* __restrict__ shared, int W, int ff, int E,
                                                                     int top) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float hs[];  // the token's `top` hidden rows
  const size_t t = blockIdx.y;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int i = threadIdx.x; i < top * ff; i += PAIR_THREADS)
    if (ids[t * top + i / ff] < E) hs[i] = to_float(hidden[t * top * ff + i]);
  __syncthreads();
  const bool vec = (ff % 8) == 0 && (((uintptr_t)w) & 15) == 0;
  const int c0 = blockIdx.x * PAIR_ROWS;
  for (int c = c0 + warp; c < min(c0 + PAIR_ROWS, W); c += PAIR_THREADS / 32) {
    float acc = 0.f;
    for (int k = 0; k < top; ++k) {
      const int e = ids[t * top + k];
      const float d = e < E ? warp_dot<T>(w + ((size_t)e * W + c) * ff, hs + (size_t)k * ff, ff, lane, vec) : to_float(x[t * W + c]);
      acc = fmaf(weights[t * top + k], d, acc);
    }
    if (lane == 0) out[t * W + c] = from_float<T>(shared ? acc + to_float(shared[t * W + c]) : acc);
  }
}

template <typename K>
inline cudaError_t allow_smem(K kernel, size_t smem, MaxPerDevice& set) {
  if ((int)smem > 48 * 1024 && set.here() < (int)smem) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
    set.here() = (int)smem;
  }
  return cudaSuccess;
}

}  // namespace

DLI_EXPORT int dli_moe_route(int* ids, float* weights, const void* x, const float* router, const float* correction, int n, int W, int E, int top,
                             int groups, int keep, float scale, int mode, int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  if (mode < ROUTE_SIGMOID || mode > ROUTE_SOFTMAX_ALL) return DLI_ERR_UNSUPPORTED;
  if (W < 1 || E < 1 || top < 1 || top > MAX_TOP || groups < 1 || E % groups || keep < 1 || keep > groups || top > keep * (E / groups))
    return DLI_ERR_UNSUPPORTED;
  const size_t smem = ((size_t)W + 2 * E + groups) * sizeof(float);
  if (smem > 200 * 1024) return DLI_ERR_UNSUPPORTED;
  const int threads = n <= ROUTE_MANY_TOKENS ? ROUTE_THREADS : 128;
  cudaError_t e;
  const size_t many_smem = (size_t)ROUTE_TOKENS * (2 * E + groups) * sizeof(float);
  if (n > ROUTE_MANY_TOKENS && (W % 8) == 0 && ((((uintptr_t)x) | ((uintptr_t)router)) & 15) == 0 && many_smem <= 48 * 1024 - ROUTE_TOKENS * MAX_TOP * sizeof(int)) {
    const dim3 grid((n + ROUTE_TOKENS - 1) / ROUTE_TOKENS), block(ROUTE_TOKENS * 32);
    if (dtype == DLI_F32)
      return (int)launch_pdl((moe_route_many_kernel<float>), grid, block, many_smem, stream, 1, ids, weights, (const float*)x, router, correction, n, W, E, top,
                             groups, keep, scale, mode);
    return (int)launch_pdl((moe_route_many_kernel<__nv_bfloat16>), grid, block, many_smem, stream, 1, ids, weights, (const __nv_bfloat16*)x, router, correction,
                           n, W, E, top, groups, keep, scale, mode);
  }
  if (dtype == DLI_F32) {
    static MaxPerDevice set;
    if ((e = allow_smem(moe_route_kernel<float>, smem, set)) != cudaSuccess) return (int)e;
    e = launch_pdl((moe_route_kernel<float>), dim3(n), dim3(threads), smem, stream, 1, ids, weights, (const float*)x, router, correction, W, E,
                   top, groups, keep, scale, mode);
  } else {
    static MaxPerDevice set;
    if ((e = allow_smem(moe_route_kernel<__nv_bfloat16>, smem, set)) != cudaSuccess) return (int)e;
    e = launch_pdl((moe_route_kernel<__nv_bfloat16>), dim3(n), dim3(threads), smem, stream, 1, ids, weights, (const __nv_bfloat16*)x, router,
                   correction, W, E, top, groups, keep, scale, mode);
  }
  return (int)e;
}

template <typename T, bool GLU>
static cudaError_t launch_pairs(void* out, void* hidden, const void* x, const int* ids, const float* weights, const void* w_up, const void* w_down,
                                const void* shared, int n, int W, int ff, int E, int top, int act, cudaStream_t stream) {
  const size_t smem_up = (size_t)W * sizeof(float), smem_down = (size_t)top * ff * sizeof(float);
  const dim3 grid_up((ff + PAIR_ROWS - 1) / PAIR_ROWS, n * top), grid_down((W + PAIR_ROWS - 1) / PAIR_ROWS, n);
  static MaxPerDevice set_up, set_down;
  cudaError_t e;
  if ((e = allow_smem(moe_pair_up_kernel<T, GLU>, smem_up, set_up)) != cudaSuccess) return e;
  if ((e = allow_smem(moe_pair_down_kernel<T>, smem_down, set_down)) != cudaSuccess) return e;
  e = launch_pdl((moe_pair_up_kernel<T, GLU>), grid_up, dim3(PAIR_THREADS), smem_up, stream, 1, (T*)hidden, (const T*)x, ids, (const T*)w_up, W, ff, E, top,
                 act);
  if (e != cudaSuccess) return e;
  return launch_pdl((moe_pair_down_kernel<T>), grid_down, dim3(PAIR_THREADS), smem_down, stream, 1, (T*)out, (const T*)hidden, ids, weights, (const T*)w_down,
                    (const T*)x, (const T*)shared, W, ff, E, top);
}

// hidden: scratch [n top][ff] in the activation dtype.  gated: w_up holds gate rows, then up rows; else up rows alone.  Experts from E on
// are identities; shared [n][W] (or null) is added to every token's sum.
DLI_EXPORT int dli_moe_pairs(void* out, void* hidden, const void* x, const int* ids, const float* weights, const void* w_up, const void* w_down,
                             const void* shared, int n, int W, int ff, int E, int top, int act, int gated, int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  const size_t smem_up = (size_t)W * sizeof(float), smem_down = (size_t)top * ff * sizeof(float);
  if (W < 1 || ff < 1 || E < 1 || top < 1 || (long long)n * top > 65535 || smem_up > 200 * 1024 || smem_down > 200 * 1024) return DLI_ERR_UNSUPPORTED;
#define DLI_PAIRS(T, GLU) launch_pairs<T, GLU>(out, hidden, x, ids, weights, w_up, w_down, shared, n, W, ff, E, top, act, stream)
  if (dtype == DLI_F32) return (int)(gated ? DLI_PAIRS(float, true) : DLI_PAIRS(float, false));
  return (int)(gated ? DLI_PAIRS(__nv_bfloat16, true) : DLI_PAIRS(__nv_bfloat16, false));
#undef DLI_PAIRS
}
