// What becomes of the experts' outputs of a routed feed-forward (float32 rows, bfloat16 model):
//   v[t] = sum_k weights[t][k] * y_k (+ shared), y_k = partial[row of pair (t, k)], or x[t] where the choice is an identity (ids >= E),
// in the order of k, float32; then either out[t] = v[t] rounded once, or, for layers that norm a sublayer's output,
//   h[t] += mult * v / sqrt(mean(v^2) + eps) * w,  y[t] = h[t] rounded (if y): the output never leaves the chip.
// pos: the row of every pair (null: the pair's own number); shared: bfloat16 rows by token, and / or shared_rows: float32 rows by token.
#include "common.cuh"

using namespace dli;
typedef __nv_bfloat16 bf16;

namespace {

struct Params {
  const float* partial;
  const int* pos;
  const int* ids;
  const float* weights;
  const bf16* x;
  const bf16* shared;
  const float* shared_rows;
  int W, E, top;
};

__device__ __forceinline__ void combined8(const Params& p, size_t t, int c, float (&acc)[8]) {
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
  for (int k = 0; k < p.top; ++k) {
    const size_t pair = t * p.top + k;
    const float w = p.weights[pair];
    float v[8];
    if (p.ids[pair] < p.E) load8(p.partial + (p.pos ? (size_t)p.pos[pair] : pair) * p.W + c, v);
    else load8(p.x + t * p.W + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] = fmaf(w, v[i], acc[i]);
  }
  if (p.shared) {
    float v[8];
    load8(p.shared + t * p.W + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] += v[i];
  }
  if (p.shared_rows) {
    float v[8];
    load8(p.shared_rows + t * p.W + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] += v[i];
  }
}

// eight columns a thread (W is a multiple of 8)
__global__ void moe_combine_kernel(bf16* __restrict__ out, const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float acc[8];
    combined8(p, t, c, acc);
    store8(out + t * p.W + c, acc);
  }
}

__global__ void moe_combine_norm_add_kernel(float* __restrict__ h, bf16* __restrict__ y, const float* __restrict__ w, float eps, float mult, const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];  // W
  __shared__ float red[33];
  const size_t t = blockIdx.x;
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {
    float acc[8];
    combined8(p, t, c, acc);
    store8(row + c, acc);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(acc[i], acc[i], ss);
  }
  const float f = mult / sqrtf(block_sum(ss, red) / (float)p.W + eps);
  for (int c = threadIdx.x * 8; c < p.W; c += blockDim.x * 8) {  // (every thread reads back what it wrote)
    float v[8], hv[8], wv[8];
    load8(row + c, v);
    load8(h + t * p.W + c, hv);
    load8(w + c, wv);
#pragma unroll
    for (int i = 0; i < 8; ++i) hv[i] += f * (v[i] * wv[i]);
    store8(h + t * p.W + c, hv);
    if (y) store8(y + t * p.W + c, hv);
  }
}

int block_threads(int W) { return W >= 4096 ? 512 : W >= 2048 ? 256 : W >= 1024 ? 128 : 64; }

}  // namespace

// h null: out [n][W]; else h [n][W] float32 (and y, or null).
DLI_EXPORT int dli_moe_combine(void* out, float* h, void* y, const float* norm_w, float eps, float mult, const float* partial, const int* pos, const int* ids,
                               const float* weights, const void* x, const void* shared, const float* shared_rows, int n, int W, int E, int top,
                               cudaStream_t stream) {
  if (n == 0) return 0;
  if (W < 8 || (W % 8) || top < 1 || E < 1 || (h ? !norm_w || W > 12160 : !out) ||
      ((((uintptr_t)out) | ((uintptr_t)h) | ((uintptr_t)y) | ((uintptr_t)norm_w) | ((uintptr_t)partial) | ((uintptr_t)x) | ((uintptr_t)shared) | ((uintptr_t)shared_rows)) & 15))
    return DLI_ERR_UNSUPPORTED;
  const Params p{partial, pos, ids, weights, (const bf16*)x, (const bf16*)shared, shared_rows, W, E, top};
  if (!h) return (int)launch_pdl(moe_combine_kernel, dim3(n), dim3(block_threads(W)), 0, stream, 1, (bf16*)out, p);
  return (int)launch_pdl(moe_combine_norm_add_kernel, dim3(n), dim3(block_threads(W)), (size_t)W * sizeof(float), stream, 1, h, (bf16*)y, norm_w, eps, mult, p);
}
