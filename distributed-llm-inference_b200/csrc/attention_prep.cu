// What lies between an attention mixer's projections and its attention kernel when queries and keys are
// normed over their whole projection or head by head, or when the keys and values are one cached latent; and what lies behind the
// attention kernel when its output is gated.
// float32 and bfloat16 instantiations; all arithmetic is float32.
#include "common.cuh"

using namespace dli;

namespace {

// Norms of q and k before the rotation: none, over the whole projection (all heads together), or over each head.
enum { NORM_NONE = 0, NORM_PROJECTION = 1, NORM_HEAD = 2 };

struct QkStoreArgs {
  long long proj_stride;
  const float* wq;  // NORM_PROJECTION: nh * d and nkv * d numbers; NORM_HEAD: d numbers each
  const float* wk;
  float eps;
  const int* positions;
  const float* inv_freq;
  const int* slots;
  int nh, nkv, d, dv;  // heads; size of a query or key, of a value
  int kd, vd;          // rows as they leave (kd >= d, vd >= dv, padded with zeros)
  int rot, page_size, write_kv, norm, values_from_keys;
};

// One block per token.  proj row: q (nh * d columns) | k (nkv * d columns) | v (nkv * dv columns), then whatever else the product
// made; without write_kv only q is read.
//   q <- q / rms(q) * wq,  k <- k / rms(k) * wk      (rms over what `norm` says)
//   rotary (rotate-half pairing, first `rot` dimensions of each head, angle float32(position) * inv_freq[i])
//   q -> q_out [n, nh, kd];  k -> k_pool at the token's slot;
//   v_pool gets the keys as projected (values_from_keys != 0; dv = d) or the nkv * dv columns behind k.
template <typename T>
__global__ void qk_norm_rotary_store_kernel(T* __restrict__ q_out, const T* __restrict__ proj, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                            const QkStoreArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];  // (nh + nkv) * d | 1 / rms of every head (NORM_HEAD)
  __shared__ float red[33];
  const int t = blockIdx.x, nh = a.nh, nkv = a.nkv, d = a.d;
  const int nq = nh * d, nk = a.write_kv ? nkv * d : 0;
  float* head_r = row + (nh + nkv) * d;
  const T* src = proj + (size_t)t * a.proj_stride;
  float sq = 0.f, sk = 0.f;
  for (int e = threadIdx.x; e < nq + nk; e += blockDim.x) {
    const float x = to_float(src[e]);
    row[e] = x;
    if (e < nq) sq = fmaf(x, x, sq); else sk = fmaf(x, x, sk);
  }
  float rq = 1.f, rk = 1.f;
  if (a.norm == NORM_PROJECTION) {
    rq = 1.f / sqrtf(block_sum(sq, red) / (float)nq + a.eps);
    if (nk) rk = 1.f / sqrtf(block_sum(sk, red) / (float)nk + a.eps);
  } else {
    __syncthreads();
    if (a.norm == NORM_HEAD) {
      for (int head = threadIdx.x >> 5; head < (nq + nk) / d; head += blockDim.x >> 5) {
        float ss = 0.f;
        for (int i = threadIdx.x & 31; i < d; i += 32) ss = fmaf(row[head * d + i], row[head * d + i], ss);
        ss = warp_sum(ss);
        if ((threadIdx.x & 31) == 0) head_r[head] = 1.f / sqrtf(ss / (float)d + a.eps);
      }
      __syncthreads();
    }
  }
  const float pos = (float)a.positions[t];
  const int half = a.rot >> 1;
  const int slot = a.write_kv ? a.slots[t] : 0;
  const long long page = slot / a.page_size;
  const int off = slot % a.page_size;
  for (int e = threadIdx.x; e < (nq + nk) / d * a.kd; e += blockDim.x) {
    const int head = e / a.kd, i = e - head * a.kd;
    const bool is_q = head < nh;
    const int hh = is_q ? head : head - nh;
    float x = 0.f;
    if (i < d) {
      const float r = a.norm == NORM_HEAD ? head_r[head] : is_q ? rq : rk;
      const float* w = (is_q ? a.wq : a.wk) + (a.norm == NORM_PROJECTION ? hh * d : 0);
      const float* h = row + head * d;
      x = h[i] * r * (a.norm ? w[i] : 1.f);
      if (i < a.rot) {
        const int j = i < half ? i : i - half, other = i < half ? i + half : i - half;
        const float xp = h[other] * r * (a.norm ? w[other] : 1.f);
        float sn, cs;
        sincosf(pos * a.inv_freq[j], &sn, &cs);
        x = i < half ? x * cs - xp * sn : x * cs + xp * sn;
      }
    }
    if (is_q) q_out[((size_t)t * nh + hh) * a.kd + i] = from_float<T>(x);
    else k_pool[((page * nkv + hh) * a.page_size + off) * a.kd + i] = from_float<T>(x);
  }
  if (!a.write_kv) return;
  const T* vsrc = src + nq + (a.values_from_keys ? 0 : nk);
  for (int e = threadIdx.x; e < nkv * a.vd; e += blockDim.x) {
    const int hh = e / a.vd, i = e - hh * a.vd;
    v_pool[((page * nkv + hh) * a.page_size + off) * a.vd + i] = i < a.dv ? vsrc[hh * a.dv + i] : from_float<T>(0.f);
  }
}

template <typename T>
__device__ __forceinline__ void copy8(T* dst, const T* src) {
#pragma unroll
  for (int i = 0; i < (int)(8 * sizeof(T) / 16); ++i) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
}

// The same with 16-byte accesses, for d, dv, kd, vd % 8 == 0, rot % 16 == 0 and 16-byte aligned rows.  A work item is a run of
// eight columns — together with its partner run, half the rotated span further, where it is rotated.  The token's
// cosines and sines are computed once, in shared memory, not once per head.
template <typename T>
__global__ void qk_norm_rotary_store_vec_kernel(T* __restrict__ q_out, const T* __restrict__ proj, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                                const QkStoreArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float cs[];  // cos [rot / 2] | sin [rot / 2] | 1 / rms of every head (NORM_HEAD)
  __shared__ float red[33];
  const int t = blockIdx.x, nh = a.nh, nkv = a.nkv, d = a.d;
  const int nq = nh * d, nk = a.write_kv ? nkv * d : 0, half = a.rot >> 1;
  const int heads = nh + (a.write_kv ? nkv : 0);
  float* head_r = cs + a.rot;
  const T* src = proj + (size_t)t * a.proj_stride;
  const float pos = (float)a.positions[t];
  for (int j = threadIdx.x; j < half; j += blockDim.x) sincosf(pos * a.inv_freq[j], &cs[half + j], &cs[j]);
  float rq = 1.f, rk = 1.f;
  if (a.norm == NORM_PROJECTION) {
    float sq = 0.f, sk = 0.f;
    for (int e = threadIdx.x * 8; e < nq + nk; e += blockDim.x * 8) {
      float x[8];
      load8(src + e, x);
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) ss = fmaf(x[k], x[k], ss);
      if (e < nq) sq += ss; else sk += ss;
    }
    rq = 1.f / sqrtf(block_sum(sq, red) / (float)nq + a.eps);
    if (nk) rk = 1.f / sqrtf(block_sum(sk, red) / (float)nk + a.eps);
  } else if (a.norm == NORM_HEAD) {
    // a head belongs to `lanes` neighbouring lanes (a power of two), each of which sums runs of eight
    const int runs = d >> 3;
    int lanes = 1;
    while (lanes < runs && lanes < 32) lanes <<= 1;
    const int lane = threadIdx.x & (lanes - 1), step = blockDim.x / lanes;
    for (int first = 0; first < heads; first += step) {  // every thread takes part in every round: the shuffles need whole warps
      const int head = first + threadIdx.x / lanes;
      float ss = 0.f;
      if (head < heads)
        for (int i = lane; i < runs; i += lanes) {
          float x[8];
          load8(src + head * d + i * 8, x);
#pragma unroll
          for (int k = 0; k < 8; ++k) ss = fmaf(x[k], x[k], ss);
        }
      for (int off = lanes >> 1; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
      if (lane == 0 && head < heads) head_r[head] = 1.f / sqrtf(ss / (float)d + a.eps);
    }
    __syncthreads();
  } else {
    __syncthreads();
  }
  const int slot = a.write_kv ? a.slots[t] : 0;
  const long long page = slot / a.page_size;
  const int off = slot % a.page_size;
  // items per head: half / 8 rotated pairs, (d - rot) / 8 runs that pass unrotated, (kd - d) / 8 runs of zeros
  const int pair_items = half >> 3, data_items = pair_items + ((d - a.rot) >> 3), per_head = data_items + ((a.kd - d) >> 3);
  for (int item = threadIdx.x; item < heads * per_head; item += blockDim.x) {
    const int head = item / per_head, it = item - head * per_head;
    const bool is_q = head < nh;
    const int hh = is_q ? head : head - nh;
    const float r = a.norm == NORM_HEAD ? head_r[head] : is_q ? rq : rk;
    const float* w = (is_q ? a.wq : a.wk) + (a.norm == NORM_PROJECTION ? hh * d : 0);
    const T* hsrc = src + head * d;  // q heads, then k heads, lie back to back
    T* dst = is_q ? q_out + ((size_t)t * nh + hh) * a.kd : k_pool + ((page * nkv + hh) * a.page_size + off) * a.kd;
    if (it < pair_items) {
      const int i = it * 8;
      float lo[8], hi[8], wl[8], wh[8], ol[8], oh[8];
      load8(hsrc + i, lo);
      load8(hsrc + i + half, hi);
      if (a.norm) {
        load8(w + i, wl);
        load8(w + i + half, wh);
      }
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float u = lo[k] * r * (a.norm ? wl[k] : 1.f), v = hi[k] * r * (a.norm ? wh[k] : 1.f);
        const float c = cs[i + k], sn = cs[half + i + k];
        ol[k] = u * c - v * sn;
        oh[k] = v * c + u * sn;
      }
      store8(dst + i, ol);
      store8(dst + i + half, oh);
    } else if (it < data_items) {
      const int i = a.rot + (it - pair_items) * 8;
      float x[8], wv[8];
      load8(hsrc + i, x);
      if (a.norm) {
        load8(w + i, wv);
#pragma unroll
        for (int k = 0; k < 8; ++k) x[k] = x[k] * r * wv[k];
      }
      store8(dst + i, x);
    } else {
      const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      store8(dst + d + (it - data_items) * 8, zero);
    }
  }
  if (!a.write_kv) return;
  const T* vsrc = src + nq + (a.values_from_keys ? 0 : nk);
  const int vper = a.vd >> 3;
  for (int item = threadIdx.x; item < nkv * vper; item += blockDim.x) {
    const int hh = item / vper, i = (item - hh * vper) * 8;
    T* dst = v_pool + ((page * nkv + hh) * a.page_size + off) * a.vd + i;
    if (i < a.dv) {
      copy8(dst, vsrc + hh * a.dv + i);
    } else {
      const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      store8(dst, zero);
    }
  }
}

// out[t, c] *= sigmoid(gate[t, c]), eight columns a thread (cols % 8 == 0, aligned rows)
template <typename T>
__global__ void sigmoid_gate_vec_kernel(T* __restrict__ out, const T* __restrict__ gate, long long gate_stride, int n, int cols) {
  pdl_launch_dependents();
  pdl_wait();
  const int per_row = cols >> 3;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)n * per_row) return;
  const int t = (int)(idx / per_row), c = (int)(idx - (long long)t * per_row) * 8;
  float o[8], g[8];
  load8(out + (size_t)t * cols + c, o);
  load8(gate + (size_t)t * gate_stride + c, g);
#pragma unroll
  for (int k = 0; k < 8; ++k) o[k] = o[k] / (1.f + expf(-g[k]));
  store8(out + (size_t)t * cols + c, o);
}

// out[t, c] *= sigmoid(gate[t * gate_stride + c])
template <typename T>
__global__ void sigmoid_gate_kernel(T* __restrict__ out, const T* __restrict__ gate, long long gate_stride, int n, int cols) {
  pdl_launch_dependents();
  pdl_wait();
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long long)n * cols) return;
  const int t = (int)(idx / cols), c = (int)(idx - (long long)t * cols);
  const float g = to_float(gate[(size_t)t * gate_stride + c]);
  out[idx] = from_float<T>(to_float(out[idx]) / (1.f + expf(-g)));
}

}  // namespace

DLI_EXPORT int dli_qk_norm_rotary_store(void* q_out, const void* proj, long long proj_stride, const float* wq, const float* wk,
                                        float eps, const int* positions, const float* inv_freq, const int* slots, void* k_pool,
                                        void* v_pool, int n, int nh, int nkv, int d, int dv, int kd, int vd, int rot, int page_size, int write_kv,
                                        int norm, int values_from_keys, int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  const size_t smem = ((size_t)(nh + nkv) * d + nh + nkv) * sizeof(float);
  if (nh < 1 || nkv < 1 || d < 1 || dv < 1 || kd < d || vd < dv || rot < 0 || rot > d || (rot & 1) || page_size < 1 || smem > 200 * 1024 ||
      (rot && !inv_freq) || norm < NORM_NONE || norm > NORM_HEAD || (norm && (!wq || (write_kv && !wk))) || (values_from_keys && dv != d) ||
      (write_kv && (!slots || !k_pool || !v_pool)))
    return DLI_ERR_UNSUPPORTED;
  const QkStoreArgs a{proj_stride, wq, wk, eps, positions, inv_freq, slots, nh, nkv, d, dv, kd, vd, rot, page_size, write_kv, norm, values_from_keys};
  const int threads = (nh + nkv) * d >= 2048 ? 512 : 256;
  const size_t esize = dtype == DLI_F32 ? 4 : 2;
  const size_t vsmem = ((size_t)rot + nh + nkv) * sizeof(float);
  const bool aligned = (d % 8) == 0 && (dv % 8) == 0 && (kd % 8) == 0 && (vd % 8) == 0 && (rot % 16) == 0 && (proj_stride % 8) == 0 && vsmem <= 47 * 1024 &&
                       (((uintptr_t)q_out | (uintptr_t)proj | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)wq | (uintptr_t)wk) & 15) == 0 &&
                       ((size_t)d * esize) % 16 == 0;
  if (aligned) {
    const int items = (nh + nkv) * (d / 8);
    const int vt = items >= 256 ? 256 : (items >= 128 ? 128 : 64);
    if (dtype == DLI_F32)
      return (int)launch_pdl((qk_norm_rotary_store_vec_kernel<float>), dim3(n), dim3(vt), vsmem, stream, 1, (float*)q_out, (const float*)proj, (float*)k_pool,
                             (float*)v_pool, a);
    return (int)launch_pdl((qk_norm_rotary_store_vec_kernel<__nv_bfloat16>), dim3(n), dim3(vt), vsmem, stream, 1, (__nv_bfloat16*)q_out,
                           (const __nv_bfloat16*)proj, (__nv_bfloat16*)k_pool, (__nv_bfloat16*)v_pool, a);
  }
  cudaError_t e;
  if (dtype == DLI_F32) {
    static MaxPerDevice set;
    if ((int)smem > 47 * 1024 && set.here() < (int)smem) {
      e = cudaFuncSetAttribute(qk_norm_rotary_store_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
      set.here() = (int)smem;
    }
    e = launch_pdl((qk_norm_rotary_store_kernel<float>), dim3(n), dim3(threads), smem, stream, 1, (float*)q_out, (const float*)proj, (float*)k_pool,
                   (float*)v_pool, a);
  } else {
    static MaxPerDevice set;
    if ((int)smem > 47 * 1024 && set.here() < (int)smem) {
      e = cudaFuncSetAttribute(qk_norm_rotary_store_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
      set.here() = (int)smem;
    }
    e = launch_pdl((qk_norm_rotary_store_kernel<__nv_bfloat16>), dim3(n), dim3(threads), smem, stream, 1, (__nv_bfloat16*)q_out,
                   (const __nv_bfloat16*)proj, (__nv_bfloat16*)k_pool, (__nv_bfloat16*)v_pool, a);
  }
  return (int)e;
}

// ---------------------------------------------------------------- attention over a cached latent
// One block per token.  proj row: per head d plain and dr rotated query numbers (nh heads), then the down projection:
// r latent numbers and dr numbers of a key part that all heads share.
//   latent <- latent / rms(latent) * w_norm                      (float32; eps inside the root)
//   the first `rot` of the dr numbers of the key part and of every head's query part are rotated by the position
//   (rotate-half pairing, angle float32(position) * inv_freq[i]); the rest pass through
//   cache row  latent | key part      -> k_pool [pages][1][page_size][r + dr] at the token's slot (if slots)
//   query parts                       -> q_out [n][nh][r + dr], columns r .. r + dr of every head
template <typename T>
__global__ void latent_prep_kernel(T* __restrict__ q_out, const T* __restrict__ proj, long long proj_stride,
                                   const float* __restrict__ w_norm, float eps, const int* __restrict__ positions,
                                   const float* __restrict__ inv_freq, const int* __restrict__ slots, T* __restrict__ k_pool, int nh,
                                   int d, int dr, int r, int rot, int page_size, float amp) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float trig[];  // cos[half] | sin[half]
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int half = rot >> 1;
  const T* src = proj + (size_t)t * proj_stride;
  const T* down = src + (size_t)nh * (d + dr);
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf(pos * inv_freq[i], &sn, &cs);
    trig[i] = cs * amp;  // amp: one factor on every cosine and sine (1: none)
    trig[half + i] = sn * amp;
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < r; i += blockDim.x) {
    const float x = to_float(down[i]);
    ss = fmaf(x, x, ss);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)r + eps);  // (the barriers inside also publish trig)
  const int slot = slots ? slots[t] : -1;
  const int row = r + dr;
  T* krow = slot >= 0 ? k_pool + (size_t)slot * row : nullptr;  // one KV head: a page is page_size rows back to back
  if (krow)
    for (int i = threadIdx.x; i < r; i += blockDim.x) krow[i] = from_float<T>(to_float(down[i]) * inv * w_norm[i]);
  // rotated parts, a pair of partners (i, i + half) a thread: head nh is the shared key part
  const int pairs = half + (dr - rot);  // per head: the rotated pairs, then the numbers that pass through
  for (int e = threadIdx.x; e < (nh + 1) * pairs; e += blockDim.x) {
    const int head = e / pairs, j = e - head * pairs;
    const T* part = head < nh ? src + (size_t)head * (d + dr) + d : down + r;
    T* dst = head < nh ? q_out + ((size_t)t * nh + head) * row + r : (krow ? krow + r : nullptr);
    if (!dst) continue;
    if (j < half) {
      const float lo = to_float(part[j]), hi = to_float(part[j + half]);
      const float cs = trig[j], sn = trig[half + j];
      dst[j] = from_float<T>(lo * cs - hi * sn);
      dst[j + half] = from_float<T>(hi * cs + lo * sn);
    } else {
      dst[rot + j - half] = part[rot + j - half];
    }
  }
}

DLI_EXPORT int dli_latent_prep(void* q_out, const void* proj, long long proj_stride, const float* w_norm, float eps, const int* positions,
                               const float* inv_freq, const int* slots, void* k_pool, int n, int nh, int d, int dr, int r, int rot,
                               int page_size, float amp, int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  if (nh < 1 || d < 1 || dr < 0 || r < 1 || rot < 0 || rot > dr || (rot & 1) || (rot && !inv_freq) || (slots && !k_pool) || page_size < 1 ||
      rot * sizeof(float) > 48 * 1024)
    return DLI_ERR_UNSUPPORTED;
  const int work = r > (nh + 1) * dr ? r : (nh + 1) * dr;
  const int threads = work >= 4096 ? 256 : 128;  // small blocks: a token's work is short, and more blocks fit an SM
  const size_t smem = (size_t)(rot > 0 ? rot : 1) * sizeof(float);
  cudaError_t e;
  if (dtype == DLI_F32)
    e = launch_pdl((latent_prep_kernel<float>), dim3(n), dim3(threads), smem, stream, 1, (float*)q_out, (const float*)proj, proj_stride,
                   w_norm, eps, positions, inv_freq, slots, (float*)k_pool, nh, d, dr, r, rot, page_size, amp);
  else
    e = launch_pdl((latent_prep_kernel<__nv_bfloat16>), dim3(n), dim3(threads), smem, stream, 1, (__nv_bfloat16*)q_out,
                   (const __nv_bfloat16*)proj, proj_stride, w_norm, eps, positions, inv_freq, slots, (__nv_bfloat16*)k_pool, nh, d, dr, r,
                   rot, page_size, amp);
  return (int)e;
}

// ---------------------------------------------------------------- rotation, then a unit root mean square per head, then the pages
// One block per token, a warp per head.  x row: q (nh heads of d) | k (nkv heads of d) | v (nkv heads of dv), as the
// convolution left them.  Every q and k head is rotated on its first `rot` dimensions (rotate-half pairing, angle
// float32(position) * inv_freq[i]) and then, if unit_eps >= 0, divided by sqrt(mean(head^2) + unit_eps), all in float32.
// Rows of D = max(d, dv) numbers leave, the shorter of keys and values padded with zeros:
//   q -> q_out [n][nh][D];   k -> k_pool, v -> v_pool [pages][nkv][page_size][D] at the token's slot (if slots)
template <typename T>
__global__ void rotary_unit_store_kernel(T* __restrict__ q_out, const T* __restrict__ x, long long x_stride, const int* __restrict__ positions,
                                         const float* __restrict__ inv_freq, const int* __restrict__ slots, T* __restrict__ k_pool,
                                         T* __restrict__ v_pool, int nh, int nkv, int d, int dv, int D, int rot, float unit_eps, int page_size) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];  // cos[half] | sin[half] | a head of d floats per warp
  const int t = blockIdx.x;
  const int half = rot >> 1;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  float* trig = sm;
  float* buf = sm + rot + (size_t)warp * d;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * inv_freq[i], &trig[half + i], &trig[i]);
  __syncthreads();
  const T* src = x + (size_t)t * x_stride;
  const int slot = slots ? slots[t] : -1;
  const long long page = slot >= 0 ? slot / page_size : 0;
  const int off = slot >= 0 ? slot % page_size : 0;
  for (int head = warp; head < nh + 2 * nkv; head += warps) {
    if (head >= nh + nkv) {  // a value head: copied, padded
      if (slot < 0) continue;
      const int g = head - nh - nkv;
      const T* part = src + (size_t)(nh + nkv) * d + (size_t)g * dv;
      T* dst = v_pool + ((page * nkv + g) * page_size + off) * D;
      for (int i = lane; i < D; i += 32) dst[i] = i < dv ? part[i] : from_float<T>(0.f);
      continue;
    }
    const T* part = src + (size_t)head * d;
    float ss = 0.f;
    for (int i = lane; i < d; i += 32) {
      float v;
      if (i < half) {
        v = to_float(part[i]) * trig[i] - to_float(part[i + half]) * trig[half + i];
      } else if (i < rot) {
        v = to_float(part[i]) * trig[i - half] + to_float(part[i - half]) * trig[i];
      } else {
        v = to_float(part[i]);
      }
      buf[i] = v;
      ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    const float inv = unit_eps >= 0.f ? 1.f / sqrtf(ss / (float)d + unit_eps) : 1.f;
    T* dst;
    if (head < nh) {
      dst = q_out + ((size_t)t * nh + head) * D;
    } else {
      if (slot < 0) { __syncwarp(); continue; }
      dst = k_pool + ((page * nkv + (head - nh)) * page_size + off) * D;
    }
    __syncwarp();
    for (int i = lane; i < D; i += 32) dst[i] = from_float<T>(i < d ? buf[i] * inv : 0.f);
    __syncwarp();
  }
}

DLI_EXPORT int dli_rotary_unit_store(void* q_out, const void* x, long long x_stride, const int* positions, const float* inv_freq,
                                     const int* slots, void* k_pool, void* v_pool, int n, int nh, int nkv, int d, int dv, int rot,
                                     float unit_eps, int page_size, int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  if (nh < 1 || nkv < 1 || d < 1 || dv < 1 || rot < 0 || rot > d || (rot & 1) || (rot && !inv_freq) || (slots && (!k_pool || !v_pool)) || page_size < 1)
    return DLI_ERR_UNSUPPORTED;
  const int D = d > dv ? d : dv;
  const int heads = nh + 2 * nkv;
  const int threads = heads >= 8 ? 256 : (heads >= 4 ? 128 : 64);
  const size_t smem = ((size_t)rot + (size_t)(threads / 32) * d) * sizeof(float);
  if (smem > 48 * 1024) return DLI_ERR_UNSUPPORTED;
  cudaError_t e;
  if (dtype == DLI_F32)
    e = launch_pdl((rotary_unit_store_kernel<float>), dim3(n), dim3(threads), smem, stream, 1, (float*)q_out, (const float*)x, x_stride, positions,
                   inv_freq, slots, (float*)k_pool, (float*)v_pool, nh, nkv, d, dv, D, rot, unit_eps, page_size);
  else
    e = launch_pdl((rotary_unit_store_kernel<__nv_bfloat16>), dim3(n), dim3(threads), smem, stream, 1, (__nv_bfloat16*)q_out,
                   (const __nv_bfloat16*)x, x_stride, positions, inv_freq, slots, (__nv_bfloat16*)k_pool, (__nv_bfloat16*)v_pool, nh, nkv, d, dv, D,
                   rot, unit_eps, page_size);
  return (int)e;
}

// ---------------------------------------------------------------- whole-projection norm, temperature, mixed values, then the pages
// One block per token.  x row: q (nh heads of d) | k (nkv heads of d) | v (nkv heads of dv), plus a float32 bias (or none).
//   q <- q / rms(q over all heads) * wq * temp,  k <- k / rms(k over all heads) * wk                        (normed != 0)
//   temp = 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1) at position p                                 (temp_coef != 0)
//   mix 1: v -> source [n][nkv dv] (float32, for the layers behind this one);  mix 2: v <- (1 - lam) v + lam source
// Rows of D >= max(d, dv) numbers leave, padded with zeros: q -> q_out [n][nh][D]; k, v -> pools [pages][nkv][page_size][D]
// at the token's slot (if slots).  VEC columns a thread at a time (8: d, dv, D multiples of 8 and aligned rows; else 1).
template <typename TI, int VEC>
__device__ __forceinline__ void load_run(const TI* __restrict__ x, const float* __restrict__ bias, int c, float (&v)[VEC]) {
  if constexpr (VEC == 8) {
    load8(x + c, v);
    if (bias) {
      float b[8];
      load8(bias + c, b);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] += b[k];
    }
  } else {
    v[0] = to_float(x[c]) + (bias ? bias[c] : 0.f);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_run(T* __restrict__ dst, const float (&v)[VEC]) {
  if constexpr (VEC == 8) store8(dst, v);
  else dst[0] = from_float<T>(v[0]);
}

template <typename TI, typename T, int VEC>
__global__ void qk_norm_mix_store_kernel(T* __restrict__ q_out, const TI* __restrict__ x, const float* __restrict__ bias, const float* __restrict__ wq,
                                         const float* __restrict__ wk, float eps, const int* __restrict__ positions, float temp_coef, float temp_every,
                                         float* __restrict__ source, float lam, const int* __restrict__ slots, T* __restrict__ k_pool,
                                         T* __restrict__ v_pool, int nh, int nkv, int d, int dv, int D, int page_size, int mix, int normed) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int nq = nh * d, nk = nkv * d, nv = nkv * dv;
  const TI* src = x + (size_t)t * (nq + nk + nv);
  float rq = 1.f, rk = 1.f;
  if (normed) {
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x * VEC; c < nq + nk; c += blockDim.x * VEC) {
      float v[VEC];
      load_run<TI, VEC>(src, bias, c, v);
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < VEC; ++k) ss = fmaf(v[k], v[k], ss);
      if (c < nq) sq += ss; else sk += ss;
    }
    rq = 1.f / sqrtf(block_sum(sq, red) / (float)nq + eps);
    rk = 1.f / sqrtf(block_sum(sk, red) / (float)nk + eps);
  }
  if (temp_coef != 0.f) rq *= 1.f + temp_coef * logf(floorf((float)(positions[t] + 1) / temp_every) + 1.f);
  const int slot = slots ? slots[t] : -1;
  const long long page = slot >= 0 ? slot / page_size : 0;
  const int off = slot >= 0 ? slot - (int)page * page_size : 0;
  const int per = D / VEC;  // runs of a head's row as it leaves
  const int heads = nh + (slot >= 0 ? 2 * nkv : (mix == 1 ? 2 * nkv : 0));
  for (int item = threadIdx.x; item < heads * per; item += blockDim.x) {
    const int head = item / per, i = (item - head * per) * VEC;
    float v[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) v[k] = 0.f;
    if (head < nh + nkv) {
      const bool is_q = head < nh;
      if (!is_q && slot < 0) continue;
      if (i < d) {
        const int c = head * d + i;  // q heads, then k heads, lie back to back
        load_run<TI, VEC>(src, bias, c, v);
        const float r = is_q ? rq : rk;
        if (normed) {
          float w[VEC];
          load_run<float, VEC>(is_q ? wq : wk, nullptr, is_q ? c : c - nq, w);
#pragma unroll
          for (int k = 0; k < VEC; ++k) v[k] = v[k] * r * w[k];
        } else {
#pragma unroll
          for (int k = 0; k < VEC; ++k) v[k] *= r;
        }
      }
      T* dst = is_q ? q_out + ((size_t)t * nh + head) * D : k_pool + ((page * nkv + (head - nh)) * page_size + off) * D;
      store_run<T, VEC>(dst + i, v);
    } else {
      const int g = head - nh - nkv;
      if (i < dv) {
        const int c = g * dv + i;
        load_run<TI, VEC>(src + nq + nk, bias ? bias + nq + nk : nullptr, c, v);
        float* s = mix ? source + (size_t)t * nv + c : nullptr;
        if (mix == 1) {
          store_run<float, VEC>(s, v);
        } else if (mix == 2) {
          float first[VEC];
          load_run<float, VEC>(s, nullptr, 0, first);
#pragma unroll
          for (int k = 0; k < VEC; ++k) v[k] = (1.f - lam) * v[k] + lam * first[k];
        }
      }
      if (slot >= 0) store_run<T, VEC>(v_pool + ((page * nkv + g) * page_size + off) * D + i, v);
    }
  }
}

template <typename TI, typename T>
static int launch_qk_norm_mix_store(void* q_out, const void* x, const float* bias, const float* wq, const float* wk, float eps, const int* positions,
                                    float temp_coef, float temp_every, float* source, float lam, const int* slots, void* k_pool, void* v_pool, int n,
                                    int nh, int nkv, int d, int dv, int D, int page_size, int mix, int normed, cudaStream_t stream) {
  const bool vec = (d % 8) == 0 && (dv % 8) == 0 && (D % 8) == 0 &&
                   (((uintptr_t)q_out | (uintptr_t)x | (uintptr_t)bias | (uintptr_t)wq | (uintptr_t)wk | (uintptr_t)source | (uintptr_t)k_pool |
                     (uintptr_t)v_pool) & 15) == 0;
  const int items = (nh + 2 * nkv) * (vec ? D / 8 : D);
  const int threads = items >= 512 ? 512 : (items >= 256 ? 256 : (items >= 128 ? 128 : 64));
#define DLI_QKM(V)                                                                                                                            \
  launch_pdl((qk_norm_mix_store_kernel<TI, T, V>), dim3(n), dim3(threads), 0, stream, 1, (T*)q_out, (const TI*)x, bias, wq, wk, eps, positions, \
             temp_coef, temp_every, source, lam, slots, (T*)k_pool, (T*)v_pool, nh, nkv, d, dv, D, page_size, mix, normed)
  return (int)(vec ? DLI_QKM(8) : DLI_QKM(1));
#undef DLI_QKM
}

DLI_EXPORT int dli_qk_norm_mix_store(void* q_out, const void* x, const float* bias, const float* wq, const float* wk, float eps, const int* positions,
                                     float temp_coef, float temp_every, float* source, float lam, const int* slots, void* k_pool, void* v_pool, int n,
                                     int nh, int nkv, int d, int dv, int D, int page_size, int mix, int normed, int in_dtype, int dtype,
                                     cudaStream_t stream) {
  if (n == 0) return 0;
  if (nh < 1 || nkv < 1 || nh % nkv || d < 1 || dv < 1 || D < d || D < dv || page_size < 1 || (slots && (!k_pool || !v_pool)) || (mix && !source) ||
      mix < 0 || mix > 2 || (normed && (!wq || !wk)) || (temp_coef != 0.f && !(temp_every > 0.f)))
    return DLI_ERR_UNSUPPORTED;
#define DLI_QKM(TI, T)                                                                                                                        \
  launch_qk_norm_mix_store<TI, T>(q_out, x, bias, wq, wk, eps, positions, temp_coef, temp_every, source, lam, slots, k_pool, v_pool, n, nh, nkv, \
                                  d, dv, D, page_size, mix, normed, stream)
  if (dtype == DLI_F32) return in_dtype == DLI_F32 ? DLI_QKM(float, float) : DLI_ERR_UNSUPPORTED;
  return in_dtype == DLI_F32 ? DLI_QKM(float, __nv_bfloat16) : DLI_QKM(__nv_bfloat16, __nv_bfloat16);
#undef DLI_QKM
}

// ---------------------------------------------------------------- a product per head, for a decode step's few tokens
// out[t, h, f] = sum_i x[t, h, i] * w[h, i, f]  (float32 sums), times sigmoid(gate[t, h, f]) if a gate is given.
// x, out and gate are column slices of wider rows (row and head strides in elements); w [heads][in][features] is
// contiguous.  One block per (token, head): the token's `in` numbers wait in shared memory; a thread takes a run of
// VEC features (8 with 16-byte loads of w, else 1) and every `slices`-th row of w, so that a thread's loads are few
// and independent of one another; the slices' partial sums meet in shared memory and are added in slice order.
template <typename T, int VEC>
__global__ void heads_matvec_kernel(T* __restrict__ out, long long out_row, int out_head, const T* __restrict__ x, long long x_row, int x_head,
                                    const T* __restrict__ w, const T* __restrict__ gate, long long gate_row, int in, int features, int slices) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float hm_smem[];
  float* xs = hm_smem;        // [in]
  float* part = xs + in;      // [slices][features]
  const int t = blockIdx.x, h = blockIdx.y;
  const T* xp = x + (size_t)t * x_row + (size_t)h * x_head;
  for (int i = threadIdx.x; i < in; i += blockDim.x) xs[i] = to_float(xp[i]);
  __syncthreads();
  const T* wp = w + (size_t)h * in * features;
  const int runs = features / VEC;
  const int run = threadIdx.x % runs, slice = threadIdx.x / runs;
  if (slice < slices) {
    float acc[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) acc[k] = 0.f;
#pragma unroll 4
    for (int i = slice; i < in; i += slices) {
      const float xi = xs[i];
      if (VEC == 8) {
        float wv[8];
        load8(wp + (size_t)i * features + run * 8, wv);
#pragma unroll
        for (int k = 0; k < 8; ++k) acc[k] = fmaf(xi, wv[k], acc[k]);
      } else {
        acc[0] = fmaf(xi, to_float(wp[(size_t)i * features + run]), acc[0]);
      }
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) part[slice * features + run * VEC + k] = acc[k];
  }
  __syncthreads();
  for (int f = threadIdx.x; f < features; f += blockDim.x) {
    float v = 0.f;
    for (int sl = 0; sl < slices; ++sl) v += part[sl * features + f];
    if (gate) v *= 1.f / (1.f + expf(-to_float(gate[(size_t)t * gate_row + (size_t)h * features + f])));
    out[(size_t)t * out_row + (size_t)h * out_head + f] = from_float<T>(v);
  }
}

template <typename T>
static int launch_heads_matvec(void* out, long long out_row, int out_head, const void* x, long long x_row, int x_head, const void* w,
                               const void* gate, long long gate_row, int n, int heads, int in, int features, cudaStream_t stream) {
  const int threads = 256;
  const bool vec = (features % 8) == 0 && features / 8 <= threads && (((uintptr_t)w) & 15) == 0;
  const int runs = vec ? features / 8 : features;
  if (!vec && runs > threads) return DLI_ERR_UNSUPPORTED;
  int slices = threads / runs;
  if (slices > in) slices = in;
  const size_t smem = (size_t)(in + slices * features) * sizeof(float);
  if (smem > 48 * 1024) return DLI_ERR_UNSUPPORTED;
  if (vec)
    return (int)launch_pdl((heads_matvec_kernel<T, 8>), dim3(n, heads), dim3(threads), smem, stream, 1, (T*)out, out_row, out_head, (const T*)x, x_row,
                           x_head, (const T*)w, (const T*)gate, gate_row, in, features, slices);
  return (int)launch_pdl((heads_matvec_kernel<T, 1>), dim3(n, heads), dim3(threads), smem, stream, 1, (T*)out, out_row, out_head, (const T*)x, x_row,
                         x_head, (const T*)w, (const T*)gate, gate_row, in, features, slices);
}

DLI_EXPORT int dli_heads_matvec(void* out, long long out_row, int out_head, const void* x, long long x_row, int x_head, const void* w,
                                const void* gate, long long gate_row, int n, int heads, int in, int features, int dtype, cudaStream_t stream) {
  if (n == 0) return 0;
  if (heads < 1 || heads > 65535 || in < 1 || features < 1) return DLI_ERR_UNSUPPORTED;
  return dtype == DLI_F32 ? launch_heads_matvec<float>(out, out_row, out_head, x, x_row, x_head, w, gate, gate_row, n, heads, in, features, stream)
                          : launch_heads_matvec<__nv_bfloat16>(out, out_row, out_head, x, x_row, x_head, w, gate, gate_row, n, heads, in, features,
                                                               stream);
}

DLI_EXPORT int dli_sigmoid_gate(void* out, const void* gate, long long gate_stride, int n, int cols, int dtype, cudaStream_t stream) {
  if (n == 0 || cols == 0) return 0;
  const long long total = (long long)n * cols;
  cudaError_t e;
  if ((cols % 8) == 0 && (gate_stride % 8) == 0 && (((uintptr_t)out | (uintptr_t)gate) & 15) == 0) {
    const int vblocks = (int)((total / 8 + 255) / 256);
    if (dtype == DLI_F32)
      e = launch_pdl((sigmoid_gate_vec_kernel<float>), dim3(vblocks), dim3(256), 0, stream, 1, (float*)out, (const float*)gate, gate_stride, n, cols);
    else
      e = launch_pdl((sigmoid_gate_vec_kernel<__nv_bfloat16>), dim3(vblocks), dim3(256), 0, stream, 1, (__nv_bfloat16*)out,
                     (const __nv_bfloat16*)gate, gate_stride, n, cols);
    return (int)e;
  }
  const int blocks = (int)((total + 255) / 256);
  if (dtype == DLI_F32)
    e = launch_pdl((sigmoid_gate_kernel<float>), dim3(blocks), dim3(256), 0, stream, 1, (float*)out, (const float*)gate, gate_stride, n, cols);
  else
    e = launch_pdl((sigmoid_gate_kernel<__nv_bfloat16>), dim3(blocks), dim3(256), 0, stream, 1, (__nv_bfloat16*)out,
                   (const __nv_bfloat16*)gate, gate_stride, n, cols);
  return (int)e;
}
