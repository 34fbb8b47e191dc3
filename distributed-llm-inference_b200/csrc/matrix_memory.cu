// A matrix memory with exponential gates: per head a matrix S (d x dv), a vector n (d) and a running maximum m, with
//   i = c tanh((gi + bi) / c),   f = logsigmoid(c tanh((gf + bf) / c)),   m' = max(f + m, i),
//   S <- exp(f + m - m') S + exp(i - m') k v^T,   n <- the same with k alone,   o = S^T q / sqrt(d),
//   divisor = max(|n . q| / sqrt(d), exp(-m')) + 1e-6.
// n is kept as one more value column of S, whose value is always 1.  Everything here is float32 on the CUDA cores: the kernel of a
// decode step (one token a sequence), and the walk, token after token, for short portions, float32 models and large heads.  (Portions
// in bfloat16 take the tiles of tokens of matrix_memory_tc.cu.)
//
// state [slots][heads][dv + 1][d]: a value column's d numbers are contiguous, n behind the last column;  top [slots][heads][dv + 1]:
// m, a copy per column, so that whoever owns a column reads and writes its own.
// u row: q (heads of d) | k (heads of d) | v (heads of dv);  gates row: gi (heads) | gf (heads), float32;  bias the same.
#include "common.cuh"
#include "matrix_memory.cuh"

using namespace dli;

namespace {

__device__ __forceinline__ float4 load4f(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4f(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

// ---------------------------------------------------------------- one token a sequence
// A warp owns 32 / LANES x COLS value columns of one head of one sequence; LANES lanes share a column, each with runs of four key
// rows 4 * (lane + LANES * c), so a column is read and written in whole lines.  VEC: d a multiple of 4 and aligned rows.
constexpr int STEP_WARPS = 4;

template <typename T, int LANES, int CHUNKS, int COLS, bool VEC>
__global__ void __launch_bounds__(STEP_WARPS * 32) matrix_memory_step_kernel(float* __restrict__ o, float* __restrict__ divisor, const T* __restrict__ u,
                                                                             long long u_stride, const float* __restrict__ gates,
                                                                             const float* __restrict__ bias, float cap, float* __restrict__ state,
                                                                             float* __restrict__ top, const int* __restrict__ q_start,
                                                                             const int* __restrict__ state_slot, int heads, int d, int dv) {
  pdl_launch_dependents();
  constexpr int PER = 32 / LANES;
  const int seq = blockIdx.z, head = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sub = lane / LANES, slice = lane - sub * LANES;
  const int cols = dv + 1;
  const int col0 = (blockIdx.x * STEP_WARPS + warp) * PER * COLS;
  if (col0 >= cols) return;
  pdl_wait();
  const int t = q_start[seq];
  if (q_start[seq + 1] <= t) return;
  const size_t base = ((size_t)state_slot[seq] * heads + head) * cols;
  const T* row = u + (size_t)t * u_stride;
  float s[COLS][CHUNKS][4], q[CHUNKS][4], k[CHUNKS][4], v[COLS];
#pragma unroll
  for (int j = 0; j < COLS; ++j) {
    const int col = col0 + j * PER + sub;
    const float* src = state + (base + col) * d;
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c) {
      const int i = 4 * (slice + LANES * c);
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][c][e] = 0.f;
      if (col < cols && i < d) {
        if (VEC) {
          const float4 x = load4f(src + i);
          s[j][c][0] = x.x; s[j][c][1] = x.y; s[j][c][2] = x.z; s[j][c][3] = x.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) if (i + e < d) s[j][c][e] = src[i + e];
        }
      }
    }
    v[j] = col < dv ? to_float(row[(size_t)2 * heads * d + (size_t)head * dv + col]) : 1.f;
  }
#pragma unroll
  for (int c = 0; c < CHUNKS; ++c) {
    const int i = 4 * (slice + LANES * c);
#pragma unroll
    for (int e = 0; e < 4; ++e) q[c][e] = k[c][e] = 0.f;
    if (i < d) {
      const T* qs = row + (size_t)head * d + i;
      const T* ks = qs + (size_t)heads * d;
      if (VEC) {
        const float4 a = load4f(qs), b = load4f(ks);
        q[c][0] = a.x; q[c][1] = a.y; q[c][2] = a.z; q[c][3] = a.w;
        k[c][0] = b.x; k[c][1] = b.y; k[c][2] = b.z; k[c][3] = b.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) if (i + e < d) { q[c][e] = to_float(qs[e]); k[c][e] = to_float(ks[e]); }
      }
    }
  }
  const float li = memory_in_gate(gates[(size_t)t * 2 * heads + head] + bias[head], cap);
  const float lf = memory_forget_gate(gates[(size_t)t * 2 * heads + heads + head] + bias[heads + head], cap);
  const float m0 = top[base + col0], m = fmaxf(lf + m0, li);
  const float keep = expf(lf + m0 - m), take = expf(li - m), scale = 1.f / sqrtf((float)d);
#pragma unroll
  for (int j = 0; j < COLS; ++j) {
    const int col = col0 + j * PER + sub;
    const float w = take * v[j];
    float acc = 0.f;
#pragma unroll
    for (int c = 0; c < CHUNKS; ++c)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[j][c][e] = fmaf(keep, s[j][c][e], w * k[c][e]);
        acc = fmaf(q[c][e], s[j][c][e], acc);
      }
#pragma unroll
    for (int off = LANES / 2; off > 0; off >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
    if (col < cols) {
      float* dst = state + (base + col) * d;
#pragma unroll
      for (int c = 0; c < CHUNKS; ++c) {
        const int i = 4 * (slice + LANES * c);
        if (i < d) {
          if (VEC) *reinterpret_cast<float4*>(dst + i) = make_float4(s[j][c][0], s[j][c][1], s[j][c][2], s[j][c][3]);
          else {
#pragma unroll
            for (int e = 0; e < 4; ++e) if (i + e < d) dst[i + e] = s[j][c][e];
          }
        }
      }
      if (slice == 0) {
        top[base + col] = m;
        if (col < dv) o[((size_t)t * heads + head) * dv + col] = acc * scale;
        else divisor[(size_t)t * heads + head] = memory_divisor(acc * scale, m);
      }
    }
  }
}

// ---------------------------------------------------------------- token after token
// One CTA: some value columns of one head of one sequence.  KS lanes share a column, each with R key rows of it in registers.  A
// tile of sixteen tokens is staged in shared memory as float32; one warp works out its gates and the running maximum in front
// of the walk.  Slices of R floats are padded by 4, so that lanes with different slices read different banks.
constexpr int WALK_R = 32, WALK_TOKENS = 16, WALK_THREADS = 128;

__host__ __device__ inline int walk_slices(int ks) { return ks * (WALK_R + 4); }
__host__ __device__ inline int walk_token_floats(int ks, int cols) { return (2 * walk_slices(ks) + cols + 3 + 3) & ~3; }

template <typename T>
__global__ void __launch_bounds__(WALK_THREADS) matrix_memory_walk_kernel(float* __restrict__ o, float* __restrict__ divisor, const T* __restrict__ u,
                                                                          long long u_stride, const float* __restrict__ gates,
                                                                          const float* __restrict__ bias, float cap, float* __restrict__ state,
                                                                          float* __restrict__ top, const int* __restrict__ q_start,
                                                                          const int* __restrict__ state_slot, int heads, int d, int dv, int ks,
                                                                          int cols_per_cta) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  const int seq = blockIdx.z, head = blockIdx.y;
  const int t0 = q_start[seq], t1 = q_start[seq + 1];
  if (t1 <= t0) return;
  const int cols = dv + 1, span = walk_slices(ks), stride = walk_token_floats(ks, cols_per_cta);
  const int tid = threadIdx.x, lane = tid & 31;
  const int col_local = tid / ks, slice = tid - col_local * ks;
  const int col0 = blockIdx.x * cols_per_cta, col = col0 + col_local;
  const bool active = col_local < cols_per_cta && col < cols;
  const int i0 = slice * WALK_R;
  const size_t base = ((size_t)state_slot[seq] * heads + head) * cols;
  float* srow = state + (base + (active ? col : 0)) * d;
  for (int e = tid; e < WALK_TOKENS * stride; e += blockDim.x) sm[e] = 0.f;  // places behind the head size stay zero
  float S[WALK_R];
#pragma unroll
  for (int r = 0; r < WALK_R; ++r) S[r] = (active && i0 + r < d) ? srow[i0 + r] : 0.f;
  float m = top[base + col0];
  const float scale = 1.f / sqrtf((float)d);
  __syncthreads();

  for (int tile = t0; tile < t1; tile += WALK_TOKENS) {
    const int cnt = min(WALK_TOKENS, t1 - tile);
    for (int e = tid; e < cnt * d; e += blockDim.x) {
      const int tok = e / d, i = e - tok * d;
      const T* row = u + (size_t)(tile + tok) * u_stride + (size_t)head * d + i;
      float* dst = sm + tok * stride + i + ((i / WALK_R) << 2);
      dst[0] = to_float(row[0]);
      dst[span] = to_float(row[(size_t)heads * d]);
    }
    for (int e = tid; e < cnt * cols_per_cta; e += blockDim.x) {
      const int tok = e / cols_per_cta, c = e - tok * cols_per_cta;
      if (col0 + c < cols)
        sm[tok * stride + 2 * span + c] =
            col0 + c < dv ? to_float(u[(size_t)(tile + tok) * u_stride + (size_t)2 * heads * d + (size_t)head * dv + col0 + c]) : 1.f;
    }
    if (tid < 32) {
      float li = 0.f, lf = 0.f;
      if (lane < cnt) {
        const float* g = gates + (size_t)(tile + lane) * 2 * heads;
        li = memory_in_gate(g[head] + bias[head], cap);
        lf = memory_forget_gate(g[heads + head] + bias[heads + head], cap);
      }
      float before = 0.f, after = 0.f;
      for (int tok = 0; tok < cnt; ++tok) {
        const float next = fmaxf(__shfl_sync(0xffffffffu, lf, tok) + m, __shfl_sync(0xffffffffu, li, tok));
        if (lane == tok) { before = m; after = next; }
        m = next;
      }
      if (lane < cnt) {
        float* dst = sm + lane * stride + 2 * span + cols_per_cta;
        dst[0] = expf(lf + before - after);
        dst[1] = expf(li - after);
        dst[2] = after;
      }
    }
    __syncthreads();
    for (int tok = 0; tok < cnt; ++tok) {
      const float* row = sm + tok * stride;
      const float4* Q = reinterpret_cast<const float4*>(row + slice * (WALK_R + 4));
      const float4* K = reinterpret_cast<const float4*>(row + span + slice * (WALK_R + 4));
      const float* tail = row + 2 * span + cols_per_cta;
      const float keep = tail[0], w = tail[1] * row[2 * span + (col_local < cols_per_cta ? col_local : 0)];
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int r = 0; r < WALK_R; r += 4) {
        const float4 qv = Q[r >> 2], kv = K[r >> 2];
        S[r] = fmaf(keep, S[r], w * kv.x);
        S[r + 1] = fmaf(keep, S[r + 1], w * kv.y);
        S[r + 2] = fmaf(keep, S[r + 2], w * kv.z);
        S[r + 3] = fmaf(keep, S[r + 3], w * kv.w);
        acc[0] = fmaf(qv.x, S[r], acc[0]);
        acc[1] = fmaf(qv.y, S[r + 1], acc[1]);
        acc[2] = fmaf(qv.z, S[r + 2], acc[2]);
        acc[3] = fmaf(qv.w, S[r + 3], acc[3]);
      }
      float sum = (acc[0] + acc[1]) + (acc[2] + acc[3]);
      for (int off = 1; off < ks; off <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      if (active && slice == 0) {
        const size_t at = (size_t)(tile + tok) * heads + head;
        if (col < dv) o[at * dv + col] = sum * scale;
        else divisor[at] = memory_divisor(sum * scale, tail[2]);
      }
    }
    if (tile + WALK_TOKENS >= t1 && active && slice == 0) top[base + col] = sm[(cnt - 1) * stride + 2 * span + cols_per_cta + 2];
    __syncthreads();
  }
  if (active) {
#pragma unroll
    for (int r = 0; r < WALK_R; ++r)
      if (i0 + r < d) srow[i0 + r] = S[r];
  }
}

template <typename T>
int launch_walk(float* o, float* divisor, const T* u, long long u_stride, const float* gates, const float* bias, float cap, float* state, float* top,
                const int* q_start, const int* state_slot, int num_seqs, int heads, int d, int dv, int max_len, cudaStream_t stream) {
  const int cols = dv + 1;
  if (max_len == 1) {
    const bool vec = (d % 4) == 0 && (u_stride % 4) == 0 && ((uintptr_t)u & (4 * sizeof(T) - 1)) == 0 && ((uintptr_t)state & 15) == 0;
#define DLI_STEP(L, C, J)                                                                                                                     \
  {                                                                                                                                           \
    const int per_cta = STEP_WARPS * (32 / L) * J;                                                                                            \
    const dim3 grid((cols + per_cta - 1) / per_cta, heads, num_seqs);                                                                         \
    if (vec)                                                                                                                                  \
      return (int)launch_pdl((matrix_memory_step_kernel<T, L, C, J, true>), grid, dim3(STEP_WARPS * 32), 0, stream, 1, o, divisor, u, u_stride, \
                             gates, bias, cap, state, top, q_start, state_slot, heads, d, dv);                                                \
    return (int)launch_pdl((matrix_memory_step_kernel<T, L, C, J, false>), grid, dim3(STEP_WARPS * 32), 0, stream, 1, o, divisor, u, u_stride, \
                           gates, bias, cap, state, top, q_start, state_slot, heads, d, dv);                                                  \
  }
    if (d <= 32) DLI_STEP(8, 1, 4)
    if (d <= 64) DLI_STEP(16, 1, 4)
    if (d <= 128) DLI_STEP(32, 1, 8)
    if (d <= 256) DLI_STEP(32, 2, 4)
    DLI_STEP(32, 4, 2)
#undef DLI_STEP
  }
  int ks = 1;
  while (ks * WALK_R < d) ks <<= 1;
  int per = WALK_THREADS / ks;
  if (per > cols) per = cols;
  while (per * ks > 32 && (long long)((cols + per - 1) / per) * heads * num_seqs < 2LL * sm_count()) per = (per + 1) / 2;
  const int blocks = (cols + per - 1) / per;
  per = (cols + blocks - 1) / blocks;  // even shares
  const int threads = (per * ks + 31) / 32 * 32;
  const size_t smem = (size_t)WALK_TOKENS * walk_token_floats(ks, per) * sizeof(float);
  static MaxPerDevice set;
  if ((int)smem > 48 * 1024 && set.here() < (int)smem) {
    cudaError_t e = cudaFuncSetAttribute(matrix_memory_walk_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    set.here() = (int)smem;
  }
  return (int)launch_pdl((matrix_memory_walk_kernel<T>), dim3(blocks, heads, num_seqs), dim3(threads), smem, stream, 1, o, divisor, u, u_stride, gates,
                         bias, cap, state, top, q_start, state_slot, heads, d, dv, ks, per);
}

}  // namespace

DLI_EXPORT int dli_matrix_memory_walk(float* o, float* divisor, const void* u, long long u_stride, const float* gates, const float* bias, float cap,
                                      float* state, float* top, const int* q_start, const int* state_slot, int num_seqs, int heads, int d, int dv,
                                      int max_len, int dtype, cudaStream_t stream) {
  if (num_seqs == 0) return 0;
  if (heads < 1 || heads > 65535 || num_seqs > 65535 || d < 1 || d > 512 || dv < 1 || !(cap > 0.f)) return DLI_ERR_UNSUPPORTED;
  return dtype == DLI_F32 ? launch_walk<float>(o, divisor, (const float*)u, u_stride, gates, bias, cap, state, top, q_start, state_slot, num_seqs, heads, d,
                                               dv, max_len, stream)
                          : launch_walk<__nv_bfloat16>(o, divisor, (const __nv_bfloat16*)u, u_stride, gates, bias, cap, state, top, q_start, state_slot,
                                                       num_seqs, heads, d, dv, max_len, stream);
}
