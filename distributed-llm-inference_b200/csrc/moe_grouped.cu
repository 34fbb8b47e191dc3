// The experts' products of a routed feed-forward for steps of many tokens (bfloat16): the (token, expert) pairs are
// sorted by expert on the device (a counting sort; no shape depends on the data), and two grouped products run over the
// sorted rows on the tensor cores (mma.sync m16n8k16 fed by ldmatrix, float32 sums), a tile of 64 rows belonging to one expert:
//   hidden[row] = act(gate_e x) * (up_e x), or act(up_e x) for experts without a gate
//                                                 (the sums rounded to bfloat16 first, as a stored product would be)
//   partial[row] = down_e hidden[row]             (float32)
// Experts numbered E and above are identities: their pairs have no row.  (moe_combine.cu adds the rows up, token by token.)
#include <math_constants.h>

#include "common.cuh"
#include "expert_act.cuh"

using namespace dli;
typedef __nv_bfloat16 bf16;

namespace {

constexpr int BM = 64, BN = 64, BK = 64, PAD = 8, THREADS = 128;
constexpr int LDS = BK + PAD;  // elements of a staged row: 144 bytes, so the eight rows of an 8 x 8 fragment lie in different banks
constexpr int TILE_ELEMS = BM * LDS;  // one staged tile of 64 rows (A, or one of B's)
enum { EPI_F32 = 0, EPI_GLU = 1, EPI_ACT = 2 };  // what a grouped product does with its sums
constexpr int SORT_SMALL_MAX_PAIRS = 2048;  // up to here one block sorts the pairs in one launch

// counts <- 0, and -1 into the tile and row maps (what no expert claims stays -1)
__global__ void moe_init_kernel(int* __restrict__ counts, int n_counts, int* __restrict__ maps, int n_maps) {
  pdl_launch_dependents();
  pdl_wait();
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n_counts + n_maps; i += gridDim.x * blockDim.x) {
    if (i < n_counts) counts[i] = 0;
    else maps[i - n_counts] = -1;
  }
}

__global__ void moe_count_kernel(const int* __restrict__ ids, int pairs, int E, int* __restrict__ counts, int* __restrict__ rank) {
  pdl_launch_dependents();
  pdl_wait();
  const int p = blockIdx.x * blockDim.x + threadIdx.x;
  if (p < pairs && ids[p] < E) rank[p] = atomicAdd(&counts[ids[p]], 1);
}

// offsets[e]: first sorted row of expert e, every expert's run padded to whole tiles; tile_expert[tile]: the tile's expert
// (-1 behind the last one: set by the caller beforehand).
__global__ void moe_plan_kernel(const int* __restrict__ counts, int E, int* __restrict__ offsets, int* __restrict__ tile_expert) {
  pdl_launch_dependents();
  pdl_wait();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < E; ++e) {
      offsets[e] = at;
      at += (counts[e] + BM - 1) / BM * BM;
    }
    offsets[E] = at;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x)
    for (int tile = offsets[e] / BM; tile < offsets[e + 1] / BM; ++tile) tile_expert[tile] = e;
}

// pos[p]: the sorted row of pair p; row_pair[row]: the pair of a sorted row (-1 for padding: set by the caller beforehand)
__global__ void moe_scatter_kernel(const int* __restrict__ ids, const int* __restrict__ rank, const int* __restrict__ offsets, int pairs, int E,
                                   int* __restrict__ pos, int* __restrict__ row_pair) {
  pdl_launch_dependents();
  pdl_wait();
  const int p = blockIdx.x * blockDim.x + threadIdx.x;
  if (p >= pairs || ids[p] >= E) return;
  const int row = offsets[ids[p]] + rank[p];
  pos[p] = row;
  row_pair[row] = p;
}

// The whole sort in one block, for steps of few pairs (a decode step): maps to -1, counts and ranks in shared memory, offsets,
// tile map, scatter.  One launch instead of four.
__global__ void moe_sort_small_kernel(const int* __restrict__ ids, int pairs, int E, int* __restrict__ offsets, int* __restrict__ pos,
                                      int* __restrict__ tile_expert, int tiles, int* __restrict__ row_pair) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ int sh[];  // counts [E] | offsets [E + 1]
  int* cnt = sh;
  int* off = sh + E;
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  for (int i = threadIdx.x; i < tiles; i += blockDim.x) tile_expert[i] = -1;
  for (int i = threadIdx.x; i < tiles * BM; i += blockDim.x) row_pair[i] = -1;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x)
    if (ids[p] < E) pos[p] = atomicAdd(&cnt[ids[p]], 1);  // the pair's rank for now
  __syncthreads();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < E; ++e) {
      off[e] = at;
      at += (cnt[e] + BM - 1) / BM * BM;
    }
    off[E] = at;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) {
    offsets[e] = off[e];
    if (e < E)
      for (int tile = off[e] / BM; tile < off[e + 1] / BM; ++tile) tile_expert[tile] = e;
  }
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    if (ids[p] >= E) continue;
    const int row = off[ids[p]] + pos[p];
    pos[p] = row;
    row_pair[row] = p;
  }
}

__device__ __forceinline__ void cp_async16(void* dst, const void* src, int bytes) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], const uint32_t (&b)[2]) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

__device__ __forceinline__ float round_bf16(float x) { return __bfloat162float(__float2bfloat16_rn(x)); }

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const bf16* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}

// C[row][n] = sum_k A[src(row)][k] * B_e[n][k] over one tile of 64 sorted rows of expert e = tile_expert[tile] and 64 NB columns.
// EPI_GLU: two B tiles (rows n and half + n of the expert's matrix) and C = act(first) * second, bfloat16 (64 columns a tile).
// EPI_ACT: C = act(sum), bfloat16; EPI_F32: C float32; with NB = 2 their second B tile is the next 64 columns, so that a tile of A
// is read once for 128.
// row_pair (the up products): the sorted row's pair, whose token pair / top is the row of A (-1: zeros); without it the row of A is the sorted row.
// k-tiles of 64 arrive by asynchronous copies STAGES deep: three for a step of few tokens, which only streams the experts' matrices
// and is bound by the bytes in flight; two for many tokens, where more CTAs an SM hide more latency.  Fragments are read with ldmatrix.
template <int EPI, int NB, int STAGES>
__global__ void __launch_bounds__(THREADS) moe_grouped_gemm_kernel(const bf16* __restrict__ A, long long a_stride, const int* __restrict__ row_pair,
                                                                   int top, const bf16* __restrict__ B, long long b_expert_stride, int half,
                                                                   void* __restrict__ C, long long c_stride, int N, int K,
                                                                   const int* __restrict__ tile_expert, int act) {
  pdl_launch_dependents();
  pdl_wait();
  const int tile_m = blockIdx.y;
  const int e = tile_expert[tile_m];
  if (e < 0) return;
  static_assert(EPI != EPI_GLU || NB == 2, "a gated product has two tiles of B");
  constexpr int STAGE_ELEMS = (1 + NB) * TILE_ELEMS;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* smem = reinterpret_cast<bf16*>(smem_raw);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int wm = warp >> 1, wn = warp & 1;
  const int g = lane >> 2, t = lane & 3;
  const int n0 = blockIdx.x * (EPI == EPI_GLU ? BN : NB * BN);
  const bf16* Be = B + (size_t)e * b_expert_stride;

  // the four 16-byte chunks of A (and of each B tile) this thread copies per k-tile: rows r0 + 16 i, one column of chunks
  const int r0 = tid >> 3, cc = (tid & 7) * 8;
  const bf16* a_src[4];
  const bf16* b_src[NB][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = r0 + 16 * i;
    const int row = tile_m * BM + r;
    if (row_pair) {
      const int p = row_pair[row];
      a_src[i] = p >= 0 ? A + (size_t)(p / top) * a_stride : nullptr;
    } else {
      a_src[i] = A + (size_t)row * a_stride;
    }
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      const int col = EPI == EPI_GLU ? n0 + r : n0 + j * BN + r;
      b_src[j][i] = col < N ? Be + (size_t)(EPI == EPI_GLU ? j * half + col : col) * K : nullptr;
    }
  }

  auto load = [&](int stage, int k0) {
    bf16* As = smem + stage * STAGE_ELEMS;
    const bool in_k = k0 + cc < K;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = r0 + 16 * i;
      const bool a_ok = in_k && a_src[i] != nullptr;
      cp_async16(As + r * LDS + cc, a_ok ? (const void*)(a_src[i] + k0 + cc) : (const void*)A, a_ok ? 16 : 0);
#pragma unroll
      for (int j = 0; j < NB; ++j) {
        const bool b_ok = in_k && b_src[j][i] != nullptr;
        cp_async16(As + (1 + j) * TILE_ELEMS + r * LDS + cc, b_ok ? (const void*)(b_src[j][i] + k0 + cc) : (const void*)B, b_ok ? 16 : 0);
      }
    }
  };

  float acc[NB][2][4][4];
#pragma unroll
  for (int j = 0; j < NB; ++j)
#pragma unroll
    for (int mi = 0; mi < 2; ++mi)
#pragma unroll
      for (int ni = 0; ni < 4; ++ni)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[j][mi][ni][q] = 0.f;

  const int k_tiles = (K + BK - 1) / BK;
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < k_tiles) load(s, s * BK);
    cp_async_commit();
  }
  for (int kt = 0; kt < k_tiles; ++kt) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();  // k-tile kt has landed, and everyone is done with the stage that is filled next
    const int next = kt + STAGES - 1;
    if (next < k_tiles) load(next % STAGES, next * BK);
    cp_async_commit();
    const bf16* As = smem + (kt % STAGES) * STAGE_ELEMS;
#pragma unroll
    for (int kk = 0; kk < BK; kk += 16) {
      uint32_t a[2][4];
#pragma unroll
      for (int mi = 0; mi < 2; ++mi) ldmatrix_x4(a[mi], As + (wm * 32 + mi * 16 + (lane & 15)) * LDS + kk + (lane >> 4) * 8);
#pragma unroll
      for (int j = 0; j < NB; ++j)
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          uint32_t b4[4];
          ldmatrix_x4(b4, As + (1 + j) * TILE_ELEMS + (wn * 32 + p * 16 + (lane & 7) + ((lane >> 4) << 3)) * LDS + kk + ((lane >> 3) & 1) * 8);
          const uint32_t blo[2] = {b4[0], b4[1]}, bhi[2] = {b4[2], b4[3]};
#pragma unroll
          for (int mi = 0; mi < 2; ++mi) {
            mma_bf16(acc[j][mi][2 * p], a[mi], blo);
            mma_bf16(acc[j][mi][2 * p + 1], a[mi], bhi);
          }
        }
    }
  }
  cp_async_wait<0>();

#pragma unroll
  for (int mi = 0; mi < 2; ++mi)
#pragma unroll
    for (int ni = 0; ni < 4; ++ni)
#pragma unroll
      for (int hrow = 0; hrow < 2; ++hrow) {
        const size_t row = (size_t)tile_m * BM + wm * 32 + mi * 16 + g + hrow * 8;
#pragma unroll
        for (int j = 0; j < (EPI == EPI_GLU ? 1 : NB); ++j) {
          const int col = n0 + j * BN + wn * 32 + ni * 8 + 2 * t;  // N is a multiple of 8: a pair of columns lies inside or outside
          if (col >= N) continue;
          const float v0 = acc[j][mi][ni][2 * hrow], v1 = acc[j][mi][ni][2 * hrow + 1];
          if (EPI == EPI_F32) {
            *reinterpret_cast<float2*>(reinterpret_cast<float*>(C) + row * c_stride + col) = make_float2(v0, v1);
          } else {
            float o0, o1;
            if (EPI == EPI_GLU) {
              o0 = glu_act(round_bf16(v0), act) * round_bf16(acc[NB - 1][mi][ni][2 * hrow]);
              o1 = glu_act(round_bf16(v1), act) * round_bf16(acc[NB - 1][mi][ni][2 * hrow + 1]);
            } else {
              o0 = plain_act(round_bf16(v0), act);
              o1 = plain_act(round_bf16(v1), act);
            }
            *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(C) + row * c_stride + col) = __floats2bfloat162_rn(o0, o1);
          }
        }
      }
}

template <int EPI, int NB, int STAGES>
cudaError_t launch_grouped(const bf16* A, long long a_stride, const int* row_pair, int top, const bf16* B, long long b_expert_stride, int half, void* C,
                           int N, int K, const int* tile_expert, int tiles, int act, cudaStream_t stream) {
  constexpr int SMEM = STAGES * (1 + NB) * TILE_ELEMS * (int)sizeof(bf16);
  static OncePerDevice configured;
  if (!configured.here()) {
    cudaError_t e = cudaFuncSetAttribute(moe_grouped_gemm_kernel<EPI, NB, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return e;
    configured.here() = true;
  }
  constexpr int COLS = EPI == EPI_GLU ? BN : NB * BN;
  return launch_pdl((moe_grouped_gemm_kernel<EPI, NB, STAGES>), dim3((N + COLS - 1) / COLS, tiles), dim3(THREADS), SMEM, stream, 1, A, a_stride, row_pair, top, B,
                    b_expert_stride, half, C, (long long)N, N, K, tile_expert, act);
}

}  // namespace

// Upper bound of the tiles the sorted rows take: every expert's run is padded to whole tiles.
DLI_EXPORT int dli_moe_grouped_tiles(int pairs, int E) { return (pairs < E ? pairs : E) + pairs / BM; }
DLI_EXPORT int dli_moe_grouped_tile_rows() { return BM; }

// ints: scratch of E + 1 (counts) + E + 1 (offsets) + 2 pairs (rank, pos) + tiles (tile_expert) + tiles * BM (row_pair) ints;
// hidden: [tiles * BM][ff] bfloat16; partial: [tiles * BM][W] float32.  stages: 2 or 3 deep copies, or 0: chosen here.
// gated: w_up holds an expert's gate rows, then its up rows; else its up rows alone.  ids from E on are identities.  The rows of
// the pairs are left behind the first 2 (E + 1) + pairs numbers of ints (those of identities undefined).
DLI_EXPORT int dli_moe_grouped(const void* x, const int* ids, const void* w_up, const void* w_down, int* ints, void* hidden, float* partial, int n, int W, int ff, int E, int top, int act, int gated, int stages, cudaStream_t stream) {
  if (n == 0) return 0;
  if (W < 8 || ff < 8 || (W % 8) || (ff % 8) || E < 1 || top < 1 || ((((uintptr_t)x) | ((uintptr_t)w_up) | ((uintptr_t)w_down) | ((uintptr_t)hidden) | ((uintptr_t)partial)) & 15))
    return DLI_ERR_UNSUPPORTED;
  const int pairs = n * top;
  const int tiles = dli_moe_grouped_tiles(pairs, E);
  if (tiles > 65535) return DLI_ERR_UNSUPPORTED;
  int* counts = ints;
  int* offsets = counts + E + 1;
  int* rank = offsets + E + 1;
  int* pos = rank + pairs;
  int* tile_expert = pos + pairs;
  int* row_pair = tile_expert + tiles;
  cudaError_t e;
  if (pairs <= SORT_SMALL_MAX_PAIRS && (2 * E + 1) * sizeof(int) <= 48 * 1024) {
    e = launch_pdl((moe_sort_small_kernel), dim3(1), dim3(256), (size_t)(2 * E + 1) * sizeof(int), stream, 1, ids, pairs, E, offsets, pos, tile_expert, tiles,
                   row_pair);
    if (e != cudaSuccess) return (int)e;
  } else {
    const int n_maps = tiles + tiles * BM;
    e = launch_pdl((moe_init_kernel), dim3((E + 1 + n_maps + 255) / 256 < 1024 ? (E + 1 + n_maps + 255) / 256 : 1024), dim3(256), 0, stream, 1, counts, E + 1,
                   tile_expert, n_maps);
    if (e != cudaSuccess) return (int)e;
    e = launch_pdl((moe_count_kernel), dim3((pairs + 255) / 256), dim3(256), 0, stream, 1, ids, pairs, E, counts, rank);
    if (e != cudaSuccess) return (int)e;
    e = launch_pdl((moe_plan_kernel), dim3(1), dim3(256), 0, stream, 1, (const int*)counts, E, offsets, tile_expert);
    if (e != cudaSuccess) return (int)e;
    e = launch_pdl((moe_scatter_kernel), dim3((pairs + 255) / 256), dim3(256), 0, stream, 1, ids, (const int*)rank, (const int*)offsets, pairs, E, pos, row_pair);
    if (e != cudaSuccess) return (int)e;
  }
  const bool many = stages == 2 || (stages != 3 && pairs > 16 * E);  // many rows an expert: the products bound the time, not the stream of the matrices
  const bf16 *bx = (const bf16*)x, *up = (const bf16*)w_up, *down = (const bf16*)w_down;
#define DLI_UP(EPI, NB, ST) \
  launch_grouped<EPI, NB, ST>(bx, W, row_pair, top, up, (long long)(gated ? 2 : 1) * ff * W, ff, hidden, ff, W, tile_expert, tiles, act, stream)
#define DLI_DOWN(NB, ST) \
  launch_grouped<EPI_F32, NB, ST>((const bf16*)hidden, ff, nullptr, top, down, (long long)W * ff, 0, partial, W, ff, tile_expert, tiles, 0, stream)
  if (gated) e = many ? DLI_UP(EPI_GLU, 2, 2) : DLI_UP(EPI_GLU, 2, 3);
  else e = !many ? DLI_UP(EPI_ACT, 1, 3) : ff > BN ? DLI_UP(EPI_ACT, 2, 2) : DLI_UP(EPI_ACT, 1, 2);
  if (e != cudaSuccess) return (int)e;
  e = !many ? DLI_DOWN(1, 3) : W > BN ? DLI_DOWN(2, 2) : DLI_DOWN(1, 2);
  if (e != cudaSuccess) return (int)e;
#undef DLI_UP
#undef DLI_DOWN
  return 0;
}
