// The (token, expert) pairs of a routed feed-forward sorted by expert on the device (a counting sort; no shape depends on the data), for
// steps of many tokens: every expert's run is padded to whole tiles of bm rows, and the rows of the input are gathered in that order,
// so that one product per expert runs over whole tiles (the grouped form in dense_gemm.cu).  Experts numbered E and above are
// identities: their pairs have no row.
#include "common.cuh"

using namespace dli;

namespace {

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
__global__ void moe_plan_kernel(const int* __restrict__ counts, int E, int bm, int* __restrict__ offsets, int* __restrict__ tile_expert) {
  pdl_launch_dependents();
  pdl_wait();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < E; ++e) {
      offsets[e] = at;
      at += (counts[e] + bm - 1) / bm * bm;
    }
    offsets[E] = at;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x)
    for (int tile = offsets[e] / bm; tile < offsets[e + 1] / bm; ++tile) tile_expert[tile] = e;
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
__global__ void moe_sort_small_kernel(const int* __restrict__ ids, int pairs, int E, int bm, int* __restrict__ offsets, int* __restrict__ pos,
                                      int* __restrict__ tile_expert, int tiles, int* __restrict__ row_pair) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ int sh[];  // counts [E] | offsets [E + 1]
  int* cnt = sh;
  int* off = sh + E;
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  for (int i = threadIdx.x; i < tiles; i += blockDim.x) tile_expert[i] = -1;
  for (int i = threadIdx.x; i < tiles * bm; i += blockDim.x) row_pair[i] = -1;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += blockDim.x)
    if (ids[p] < E) pos[p] = atomicAdd(&cnt[ids[p]], 1);  // the pair's rank for now
  __syncthreads();
  if (threadIdx.x == 0) {
    int at = 0;
    for (int e = 0; e < E; ++e) {
      off[e] = at;
      at += (cnt[e] + bm - 1) / bm * bm;
    }
    off[E] = at;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) {
    offsets[e] = off[e];
    if (e < E)
      for (int tile = off[e] / bm; tile < off[e + 1] / bm; ++tile) tile_expert[tile] = e;
  }
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    if (ids[p] >= E) continue;
    const int row = off[ids[p]] + pos[p];
    pos[p] = row;
    row_pair[row] = p;
  }
}

// Upper bound of the tiles of bm rows that the sorted rows take: every expert's run is padded to whole tiles.
int tiles_of(int pairs, int E, int bm) { return (pairs < E ? pairs : E) + pairs / bm; }

// The arrays of a sort in the caller's scratch: E + 1 (counts) + E + 1 (offsets) + 2 pairs (rank, pos) + tiles (tile_expert) + tiles * bm (row_pair)
// ints.  offsets[E]: rows in use.
struct Sorted {
  int *counts, *offsets, *rank, *pos, *tile_expert, *row_pair;
  int tiles;
};
cudaError_t sort_pairs(const int* ids, int pairs, int E, int bm, int* ints, Sorted& s, cudaStream_t stream) {
  s.tiles = tiles_of(pairs, E, bm);
  s.counts = ints;
  s.offsets = s.counts + E + 1;
  s.rank = s.offsets + E + 1;
  s.pos = s.rank + pairs;
  s.tile_expert = s.pos + pairs;
  s.row_pair = s.tile_expert + s.tiles;
  if (pairs <= SORT_SMALL_MAX_PAIRS && (2 * E + 1) * sizeof(int) <= 48 * 1024)
    return launch_pdl((moe_sort_small_kernel), dim3(1), dim3(256), (size_t)(2 * E + 1) * sizeof(int), stream, 1, ids, pairs, E, bm, s.offsets, s.pos, s.tile_expert,
                      s.tiles, s.row_pair);
  const int n_maps = s.tiles + s.tiles * bm;
  cudaError_t e = launch_pdl((moe_init_kernel), dim3((E + 1 + n_maps + 255) / 256 < 1024 ? (E + 1 + n_maps + 255) / 256 : 1024), dim3(256), 0, stream, 1, s.counts,
                             E + 1, s.tile_expert, n_maps);
  if (e != cudaSuccess) return e;
  e = launch_pdl((moe_count_kernel), dim3((pairs + 255) / 256), dim3(256), 0, stream, 1, ids, pairs, E, s.counts, s.rank);
  if (e != cudaSuccess) return e;
  e = launch_pdl((moe_plan_kernel), dim3(1), dim3(256), 0, stream, 1, (const int*)s.counts, E, bm, s.offsets, s.tile_expert);
  if (e != cudaSuccess) return e;
  return launch_pdl((moe_scatter_kernel), dim3((pairs + 255) / 256), dim3(256), 0, stream, 1, ids, (const int*)s.rank, (const int*)s.offsets, pairs, E, s.pos,
                    s.row_pair);
}

// xs[row] = x[token of the row's pair], 16 bytes a thread (rows without a pair keep what they hold)
__global__ void moe_gather_kernel(uint4* __restrict__ xs, const uint4* __restrict__ x, const int* __restrict__ row_pair, int top, int chunks) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = blockIdx.x;
  const int pair = row_pair[row];
  if (pair < 0) return;
  const uint4* src = x + (size_t)(pair / top) * chunks;
  for (int c = threadIdx.x; c < chunks; c += blockDim.x) xs[row * chunks + c] = src[c];
}

}  // namespace

// The pairs sorted by expert, every expert's run padded to whole tiles of bm rows (ints: see Sorted), and the rows of x in that order:
// xs [tiles * bm][W].
DLI_EXPORT int dli_moe_sort_gather(void* xs, const void* x, const int* ids, int* ints, int n, int W, int E, int top, int bm, cudaStream_t stream) {
  if (n == 0) return 0;
  if (W < 8 || W % 8 || E < 1 || top < 1 || bm < 1 || ((uintptr_t)xs | (uintptr_t)x) & 15) return DLI_ERR_UNSUPPORTED;
  Sorted s;
  cudaError_t e = sort_pairs(ids, n * top, E, bm, ints, s, stream);
  if (e != cudaSuccess) return (int)e;
  const int chunks = W / 8;
  return (int)launch_pdl(moe_gather_kernel, dim3(s.tiles * bm), dim3(chunks >= 256 ? 256 : 128), 0, stream, 1, (uint4*)xs, (const uint4*)x, (const int*)s.row_pair, top,
                         chunks);
}
