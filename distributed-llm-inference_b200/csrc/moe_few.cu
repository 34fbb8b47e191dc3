// The experts' products of a routed feed-forward for a step of few tokens (bfloat16, up to 64), which is bound by the stream of the
// experts' matrices: every chosen expert's matrix is read once, whatever number of tokens chose it, and nothing is sorted.
//   hidden[p] = act(gate_e x) * (up_e x), or act(up_e x) for experts without a gate      p: a (token, choice) pair, e its expert
//                                         (the sums rounded to bfloat16 first, as a stored product would be)
//   partial[p] = down_e hidden[p]         (float32)
// A feed-forward without a gate that runs for every token may ride along as one more expert with a size of its own: its rows of hidden
// and partial lie behind the pairs'.  Experts numbered E and above (identities) have no rows.
//
// A CTA owns 64 rows of one expert's matrix.  It finds the expert's pairs by looking through the step's choices itself, and the pairs'
// rows become the rows of an mma.sync m16n8k16 tile (float32 sums): MI tiles of 16, so that no token count up to 16 MI reads a
// matrix twice; tiles without a row are skipped.  k-tiles of 64 arrive by asynchronous copies, four to six deep.
#include "common.cuh"
#include "expert_act.cuh"

using namespace dli;
typedef __nv_bfloat16 bf16;

namespace {

constexpr int BN = 64, BK = 64, PAD = 8, THREADS = 128;
constexpr int LDS = BK + PAD;  // elements of a staged row: 144 bytes, so the eight rows of an 8 x 8 fragment lie in different banks
enum { EPI_F32 = 0, EPI_GLU = 1, EPI_ACT = 2 };  // what a product does with its sums

struct Matrix {  // of the experts, or of the feed-forward that rides along
  const bf16* w;
  long long expert_stride;
  int rows, k;  // output rows (of the up half, for a gated product) and columns
};

struct Params {
  const int* ids;  // [n][top]
  int n, top, E;
  const bf16* a;          // rows of the inputs: x by token (up), or hidden by pair (down)
  const bf16* a_extra;    // of the feed-forward that rides along: x by token (up), its hidden by token (down)
  int by_token;           // a's rows are tokens
  Matrix experts, extra;  // extra.w null: nothing rides along
  void* c;                // rows by pair: bfloat16 [pairs][experts.rows] or float32
  void* c_extra;          // rows by token
  int act, extra_act;
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src, int bytes) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const bf16* p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ float round_bf16(float x) { return __bfloat162float(__float2bfloat16_rn(x)); }

template <int EPI, int MI>
struct Shape {
  static constexpr int NB = EPI == EPI_GLU ? 2 : 1;
  static constexpr int STAGE = (16 * MI + NB * BN) * LDS;  // elements
  static constexpr int STAGES = EPI == EPI_GLU ? 4 : MI == 1 ? 6 : MI == 2 ? 5 : 4;
  static constexpr int SMEM = STAGES * STAGE * (int)sizeof(bf16);
};

// grid (blocks of 64 output rows, experts and, behind them, the feed-forward that rides along)
template <int EPI, int MI>
__global__ void __launch_bounds__(THREADS) moe_few_kernel(const Params p) {
  using S = Shape<EPI, MI>;
  constexpr int NB = S::NB, STAGES = S::STAGES;
  pdl_launch_dependents();
  const int e = blockIdx.y;
  const bool extra = e == p.E;
  const int n0 = blockIdx.x * BN, K = extra ? p.extra.k : p.experts.k, N = extra ? p.extra.rows : p.experts.rows;
  if (n0 >= N) return;  // (this grid is as wide as the wider of the two)
  pdl_wait();
  extern __shared__ __align__(16) unsigned char smem_raw[];
  bf16* smem = reinterpret_cast<bf16*>(smem_raw);
  __shared__ int list[16 * MI];  // the expert's pairs, in order (extra: the tokens)
  __shared__ int hits[THREADS / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  int count = 0;
  if (extra) {
    count = p.n;
    for (int i = tid; i < count; i += THREADS) list[i] = i;
    __syncthreads();
  } else {
    const int pairs = p.n * p.top;
    for (int first = 0; first < pairs; first += THREADS) {
      const bool hit = first + tid < pairs && p.ids[first + tid] == e;
      const unsigned mask = __ballot_sync(0xffffffffu, hit);
      if (lane == 0) hits[warp] = __popc(mask);
      __syncthreads();
      int at = count + __popc(mask & ((1u << lane) - 1));
      for (int w = 0; w < THREADS / 32; ++w) {
        if (w < warp) at += hits[w];
        count += hits[w];
      }
      if (hit && at < 16 * MI) list[at] = first + tid;  // (a token names an expert once, and there are at most 16 MI tokens)
      __syncthreads();
    }
    if (count == 0) return;
    count = min(count, 16 * MI);
  }

  // the 16-byte chunks this thread copies per k-tile: rows r0 + 16 i of A and of B, one column of chunks
  const int r0 = tid >> 3, cc = (tid & 7) * 8;
  const bf16* A = extra ? p.a_extra : p.a;
  const bf16* W = extra ? p.extra.w : p.experts.w + (size_t)e * p.experts.expert_stride;
  const bf16* a_src[MI];
  const bf16* b_src[NB][4];
#pragma unroll
  for (int i = 0; i < MI; ++i) {
    const int r = r0 + 16 * i;
    a_src[i] = r < count ? A + (size_t)(p.by_token && !extra ? list[r] / p.top : list[r]) * K : nullptr;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < NB; ++j) b_src[j][i] = n0 + r0 + 16 * i < N ? W + (size_t)(j * N + n0 + r0 + 16 * i) * K : nullptr;

  auto load = [&](int stage, int k0) {
    bf16* As = smem + stage * S::STAGE;
    const bool in_k = k0 + cc < K;
#pragma unroll
    for (int j = 0; j < NB; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const bool ok = in_k && b_src[j][i] != nullptr;
        cp_async16(As + (16 * MI + j * BN + r0 + 16 * i) * LDS + cc, ok ? (const void*)(b_src[j][i] + k0 + cc) : (const void*)W, ok ? 16 : 0);
      }
#pragma unroll
    for (int i = 0; i < MI; ++i)
      if (16 * i < count) {
        const bool ok = in_k && a_src[i] != nullptr;
        cp_async16(As + (r0 + 16 * i) * LDS + cc, ok ? (const void*)(a_src[i] + k0 + cc) : (const void*)W, ok ? 16 : 0);
      }
  };

  float acc[NB][MI][2][4];
#pragma unroll
  for (int j = 0; j < NB; ++j)
#pragma unroll
    for (int i = 0; i < MI; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h)
#pragma unroll
        for (int q = 0; q < 4; ++q) acc[j][i][h][q] = 0.f;

  const int k_tiles = (K + BK - 1) / BK;
#pragma unroll
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < k_tiles) load(s, s * BK);
    cp_async_commit();
  }
  int at = 0, fill = STAGES - 1;  // the stage that is read next, and the one that is filled next
  for (int kt = 0; kt < k_tiles; ++kt) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();  // k-tile kt has landed, and everyone is done with the stage that is filled next
    if (kt + STAGES - 1 < k_tiles) load(fill, (kt + STAGES - 1) * BK);
    cp_async_commit();
    const bf16* As = smem + at * S::STAGE;
#pragma unroll
    for (int kk = 0; kk < BK; kk += 16) {
      uint32_t b[NB][4];
#pragma unroll
      for (int j = 0; j < NB; ++j)
        ldmatrix_x4(b[j], As + (16 * MI + j * BN + warp * 16 + (lane & 7) + ((lane >> 4) << 3)) * LDS + kk + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int i = 0; i < MI; ++i)
        if (16 * i < count) {
          uint32_t a[4];
          ldmatrix_x4(a, As + (i * 16 + (lane & 15)) * LDS + kk + (lane >> 4) * 8);
#pragma unroll
          for (int j = 0; j < NB; ++j) {
            mma_bf16(acc[j][i][0], a, b[j][0], b[j][1]);
            mma_bf16(acc[j][i][1], a, b[j][2], b[j][3]);
          }
        }
    }
    if (++at == STAGES) at = 0;
    if (++fill == STAGES) fill = 0;
  }
  cp_async_wait<0>();

  const int g = lane >> 2, t = lane & 3, act = extra ? p.extra_act : p.act;
  void* C = extra ? p.c_extra : p.c;
#pragma unroll
  for (int i = 0; i < MI; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = i * 16 + g + half * 8;
      if (r >= count) continue;
      const size_t row = (size_t)list[r] * N;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int col = n0 + warp * 16 + h * 8 + 2 * t;  // N is a multiple of 8: a pair of columns lies inside or outside
        if (col >= N) continue;
        const float v0 = acc[0][i][h][2 * half], v1 = acc[0][i][h][2 * half + 1];
        if (EPI == EPI_F32) {
          *reinterpret_cast<float2*>(reinterpret_cast<float*>(C) + row + col) = make_float2(v0, v1);
        } else {
          float o0, o1;
          if (EPI == EPI_GLU) {
            o0 = glu_act(round_bf16(v0), act) * round_bf16(acc[NB - 1][i][h][2 * half]);
            o1 = glu_act(round_bf16(v1), act) * round_bf16(acc[NB - 1][i][h][2 * half + 1]);
          } else {
            o0 = plain_act(round_bf16(v0), act);
            o1 = plain_act(round_bf16(v1), act);
          }
          *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(C) + row + col) = __floats2bfloat162_rn(o0, o1);
        }
      }
    }
}

template <int EPI, int MI>
cudaError_t launch_few(const Params& p, cudaStream_t stream) {
  using S = Shape<EPI, MI>;
  static OncePerDevice configured;
  if (!configured.here()) {
    cudaError_t e = cudaFuncSetAttribute(moe_few_kernel<EPI, MI>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::SMEM);
    if (e != cudaSuccess) return e;
    configured.here() = true;
  }
  const int widest = p.extra.w && p.extra.rows > p.experts.rows ? p.extra.rows : p.experts.rows;
  return launch_pdl((moe_few_kernel<EPI, MI>), dim3((widest + BN - 1) / BN, p.E + (p.extra.w ? 1 : 0)), dim3(THREADS), S::SMEM, stream, 1, p);
}

template <int EPI>
cudaError_t launch_tokens(const Params& p, cudaStream_t stream) {
  if (p.n <= 16) return launch_few<EPI, 1>(p, stream);
  if (p.n <= 32) return launch_few<EPI, 2>(p, stream);
  return launch_few<EPI, 4>(p, stream);
}

}  // namespace

DLI_EXPORT int dli_moe_few_max_tokens() { return 64; }

// hidden: scratch [pairs][ff] bfloat16 and, behind it, [n][extra_ff]; partial: [pairs (+ n)][W] float32.  gated: w_up holds an expert's gate
// rows, then its up rows; else its up rows alone.  extra_up [extra_ff][W], extra_down [W][extra_ff] (null: nothing rides along; only
// beside experts without a gate).  ids from E on are identities.
DLI_EXPORT int dli_moe_few(float* partial, void* hidden, const void* x, const int* ids, const void* w_up, const void* w_down, const void* extra_up,
                           const void* extra_down, int n, int W, int ff, int E, int top, int act, int gated, int extra_ff, int extra_act, cudaStream_t stream) {
  if (n == 0) return 0;
  if (n > 64 || W < 8 || ff < 8 || (W % 8) || (ff % 8) || E < 1 || E > 65534 || top < 1 || (extra_up && (gated || !extra_down || extra_ff < 8 || extra_ff % 8)))
    return DLI_ERR_UNSUPPORTED;
  if ((((uintptr_t)x) | ((uintptr_t)w_up) | ((uintptr_t)w_down) | ((uintptr_t)extra_up) | ((uintptr_t)extra_down) | ((uintptr_t)hidden) | ((uintptr_t)partial)) & 15)
    return DLI_ERR_UNSUPPORTED;
  const size_t pairs = (size_t)n * top;
  bf16* hid = (bf16*)hidden;
  bf16* hid_extra = hid + pairs * ff;
  Params p{};
  p.ids = ids; p.n = n; p.top = top; p.E = E;
  p.a = p.a_extra = (const bf16*)x;
  p.by_token = 1;
  p.experts = Matrix{(const bf16*)w_up, (long long)(gated ? 2 : 1) * ff * W, ff, W};
  p.extra = Matrix{(const bf16*)extra_up, 0, extra_ff, W};
  p.c = hid; p.c_extra = hid_extra; p.act = act; p.extra_act = extra_act;
  cudaError_t e = gated ? launch_tokens<EPI_GLU>(p, stream) : launch_tokens<EPI_ACT>(p, stream);
  if (e != cudaSuccess) return (int)e;
  p.a = hid; p.a_extra = hid_extra;
  p.by_token = 0;
  p.experts = Matrix{(const bf16*)w_down, (long long)W * ff, W, ff};
  p.extra = Matrix{(const bf16*)extra_down, 0, W, extra_ff};
  p.c = partial; p.c_extra = partial + pairs * W;
  return (int)launch_tokens<EPI_F32>(p, stream);
}
