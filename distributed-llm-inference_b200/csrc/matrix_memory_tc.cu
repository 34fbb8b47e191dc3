// The matrix memory with exponential gates (matrix_memory.cu says what is computed) for prompt portions in bfloat16: tiles of 64
// tokens in closed form on the tensor cores, for one key size (-DKEY_DIM=<the head size rounded up to a multiple of 16>).
//
// Inside a tile that starts from (S0, n0, m0), with b_t the sum of the log forget gates up to t, a_j = i_j - b_j and
// g_t = max(m0, max_{j <= t} a_j), the running maximum is m_t = b_t + g_t and
//   S_t = exp(m0 - g_t) S0 + sum_{j <= t} exp(a_j - g_t) k_j v_j^T,
// so the tile's read-outs are  exp(m0 - g_t) q_t S0 + sum_{j <= t} exp(a_j - g_t) (q_t . k_j) v_j.
//
// q, k and v are bfloat16 as the projection left them; gates, weights, state and every sum are float32, and nothing float32 is
// rounded on its way into a product: a float32 operand (the state, the weighted scores, the weighted values) is cut into three
// bfloat16 numbers whose sum it is (8 bits of mantissa each), and each goes through an mma.sync of its own into the same
// float32 accumulator.  The products of two bfloat16 numbers are exact in float32.
//
// A warp owns 16 value columns of one head of one sequence; S^T of those columns stays in its registers as the accumulator of
// mma.sync m16n8k16 over all tiles (the layout of an accumulator of S^T is that of the B operand of Q S, so nothing moves).  The
// vector n is one more value column, whose value is always 1.  Tokens arrive by cp.async a tile ahead; a CTA's warps share them.
//
// A few long sequences leave most of the GPU idle, because a sequence's tiles follow one another.  They are then cut into segments of
// whole tiles, in two launches: the first computes what every segment but the last adds to a state (L, its maximum, the sum B of its
// log forget gates; no read-outs), the second starts every segment from the states in front of it,
//   m' = max(m + B, m_L),   S <- exp(m + B - m') S + exp(m_L - m') L,   segment after segment,
// and walks all segments side by side.
#include "common.cuh"
#include "matrix_memory.cuh"
#include <math_constants.h>

#ifndef KEY_DIM
#error "compile with -DKEY_DIM=<multiple of 16>"
#endif

using namespace dli;
typedef __nv_bfloat16 bf16;

namespace {

constexpr int DK = KEY_DIM;
static_assert(DK % 16 == 0 && DK >= 16 && DK <= 256, "key size: a multiple of 16 up to 256");
constexpr int TOKENS = 64;
constexpr int MAX_WARPS = 4;
constexpr int QK_ROW = DK * 2 + 16;                  // bytes of a staged row of q or k: padded so that ldmatrix reads different banks
constexpr int QK_TILE = TOKENS * QK_ROW;
constexpr int V_ROW = MAX_WARPS * 16 * 2 + 16;
constexpr int V_TILE = TOKENS * V_ROW;
constexpr int STAGE = 2 * QK_TILE + V_TILE;
constexpr int GATE_FLOATS = 2 * TOKENS + 2;          // per warp: a_j | g_t (log2 units)
constexpr int SMEM = 2 * STAGE + MAX_WARPS * GATE_FLOATS * 4 + 16;
static_assert(SMEM <= 227 * 1024, "two stages must fit");
constexpr float LOG2E = 1.4426950408889634f;

struct Params {
  float* o;               // [n][heads dv]
  float* divisor;         // [n][heads]
  const bf16* u;          // rows: q | k | v
  long long u_stride;
  const float* gates;     // [n][2 heads]
  const float* bias;      // [2 heads]
  float cap;
  float* state;           // [slots][heads][dv + 1][d]
  float* top;             // [slots][heads][dv + 1]
  const int* q_start;
  const int* state_slot;
  int heads, d, dv, warps, vec;
  int segments;           // of a sequence; with more than one:
  float* part;            // [seqs][segments][heads][dv + 1][d]: slot 0 the state at the start, slot g + 1 what segment g adds
  float* part_m;          // [seqs][segments][heads][dv + 1][2]: its maximum, the sum of its log forget gates (a copy per column)
};

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float2 unpack2(uint32_t v) { return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }
// x, y as three bfloat16 pairs whose sum they are (to the last bit of float32)
__device__ __forceinline__ void split3(float x, float y, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  hi = pack2(x, y);
  const float2 h = unpack2(hi);
  x -= h.x; y -= h.y;
  mid = pack2(x, y);
  const float2 m = unpack2(mid);
  lo = pack2(x - m.x, y - m.y);
}

// LOCAL: the first of the two launches over segments (what a segment adds to a state, no read-outs).
template <bool LOCAL>
__global__ void __launch_bounds__(MAX_WARPS * 32) matrix_memory_chunk_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(128) unsigned char smem[];
  const int launched = LOCAL ? p.segments - 1 : p.segments;
  const int seq = blockIdx.z / launched, seg = blockIdx.z - seq * launched, head = blockIdx.y;
  const int first = p.q_start[seq], last = p.q_start[seq + 1];
  const int per_segment = ((last - first + TOKENS - 1) / TOKENS + p.segments - 1) / p.segments * TOKENS;
  const int t0 = first + seg * per_segment, t1 = min(last, t0 + per_segment);  // this CTA's tokens
  if (t1 <= t0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthreads = p.warps * 32;
  const int d = p.d, dv = p.dv, cols = dv + 1, heads = p.heads;
  const int vcol0 = blockIdx.x * p.warps * 16;       // the CTA's first value column
  const int col0 = vcol0 + warp * 16;                // this warp's
  const bool active = col0 < cols;
  float* sA = reinterpret_cast<float*>(smem + 2 * STAGE) + warp * GATE_FLOATS;  // a_j
  float* sG = sA + TOKENS;                                                       // g_t

  const bf16* ubase = p.u + (size_t)head * d;
  const bf16* vbase = p.u + (size_t)2 * heads * d + (size_t)head * dv;
  auto load_tile = [&](int stage, int base) {
    unsigned char* sQ = smem + stage * STAGE;
    unsigned char* sK = sQ + QK_TILE;
    unsigned char* sV = sK + QK_TILE;
    const int vcols = p.warps * 16;
    if (p.vec) {  // d and dv multiples of 8, aligned rows: 16 bytes a copy
      for (int e = tid; e < TOKENS * (DK / 8); e += nthreads) {
        const int r = e / (DK / 8), c = e - r * (DK / 8);
        const bool ok = base + r < t1 && c * 8 < d;
        const bf16* src = ubase + (ok ? (size_t)(base + r) * p.u_stride + c * 8 : 0);
        if (!LOCAL) cp_async16(smem_u32(sQ + r * QK_ROW + c * 16), src, ok ? 16 : 0);
        cp_async16(smem_u32(sK + r * QK_ROW + c * 16), src + (size_t)heads * d, ok ? 16 : 0);
      }
      const int chunks = vcols / 8;
      for (int e = tid; e < TOKENS * chunks; e += nthreads) {
        const int r = e / chunks, c = e - r * chunks, col = vcol0 + c * 8;
        if (col == dv) {  // the column of ones, and nothing behind it
          *reinterpret_cast<uint4*>(sV + r * V_ROW + c * 16) = make_uint4(0x3f80u, 0, 0, 0);
        } else {
          const bool ok = base + r < t1 && col < dv;
          cp_async16(smem_u32(sV + r * V_ROW + c * 16), vbase + (ok ? (size_t)(base + r) * p.u_stride + col : 0), ok ? 16 : 0);
        }
      }
    } else {
      const bf16 zero = __float2bfloat16_rn(0.f);
      for (int e = tid; e < TOKENS * DK; e += nthreads) {
        const int r = e / DK, i = e - r * DK;
        const bool ok = base + r < t1 && i < d;
        const bf16* src = ubase + (ok ? (size_t)(base + r) * p.u_stride + i : 0);
        *reinterpret_cast<bf16*>(sQ + r * QK_ROW + i * 2) = ok ? src[0] : zero;
        *reinterpret_cast<bf16*>(sK + r * QK_ROW + i * 2) = ok ? src[(size_t)heads * d] : zero;
      }
      for (int e = tid; e < TOKENS * vcols; e += nthreads) {
        const int r = e / vcols, c = e - r * vcols, col = vcol0 + c;
        bf16 x = zero;
        if (base + r < t1) x = col < dv ? vbase[(size_t)(base + r) * p.u_stride + col] : (col == dv ? __float2bfloat16_rn(1.f) : zero);
        *reinterpret_cast<bf16*>(sV + r * V_ROW + c * 2) = x;
      }
    }
  };
  // raw gates of this lane's two tokens of a tile (2 lane, 2 lane + 1)
  auto load_gates = [&](int base, float (&raw)[4]) {
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int t = base + 2 * lane + k;
      const bool ok = t < t1;
      const float* g = p.gates + (ok ? (size_t)t * 2 * heads : 0);
      raw[k] = ok ? g[head] : 0.f;
      raw[2 + k] = ok ? g[heads + head] : 0.f;
    }
  };

  load_tile(0, t0);
  cp_async_commit();

  // ---- the state: S^T, rows = this warp's value columns, columns = key rows, in accumulators of 16 x 8
  const size_t sbase = ((size_t)p.state_slot[seq] * heads + head) * cols;
  auto pbase = [&](int slot) { return (((size_t)seq * p.segments + slot) * heads + head) * cols; };
  float S[DK / 8][4];
  const int row_lo = col0 + (lane >> 2), row_hi = row_lo + 8, kcol = (lane & 3) * 2;
  auto each = [&](auto&& fn) {  // fn(accumulator j, element e, offset of that number in a [dv + 1][d] block) for the numbers that exist
#pragma unroll
    for (int j = 0; j < DK / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int col = e < 2 ? row_lo : row_hi, i = j * 8 + kcol + (e & 1);
        if (col < cols && i < d) fn(j, e, (size_t)col * d + i);
      }
  };
#pragma unroll
  for (int j = 0; j < DK / 8; ++j) S[j][0] = S[j][1] = S[j][2] = S[j][3] = 0.f;
  float m0 = -CUDART_INF_F, forgot = 0.f;  // forgot: the sum of the log forget gates so far (LOCAL)
  if (LOCAL) {
    if (seg == 0 && active) {  // the state at the start, set aside: the second launch's last segment writes over it
      float* dst = p.part + pbase(0) * d;
      const float* src = p.state + sbase * d;
      each([&](int, int, size_t at) { dst[at] = src[at]; });
      if (lane < 16 && col0 + lane < cols) p.part_m[(pbase(0) + col0 + lane) * 2] = p.top[sbase + col0 + lane];
    }
  } else if (active) {
    const float* src = p.segments == 1 ? p.state + sbase * d : p.part + pbase(0) * d;
    each([&](int j, int e, size_t at) { S[j][e] = src[at]; });
    m0 = p.segments == 1 ? p.top[sbase + col0] : p.part_m[(pbase(0) + col0) * 2];
    for (int g = 1; g <= seg; ++g) {
      const float* meta = p.part_m + (pbase(g) + col0) * 2;
      const float mb = m0 + meta[1], next = fmaxf(mb, meta[0]);
      const float keep = expf(mb - next), take = expf(meta[0] - next);
      const float* add = p.part + pbase(g) * d;
      each([&](int j, int e, size_t at) { S[j][e] = fmaf(keep, S[j][e], take * add[at]); });
      m0 = next;
    }
  }
  const float bias_i = p.bias[head], bias_f = p.bias[heads + head];
  const float scale = 1.f / sqrtf((float)d);
  float raw[4];
  load_gates(t0, raw);

  int stage = 0;
  for (int base = t0; base < t1; base += TOKENS, stage ^= 1) {
    const int len = min(TOKENS, t1 - base);
    if (base + TOKENS < t1) load_tile(stage ^ 1, base + TOKENS);  // (its readers finished before the barrier that ended the last round)
    cp_async_commit();

    // ---- gates of the tile, every warp for itself: b, a, g by two scans over pairs of tokens (log2 units from here on)
    float bC, gC;
    {
      float lf[2], li[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const bool ok = 2 * lane + k < len;
        lf[k] = ok ? memory_forget_gate(raw[2 + k] + bias_f, p.cap) * LOG2E : 0.f;
        li[k] = ok ? memory_in_gate(raw[k] + bias_i, p.cap) * LOG2E : -CUDART_INF_F;
      }
      float incl = lf[0] + lf[1];
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const float other = __shfl_up_sync(0xffffffffu, incl, off);
        if (lane >= off) incl += other;
      }
      float before = __shfl_up_sync(0xffffffffu, incl, 1);
      if (lane == 0) before = 0.f;
      const float b0 = before + lf[0], b1 = b0 + lf[1];
      const float a0 = li[0] - b0, a1 = li[1] - b1;
      float mx = fmaxf(a0, a1);
#pragma unroll
      for (int off = 1; off < 32; off <<= 1) {
        const float other = __shfl_up_sync(0xffffffffu, mx, off);
        if (lane >= off) mx = fmaxf(mx, other);
      }
      float mbefore = __shfl_up_sync(0xffffffffu, mx, 1);
      const float m02 = m0 * LOG2E;
      if (lane == 0) mbefore = m02;
      const float g0 = fmaxf(fmaxf(m02, mbefore), a0), g1 = fmaxf(g0, a1);
      sA[2 * lane] = a0;
      sA[2 * lane + 1] = a1;
      sG[2 * lane] = g0;
      sG[2 * lane + 1] = g1;
      bC = __shfl_sync(0xffffffffu, b1, 31);
      gC = __shfl_sync(0xffffffffu, g1, 31);
      raw[0] = b0 + g0;  // m_t (log2 units) of this lane's tokens, until the next tile's gates are loaded
      raw[1] = b1 + g1;
    }
    __syncwarp();
    cp_async_wait<1>();
    __syncthreads();

    if (active) {
      const unsigned char* sQ = smem + stage * STAGE;
      const unsigned char* sK = sQ + QK_TILE;
      const unsigned char* sV = sK + QK_TILE + warp * 32;
      const uint32_t q_addr = smem_u32(sQ) + (lane & 15) * QK_ROW + (lane >> 4) * 16;
      const float m02 = m0 * LOG2E;

      if constexpr (!LOCAL) {
      // ---- what the state at the tile's start gives: O = Q S0, 64 tokens x 16 columns
      float O[TOKENS / 16][2][4];
#pragma unroll
      for (int mt = 0; mt < TOKENS / 16; ++mt)
#pragma unroll
        for (int e = 0; e < 4; ++e) O[mt][0][e] = O[mt][1][e] = 0.f;
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t B[3][4];  // three terms: columns 0..7 (k 0..7, k 8..15), columns 8..15
        split3(S[2 * kk][0], S[2 * kk][1], B[0][0], B[1][0], B[2][0]);
        split3(S[2 * kk + 1][0], S[2 * kk + 1][1], B[0][1], B[1][1], B[2][1]);
        split3(S[2 * kk][2], S[2 * kk][3], B[0][2], B[1][2], B[2][2]);
        split3(S[2 * kk + 1][2], S[2 * kk + 1][3], B[0][3], B[1][3], B[2][3]);
        uint32_t a[TOKENS / 16][4];
#pragma unroll
        for (int mt = 0; mt < TOKENS / 16; ++mt) ldsm_x4(a[mt], q_addr + mt * 16 * QK_ROW + kk * 32);
#pragma unroll
        for (int s = 2; s >= 0; --s)  // the small terms first; eight accumulators in turn, so that no product waits for the one before
#pragma unroll
          for (int mt = 0; mt < TOKENS / 16; ++mt) {
            mma(O[mt][0], a[mt], B[s][0], B[s][1]);
            mma(O[mt][1], a[mt], B[s][2], B[s][3]);
          }
      }

      // ---- what the tile's own tokens give, sixteen rows at a time
#pragma unroll
      for (int mt = 0; mt < TOKENS / 16; ++mt) {
        if (mt * 16 < len) {
          const int r_lo = mt * 16 + (lane >> 2), r_hi = r_lo + 8;
          const float g_lo = sG[r_lo], g_hi = sG[r_hi];
          const float e_lo = ex2(m02 - g_lo), e_hi = ex2(m02 - g_hi);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            O[mt][nt][0] *= e_lo; O[mt][nt][1] *= e_lo;
            O[mt][nt][2] *= e_hi; O[mt][nt][3] *= e_hi;
          }
          float P[8][4];  // q . k of these rows with the tile's tokens up to them
#pragma unroll
          for (int j = 0; j < 2 * (mt + 1); ++j) P[j][0] = P[j][1] = P[j][2] = P[j][3] = 0.f;
#pragma unroll
          for (int kk = 0; kk < DK / 16; ++kk) {
            uint32_t a[4];
            ldsm_x4(a, q_addr + mt * 16 * QK_ROW + kk * 32);
#pragma unroll
            for (int jp = 0; jp <= mt; ++jp) {
              uint32_t b[4];
              ldsm_x4(b, smem_u32(sK) + (jp * 16 + (lane & 7) + (lane >> 4) * 8) * QK_ROW + (kk * 16 + ((lane >> 3) & 1) * 8) * 2);
              mma(P[2 * jp], a, b[0], b[1]);
              mma(P[2 * jp + 1], a, b[2], b[3]);
            }
          }
#pragma unroll
          for (int j = 0; j < 2 * (mt + 1); ++j) {
            const int tok = j * 8 + kcol;
            const float a0 = sA[tok], a1 = sA[tok + 1];
            P[j][0] = tok <= r_lo ? P[j][0] * ex2(a0 - g_lo) : 0.f;
            P[j][1] = tok + 1 <= r_lo ? P[j][1] * ex2(a1 - g_lo) : 0.f;
            P[j][2] = tok <= r_hi ? P[j][2] * ex2(a0 - g_hi) : 0.f;
            P[j][3] = tok + 1 <= r_hi ? P[j][3] * ex2(a1 - g_hi) : 0.f;
          }
          float T[3][2][4];  // the three terms' sums apart: six accumulators in turn
#pragma unroll
          for (int s = 0; s < 3; ++s)
#pragma unroll
            for (int e = 0; e < 4; ++e) T[s][0][e] = T[s][1][e] = 0.f;
#pragma unroll
          for (int kk = 0; kk <= mt; ++kk) {
            uint32_t A[3][4], b[4];
            split3(P[2 * kk][0], P[2 * kk][1], A[0][0], A[1][0], A[2][0]);
            split3(P[2 * kk][2], P[2 * kk][3], A[0][1], A[1][1], A[2][1]);
            split3(P[2 * kk + 1][0], P[2 * kk + 1][1], A[0][2], A[1][2], A[2][2]);
            split3(P[2 * kk + 1][2], P[2 * kk + 1][3], A[0][3], A[1][3], A[2][3]);
            ldsm_x4_trans(b, smem_u32(sV) + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * V_ROW + (lane >> 4) * 16);
#pragma unroll
            for (int s = 2; s >= 0; --s) {
              mma(T[s][0], A[s], b[0], b[1]);
              mma(T[s][1], A[s], b[2], b[3]);
            }
          }
#pragma unroll
          for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) O[mt][nt][e] += (T[2][nt][e] + T[1][nt][e]) + T[0][nt][e];
        }
      }

      // ---- leave the read-outs: a thread holds columns kcol, kcol + 1 (and 8 on) of two rows of every sixteen
#pragma unroll
      for (int mt = 0; mt < TOKENS / 16; ++mt) {
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int r = mt * 16 + (lane >> 2) + hf * 8;
          // m_t of row r sits with lane r / 2 (every lane takes part in the exchange)
          const float m_even = __shfl_sync(0xffffffffu, raw[0], r >> 1), m_odd = __shfl_sync(0xffffffffu, raw[1], r >> 1);
          if (r < len) {
            const size_t at = (size_t)(base + r) * heads + head;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
              const int col = col0 + nt * 8 + kcol;
              const float x0 = O[mt][nt][2 * hf] * scale, x1 = O[mt][nt][2 * hf + 1] * scale;
              if (col + 1 < dv && (dv & 1) == 0) {
                *reinterpret_cast<float2*>(p.o + at * dv + col) = make_float2(x0, x1);
              } else {
                if (col < dv) p.o[at * dv + col] = x0;
                if (col + 1 < dv) p.o[at * dv + col + 1] = x1;
                if (col == dv || col + 1 == dv) {
                  const float floor_ = ex2(-((r & 1) ? m_odd : m_even));
                  p.divisor[at] = fmaxf(fabsf(col == dv ? x0 : x1), floor_) + 1e-6f;
                }
              }
            }
          }
        }
      }

      }
      // ---- the state at the tile's end: S^T <- exp(m0 - g_C) S^T + (w V)^T K, w_j = exp(a_j - g_C)
      const float eC = ex2(m02 - gC);
#pragma unroll
      for (int j = 0; j < DK / 8; ++j) { S[j][0] *= eC; S[j][1] *= eC; S[j][2] *= eC; S[j][3] *= eC; }
#pragma unroll
      for (int kk = 0; kk < TOKENS / 16; ++kk) {
        if (kk * 16 < len) {
          uint32_t v[4], A[3][4];
          ldsm_x4_trans(v, smem_u32(sV) + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * V_ROW + ((lane >> 3) & 1) * 16);
          const float w0 = ex2(sA[kk * 16 + kcol] - gC), w1 = ex2(sA[kk * 16 + kcol + 1] - gC);
          const float w8 = ex2(sA[kk * 16 + kcol + 8] - gC), w9 = ex2(sA[kk * 16 + kcol + 9] - gC);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 x = unpack2(v[e]);
            split3(x.x * (e < 2 ? w0 : w8), x.y * (e < 2 ? w1 : w9), A[0][e], A[1][e], A[2][e]);
          }
          constexpr int GROUP = (DK / 16) % 4 == 0 ? 4 : ((DK / 16) % 3 == 0 ? 3 : ((DK / 16) % 2 == 0 ? 2 : 1));
#pragma unroll
          for (int j0 = 0; j0 < DK / 16; j0 += GROUP) {  // 2 GROUP accumulators in turn
            uint32_t b[GROUP][4];
#pragma unroll
            for (int g = 0; g < GROUP; ++g)
              ldsm_x4_trans(b[g], smem_u32(sK) + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * QK_ROW + ((j0 + g) * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
            for (int s = 2; s >= 0; --s)
#pragma unroll
              for (int g = 0; g < GROUP; ++g) {
                mma(S[2 * (j0 + g)], A[s], b[g][0], b[g][1]);
                mma(S[2 * (j0 + g) + 1], A[s], b[g][2], b[g][3]);
              }
          }
        }
      }
    }
    m0 = (bC + gC) * (1.f / LOG2E);
    if (LOCAL) forgot += bC * (1.f / LOG2E);
    if (base + TOKENS < t1) load_gates(base + TOKENS, raw);
    __syncthreads();  // this stage is copied into again in the round after next; sA and sG are written anew
  }
  cp_async_wait<0>();
  if (!active) return;
  if (LOCAL) {
    float* dst = p.part + pbase(seg + 1) * d;
    each([&](int j, int e, size_t at) { dst[at] = S[j][e]; });
    if (lane < 16 && col0 + lane < cols) {
      p.part_m[(pbase(seg + 1) + col0 + lane) * 2] = m0;
      p.part_m[(pbase(seg + 1) + col0 + lane) * 2 + 1] = forgot;
    }
  } else if (t1 == last) {
    float* dst = p.state + sbase * d;
    each([&](int j, int e, size_t at) { dst[at] = S[j][e]; });
    if (lane < 16 && col0 + lane < cols) p.top[sbase + col0 + lane] = m0;
  }
}

}  // namespace

namespace {
// CTAs of a sequence's head, and warps of a CTA (even shares of the value columns' tiles of sixteen)
inline void shares(int dv, int& ctas, int& warps) {
  const int tiles = (dv + 1 + 15) / 16;
  ctas = (tiles + MAX_WARPS - 1) / MAX_WARPS;
  warps = (tiles + ctas - 1) / ctas;
}
}  // namespace

// Into how many segments the sequences of a step are cut: as many as give every SM two CTAs, none shorter than four tiles.
DLI_EXPORT int dli_matrix_memory_segments(int num_seqs, int heads, int dv, int max_len) {
  int ctas, warps;
  shares(dv, ctas, warps);
  long long fill = 2LL * sm_count() / ((long long)ctas * heads * (num_seqs > 0 ? num_seqs : 1));
  const int most = (max_len + TOKENS - 1) / TOKENS / 4;
  if (fill > most) fill = most;
  return fill < 1 ? 1 : (fill > 64 ? 64 : (int)fill);
}

// segments > 1: part [num_seqs segments heads (dv + 1) d] and part_m [num_seqs segments heads (dv + 1) 2] are scratch.
DLI_EXPORT int dli_matrix_memory_chunk(float* o, float* divisor, const void* u, long long u_stride, const float* gates, const float* bias, float cap,
                                       float* state, float* top, const int* q_start, const int* state_slot, int num_seqs, int heads, int d, int dv,
                                       int segments, float* part, float* part_m, cudaStream_t stream) {
  if (num_seqs == 0) return 0;
  if (heads < 1 || heads > 65535 || segments < 1 || (long long)num_seqs * segments > 65535 || d < 1 || d > DK || dv < 1 || !(cap > 0.f) ||
      (segments > 1 && (!part || !part_m)))
    return DLI_ERR_UNSUPPORTED;
  static OncePerDevice configured;
  if (!configured.here()) {
    cudaError_t e = cudaFuncSetAttribute(matrix_memory_chunk_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(matrix_memory_chunk_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return (int)e;
    configured.here() = true;
  }
  Params p;
  p.o = o; p.divisor = divisor; p.u = (const bf16*)u; p.u_stride = u_stride; p.gates = gates; p.bias = bias; p.cap = cap;
  p.state = state; p.top = top; p.q_start = q_start; p.state_slot = state_slot; p.heads = heads; p.d = d; p.dv = dv;
  p.vec = (d % 8) == 0 && (dv % 8) == 0 && (u_stride % 8) == 0 && ((uintptr_t)u & 15) == 0;
  p.segments = segments; p.part = part; p.part_m = part_m;
  int ctas;
  shares(dv, ctas, p.warps);
  if (segments > 1) {
    const cudaError_t e = launch_pdl((matrix_memory_chunk_kernel<true>), dim3(ctas, heads, num_seqs * (segments - 1)), dim3(p.warps * 32), (size_t)SMEM,
                                     stream, 1, p);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl((matrix_memory_chunk_kernel<false>), dim3(ctas, heads, num_seqs * segments), dim3(p.warps * 32), (size_t)SMEM, stream, 1, p);
}
