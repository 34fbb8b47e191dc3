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

__global__ void __launch_bounds__(MAX_WARPS * 32) matrix_memory_chunk_kernel(const Params p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(128) unsigned char smem[];
  const int seq = blockIdx.z, head = blockIdx.y;
  const int t0 = p.q_start[seq], t1 = p.q_start[seq + 1];
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
        cp_async16(smem_u32(sQ + r * QK_ROW + c * 16), src, ok ? 16 : 0);
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
  float S[DK / 8][4];
  const int row_lo = col0 + (lane >> 2), row_hi = row_lo + 8, kcol = (lane & 3) * 2;
#pragma unroll
  for (int j = 0; j < DK / 8; ++j) {
    const int i = j * 8 + kcol;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int col = e < 2 ? row_lo : row_hi, ii = i + (e & 1);
      S[j][e] = (col < cols && ii < d) ? p.state[(sbase + col) * d + ii] : 0.f;
    }
  }
  float m0 = active ? p.top[sbase + col0] : 0.f;
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
#pragma unroll
        for (int mt = 0; mt < TOKENS / 16; ++mt) {
          if (mt * 16 < len) {
            uint32_t a[4];
            ldsm_x4(a, q_addr + mt * 16 * QK_ROW + kk * 32);
#pragma unroll
            for (int s = 2; s >= 0; --s) {  // the small terms first
              mma(O[mt][0], a, B[s][0], B[s][1]);
              mma(O[mt][1], a, B[s][2], B[s][3]);
            }
          }
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
              mma(O[mt][0], A[s], b[0], b[1]);
              mma(O[mt][1], A[s], b[2], b[3]);
            }
          }
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
#pragma unroll
          for (int jp = 0; jp < DK / 16; ++jp) {
            uint32_t b[4];
            ldsm_x4_trans(b, smem_u32(sK) + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * QK_ROW + (jp * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
            for (int s = 2; s >= 0; --s) {
              mma(S[2 * jp], A[s], b[0], b[1]);
              mma(S[2 * jp + 1], A[s], b[2], b[3]);
            }
          }
        }
      }
    }
    m0 = (bC + gC) * (1.f / LOG2E);
    if (base + TOKENS < t1) load_gates(base + TOKENS, raw);
    __syncthreads();  // this stage is copied into again in the round after next; sA and sG are written anew
  }
  cp_async_wait<0>();
  if (!active) return;
#pragma unroll
  for (int j = 0; j < DK / 8; ++j) {
    const int i = j * 8 + kcol;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int col = e < 2 ? row_lo : row_hi, ii = i + (e & 1);
      if (col < cols && ii < d) p.state[(sbase + col) * d + ii] = S[j][e];
    }
  }
  if (lane < 16 && col0 + lane < cols) p.top[sbase + col0 + lane] = m0;
}

}  // namespace

DLI_EXPORT int dli_matrix_memory_chunk(float* o, float* divisor, const void* u, long long u_stride, const float* gates, const float* bias, float cap,
                                       float* state, float* top, const int* q_start, const int* state_slot, int num_seqs, int heads, int d, int dv,
                                       int max_len, cudaStream_t stream) {
  (void)max_len;
  if (num_seqs == 0) return 0;
  if (heads < 1 || heads > 65535 || num_seqs > 65535 || d < 1 || d > DK || dv < 1 || !(cap > 0.f)) return DLI_ERR_UNSUPPORTED;
  static OncePerDevice configured;
  if (!configured.here()) {
    cudaError_t e = cudaFuncSetAttribute(matrix_memory_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return (int)e;
    configured.here() = true;
  }
  Params p;
  p.o = o; p.divisor = divisor; p.u = (const bf16*)u; p.u_stride = u_stride; p.gates = gates; p.bias = bias; p.cap = cap;
  p.state = state; p.top = top; p.q_start = q_start; p.state_slot = state_slot; p.heads = heads; p.d = d; p.dv = dv;
  p.vec = (d % 8) == 0 && (dv % 8) == 0 && (u_stride % 8) == 0 && ((uintptr_t)u & 15) == 0;
  const int tiles = (dv + 1 + 15) / 16, ctas = (tiles + MAX_WARPS - 1) / MAX_WARPS;
  p.warps = (tiles + ctas - 1) / ctas;  // even shares
  return (int)launch_pdl(matrix_memory_chunk_kernel, dim3(ctas, heads, num_seqs), dim3(p.warps * 32), (size_t)SMEM, stream, 1, p);
}
