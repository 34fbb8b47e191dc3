// Attention scores that are bent before the softmax: a soft cap, s -> c tanh(s / c), and a penalty that grows with the distance,
// s -> s - slope (i - j) with a slope per query head.  Kernels compiled with -DBENT_SCORES=1 apply both to the float32 scores as
// they leave the Q K^T product, and work in log2 units with a scale of 1 from there on.
#pragma once
#include "common.cuh"

#ifndef BENT_SCORES
#define BENT_SCORES 0
#endif

namespace dli {

struct ScoreBend {
  float scale_log2;     // softmax scale times log2(e)
  float exp_scale;      // 2 log2(e) scale / softcap: 2^(raw exp_scale) = e^(2 s / c)
  float cap_log2;       // softcap times log2(e); 0: no cap
  const float* slopes;  // per query head (natural units), or null
};

inline ScoreBend make_score_bend(float scale, float softcap, const float* slopes) {
  const float log2e = 1.4426950408889634f;
  ScoreBend b;
  b.scale_log2 = scale * log2e;
  b.exp_scale = softcap > 0.f ? 2.f * log2e * scale / softcap : 0.f;
  b.cap_log2 = softcap > 0.f ? softcap * log2e : 0.f;
  b.slopes = slopes;
  return b;
}

__device__ __forceinline__ float bend_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float bend_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// c tanh(s / c) = c - 2 c / (1 + e^(2 s / c)), plus `bias`, all in log2 units.  (Large arguments end at c and -c: the power becomes
// infinite or zero.)
__device__ __forceinline__ float capped_score(float raw, const ScoreBend& b, float bias) {
  return fmaf(-2.f * b.cap_log2, bend_rcp(1.f + bend_ex2(raw * b.exp_scale)), b.cap_log2 + bias);
}
__device__ __forceinline__ float bent_score(float raw, const ScoreBend& b, float bias) {
  return b.cap_log2 != 0.f ? capped_score(raw, b, bias) : fmaf(raw, b.scale_log2, bias);
}
// the slope of a query head in log2 units
__device__ __forceinline__ float bend_slope(const ScoreBend& b, int head) { return b.slopes ? b.slopes[head] * 1.4426950408889634f : 0.f; }

}  // namespace dli
