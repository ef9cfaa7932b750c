// What may happen to a scaled score s = (q . k) * scale before the softmax; d = p - key, the distance (>= 0 where seen).
// A template parameter of the tensor-core attention kernels, `kind` at their entry points:
//
//   SCORE_PLAIN   nothing
//   SCORE_LOG     s - r1_h ln(1 + r2_h d)                  numbers per head from `dist` [2, heads], r1 of all heads, then r2
//   SCORE_BOUND   cap tanh(s / cap) - slope_h d            slopes from `dist` [heads]; cap <= 0: s itself in place of the tanh
//
// The kernels work on scores times log2 e ("units" below): the softmax is then powers of two.
#pragma once

#define SCORE_PLAIN 0
#define SCORE_LOG 1
#define SCORE_BOUND 2

// The bound in units: with c = cap log2 e, cap tanh(s / cap) is c - 2 c / (1 + 2^(v k)), k = 2 log2(e) / c, v in units.
struct ScoreBound {
  float c, k;
};
__device__ __forceinline__ ScoreBound score_bound(float cap) {
  ScoreBound b;
  b.c = cap * 1.4426950408889634f;
  b.k = cap > 0.f ? 2.0f / cap : 0.f;
  return b;
}
__device__ __forceinline__ float score_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float score_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// v in units -> the bounded score in units (2^x overflows to infinity for large x: the fraction is then 0)
__device__ __forceinline__ float bounded_score(float v, const ScoreBound& b) {
  return b.c > 0.f ? fmaf(-2.0f * b.c, score_rcp(1.0f + score_exp2(v * b.k)), b.c) : v;
}

// the entry points' check of `kind`, `dist` and `cap`
static inline bool score_kind_ok(int kind, const float* dist) {
  return kind == SCORE_PLAIN || ((kind == SCORE_LOG || kind == SCORE_BOUND) && dist != nullptr);
}
