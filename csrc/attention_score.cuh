// How a raw score (q . k) becomes a softmax exponent or a weight, for the attention kernels. All arithmetic is fp32.
//
//   kPlain    exponent = scale * s
//   kCapped   exponent = cap * tanh(scale * s / cap)            (tanh through one exponential and one reciprocal)
//   kSigmoid  weight   = sigmoid(scale * s + bias of the head)  (no maximum, no sum: nothing normalises the weights)
#pragma once

#include "common.cuh"

namespace pxl {

enum ScoreMode : int { kPlain = 0, kCapped = 1, kSigmoid = 2 };

struct ScoreArgs {
  float cap2;         // kCapped: cap * log2(e)
  float gain;         // kCapped: 2 log2(e) * scale / cap
  const float* bias;  // kSigmoid: [query heads]
};

inline ScoreArgs score_args(float scale, float softcap, const float* bias) {
  constexpr float log2e = 1.4426950408889634f;
  return {softcap * log2e, softcap > 0.f ? 2.f * log2e * scale / softcap : 0.f, bias};
}
inline int score_mode(float softcap, const float* bias) { return bias ? kSigmoid : softcap > 0.f ? kCapped : kPlain; }

__device__ __forceinline__ float score_ex2(float x) {  // 2^x; -inf -> 0, large -> inf
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float score_rcp(float x) {  // 1 / x; inf -> 0
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// exponent in units of log2
template <int SM>
__device__ __forceinline__ float score_log2(float s, float scale_log2, const ScoreArgs& a) {
  if constexpr (SM == kCapped) return fmaf(-2.f * a.cap2, score_rcp(1.f + score_ex2(s * a.gain)), a.cap2);
  return s * scale_log2;
}
__device__ __forceinline__ float sigmoid_weight(float s, float scale_log2, float bias_log2) {
  return score_rcp(1.f + score_ex2(-fmaf(s, scale_log2, bias_log2)));
}

}  // namespace pxl
