// Scores of talking-heads attention: capped, with a bias that grows with the logarithm of the distance, as e^s.
#pragma once
#include "common.cuh"

namespace mv {

// Largest cap whose e^s and sums of them fit into fp32 with a wide margin on both sides.
constexpr float kTalkCap = 60.f;

__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// e^(cap tanh(x scale / cap) - bias) in powers of two: tanh(z) = 1 - 2 / (e^2z + 1), whose absolute error is that of fp32.
struct TalkScore {
  float in, out, top;
  __device__ __forceinline__ TalkScore(float scale, float cap)
      : in(2.f * scale / cap * 1.4426950408889634f), out(-2.f * cap * 1.4426950408889634f), top(cap * 1.4426950408889634f) {}
  // log2 of the factor that a distance puts on a weight, plus the cap's constant term
  __device__ __forceinline__ float bias(float r1, float r2, int distance) const {
    return fmaf(-r1, __log2f(fmaf(r2, static_cast<float>(distance), 1.f)), top);
  }
  __device__ __forceinline__ float weight(float dot, float bias) const {
    return fast_exp2(fmaf(fast_rcp(fast_exp2(dot * in) + 1.f), out, bias));
  }
};

}  // namespace mv
