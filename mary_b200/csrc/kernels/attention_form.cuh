// What a call of the attention kernels may ask for beyond causal softmax attention with a window: chunks, capped scores, a sink, a query
// temperature by position, and the difference of two softmax maps over the same values.
#pragma once
#include "common.cuh"

// Passed by host pointer to the launchers (null: none of it).  Two maps: the query and key rows of a head are [map 0 | map 1], both maps read
// the head's values, and the result is rms(a0 - mix * a1) * post over the value width.
struct MaryAttnForm {
  const float* sink;     // [Hq]: a learned score per head that enters the sum of weights only; or null
  int64_t q_ld;          // elements between the query rows of two tokens (0: contiguous)
  int chunk;             // > 0: a query sees the keys of its own chunk of this many positions, counted from position 0
  int maps;              // 1 or 2
  int temp_every;        // > 0: the query at position p is multiplied by 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)
  float temp_coef;
  float cap;             // > 0: score <- cap * tanh(score / cap)
  float mix, post, eps;  // two maps
};

namespace mary {

__device__ __forceinline__ float query_temperature(const MaryAttnForm& f, int pos) {
  return f.temp_every > 0 ? fmaf(f.temp_coef, logf((float)((pos + 1) / f.temp_every + 1)), 1.0f) : 1.0f;
}
__device__ __forceinline__ int first_key(const MaryAttnForm& f, int pos) { return f.chunk > 0 ? pos / f.chunk * f.chunk : 0; }

// tanh in 32 bits whatever the compiler's math mode (its fast tanh has 11 bits): the power series for small arguments, elsewhere
// 1 - 2 / (exp(2 |x|) + 1), whose result is at least 0.46 there, so the subtraction loses nothing.
__device__ __forceinline__ float tanh_series(float x) {      // |x| <= 0.5
  const float y = x * x;
  float p = fmaf(y, 21844.0f / 6081075.0f, -1382.0f / 155925.0f);
  p = fmaf(p, y, 62.0f / 2835.0f);
  p = fmaf(p, y, -17.0f / 315.0f);
  p = fmaf(p, y, 2.0f / 15.0f);
  p = fmaf(p, y, -1.0f / 3.0f);
  return fmaf(p * y, x, x);
}
__device__ __forceinline__ float tanh_32(float x) {
  const float a = fabsf(x);
  if (a <= 0.5f) return tanh_series(x);
  return copysignf(1.0f - __fdividef(2.0f, __expf(2.0f * fminf(a, 20.0f)) + 1.0f), x);
}
__device__ __forceinline__ float cap_score(float s, float cap) { return cap > 0.f ? cap * tanh_32(s / cap) : s; }

}  // namespace mary
