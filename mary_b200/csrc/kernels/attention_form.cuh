// What a call of the attention kernels may ask for beyond causal softmax attention with a window: chunks, capped scores, a sink, a query
// temperature by position, the difference of two softmax maps over the same values, and a rotation of the result by the query's position.
#pragma once
#include "common.cuh"

// Passed by host pointer to the launchers (null: none of it).  Two maps: the query and key rows of a head are [map 0 | map 1], both maps read
// the head's values, and the result is rms(a0 - mix * a1) * post over the value width.
struct MaryAttnForm {
  const float2* turn;    // [T][DV / 2] (cosine, sine): pair (2 m, 2 m + 1) of every head's result at token row t is turned back by that angle; or null
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

// The result's pair (a, b) turned back by the angle of cs.
__device__ __forceinline__ float2 turned_back(float2 cs, float a, float b) { return make_float2(fmaf(a, cs.x, b * cs.y), fmaf(b, cs.x, -a * cs.y)); }
// The same where neighbouring lanes hold neighbouring columns: every lane of the warp calls it with its value of token row t, column d of a head.
__device__ __forceinline__ float turned_back_lane(const MaryAttnForm& f, float v, int64_t t, int d, int DV, bool in) {
  if (!f.turn) return v;
  const float other = __shfl_xor_sync(0xffffffffu, v, 1);
  if (!in) return v;
  const float2 cs = f.turn[t * (DV / 2) + d / 2];
  return fmaf(v, cs.x, (d & 1 ? -other : other) * cs.y);
}

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
// Two values at a time through the packed 32-bit pipes: a * b + c.
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(*(const uint64_t*)&a), "l"(*(const uint64_t*)&b), "l"(*(const uint64_t*)&c));
  return *(float2*)&d;
}

// N raw scores of a lane's row -> cap * tanh(score * scale / cap) in units of log2, given scale_log2 = scale * log2(e).  Where no score of the
// warp is beyond a quarter of the cap (lanes that hold no scores: `held` false) the series of tanh to the ninth power is exact to 32 bits.
template <int N>
__device__ __forceinline__ void cap_scores(float (&s)[N], float scale_log2, float cap, bool held = true) {
  float top = 0.f;
#pragma unroll
  for (int j = 0; j < N; ++j) top = fmaxf(top, fabsf(s[j]));
  const float c = cap * 1.4426950408889634f, k = scale_log2 / c;                // raw score -> argument of tanh
  if (__all_sync(0xffffffffu, !held || top * fabsf(k) <= 0.25f)) {
    const float k2 = k * k, c1 = scale_log2, c3 = c1 * k2 * (-1.0f / 3.0f), c5 = c1 * k2 * k2 * (2.0f / 15.0f);
    const float c7 = c1 * k2 * k2 * k2 * (-17.0f / 315.0f), c9 = c1 * k2 * k2 * k2 * k2 * (62.0f / 2835.0f);
    const float2 zero = make_float2(0.f, 0.f);
#pragma unroll
    for (int j = 0; j < N; j += 2) {
      const float2 x = make_float2(s[j], s[j + 1]), y = fma2(x, x, zero);
      float2 q = fma2(y, make_float2(c9, c9), make_float2(c7, c7));
      q = fma2(q, y, make_float2(c5, c5));
      q = fma2(q, y, make_float2(c3, c3));
      q = fma2(q, y, make_float2(c1, c1));
      q = fma2(q, x, zero);
      s[j] = q.x;
      s[j + 1] = q.y;
    }
  } else {
#pragma unroll
    for (int j = 0; j < N; ++j) s[j] = c * tanh_32(s[j] * k);
  }
}
__device__ __forceinline__ float cap_score(float s, float cap) { return cap > 0.f ? cap * tanh_32(s / cap) : s; }

}  // namespace mary
