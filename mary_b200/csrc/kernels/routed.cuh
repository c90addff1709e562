// The outputs of a batch's routed experts as the residual step reads them: weighted and summed per token while the stream is updated.
#pragma once
#include "typed.cuh"

namespace mary {

constexpr int ROUTED_MAX = 32;       // experts per token

// Where the weighted outputs of a token's routed experts come from: padded rows (row_of[t * k + j], y) or their finished sum; entries whose
// expert index is n_experts or more stand for the normed input x itself.
template <typename T> struct Routed {
  const T* y; int64_t ldy; const int* row_of;
  const float* sum;
  const int* idx; const float* w; const T* x;
  int k, n_experts;
};

// The rows of one token, listed in shared memory.
struct RoutedRows {
  float weight[ROUTED_MAX], self;
  int src[ROUTED_MAX], n;
};

// Called by one thread; the block synchronises before the list is read.
template <typename T>
__device__ __forceinline__ void list_routed(const Routed<T>& r, int64_t t, RoutedRows& l) {
  l.self = 0.f;
  l.n = 0;
  for (int j = 0; j < r.k; ++j) {
    const float w = r.w[t * r.k + j];
    if (r.idx[t * r.k + j] >= r.n_experts) l.self += w;
    else if (r.y) {
      const int s = r.row_of[t * r.k + j];
      if (s >= 0) { l.src[l.n] = s; l.weight[l.n++] = w; }
    }
  }
}

// s += the routed outputs of token t at columns i .. i + E - 1 of H; n and self as listed (0 without routed experts).
template <typename T, int E>
__device__ __forceinline__ void add_routed(const Routed<T>& r, const RoutedRows& l, int n, float self, int64_t t, int i, int H, float (&s)[E]) {
  float g[E];
  if (r.sum) {
    load_v<float, E>(r.sum + t * H + i, g);
#pragma unroll
    for (int j = 0; j < E; ++j) s[j] += g[j];
  }
  for (int e = 0; e < n; ++e) {
    load_v<T, E>(r.y + l.src[e] * r.ldy + i, g);
#pragma unroll
    for (int j = 0; j < E; ++j) s[j] = fmaf(l.weight[e], g[j], s[j]);
  }
  if (self != 0.f) {
    load_v<T, E>(r.x + t * H + i, g);
#pragma unroll
    for (int j = 0; j < E; ++j) s[j] = fmaf(self, g[j], s[j]);
  }
}

}  // namespace mary
