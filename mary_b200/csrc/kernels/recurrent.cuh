// What the kernels of recurrent layers share: short convolutions with their history, and the one-token update of a head's state.
//
// Convolution history: the last `taps` inputs of every channel in a ring addressed by absolute position, [slot][taps][channels].  A
// token at position p reads the entries of p - 1 .. p - (taps - 1) and writes the entry of p, which none of those reads touches.
#pragma once
#include "typed.cuh"

namespace mary {

constexpr int STEP_THREADS = 256;                                  // threads of a one-token kernel

// How a state decays and what is written to it: a decay per key channel; the delta rule with a decay per head; a decay per head.
enum DecayMode { DECAY_CHANNEL, DECAY_DELTA, DECAY_HEAD };

// silu of the depthwise causal convolution of channel c at row t (position pos of its sequence, whose portion starts at row first)
template <typename T>
__device__ __forceinline__ float conv_silu(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, const T* __restrict__ bias,
                                           const T* __restrict__ ring, int taps, int C,
                                           int c, int t, int first, int pos) {
  float acc = bias ? to_f<T>(bias[c]) : 0.f;
  for (int d = 0; d < taps; ++d) {                     // d tokens back
    float v = 0.f;
    if (t - d >= first) v = to_f<T>(x[(int64_t)(t - d) * ldx + c]);
    else if (pos - d >= 0) v = to_f<T>(ring[(int64_t)((pos - d) % taps) * C + c]);
    acc = fmaf(to_f<T>(w[(int64_t)c * taps + taps - 1 - d]), v, acc);
  }
  return silu_t<T>(acc);
}

// silu(conv) of E channels from c on for the four tokens of a block: rows rb .. rb + 3 (a sequence's portion is rows first .. end - 1),
// the block's first token at position pos.  Rows before the portion come from the ring, positions before 0 are zero.
template <typename T, int TAPS, int E>
__device__ __forceinline__ void conv_block(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, const T* __restrict__ bias,
                                           const T* __restrict__ ring, int n_taps, int C,
                                           int c, int rb, int first, int end, int pos, float (&y)[4][E]) {
  const int taps = TAPS > 0 ? TAPS : n_taps;
  float wr[E][TAPS > 0 ? TAPS : 1];
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int e = 0; e < E; ++e) {
      if constexpr (TAPS == 4 && E == 4) {
        load_e<T, 4>(w + (int64_t)(c + e) * 4, wr[e]);
      } else {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) wr[e][j] = to_f<T>(w[(int64_t)(c + e) * TAPS + j]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < E; ++e) y[i][e] = bias ? to_f<T>(bias[c + e]) : 0.f;
  if constexpr (TAPS > 0) {
    // all rows are requested before the first is used
    float v[TAPS + 3][E];
#pragma unroll
    for (int r = 1 - TAPS; r < 4; ++r) {
      const bool here = rb + r >= first;
      const T* src = here ? x + (int64_t)(rb + r) * ldx + c : ring + (int64_t)((pos + r + TAPS) % TAPS) * C + c;
      if (rb + r < end && pos + r >= 0) load_e<T, E>(src, v[r + TAPS - 1]);
      else
#pragma unroll
        for (int e = 0; e < E; ++e) v[r + TAPS - 1][e] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int d = 0; d < TAPS; ++d)
#pragma unroll
        for (int e = 0; e < E; ++e) y[i][e] = fmaf(wr[e][TAPS - 1 - d], v[i - d + TAPS - 1][e], y[i][e]);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < E; ++e) y[i][e] = silu_t<T>(y[i][e]);
    return;
  }
  for (int r = 1 - taps; r < 4; ++r) {
    float v[E] = {};
    if (rb + r >= end) break;
    if (rb + r >= first) load_e<T, E>(x + (int64_t)(rb + r) * ldx + c, v);
    else if (pos + r >= 0) load_e<T, E>(ring + (int64_t)((pos + r) % taps) * C + c, v);
    else continue;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = i - r;
      if (d < 0 || d >= taps) continue;
#pragma unroll
      for (int e = 0; e < E; ++e) {
        y[i][e] = fmaf(to_f<T>(w[(int64_t)(c + e) * taps + taps - 1 - d]), v[e], y[i][e]);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < E; ++e) y[i][e] = silu_t<T>(y[i][e]);
}

// One CTA per (sequence, head): 8 lanes per state column, 32 columns at a time, the next columns' state in flight while the
// current ones are updated.  The read-out of all columns meets in shared memory for the head norm.
template <int NR4>
__device__ __forceinline__ void load_cols(float4 (&st)[NR4], const float* state, int col, int DV, int DKS, bool fresh, int lane8) {
#pragma unroll
  for (int r = 0; r < NR4; ++r) {
    const int c = (r * 8 + lane8) * 4;
    st[r] = (!fresh && col < DV && c < DKS) ? __ldcs((const float4*)(state + (int64_t)col * DKS + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
}

__device__ __forceinline__ float sum8(float v) {
#pragma unroll
  for (int o = 4; o >= 1; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// sq / sk [NR4 * 32] (zero beyond DK), sa [NR4 * 32] channel decays (delta rule and decay per head: the scalars g and b instead; b scales what
// is written), sv [DV]; leaves o in so[DV].
template <int NR4, int MODE>
__device__ __forceinline__ void step_columns(float4 (&st)[NR4], float* state, int DV, int DKS, bool fresh, const float* sq, const float* sk,
                                             const float* sa, float g, float b, const float* sv, float* so) {
  const int lane8 = threadIdx.x & 7;
  for (int col = threadIdx.x >> 3, c0 = 0; c0 < DV; c0 += STEP_THREADS / 8, col += STEP_THREADS / 8) {
    float4 nx[NR4];
    if (c0 + STEP_THREADS / 8 < DV) load_cols<NR4>(nx, state, col + STEP_THREADS / 8, DV, DKS, fresh, lane8);
    const float vt = col < DV ? sv[col] : 0.f;
    float w = vt;
    if constexpr (MODE == DECAY_DELTA) {
      float pred = 0.f;
#pragma unroll
      for (int r = 0; r < NR4; ++r) {
        const float4 k4 = *(const float4*)(sk + (r * 8 + lane8) * 4);
        st[r].x *= g; st[r].y *= g; st[r].z *= g; st[r].w *= g;
        pred = fmaf(k4.x, st[r].x, fmaf(k4.y, st[r].y, fmaf(k4.z, st[r].z, fmaf(k4.w, st[r].w, pred))));
      }
      w = b * (vt - sum8(pred));
    } else if constexpr (MODE == DECAY_HEAD) {
      w = b * vt;
#pragma unroll
      for (int r = 0; r < NR4; ++r) { st[r].x *= g; st[r].y *= g; st[r].z *= g; st[r].w *= g; }
    }
    float acc = 0.f;
#pragma unroll
    for (int r = 0; r < NR4; ++r) {
      const int c = (r * 8 + lane8) * 4;
      const float4 k4 = *(const float4*)(sk + c), q4 = *(const float4*)(sq + c);
      if constexpr (MODE == DECAY_CHANNEL) {
        const float4 a4 = *(const float4*)(sa + c);
        st[r].x *= a4.x; st[r].y *= a4.y; st[r].z *= a4.z; st[r].w *= a4.w;
      }
      st[r].x = fmaf(k4.x, w, st[r].x); st[r].y = fmaf(k4.y, w, st[r].y); st[r].z = fmaf(k4.z, w, st[r].z); st[r].w = fmaf(k4.w, w, st[r].w);
      acc = fmaf(q4.x, st[r].x, fmaf(q4.y, st[r].y, fmaf(q4.z, st[r].z, fmaf(q4.w, st[r].w, acc))));
      if (col < DV && c < DKS) __stcs((float4*)(state + (int64_t)col * DKS + c), st[r]);
    }
    acc = sum8(acc);
    if (lane8 == 0 && col < DV) so[col] = acc;
#pragma unroll
    for (int r = 0; r < NR4; ++r) st[r] = nx[r];
  }
}

}  // namespace mary
