// Everything around the linear recurrences of recurrent_scan.cu, for bf16 and for 32-bit activations: the per-channel decay from its
// low-rank projection, the short convolutions with their unit norms and gates, the convolution history, the gated norm of the
// read-out, and the fused one-token steps that do all of it in one launch per layer.  Decays, gates, unit norms and the state are in
// exact 32-bit arithmetic.
#include "host_utils.h"
#include "recurrent.cuh"

using namespace mary;

namespace {

constexpr int NT = STEP_THREADS;

// decay[t, c] = sigmoid(a2[c] . x[t] + bias[c]) ^ inv_tau, x[t] of `rank` values
template <typename T>
__global__ void __launch_bounds__(NT) channel_decay_kernel(const T* __restrict__ x, int64_t ldx, int rank, const T* __restrict__ a2,
                                                           const T* __restrict__ bias, float* __restrict__ decay, int n_tok, int C, float inv_tau) {
  pdl_sync();
  constexpr int TT = 16, RC = 16;
  __shared__ __align__(16) float sx[RC][TT];
  __shared__ float sw[NT][RC + 1];
  const int c = blockIdx.x * NT + threadIdx.x, t0 = blockIdx.y * TT;
  float acc[TT] = {};
  for (int r0 = 0; r0 < rank; r0 += RC) {
    __syncthreads();
    {
      const int t = threadIdx.x / RC, r = threadIdx.x % RC;
      sx[r][t] = (t0 + t < n_tok && r0 + r < rank) ? to_f<T>(x[(int64_t)(t0 + t) * ldx + r0 + r]) : 0.f;
    }
    for (int i = threadIdx.x; i < NT * RC; i += NT) {
      const int cc = blockIdx.x * NT + i / RC, r = r0 + i % RC;
      sw[i / RC][i % RC] = (cc < C && r < rank) ? to_f<T>(a2[(int64_t)cc * rank + r]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < RC; ++r) {
      const float w = sw[threadIdx.x][r];
#pragma unroll
      for (int t = 0; t < TT; t += 4) {
        const float4 x4 = *(const float4*)&sx[r][t];
        acc[t] = fmaf(w, x4.x, acc[t]); acc[t + 1] = fmaf(w, x4.y, acc[t + 1]);
        acc[t + 2] = fmaf(w, x4.z, acc[t + 2]); acc[t + 3] = fmaf(w, x4.w, acc[t + 3]);
      }
    }
  }
  if (c >= C) return;
  const float b = to_f<T>(bias[c]);
#pragma unroll
  for (int t = 0; t < TT; ++t)
    if (t0 + t < n_tok) decay[(int64_t)(t0 + t) * C + c] = exp_t<T>(log_sigmoid_t<T>(acc[t] + b) * inv_tau);
}

struct ConvIn {
  int HK, H, DK, DV, taps, C;      // C = 2 HK DK + H DV channels, in the order q, k, v; taps [C][taps], last one the current token's
};

// One warp per (sequence, block of four tokens, item); items: HK query / key heads (unit vectors, and the products of the block's keys
// with its keys and queries), H value heads (with their gates).  VEC: widths, pitch and addresses allow accesses of four values.
template <typename T, int TAPS, bool VEC>
__global__ void __launch_bounds__(256) delta_prep_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, const T* __restrict__ ring_all,
                                                         const T* __restrict__ b_in, const T* __restrict__ a_in, const float* __restrict__ a_log,
                                                         const float* __restrict__ dt_bias, const int* __restrict__ q_start,
                                                         const int* __restrict__ kv_len, const int* __restrict__ slots, float* __restrict__ q,
                                                         float* __restrict__ k, float* __restrict__ v, float* __restrict__ g, float* __restrict__ beta,
                                                         float* __restrict__ pairs, ConvIn ci) {
  pdl_sync();
  constexpr int E = VEC ? 4 : 1, NI = 8 / E;          // DK <= 256: eight channels per lane
  const int items = ci.HK + ci.H;
  const int gw = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int blk = gw / items, it = gw % items, lane = threadIdx.x & 31, seq = blockIdx.y;
  const int first = q_start[seq], end = q_start[seq + 1], rb = first + blk * 4;
  if (rb >= end) return;
  const int nt = min(4, end - rb);
  const int pos = kv_len[seq] - (end - first) + blk * 4;
  const T* ring = ring_all + (int64_t)slots[seq] * ci.taps * ci.C;
  if (it < ci.HK) {
    float yq[NI][4][E], yk[NI][4][E];
    // 32 sums in the places of the output rows: dot[8 t + j] = k_j . k_t for j < t, dot[8 t + 4 + j] = k_j . q_t for j <= t,
    // dot[8 t + 3] = k_t . k_t, and q_t . q_t in four of the places that no product takes
    constexpr int QQ[4] = {0, 1, 2, 5};
    float dot[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) dot[i] = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = i * 32 * E + lane * E;
      if (c < ci.DK) {
        conv_block<T, TAPS, E>(x, ldx, w, (const T*)nullptr, ring, ci.taps, ci.C, it * ci.DK + c, rb, first, end, pos, yq[i]);
        conv_block<T, TAPS, E>(x, ldx, w, (const T*)nullptr, ring, ci.taps, ci.C, (ci.HK + it) * ci.DK + c, rb, first, end, pos, yk[i]);
      } else {
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
          for (int e = 0; e < E; ++e) yq[i][t][e] = yk[i][t][e] = 0.f;
      }
#pragma unroll
      for (int t = 0; t < 4; ++t)
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const float qv = yq[i][t][e], kv = yk[i][t][e];
          dot[QQ[t]] = fmaf(qv, qv, dot[QQ[t]]);
          dot[8 * t + 3] = fmaf(kv, kv, dot[8 * t + 3]);
#pragma unroll
          for (int j = 0; j <= t; ++j) {
            if (j < t) dot[8 * t + j] = fmaf(yk[i][j][e], kv, dot[8 * t + j]);
            dot[8 * t + 4 + j] = fmaf(yk[i][j][e], qv, dot[8 * t + 4 + j]);
          }
        }
    }
    halve<32>(dot, lane, 16);
    halve<16>(dot, lane, 8);
    halve<8>(dot, lane, 4);
    halve<4>(dot, lane, 2);
    halve<2>(dot, lane, 1);                            // lane i holds sum i
    const float r = 1.0f / sqrtf(dot[0] + 1e-6f), qs = 1.0f / sqrtf((float)ci.DK);
    float iq[4], ik[4];
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      iq[t] = __shfl_sync(0xffffffffu, r, QQ[t]) * qs;
      ik[t] = __shfl_sync(0xffffffffu, r, 8 * t + 3);
    }
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = i * 32 * E + lane * E;
#pragma unroll
      for (int t = 0; t < 4; ++t) {
#pragma unroll
        for (int e = 0; e < E; ++e) { yq[i][t][e] *= iq[t]; yk[i][t][e] *= ik[t]; }
        if (t < nt && c < ci.DK) {
          const int64_t o = ((int64_t)(rb + t) * ci.HK + it) * ci.DK + c;
          store_e<float, E>(q + o, yq[i][t]);
          store_e<float, E>(k + o, yk[i][t]);
        }
      }
    }
    const int pt = lane >> 3, pj = lane & 3;
    float si = 0.f, sj = 0.f;
#pragma unroll
    for (int t = 0; t < 4; ++t) {
      if (t == pt) si = (lane & 4) ? iq[t] : ik[t];
      if (t == pj) sj = ik[t];
    }
    if (pt < nt) pairs[((int64_t)(rb + pt) * ci.HK + it) * 8 + (lane & 7)] = dot[0] * si * sj;
    return;
  }
  const int h = it - ci.HK;
  const int c0 = 2 * ci.HK * ci.DK + h * ci.DV;
  for (int c = lane * E; c < ci.DV; c += 32 * E) {
    float y[4][E];
    conv_block<T, TAPS, E>(x, ldx, w, (const T*)nullptr, ring, ci.taps, ci.C, c0 + c, rb, first, end, pos, y);
#pragma unroll
    for (int t = 0; t < 4; ++t)
      if (t < nt) store_e<float, E>(v + ((int64_t)(rb + t) * ci.H + h) * ci.DV + c, y[t]);
  }
  if (lane < nt) {
    const int64_t t = rb + lane;
    beta[t * ci.H + h] = sigmoid_x(to_f<T>(b_in[t * ldx + h]));
    g[t * ci.H + h] = expf(-expf(a_log[h]) * softplus_x(to_f<T>(a_in[t * ldx + h]) + dt_bias[h]));
  }
}

// The ring entries of the last `taps` tokens of every portion (after all reads of the older entries).
template <typename T>
__global__ void conv_history_kernel(const T* __restrict__ x, int64_t ldx, T* __restrict__ ring_all, const int* __restrict__ q_start,
                                    const int* __restrict__ kv_len, const int* __restrict__ slots, int taps, int C) {
  pdl_sync();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, seq = blockIdx.y;
  if (c >= C) return;
  const int first = q_start[seq], end = q_start[seq + 1];
  T* ring = ring_all + (int64_t)slots[seq] * taps * C;
  for (int d = 0; d < taps && end - 1 - d >= first; ++d) ring[(int64_t)((kv_len[seq] - 1 - d) % taps) * C + c] = x[(int64_t)(end - 1 - d) * ldx + c];
}

// y[t, h, :] = rms(o[t, h, :]) * gain * silu(gate[t, h, :]) * scale, one warp per (token, head); E values per access
template <typename T, int E>
__global__ void gated_head_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, int64_t ldg, const T* __restrict__ gain,
                                       T* __restrict__ y, int64_t ldy, int n_tok, int H, int DV, float eps, float scale) {
  pdl_sync();
  const int64_t gw = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (gw >= (int64_t)n_tok * H) return;
  const int t = (int)(gw / H), h = (int)(gw % H), lane = threadIdx.x & 31;
  const float* src = o + gw * DV;
  const T* gr = gate + (int64_t)t * ldg + (int64_t)h * DV;
  T* yr = y + (int64_t)t * ldy + (int64_t)h * DV;
  if (E == 4 && DV == 128) {                 // one access per lane, all of them requested before the reduction
    float f[E], gt[E], gn[E];
    load_e<float, E>(src + lane * E, f);
    load_e<T, E>(gr + lane * E, gt);
    load_e<T, E>(gain + lane * E, gn);
    float s2 = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) s2 = fmaf(f[e], f[e], s2);
    const float r = 1.0f / sqrtf(warp_sum(s2) / DV + eps) * scale;
#pragma unroll
    for (int e = 0; e < E; ++e) f[e] *= r * gn[e] * silu_t<T>(gt[e]);
    store_e<T, E>(yr + lane * E, f);
    return;
  }
  float ss = 0.f;
  for (int c = lane * E; c < DV; c += 32 * E) {
    float f[E];
    load_e<float, E>(src + c, f);
#pragma unroll
    for (int e = 0; e < E; ++e) ss = fmaf(f[e], f[e], ss);
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / DV + eps) * scale;
  for (int c = lane * E; c < DV; c += 32 * E) {
    float f[E], gt[E], gn[E];
    load_e<float, E>(src + c, f);
    load_e<T, E>(gr + c, gt);
    load_e<T, E>(gain + c, gn);
#pragma unroll
    for (int e = 0; e < E; ++e) f[e] *= inv * gn[e] * silu_t<T>(gt[e]);
    store_e<T, E>(yr + c, f);
  }
}

// ----------------------------------------------------------------------------------------------- fused one-token steps
template <typename T>
__device__ __forceinline__ void finish_head(const float* so, float* red, const T* gate, const T* gain, T* y, int DV, float eps, float scale) {
  float ss = 0.f;
  for (int c = threadIdx.x; c < DV; c += NT) ss += so[c] * so[c];
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / DV + eps) * scale;
  for (int c = threadIdx.x; c < DV; c += NT) y[c] = from_f<T>(so[c] * inv * to_f<T>(gain[c]) * silu_t<T>(to_f<T>(gate[c])));
}

struct StepIo {
  const int* q_start; const int* positions; const int* slots;
  float* state;
  int H, HK, DK, DV, DKS;
  float eps, out_scale;
};

template <typename T, int NR4>
__global__ void __launch_bounds__(NT) decay_step_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                                                        const T* __restrict__ gate, const T* __restrict__ low, int64_t ld, int rank,
                                                        const T* __restrict__ a2, const T* __restrict__ a2_bias, float inv_tau,
                                                        const T* __restrict__ gain, T* __restrict__ y, int64_t ldy, float q_scale, StepIo io) {
  pdl_sync();
  constexpr int DKP = NR4 * 32;
  extern __shared__ __align__(16) float sm[];
  float *sq = sm, *sk = sq + DKP, *sa = sk + DKP, *sv = sa + DKP, *so = sv + io.DV;
  __shared__ float red[32];
  const int seq = blockIdx.x, h = blockIdx.y, t = io.q_start[seq];
  const bool fresh = io.positions[t] == 0;
  float* state = io.state + ((int64_t)io.slots[seq] * io.H + h) * io.DV * io.DKS;
  float4 st[NR4];
  load_cols<NR4>(st, state, threadIdx.x >> 3, io.DV, io.DKS, fresh, threadIdx.x & 7);
  const int64_t row = (int64_t)t * ld;
  for (int c = threadIdx.x; c < DKP; c += NT) {
    float a = 1.f, qv = 0.f, kv = 0.f;
    if (c < io.DK) {
      const int ch = h * io.DK + c;
      float z = to_f<T>(a2_bias[ch]);
      for (int r = 0; r < rank; ++r) z = fmaf(to_f<T>(a2[(int64_t)ch * rank + r]), to_f<T>(low[row + r]), z);
      a = exp_t<T>(log_sigmoid_t<T>(z) * inv_tau);
      qv = to_f<T>(q[row + ch]) * q_scale;
      kv = to_f<T>(k[row + ch]);
    }
    sa[c] = a; sq[c] = qv; sk[c] = kv;
  }
  for (int c = threadIdx.x; c < io.DV; c += NT) sv[c] = to_f<T>(v[row + (int64_t)h * io.DV + c]);
  __syncthreads();
  step_columns<NR4, DECAY_CHANNEL>(st, state, io.DV, io.DKS, fresh, sq, sk, sa, 0.f, 0.f, sv, so);
  __syncthreads();
  finish_head<T>(so, red, gate + row + (int64_t)h * io.DV, gain, y + (int64_t)t * ldy + (int64_t)h * io.DV, io.DV, io.eps, io.out_scale);
}

// Linear attention with a constant decay per head.  The norm spans the heads of a token: the CTA that finishes the token's last head norms the row
// and gates it, y = rms(o) * gain * sigmoid(gate).
template <typename T, int NR4>
__global__ void __launch_bounds__(NT) lightning_step_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v,
                                                            const T* __restrict__ gate, int64_t ld, const float* __restrict__ decay,
                                                            const T* __restrict__ gain, T* __restrict__ y, int64_t ldy, float* __restrict__ rows,
                                                            int* __restrict__ arrived, StepIo io) {
  pdl_sync();
  constexpr int DKP = NR4 * 32;
  extern __shared__ __align__(16) float sm[];
  float *sq = sm, *sk = sq + DKP, *sv = sk + DKP, *so = sv + io.DV;
  __shared__ float red[32];
  __shared__ int last;
  const int seq = blockIdx.x, h = blockIdx.y, t = io.q_start[seq], inner = io.H * io.DV;
  const bool fresh = io.positions[t] == 0;
  float* state = io.state + ((int64_t)io.slots[seq] * io.H + h) * io.DV * io.DKS;
  float4 st[NR4];
  load_cols<NR4>(st, state, threadIdx.x >> 3, io.DV, io.DKS, fresh, threadIdx.x & 7);
  const int64_t row = (int64_t)t * ld;
  for (int c = threadIdx.x; c < DKP; c += NT) {
    sq[c] = c < io.DK ? to_f<T>(q[row + h * io.DK + c]) : 0.f;
    sk[c] = c < io.DK ? to_f<T>(k[row + h * io.DK + c]) : 0.f;
  }
  for (int c = threadIdx.x; c < io.DV; c += NT) sv[c] = to_f<T>(v[row + h * io.DV + c]);
  __syncthreads();
  step_columns<NR4, DECAY_HEAD>(st, state, io.DV, io.DKS, fresh, sq, sk, nullptr, decay[h], 1.f, sv, so);
  __syncthreads();
  float* yr = rows + (int64_t)seq * inner;
  for (int c = threadIdx.x; c < io.DV; c += NT) yr[h * io.DV + c] = so[c];
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    last = atomicAdd(arrived + seq, 1) == io.H - 1;
    if (last) arrived[seq] = 0;
  }
  __syncthreads();
  if (!last) return;
  __threadfence();
  T* o = y + (int64_t)t * ldy;
  const T* gr = gate + row;
  auto put = [&](int i, float x, float inv) { o[i] = from_f<T>(x * inv * to_f<T>(gain[i]) * sigmoid_t<T>(to_f<T>(gr[i]))); };
  constexpr int KEEP = 16;                             // values a thread keeps between the two passes, all requested before the first is used
  float held[KEEP], ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = threadIdx.x + j * NT;
    held[j] = i < inner ? __ldcg(yr + i) : 0.f;
  }
#pragma unroll
  for (int j = 0; j < KEEP; ++j) ss = fmaf(held[j], held[j], ss);
  for (int i = threadIdx.x + KEEP * NT; i < inner; i += NT) { const float x = __ldcg(yr + i); ss = fmaf(x, x, ss); }
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / inner + io.eps);
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if ((int)threadIdx.x + j * NT < inner) put(threadIdx.x + j * NT, held[j], inv);
  for (int i = threadIdx.x + KEEP * NT; i < inner; i += NT) put(i, __ldcg(yr + i), inv);
}

template <typename T, int NR4>
__global__ void __launch_bounds__(NT) delta_step_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, T* __restrict__ ring_all,
                                                        int taps, const T* __restrict__ b_in, const T* __restrict__ a_in,
                                                        const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                                        const T* __restrict__ gate, const T* __restrict__ gain, T* __restrict__ y, int64_t ldy,
                                                        StepIo io) {
  pdl_sync();
  constexpr int DKP = NR4 * 32;
  extern __shared__ __align__(16) float sm[];
  float *sq = sm, *sk = sq + DKP, *sv = sk + DKP, *so = sv + io.DV;
  __shared__ float red[32];
  const int seq = blockIdx.x, h = blockIdx.y, rep = io.H / io.HK, hk = h / rep, t = io.q_start[seq];
  const int pos = io.positions[t];
  const bool fresh = pos == 0;
  float* state = io.state + ((int64_t)io.slots[seq] * io.H + h) * io.DV * io.DKS;
  float4 st[NR4];
  load_cols<NR4>(st, state, threadIdx.x >> 3, io.DV, io.DKS, fresh, threadIdx.x & 7);
  const int C = 2 * io.HK * io.DK + io.H * io.DV;
  T* ring = ring_all + (int64_t)io.slots[seq] * taps * C;
  const int64_t row = (int64_t)t * ldx;
  float sq2 = 0.f, sk2 = 0.f;
  for (int i = threadIdx.x; i < 2 * DKP + io.DV; i += NT) {
    const int part = i < DKP ? 0 : (i < 2 * DKP ? 1 : 2);
    const int c = i - (part == 0 ? 0 : (part == 1 ? DKP : 2 * DKP));
    float f = 0.f;
    if (part == 2 || c < io.DK) {
      const int ch = part == 2 ? 2 * io.HK * io.DK + h * io.DV + c : (part * io.HK + hk) * io.DK + c;
      f = conv_silu<T>(x, ldx, w, (const T*)nullptr, ring, taps, C, ch, t, t, pos);
      if (part == 2 || h % rep == 0) ring[(int64_t)(pos % taps) * C + ch] = x[row + ch];   // one head of the group records the shared channels
    }
    if (part == 0) { sq[c] = f; sq2 += f * f; }
    else if (part == 1) { sk[c] = f; sk2 += f * f; }
    else sv[c] = f;
  }
  const float qi = 1.0f / sqrtf(block_sum_x(sq2, red) + 1e-6f) * (1.0f / sqrtf((float)io.DK));
  const float ki = 1.0f / sqrtf(block_sum_x(sk2, red) + 1e-6f);
  for (int i = threadIdx.x; i < DKP; i += NT) { sq[i] *= qi; sk[i] *= ki; }
  const float b = sigmoid_x(to_f<T>(b_in[row + h]));
  const float g = expf(-expf(a_log[h]) * softplus_x(to_f<T>(a_in[row + h]) + dt_bias[h]));
  __syncthreads();
  step_columns<NR4, DECAY_DELTA>(st, state, io.DV, io.DKS, fresh, sq, sk, nullptr, g, b, sv, so);
  __syncthreads();
  finish_head<T>(so, red, gate + row + (int64_t)h * io.DV, gain, y + (int64_t)t * ldy + (int64_t)h * io.DV, io.DV, io.eps, io.out_scale);
}

}  // namespace

#define BY_TYPE(f32, ...)                                      \
  do {                                                         \
    if (f32) { using T = float; __VA_ARGS__; }                 \
    else { using T = __nv_bfloat16; __VA_ARGS__; }             \
  } while (0)
#define BY_WIDTH(DK, ...)                                           \
  do {                                                              \
    if (DK <= 32) { constexpr int NR4 = 1; __VA_ARGS__; }           \
    else if (DK <= 64) { constexpr int NR4 = 2; __VA_ARGS__; }      \
    else if (DK <= 128) { constexpr int NR4 = 4; __VA_ARGS__; }     \
    else { constexpr int NR4 = 8; __VA_ARGS__; }                    \
  } while (0)

MARY_API int mary_channel_decay(const void* x, int64_t ldx, int rank, const void* a2, const void* bias, float* decay, int n_tok, int C,
                                float inv_tau, int f32, cudaStream_t s) {
  if (n_tok <= 0) return MARY_OK;
  if (rank < 1 || C < 1 || (n_tok + 15) / 16 > 65535) return MARY_ERR_BAD_ARG;
  const dim3 grid((C + NT - 1) / NT, (n_tok + 15) / 16);
  BY_TYPE(f32, MARY_LAUNCH((channel_decay_kernel<T>), grid, NT, 0, s, (const T*)x, ldx, rank, (const T*)a2, (const T*)bias, decay, n_tok, C, inv_tau));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// x: projection rows whose first 2 HK DK + H DV columns are the q, k, v inputs; b_in / a_in: columns of the same rows.  S sequences of at
// most max_q rows each.  pairs [T, HK, 8] as mary_delta_scan takes it.
MARY_API int mary_delta_prep(const void* x, int64_t ldx, const void* taps_w, const void* ring, const void* b_in, const void* a_in,
                             const float* a_log, const float* dt_bias, const int* q_start, const int* kv_len, const int* slots, float* q, float* k,
                             float* v, float* g, float* beta, float* pairs, int S, int max_q, int HK, int H, int DK, int DV, int taps, int f32,
                             cudaStream_t s) {
  if (S <= 0 || max_q <= 0) return MARY_OK;
  if (HK < 1 || H < 1 || H % HK || DK < 1 || DK > 256 || DV < 1 || taps < 1 || S > 65535 || ((uintptr_t)pairs & 15)) return MARY_ERR_BAD_ARG;
  const ConvIn ci = {HK, H, DK, DV, taps, 2 * HK * DK + H * DV};
  const int64_t warps = (int64_t)((max_q + 3) / 4) * (HK + H);
  const dim3 grid((unsigned)((warps + 7) / 8), S);
  BY_TYPE(f32, {
    const uintptr_t mask = 4 * sizeof(T) - 1;
    const bool vec = DK % 4 == 0 && DV % 4 == 0 && ldx % 4 == 0 && !(((uintptr_t)x | (uintptr_t)ring | (uintptr_t)taps_w) & mask);
    auto fn = taps == 4 ? (vec ? delta_prep_kernel<T, 4, true> : delta_prep_kernel<T, 4, false>)
                        : (vec ? delta_prep_kernel<T, 0, true> : delta_prep_kernel<T, 0, false>);
    MARY_LAUNCH(fn, grid, 256, 0, s, (const T*)x, ldx, (const T*)taps_w, (const T*)ring, (const T*)b_in, (const T*)a_in, a_log, dt_bias, q_start, kv_len,
                slots, q, k, v, g, beta, pairs, ci);
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_conv_history(const void* x, int64_t ldx, void* ring, const int* q_start, const int* kv_len, const int* slots, int S, int taps,
                               int C, int f32, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (taps < 1 || C < 1 || S > 65535) return MARY_ERR_BAD_ARG;
  BY_TYPE(f32, MARY_LAUNCH((conv_history_kernel<T>), dim3((C + NT - 1) / NT, S), NT, 0, s, (const T*)x, ldx, (T*)ring, q_start, kv_len, slots, taps, C));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_gated_head_norm(const float* o, const void* gate, int64_t ldg, const void* gain, void* y, int64_t ldy, int n_tok, int H, int DV,
                                  float eps, float scale, int f32, cudaStream_t s) {
  if (n_tok <= 0) return MARY_OK;
  const int64_t warps = (int64_t)n_tok * H;
  BY_TYPE(f32, {
    const uintptr_t mask = 4 * sizeof(T) - 1;
    const bool vec = DV % 4 == 0 && ldg % 4 == 0 && ldy % 4 == 0 && !(((uintptr_t)gate | (uintptr_t)gain | (uintptr_t)y) & mask) && !((uintptr_t)o & 15);
    auto fn = vec ? gated_head_norm_kernel<T, 4> : gated_head_norm_kernel<T, 1>;
    MARY_LAUNCH(fn, (unsigned)((warps + 7) / 8), 256, 0, s, o, (const T*)gate, ldg, (const T*)gain, (T*)y, ldy, n_tok, H, DV, eps, scale);
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// One token of each of S sequences: decay, recurrence, head norm and output gate of a decayed-linear-attention layer.  q / k / v / gate /
// low are columns of projection rows with pitch ld.
MARY_API int mary_decay_step(const void* q, const void* k, const void* v, const void* gate, const void* low, int64_t ld, int rank, const void* a2,
                             const void* a2_bias, float inv_tau, const void* gain, void* y, int64_t ldy, float q_scale, float* state,
                             const int* q_start, const int* positions, const int* slots, int S, int H, int DK, int DV, float eps,
                             float out_scale, int f32, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (H < 1 || H > 65535 || DK < 1 || DK > 256 || DV < 1 || DV > 4096 || rank < 1) return MARY_ERR_BAD_ARG;
  const StepIo io = {q_start, positions, slots, state, H, H, DK, DV, (DK + 3) / 4 * 4, eps, out_scale};
  BY_TYPE(f32, BY_WIDTH(DK, MARY_LAUNCH((decay_step_kernel<T, NR4>), dim3(S, H), NT, (3 * NR4 * 32 + 2 * DV) * 4, s, (const T*)q, (const T*)k, (const T*)v,
                                        (const T*)gate, (const T*)low, ld, rank, (const T*)a2, (const T*)a2_bias, inv_tau, (const T*)gain, (T*)y, ldy,
                                        q_scale, io)));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// One token of each of S sequences of a gated-delta-rule layer: convolutions, unit norms, gates, recurrence, head norm and output gate.
MARY_API int mary_delta_step(const void* x, int64_t ldx, const void* taps_w, void* ring, int taps, const void* b_in, const void* a_in,
                             const float* a_log, const float* dt_bias, const void* gate, const void* gain, void* y, int64_t ldy, float* state,
                             const int* q_start, const int* positions, const int* slots, int S, int HK, int H, int DK, int DV, float eps,
                             float out_scale, int f32, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (HK < 1 || H < 1 || H % HK || H > 65535 || DK < 1 || DK > 256 || DV < 1 || DV > 4096 || taps < 1) return MARY_ERR_BAD_ARG;
  const StepIo io = {q_start, positions, slots, state, H, HK, DK, DV, (DK + 3) / 4 * 4, eps, out_scale};
  BY_TYPE(f32, BY_WIDTH(DK, MARY_LAUNCH((delta_step_kernel<T, NR4>), dim3(S, H), NT, (2 * NR4 * 32 + 2 * DV) * 4, s, (const T*)x, ldx, (const T*)taps_w, (T*)ring,
                                        taps, (const T*)b_in, (const T*)a_in, a_log, dt_bias, (const T*)gate, (const T*)gain, (T*)y, ldy, io)));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// One token of each of S sequences of linear attention with a constant decay per head (decay [H]): recurrence, norm of the whole row, gate.  q, k, v,
// gate: columns of projection rows with pitch ld; rows: scratch [S, H DV]; arrived: S counters, zero before and after.
MARY_API int mary_lightning_step(const void* q, const void* k, const void* v, const void* gate, int64_t ld, const float* decay, const void* gain, void* y,
                                 int64_t ldy, float* state, float* rows, int* arrived, const int* q_start, const int* positions, const int* slots, int S,
                                 int H, int DK, int DV, float eps, int f32, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (H < 1 || H > 65535 || DK < 1 || DK > 256 || DV < 1 || DV > 4096 || !rows || !arrived) return MARY_ERR_BAD_ARG;
  const StepIo io = {q_start, positions, slots, state, H, H, DK, DV, (DK + 3) / 4 * 4, eps, 1.f};
  BY_TYPE(f32, BY_WIDTH(DK, MARY_LAUNCH((lightning_step_kernel<T, NR4>), dim3(S, H), NT, (2 * NR4 * 32 + 2 * DV) * 4, s, (const T*)q, (const T*)k,
                                        (const T*)v, (const T*)gate, ld, decay, (const T*)gain, (T*)y, ldy, rows, arrived, io)));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
