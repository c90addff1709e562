// Everything around the linear recurrences of recurrent_scan.cu, for bf16 and for 32-bit activations: the per-channel decay from its
// low-rank projection, the short convolutions with their unit norms and gates, the convolution history, the gated norm of the
// read-out, and the fused one-token steps that do all of it in one launch per layer.  Decays, gates, unit norms and the state are in
// exact 32-bit arithmetic.
//
// Convolution history: the last `taps` inputs of every channel in a ring addressed by absolute position, [slot][taps][channels].  A
// token at position p reads the entries of p - 1 .. p - (taps - 1) and writes the entry of p, which none of those reads touches.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int NT = 256;

// decay[t, c] = sigmoid(a2[c] . x[t] + bias[c]) ^ inv_tau, x[t] of `rank` values
template <typename T>
__global__ void __launch_bounds__(NT) channel_decay_kernel(const T* __restrict__ x, int64_t ldx, int rank, const T* __restrict__ a2,
                                                           const T* __restrict__ bias, float* __restrict__ decay, int n_tok, int C, float inv_tau) {
  pdl_sync();
  constexpr int TT = 16, RC = 16;
  __shared__ float sx[TT][RC], sw[NT][RC + 1];
  const int c = blockIdx.x * NT + threadIdx.x, t0 = blockIdx.y * TT;
  float acc[TT] = {};
  for (int r0 = 0; r0 < rank; r0 += RC) {
    __syncthreads();
    {
      const int t = threadIdx.x / RC, r = threadIdx.x % RC;
      sx[t][r] = (t0 + t < n_tok && r0 + r < rank) ? to_f<T>(x[(int64_t)(t0 + t) * ldx + r0 + r]) : 0.f;
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
      for (int t = 0; t < TT; ++t) acc[t] = fmaf(w, sx[t][r], acc[t]);
    }
  }
  if (c >= C) return;
  const float b = to_f<T>(bias[c]);
#pragma unroll
  for (int t = 0; t < TT; ++t)
    if (t0 + t < n_tok) decay[(int64_t)(t0 + t) * C + c] = expf(log_sigmoid_x(acc[t] + b) * inv_tau);
}

struct ConvIn {
  int HK, H, DK, DV, taps, C;      // C = 2 HK DK + H DV channels, in the order q, k, v; taps [C][taps], last one the current token's
};

// silu of the depthwise causal convolution of channel c at row t (position pos of its sequence, whose portion starts at row first)
template <typename T>
__device__ __forceinline__ float conv_silu(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, const T* __restrict__ ring, int taps, int C,
                                           int c, int t, int first, int pos) {
  float acc = 0.f;
  for (int d = 0; d < taps; ++d) {                     // d tokens back
    float v = 0.f;
    if (t - d >= first) v = to_f<T>(x[(int64_t)(t - d) * ldx + c]);
    else if (pos - d >= 0) v = to_f<T>(ring[(int64_t)((pos - d) % taps) * C + c]);
    acc = fmaf(to_f<T>(w[(int64_t)c * taps + taps - 1 - d]), v, acc);
  }
  return silu_x(acc);
}

// One warp per (token, item); items: HK query heads, HK key heads (both made unit vectors), H value heads (with their gates).
template <typename T>
__global__ void delta_prep_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, const T* __restrict__ ring_all,
                                  const T* __restrict__ b_in, const T* __restrict__ a_in, const float* __restrict__ a_log,
                                  const float* __restrict__ dt_bias, const int* __restrict__ positions, const int* __restrict__ seq_index,
                                  const int* __restrict__ q_start, const int* __restrict__ slots, float* __restrict__ q, float* __restrict__ k,
                                  float* __restrict__ v, float* __restrict__ g, float* __restrict__ beta, int n_tok, ConvIn ci) {
  pdl_sync();
  const int items = 2 * ci.HK + ci.H;
  const int64_t gw = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (gw >= (int64_t)n_tok * items) return;
  const int t = (int)(gw / items), it = (int)(gw % items), lane = threadIdx.x & 31;
  const int seq = seq_index[t], first = q_start[seq], pos = positions[t];
  const T* ring = ring_all + (int64_t)slots[seq] * ci.taps * ci.C;
  if (it < 2 * ci.HK) {
    const bool is_q = it < ci.HK;
    const int c0 = it * ci.DK;                         // q channels first, then k channels
    float y[8], ss = 0.f;                              // DK <= 256
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = lane + 32 * i;
      y[i] = c < ci.DK ? conv_silu<T>(x, ldx, w, ring, ci.taps, ci.C, c0 + c, t, first, pos) : 0.f;
      ss += y[i] * y[i];
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) + 1e-6f) * (is_q ? 1.0f / sqrtf((float)ci.DK) : 1.0f);
    float* dst = (is_q ? q : k) + ((int64_t)t * ci.HK + (is_q ? it : it - ci.HK)) * ci.DK;
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (lane + 32 * i < ci.DK) dst[lane + 32 * i] = y[i] * inv;
    return;
  }
  const int h = it - 2 * ci.HK;
  const int c0 = 2 * ci.HK * ci.DK + h * ci.DV;
  for (int c = lane; c < ci.DV; c += 32)
    v[((int64_t)t * ci.H + h) * ci.DV + c] = conv_silu<T>(x, ldx, w, ring, ci.taps, ci.C, c0 + c, t, first, pos);
  if (lane == 0) {
    beta[(int64_t)t * ci.H + h] = sigmoid_x(to_f<T>(b_in[(int64_t)t * ldx + h]));
    g[(int64_t)t * ci.H + h] = expf(-expf(a_log[h]) * softplus_x(to_f<T>(a_in[(int64_t)t * ldx + h]) + dt_bias[h]));
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

// y[t, h, :] = rms(o[t, h, :]) * gain * silu(gate[t, h, :]) * scale, one warp per (token, head)
template <typename T>
__global__ void gated_head_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, int64_t ldg, const T* __restrict__ gain,
                                       T* __restrict__ y, int64_t ldy, int n_tok, int H, int DV, float eps, float scale) {
  pdl_sync();
  const int64_t gw = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (gw >= (int64_t)n_tok * H) return;
  const int t = (int)(gw / H), h = (int)(gw % H), lane = threadIdx.x & 31;
  const float* src = o + gw * DV;
  float ss = 0.f;
  for (int c = lane; c < DV; c += 32) ss += src[c] * src[c];
  const float inv = 1.0f / sqrtf(warp_sum(ss) / DV + eps) * scale;
  for (int c = lane; c < DV; c += 32)
    y[(int64_t)t * ldy + (int64_t)h * DV + c] = from_f<T>(src[c] * inv * to_f<T>(gain[c]) * silu_x(to_f<T>(gate[(int64_t)t * ldg + (int64_t)h * DV + c])));
}

// ----------------------------------------------------------------------------------------------- fused one-token steps
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

// sq / sk [NR4 * 32] (zero beyond DK), sa [NR4 * 32] channel decays (DELTA: the scalars g and b instead), sv [DV]; leaves o in so[DV].
template <int NR4, bool DELTA>
__device__ __forceinline__ void step_columns(float4 (&st)[NR4], float* state, int DV, int DKS, bool fresh, const float* sq, const float* sk,
                                             const float* sa, float g, float b, const float* sv, float* so) {
  const int lane8 = threadIdx.x & 7;
  for (int col = threadIdx.x >> 3, c0 = 0; c0 < DV; c0 += NT / 8, col += NT / 8) {
    float4 nx[NR4];
    if (c0 + NT / 8 < DV) load_cols<NR4>(nx, state, col + NT / 8, DV, DKS, fresh, lane8);
    const float vt = col < DV ? sv[col] : 0.f;
    float w = vt;
    if constexpr (DELTA) {
      float pred = 0.f;
#pragma unroll
      for (int r = 0; r < NR4; ++r) {
        const float4 k4 = *(const float4*)(sk + (r * 8 + lane8) * 4);
        st[r].x *= g; st[r].y *= g; st[r].z *= g; st[r].w *= g;
        pred = fmaf(k4.x, st[r].x, fmaf(k4.y, st[r].y, fmaf(k4.z, st[r].z, fmaf(k4.w, st[r].w, pred))));
      }
      w = b * (vt - sum8(pred));
    }
    float acc = 0.f;
#pragma unroll
    for (int r = 0; r < NR4; ++r) {
      const int c = (r * 8 + lane8) * 4;
      const float4 k4 = *(const float4*)(sk + c), q4 = *(const float4*)(sq + c);
      if constexpr (!DELTA) {
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

template <typename T>
__device__ __forceinline__ void finish_head(const float* so, float* red, const T* gate, const T* gain, T* y, int DV, float eps, float scale) {
  float ss = 0.f;
  for (int c = threadIdx.x; c < DV; c += NT) ss += so[c] * so[c];
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / DV + eps) * scale;
  for (int c = threadIdx.x; c < DV; c += NT) y[c] = from_f<T>(so[c] * inv * to_f<T>(gain[c]) * silu_x(to_f<T>(gate[c])));
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
      a = expf(log_sigmoid_x(z) * inv_tau);
      qv = to_f<T>(q[row + ch]) * q_scale;
      kv = to_f<T>(k[row + ch]);
    }
    sa[c] = a; sq[c] = qv; sk[c] = kv;
  }
  for (int c = threadIdx.x; c < io.DV; c += NT) sv[c] = to_f<T>(v[row + (int64_t)h * io.DV + c]);
  __syncthreads();
  step_columns<NR4, false>(st, state, io.DV, io.DKS, fresh, sq, sk, sa, 0.f, 0.f, sv, so);
  __syncthreads();
  finish_head<T>(so, red, gate + row + (int64_t)h * io.DV, gain, y + (int64_t)t * ldy + (int64_t)h * io.DV, io.DV, io.eps, io.out_scale);
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
      f = conv_silu<T>(x, ldx, w, ring, taps, C, ch, t, t, pos);
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
  step_columns<NR4, true>(st, state, io.DV, io.DKS, fresh, sq, sk, nullptr, g, b, sv, so);
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

// x: projection rows whose first 2 HK DK + H DV columns are the q, k, v inputs; b_in / a_in: columns of the same rows
MARY_API int mary_delta_prep(const void* x, int64_t ldx, const void* taps_w, const void* ring, const void* b_in, const void* a_in,
                             const float* a_log, const float* dt_bias, const int* positions, const int* seq_index, const int* q_start,
                             const int* slots, float* q, float* k, float* v, float* g, float* beta, int n_tok, int HK, int H, int DK, int DV,
                             int taps, int f32, cudaStream_t s) {
  if (n_tok <= 0) return MARY_OK;
  if (HK < 1 || H < 1 || H % HK || DK < 1 || DK > 256 || DV < 1 || taps < 1) return MARY_ERR_BAD_ARG;
  const ConvIn ci = {HK, H, DK, DV, taps, 2 * HK * DK + H * DV};
  const int64_t warps = (int64_t)n_tok * (2 * HK + H);
  BY_TYPE(f32, MARY_LAUNCH((delta_prep_kernel<T>), (unsigned)((warps + 7) / 8), 256, 0, s, (const T*)x, ldx, (const T*)taps_w, (const T*)ring, (const T*)b_in,
                           (const T*)a_in, a_log, dt_bias, positions, seq_index, q_start, slots, q, k, v, g, beta, n_tok, ci));
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
  BY_TYPE(f32, MARY_LAUNCH((gated_head_norm_kernel<T>), (unsigned)((warps + 7) / 8), 256, 0, s, o, (const T*)gate, ldg, (const T*)gain, (T*)y, ldy, n_tok, H, DV,
                           eps, scale));
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
