// Everything around the recurrence of a Mamba-2 layer, for bf16 and for 32-bit activations: the short convolutions with bias, step sizes
// and decays, the products the scan takes (recurrent_scan.cu), the gate and the norm in equal parts of the read-out, and the fused
// one-token step that does all of it in one launch per layer.  Step sizes, decays, the state and the norm are in exact 32-bit arithmetic.
//
// Convolution channels: [x: H P | B: G N | C: G N]; head h uses the B and C of group h / (H / G).
#include "host_utils.h"
#include "recurrent.cuh"

using namespace mary;

namespace {

constexpr int NT = STEP_THREADS;

struct SsIo {
  int G, H, N, P, taps, C;             // C = H P + 2 G N channels
};

__device__ __forceinline__ float step_size(float raw, float bias) { return softplus_x(raw + bias); }
// Decays close to 1 are multiplied over thousands of tokens, so theirs is the exponential with the smaller error there.
__device__ __forceinline__ float step_decay(float a_log, float dt) {
  const float x = -expf(a_log) * dt;
  return x > -0.5f ? 1.0f + expm1f(x) : expf(x);
}

// One warp per (sequence, block of four tokens, item); items: G groups (B, C and the products B_j . C_i of the block), chunks of x
// channels, chunks of 32 heads (step sizes and decays).  VEC: widths, pitch and addresses allow accesses of four values.
template <typename T, int TAPS, bool VEC>
__global__ void __launch_bounds__(256) ss_prep_kernel(const T* __restrict__ xbc, int64_t ldx, const T* __restrict__ w, const T* __restrict__ bias,
                                                      const T* __restrict__ ring_all, const T* __restrict__ dt_in, const float* __restrict__ dt_bias,
                                                      const float* __restrict__ a_log, const int* __restrict__ q_start,
                                                      const int* __restrict__ kv_len, const int* __restrict__ slots, float* __restrict__ x,
                                                      float* __restrict__ b, float* __restrict__ c, float* __restrict__ dt, float* __restrict__ decay,
                                                      float* __restrict__ pairs, SsIo io) {
  pdl_sync();
  constexpr int E = VEC ? 4 : 1, NI = 8 / E;          // N <= 256: eight channels per lane
  const int inner = io.H * io.P;
  const int xi = (inner + 32 * E - 1) / (32 * E), items = io.G + xi + (io.H + 31) / 32;
  const int gw = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int blk = gw / items, it = gw % items, lane = threadIdx.x & 31, seq = blockIdx.y;
  const int first = q_start[seq], end = q_start[seq + 1], rb = first + blk * 4;
  if (rb >= end) return;
  const int nt = min(4, end - rb);
  const int pos = kv_len[seq] - (end - first) + blk * 4;
  const T* ring = ring_all + (int64_t)slots[seq] * io.taps * io.C;
  if (it < io.G) {
    float dot[16];                                    // B_j . C_i at 4 i + j, j <= i
#pragma unroll
    for (int i = 0; i < 16; ++i) dot[i] = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int ch = i * 32 * E + lane * E;
      if (ch >= io.N) break;
      float yb[4][E], yc[4][E];
      conv_block<T, TAPS, E>(xbc, ldx, w, bias, ring, io.taps, io.C, inner + it * io.N + ch, rb, first, end, pos, yb);
      conv_block<T, TAPS, E>(xbc, ldx, w, bias, ring, io.taps, io.C, inner + (io.G + it) * io.N + ch, rb, first, end, pos, yc);
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        if (t < nt) {
          const int64_t o = ((int64_t)(rb + t) * io.G + it) * io.N + ch;
          store_e<float, E>(b + o, yb[t]);
          store_e<float, E>(c + o, yc[t]);
        }
#pragma unroll
        for (int j = 0; j <= t; ++j)
#pragma unroll
          for (int e = 0; e < E; ++e) dot[4 * t + j] = fmaf(yb[j][e], yc[t][e], dot[4 * t + j]);
      }
    }
    __syncwarp();
    halve<16>(dot, lane, 16);
    halve<8>(dot, lane, 8);
    halve<4>(dot, lane, 4);
    halve<2>(dot, lane, 2);
    dot[0] += __shfl_xor_sync(0xffffffffu, dot[0], 1);       // lanes 2 i and 2 i + 1 hold product i
    const int i = lane >> 3, j = (lane >> 1) & 3;
    if (!(lane & 1) && i < nt) pairs[((int64_t)(rb + i) * io.G + it) * 4 + j] = dot[0];
    return;
  }
  if (it < io.G + xi) {
    const int ch = ((it - io.G) * 32 + lane) * E;
    if (ch >= inner) return;
    float y[4][E];
    conv_block<T, TAPS, E>(xbc, ldx, w, bias, ring, io.taps, io.C, ch, rb, first, end, pos, y);
#pragma unroll
    for (int t = 0; t < 4; ++t)
      if (t < nt) store_e<float, E>(x + (int64_t)(rb + t) * inner + ch, y[t]);
    return;
  }
  const int h = (it - io.G - xi) * 32 + lane;
  if (h >= io.H) return;
  for (int t = 0; t < nt; ++t) {
    const float d = step_size(to_f<T>(dt_in[(int64_t)(rb + t) * ldx + h]), dt_bias[h]);
    dt[(int64_t)(rb + t) * io.H + h] = d;
    decay[(int64_t)(rb + t) * io.H + h] = step_decay(a_log[h], d);
  }
}

// out[t, part] = rms(y[t, part] * silu(z[t, part])) * gain, one CTA per (token, part) of n values; E values per access.  NORM_FIRST: rms(y[t, part])
// * gain * sigmoid(z[t, part]) instead
template <typename T, int E, bool NORM_FIRST>
__global__ void gated_part_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, int64_t ldz, const T* __restrict__ gain, T* __restrict__ out,
                                       int64_t ldo, int inner, int n, float eps) {
  pdl_sync();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int c0 = blockIdx.y * n;
  const float* yr = y + t * inner + c0;
  const T* zr = z + t * ldz + c0;
  T* o = out + t * ldo + c0;
  constexpr int KEEP = E == 1 ? 8 : 2;                // accesses a thread keeps between the two passes
  const int step = blockDim.x * E;
  float v[KEEP][E], ss = 0.f;
  auto value = [&](int i, float (&u)[E]) {
    float zv[E];
    load_e<float, E>(yr + i, u);
    if constexpr (!NORM_FIRST) load_e<T, E>(zr + i, zv);
#pragma unroll
    for (int e = 0; e < E; ++e) {
      if constexpr (!NORM_FIRST) u[e] *= silu_t<T>(zv[e]);
      ss = fmaf(u[e], u[e], ss);
    }
  };
  auto put = [&](int i, float (&u)[E], float inv) {
    float g[E];
    load_e<T, E>(gain + c0 + i, g);
#pragma unroll
    for (int e = 0; e < E; ++e) u[e] *= inv * g[e];
    if constexpr (NORM_FIRST) {
      load_e<T, E>(zr + i, g);
#pragma unroll
      for (int e = 0; e < E; ++e) u[e] *= sigmoid_t<T>(g[e]);
    }
    store_e<T, E>(o + i, u);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (threadIdx.x * E + j * step < n) value(threadIdx.x * E + j * step, v[j]);
  for (int i = threadIdx.x * E + KEEP * step; i < n; i += step) {
    float u[E];
    value(i, u);
  }
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / n + eps);
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (threadIdx.x * E + j * step < n) put(threadIdx.x * E + j * step, v[j], inv);
  for (int i = threadIdx.x * E + KEEP * step; i < n; i += step) {
    float u[E];
    value(i, u);
    put(i, u, inv);
  }
}

struct SsStep {
  const int* q_start; const int* positions; const int* slots;
  float* state; float* row; int* arrived;             // row [S][H P]: gated read-outs; arrived [S * parts]: zero between launches
  int parts;
  float eps;
};

// One CTA per (sequence, head).  The norm spans the heads of a part: the CTA that finishes a part last norms it.
template <typename T, int NR4>
__global__ void __launch_bounds__(NT) ss_step_kernel(const T* __restrict__ xbc, int64_t ldx, const T* __restrict__ w, const T* __restrict__ bias,
                                                     T* __restrict__ ring_all, const T* __restrict__ dt_in, const float* __restrict__ dt_bias,
                                                     const float* __restrict__ a_log, const float* __restrict__ skip, const T* __restrict__ z,
                                                     const T* __restrict__ gain, T* __restrict__ out, int64_t ldo, SsIo io, SsStep st_io) {
  pdl_sync();
  constexpr int NP = NR4 * 32;
  extern __shared__ __align__(16) float sm[];
  float *sc = sm, *sb = sc + NP, *sx = sb + NP, *so = sx + io.P;
  __shared__ float red[32];
  __shared__ int last;
  const int seq = blockIdx.x, h = blockIdx.y, rep = io.H / io.G, g = h / rep, t = st_io.q_start[seq];
  const int pos = st_io.positions[t], inner = io.H * io.P, NS = (io.N + 3) / 4 * 4;
  const bool fresh = pos == 0;
  float* state = st_io.state + ((int64_t)st_io.slots[seq] * io.H + h) * io.P * NS;
  float4 st[NR4];
  load_cols<NR4>(st, state, threadIdx.x >> 3, io.P, NS, fresh, threadIdx.x & 7);
  T* ring = ring_all + (int64_t)st_io.slots[seq] * io.taps * io.C;
  const int64_t row = (int64_t)t * ldx;
  for (int i = threadIdx.x; i < 2 * NP + io.P; i += NT) {
    const int part = i < NP ? 0 : (i < 2 * NP ? 1 : 2);
    const int c = i - (part == 0 ? 0 : (part == 1 ? NP : 2 * NP));
    float f = 0.f;
    if (part == 2 || c < io.N) {
      const int ch = part == 2 ? h * io.P + c : inner + ((part == 0 ? io.G : 0) + g) * io.N + c;
      f = conv_silu<T>(xbc, ldx, w, bias, ring, io.taps, io.C, ch, t, t, pos);
      if (part == 2 || h % rep == 0) ring[(int64_t)(pos % io.taps) * io.C + ch] = xbc[row + ch];   // one head of the group records the shared channels
    }
    if (part == 0) sc[c] = f;
    else if (part == 1) sb[c] = f;
    else sx[c] = f;
  }
  const float dt = step_size(to_f<T>(dt_in[row + h]), dt_bias[h]), decay = step_decay(a_log[h], dt);
  __syncthreads();
  step_columns<NR4, DECAY_HEAD>(st, state, io.P, NS, fresh, sc, sb, nullptr, decay, dt, sx, so);
  __syncthreads();
  float* yr = st_io.row + (int64_t)seq * inner;
  for (int c = threadIdx.x; c < io.P; c += NT)
    yr[h * io.P + c] = fmaf(skip[h], sx[c], so[c]) * silu_t<T>(to_f<T>(z[row + h * io.P + c]));
  __threadfence();
  __syncthreads();
  const int n = inner / st_io.parts;
  const bool aligned = n % io.P == 0;                 // a part is a whole number of heads: parts finish on their own
  const int per = aligned ? n / io.P : io.H, p_lo = aligned ? h / per : 0, p_hi = aligned ? p_lo + 1 : st_io.parts;
  if (threadIdx.x == 0) {
    int* cnt = st_io.arrived + (int64_t)seq * st_io.parts + p_lo;
    last = atomicAdd(cnt, 1) == per - 1;
    if (last) *cnt = 0;
  }
  __syncthreads();
  if (!last) return;
  __threadfence();
  T* o = out + (int64_t)t * ldo;
  for (int p = p_lo; p < p_hi; ++p) {
    float ss = 0.f;
    for (int i = p * n + threadIdx.x; i < (p + 1) * n; i += NT) { const float v = __ldcg(yr + i); ss = fmaf(v, v, ss); }
    const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / n + st_io.eps);
    for (int i = p * n + threadIdx.x; i < (p + 1) * n; i += NT) o[i] = from_f<T>(__ldcg(yr + i) * inv * to_f<T>(gain[i]));
  }
}

bool bad_shape(const SsIo& io) { return io.G < 1 || io.H < 1 || io.H % io.G || io.H > 65535 || io.N < 1 || io.N > 256 || io.P < 1 || io.P > 4096 || io.taps < 1; }

}  // namespace

#define BY_TYPE(f32, ...)                                      \
  do {                                                         \
    if (f32) { using T = float; __VA_ARGS__; }                 \
    else { using T = __nv_bfloat16; __VA_ARGS__; }             \
  } while (0)
#define BY_WIDTH(N, ...)                                           \
  do {                                                              \
    if (N <= 32) { constexpr int NR4 = 1; __VA_ARGS__; }            \
    else if (N <= 64) { constexpr int NR4 = 2; __VA_ARGS__; }       \
    else if (N <= 128) { constexpr int NR4 = 4; __VA_ARGS__; }      \
    else { constexpr int NR4 = 8; __VA_ARGS__; }                    \
  } while (0)

// xbc, dt_in: columns of projection rows with pitch ldx.  S sequences of at most max_q rows each.  f32 results: x [T, H P], b, c [T, G N],
// dt, decay [T, H], pairs [T, G, 4] as mary_head_decay_scan takes them.
MARY_API int mary_ss_prep(const void* xbc, int64_t ldx, const void* taps_w, const void* taps_b, const void* ring, const void* dt_in,
                          const float* dt_bias, const float* a_log, const int* q_start, const int* kv_len, const int* slots, float* x, float* b,
                          float* c, float* dt, float* decay, float* pairs, int S, int max_q, int G, int H, int N, int P, int taps, int f32,
                          cudaStream_t s) {
  if (S <= 0 || max_q <= 0) return MARY_OK;
  const SsIo io = {G, H, N, P, taps, H * P + 2 * G * N};
  if (bad_shape(io) || S > 65535) return MARY_ERR_BAD_ARG;
  BY_TYPE(f32, {
    const uintptr_t mask = 4 * sizeof(T) - 1;
    const bool vec = N % 4 == 0 && (H * P) % 4 == 0 && ldx % 4 == 0 && !(((uintptr_t)xbc | (uintptr_t)ring | (uintptr_t)taps_w) & mask);
    const int E = vec ? 4 : 1;
    const int64_t items = G + (H * P + 32 * E - 1) / (32 * E) + (H + 31) / 32, warps = (int64_t)((max_q + 3) / 4) * items;
    auto fn = taps == 4 ? (vec ? ss_prep_kernel<T, 4, true> : ss_prep_kernel<T, 4, false>)
                        : (vec ? ss_prep_kernel<T, 0, true> : ss_prep_kernel<T, 0, false>);
    MARY_LAUNCH(fn, dim3((unsigned)((warps + 7) / 8), S), 256, 0, s, (const T*)xbc, ldx, (const T*)taps_w, (const T*)taps_b, (const T*)ring, (const T*)dt_in,
                dt_bias, a_log, q_start, kv_len, slots, x, b, c, dt, decay, pairs, io);
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// norm_first = 0: rms(y * silu(z)) * gain, 1: rms(y) * gain * sigmoid(z), in `parts` equal parts of a row
MARY_API int mary_gated_part_norm(const float* y, const void* z, int64_t ldz, const void* gain, void* out, int64_t ldo, int n_tok, int inner, int parts,
                                  float eps, int norm_first, int f32, cudaStream_t s) {
  if (n_tok <= 0) return MARY_OK;
  if (parts < 1 || inner % parts || parts > 65535) return MARY_ERR_BAD_ARG;
  const int n = inner / parts;
  int nt = (n + 7) / 8;
  nt = nt <= 32 ? 32 : (nt >= 512 ? 512 : (nt + 31) / 32 * 32);
  BY_TYPE(f32, {
    const uintptr_t mask = 4 * sizeof(T) - 1;
    const bool vec = n % 4 == 0 && ldz % 4 == 0 && ldo % 4 == 0 && !(((uintptr_t)z | (uintptr_t)gain | (uintptr_t)out) & mask) && !((uintptr_t)y & 15);
    auto fn = norm_first ? (vec ? gated_part_norm_kernel<T, 4, true> : gated_part_norm_kernel<T, 1, true>)
                         : (vec ? gated_part_norm_kernel<T, 4, false> : gated_part_norm_kernel<T, 1, false>);
    MARY_LAUNCH(fn, dim3(n_tok, parts), nt, 0, s, y, (const T*)z, ldz, (const T*)gain, (T*)out, ldo, inner, n, eps);
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// One token of each of S sequences of a Mamba-2 layer: convolutions, step size, recurrence, skip, gate and norm.  xbc, dt_in, z: columns of
// projection rows with pitch ldx.  row: scratch [S, H P]; arrived: S * parts counters, zero before and after.
MARY_API int mary_ss_step(const void* xbc, int64_t ldx, const void* taps_w, const void* taps_b, void* ring, const void* dt_in, const float* dt_bias,
                          const float* a_log, const float* skip, const void* z, const void* gain, int parts, void* out, int64_t ldo, float* state,
                          float* row, int* arrived, const int* q_start, const int* positions, const int* slots, int S, int G, int H, int N, int P,
                          int taps, float eps, int f32, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  const SsIo io = {G, H, N, P, taps, H * P + 2 * G * N};
  if (bad_shape(io) || parts < 1 || (H * P) % parts) return MARY_ERR_BAD_ARG;
  const SsStep st = {q_start, positions, slots, state, row, arrived, parts, eps};
  BY_TYPE(f32, BY_WIDTH(N, MARY_LAUNCH((ss_step_kernel<T, NR4>), dim3(S, H), NT, (2 * NR4 * 32 + 2 * P) * 4, s, (const T*)xbc, ldx, (const T*)taps_w,
                                       (const T*)taps_b, (T*)ring, (const T*)dt_in, dt_bias, a_log, skip, (const T*)z, (const T*)gain, (T*)out, ldo, io, st)));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
