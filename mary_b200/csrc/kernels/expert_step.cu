// Routed experts around the grouped products: rows gathered into a routing plan's order (any storage type), and for batches of few
// entries the experts as matrix-vector products driven by the (token, slot) entries, without a plan: gate and up rows with the GLU in one
// launch, the weighted sum of the down projections of a token's experts in another.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int NT = 256, WARPS = NT / 32;

// One CTA per token: its row to the padded row of each of its k entries (row_of < 0: not routed here).
template <typename V>                          // V: the unit of the copy
__global__ void __launch_bounds__(NT) gather_rows_kernel(const V* __restrict__ x, int64_t ldx, const int* __restrict__ row_of, int k, V* __restrict__ out,
                                                         int n) {
  pdl_sync();
  const int64_t t = blockIdx.x;
  for (int i = threadIdx.x; i < n; i += NT) {
    const V v = x[t * ldx + i];
    for (int j = 0; j < k; ++j) {
      const int r = row_of[t * k + j];
      if (r >= 0) out[(int64_t)r * n + i] = v;
    }
  }
}

// Dot products of four weight rows (null: skipped) with four vectors in shared memory, lanes striding over K in 16-byte chunks; two
// chunks per row are requested before the first is used.
__device__ __forceinline__ void dot4(const __nv_bfloat16* const (&w)[4], const float* const (&x)[4], int K, float (&out)[4]) {
  const int lane = threadIdx.x & 31;
  constexpr int U = 2;
  float acc[4] = {};
  for (int c0 = lane * 8; c0 < K; c0 += 256 * U) {
    uint4 v[U][4];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int r = 0; r < 4; ++r)
        if (w[r] && c0 + u * 256 < K) v[u][r] = __ldg((const uint4*)(w[r] + c0 + u * 256));
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int c = c0 + u * 256;
      if (c < K) {
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          if (!w[r]) continue;
          float f[8];
          unpack16(v[u][r], f);
          const float4 a = *(const float4*)(x[r] + c), b = *(const float4*)(x[r] + c + 4);
          acc[r] = fmaf(f[0], a.x, fmaf(f[1], a.y, fmaf(f[2], a.z, fmaf(f[3], a.w, acc[r]))));
          acc[r] = fmaf(f[4], b.x, fmaf(f[5], b.y, fmaf(f[6], b.z, fmaf(f[7], b.w, acc[r]))));
        }
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 4; ++r) out[r] = warp_sum(acc[r]);
}

// h[entry] = act(gate x_t) * (up x_t) of the entry's expert; w [E][2 F][K].  blockIdx.y: entry; a warp owns two outputs.
__global__ void __launch_bounds__(NT) expert_glu_kernel(const __nv_bfloat16* __restrict__ x, int64_t ldx, const int* __restrict__ idx, int k, int E,
                                                        const __nv_bfloat16* __restrict__ w, int64_t bsw, __nv_bfloat16* __restrict__ h, int F, int K,
                                                        int act, float limit) {
  pdl_sync();
  extern __shared__ float xs[];
  const int64_t en = blockIdx.y;
  const int e = idx[en];
  if (e < 0 || e >= E) return;
  const __nv_bfloat16* xr = x + en / k * ldx;
  for (int c = threadIdx.x * 8; c < K; c += NT * 8) {
    float f[8];
    unpack16(*(const uint4*)(xr + c), f);
#pragma unroll
    for (int j = 0; j < 8; ++j) xs[c + j] = f[j];
  }
  __syncthreads();
  const int f0 = (blockIdx.x * WARPS + (threadIdx.x >> 5)) * 2;
  if (f0 >= F) return;
  const bool two = f0 + 1 < F;
  const __nv_bfloat16* g = w + e * bsw + (int64_t)f0 * K;
  const __nv_bfloat16* u = g + (int64_t)F * K;
  const __nv_bfloat16* const rows[4] = {g, u, two ? g + K : nullptr, two ? u + K : nullptr};
  const float* const in[4] = {xs, xs, xs, xs};
  float d[4];
  dot4(rows, in, K, d);
  if ((threadIdx.x & 31) == 0) {
    h[en * F + f0] = __float2bfloat16(glu_f(act, d[0], d[1], limit));
    if (two) h[en * F + f0 + 1] = __float2bfloat16(glu_f(act, d[2], d[3], limit));
  }
}

// out[t][n] = sum_j weight_j * (row n of the down matrix of entry j's expert) . h[entry j]; w [E][N][F].  blockIdx.y: token; a warp owns one n.
__global__ void __launch_bounds__(NT) expert_down_kernel(const __nv_bfloat16* __restrict__ h, const int* __restrict__ idx, const float* __restrict__ weight,
                                                         int k, int E, const __nv_bfloat16* __restrict__ w, int64_t bsw, float* __restrict__ out, int N,
                                                         int F) {
  pdl_sync();
  extern __shared__ float hs[];                  // [entries that are experts][F]
  __shared__ int ex[32], n_ex;
  __shared__ float wt[32];
  const int64_t t = blockIdx.y;
  if (threadIdx.x < 32) {
    const int e = threadIdx.x < k ? idx[t * k + threadIdx.x] : -1;
    const bool in = e >= 0 && e < E;
    const unsigned mask = __ballot_sync(0xffffffffu, in);
    const int at = __popc(mask & ((1u << threadIdx.x) - 1));
    if (in) { ex[at] = e | (threadIdx.x << 16); wt[at] = weight[t * k + threadIdx.x]; }
    if (threadIdx.x == 0) n_ex = __popc(mask);
  }
  __syncthreads();
  const int n = n_ex;
  for (int i = threadIdx.x * 8; i < n * F; i += NT * 8) {
    float f[8];
    unpack16(*(const uint4*)(h + (t * k + (ex[i / F] >> 16)) * F + i % F), f);
#pragma unroll
    for (int j = 0; j < 8; ++j) hs[i + j] = f[j];
  }
  __syncthreads();
  const int col = blockIdx.x * WARPS + (threadIdx.x >> 5);
  if (col >= N) return;
  float acc = 0.f;
  for (int j0 = 0; j0 < n; j0 += 4) {
    const __nv_bfloat16* rows[4];
    const float* in[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const int j = min(j0 + r, n - 1);
      rows[r] = j0 + r < n ? w + (ex[j] & 0xffff) * bsw + (int64_t)col * F : nullptr;
      in[r] = hs + j * F;
    }
    float d[4];
    dot4(rows, in, F, d);
#pragma unroll
    for (int r = 0; r < 4; ++r)
      if (j0 + r < n) acc = fmaf(wt[j0 + r], d[r], acc);
  }
  if ((threadIdx.x & 31) == 0) out[t * N + col] = acc;
}

}  // namespace

// out[row_of[t * k + j]] = x[t], rows of n bytes (a multiple of 4) at x + t * ld bytes.
MARY_API int mary_gather_rows(const void* x, int64_t ld, const int* row_of, int T_, int k, void* out, int n, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (n < 1 || k < 1 || n % 2 || ld % 2) return MARY_ERR_BAD_ARG;
  if (n % 16 == 0 && ld % 16 == 0 && !(((uintptr_t)x | (uintptr_t)out) & 15))
    MARY_LAUNCH((gather_rows_kernel<uint4>), T_, NT, 0, s, (const uint4*)x, ld / 16, row_of, k, (uint4*)out, n / 16);
  else
    MARY_LAUNCH((gather_rows_kernel<uint16_t>), T_, NT, 0, s, (const uint16_t*)x, ld / 2, row_of, k, (uint16_t*)out, n / 2);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// bf16; K % 8 == 0, 16-byte aligned rows.  h [T * k][F]; entries with idx outside [0, E) are left alone.
MARY_API int mary_expert_glu(const void* x, int64_t ldx, const int* idx, int T_, int k, int E, const void* w, int64_t bsw, void* h, int F, int K, int act,
                             float limit, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if ((int64_t)T_ * k > 65535 || F < 1 || K % 8 || ldx % 8 || bsw % 8 || K > 16384) return MARY_ERR_BAD_ARG;
  static MarySmemSlots smem_set = {};
  const size_t sm = (size_t)K * 4;
  if (int rc = sm > 48 * 1024 ? mary_ensure_dyn_smem((const void*)expert_glu_kernel, sm, &smem_set) : 0) return rc;
  MARY_LAUNCH(expert_glu_kernel, dim3((F + 2 * WARPS - 1) / (2 * WARPS), T_ * k), NT, sm, s, (const __nv_bfloat16*)x, ldx, idx, k, E,
              (const __nv_bfloat16*)w, bsw, (__nv_bfloat16*)h, F, K, act, limit);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// bf16 h [T * k][F] and w [E][N][F] -> f32 out [T][N]; F % 8 == 0, k * F <= 49152, E <= 65536.
MARY_API int mary_expert_down(const void* h, const int* idx, const float* weight, int T_, int k, int E, const void* w, int64_t bsw, float* out, int N, int F,
                              cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (T_ > 65535 || N < 1 || F % 8 || bsw % 8 || k < 1 || k > 32 || E > 65536 || (int64_t)k * F > 49152) return MARY_ERR_BAD_ARG;
  static MarySmemSlots smem_set = {};
  const size_t sm = (size_t)k * F * 4;
  if (int rc = sm > 46 * 1024 ? mary_ensure_dyn_smem((const void*)expert_down_kernel, sm, &smem_set) : 0) return rc;
  MARY_LAUNCH(expert_down_kernel, dim3((N + WARPS - 1) / WARPS, T_), NT, sm, s, (const __nv_bfloat16*)h, idx, weight, k, E, (const __nv_bfloat16*)w, bsw, out,
              N, F);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
