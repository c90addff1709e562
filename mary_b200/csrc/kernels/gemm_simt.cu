// General matrix product on the CUDA cores with 32-bit accumulation: out[M, N] = alpha * X[M, K] W[N, K]^T (+ out).  It serves 32-bit
// models (no reduced-precision tensor-core mode is involved) and the shapes that TMA addressing excludes (row pitches that are not
// multiples of 16 bytes); everything else belongs to gemm_bf16.cu.  64 x 64 tile, 256 threads, 4 x 4 outputs each, register prefetch.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int BM = 64, BN = 64, BK = 16, NT = 256;

template <typename TI, typename TO>
__device__ __forceinline__ void simt_tile(const TI* __restrict__ X, const TI* __restrict__ W, TO* __restrict__ out, int M, int N, int K, int64_t ldx,
                                          int64_t ldw, int64_t ldo, float alpha, int accumulate, int m0, int n0) {
  __shared__ float sx[2][BK][BM + 4], sw[2][BK][BN + 4];
  const int tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  const int lk = threadIdx.x % BK, lr = threadIdx.x / BK;          // loader: one k, rows lr, lr + 16, ...
  float acc[4][4] = {};
  float px[4], pw[4];
  auto fetch = [&](int k0) {
    const int k = k0 + lk;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int m = m0 + lr + 16 * i, n = n0 + lr + 16 * i;
      px[i] = (k < K && m < M) ? to_f<TI>(X[(int64_t)m * ldx + k]) : 0.f;
      pw[i] = (k < K && n < N) ? to_f<TI>(W[(int64_t)n * ldw + k]) : 0.f;
    }
  };
  auto stash = [&](int b) {
#pragma unroll
    for (int i = 0; i < 4; ++i) { sx[b][lk][lr + 16 * i] = px[i]; sw[b][lk][lr + 16 * i] = pw[i]; }
  };
  fetch(0);
  stash(0);
  __syncthreads();
  const int nk = (K + BK - 1) / BK;
  for (int kb = 0; kb < nk; ++kb) {
    const int b = kb & 1;
    if (kb + 1 < nk) fetch((kb + 1) * BK);
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      const float4 a = *(const float4*)&sx[b][k][ty * 4], c = *(const float4*)&sw[b][k][tx * 4];
      const float av[4] = {a.x, a.y, a.z, a.w}, cv[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], cv[j], acc[i][j]);
    }
    if (kb + 1 < nk) stash(b ^ 1);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      TO* o = out + (int64_t)m * ldo + n;
      const float v = alpha * acc[i][j];
      *o = from_f<TO>(accumulate ? to_f<TO>(*o) + v : v);
    }
  }
}

template <typename TI, typename TO>
__global__ void __launch_bounds__(NT) gemm_simt_kernel(const TI* __restrict__ X, const TI* __restrict__ W, TO* __restrict__ out, int M, int N, int K,
                                                       int64_t ldx, int64_t ldw, int64_t ldo, float alpha, int accumulate, int64_t bsx, int64_t bsw,
                                                       int64_t bso) {
  pdl_sync();
  simt_tile<TI, TO>(X + blockIdx.z * bsx, W + blockIdx.z * bsw, out + blockIdx.z * bso, M, N, K, ldx, ldw, ldo, alpha, accumulate, blockIdx.y * BM,
                    blockIdx.x * BN);
}

// Rows sorted into tiles of one expert each (tiles: {expert, first row, rows, -}, meta[0] of them in use): every tile times its expert's matrix.
template <typename TI>
__global__ void __launch_bounds__(NT) gemm_simt_grouped_kernel(const TI* __restrict__ X, const TI* __restrict__ W, TI* __restrict__ out, int N, int K,
                                                               int64_t ldx, int64_t ldw, int64_t ldo, int E, int64_t bsw, const int* __restrict__ tiles,
                                                               const int* __restrict__ meta) {
  pdl_sync();
  if ((int)blockIdx.y >= meta[0]) return;
  const int* t = tiles + 4 * blockIdx.y;
  const int e = min(max(t[0], 0), E - 1);
  simt_tile<TI, TI>(X + (int64_t)t[1] * ldx, W + e * bsw, out + (int64_t)t[1] * ldo, min(t[2], BM), N, K, ldx, ldw, ldo, 1.0f, 0, 0, blockIdx.x * BN);
}

}  // namespace

// `batch` products over strided views (element strides bsx / bsw / bso).  x_f32: X and W are f32 (else both bf16); out_f32: out is f32 (else bf16)
MARY_API int mary_gemm_simt_batched(const void* X, const void* W, void* out, int M, int N, int K, int64_t ldx, int64_t ldw, int64_t ldo, int batch,
                                    int64_t bsx, int64_t bsw, int64_t bso, float alpha, int accumulate, int x_f32, int out_f32, cudaStream_t s) {
  if (M <= 0) return MARY_OK;
  if (N <= 0 || K <= 0 || (M + BM - 1) / BM > 65535 || batch < 1 || batch > 65535) return MARY_ERR_BAD_ARG;
  const dim3 grid((N + BN - 1) / BN, (M + BM - 1) / BM, batch);
  using B = __nv_bfloat16;
  if (x_f32 && out_f32)
    MARY_LAUNCH((gemm_simt_kernel<float, float>), grid, NT, 0, s, (const float*)X, (const float*)W, (float*)out, M, N, K, ldx, ldw, ldo, alpha, accumulate, bsx, bsw, bso);
  else if (x_f32) return MARY_ERR_BAD_ARG;
  else if (out_f32)
    MARY_LAUNCH((gemm_simt_kernel<B, float>), grid, NT, 0, s, (const B*)X, (const B*)W, (float*)out, M, N, K, ldx, ldw, ldo, alpha, accumulate, bsx, bsw, bso);
  else
    MARY_LAUNCH((gemm_simt_kernel<B, B>), grid, NT, 0, s, (const B*)X, (const B*)W, (B*)out, M, N, K, ldx, ldw, ldo, alpha, accumulate, bsx, bsw, bso);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_gemm_simt(const void* X, const void* W, void* out, int M, int N, int K, int64_t ldx, int64_t ldw, int64_t ldo, float alpha,
                            int accumulate, int x_f32, int out_f32, cudaStream_t s) {
  return mary_gemm_simt_batched(X, W, out, M, N, K, ldx, ldw, ldo, 1, 0, 0, 0, alpha, accumulate, x_f32, out_f32, s);
}

// out[r] = X[r] W[expert of r's tile]^T over the rows of a routing plan with tiles of at most 64 rows (`max_tiles` of them); X, W [E][N][K] (bsw elements
// between experts) and out have one storage type.
MARY_API int mary_gemm_simt_grouped(const void* X, const void* W, void* out, int N, int K, int64_t ldx, int64_t ldw, int64_t ldo, int E, int64_t bsw,
                                    const int* tiles, const int* meta, int max_tiles, int f32, cudaStream_t s) {
  if (max_tiles <= 0) return MARY_OK;
  if (N <= 0 || K <= 0 || E < 1 || max_tiles > 65535) return MARY_ERR_BAD_ARG;
  const dim3 grid((N + BN - 1) / BN, max_tiles);
  using B = __nv_bfloat16;
  if (f32) MARY_LAUNCH((gemm_simt_grouped_kernel<float>), grid, NT, 0, s, (const float*)X, (const float*)W, (float*)out, N, K, ldx, ldw, ldo, E, bsw, tiles, meta);
  else MARY_LAUNCH((gemm_simt_grouped_kernel<B>), grid, NT, 0, s, (const B*)X, (const B*)W, (B*)out, N, K, ldx, ldw, ldo, E, bsw, tiles, meta);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
