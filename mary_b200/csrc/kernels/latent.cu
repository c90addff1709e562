// Row kernels of latent attention with any widths, for bf16 and for 32-bit activations: norms of the query latent and of the key/value
// latent with rotation and cache append, rotation of the queries' rotated parts.  A pair of a rotation is (2i, 2i + 1); cosine and sine
// carry a common factor.  Norms, angles and rotations in exact 32-bit arithmetic.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int NT = 256;

__device__ __forceinline__ void turn(float& u, float& v, int pos, float freq, float gain) {
  float s, c;
  sincosf((float)pos * freq, &s, &c);
  s *= gain; c *= gain;
  const float a = u * c - v * s, b = v * c + u * s;
  u = a; v = b;
}

// y_q [q_rank] -> rms * q_gain -> c;  y_kv [rank + rot] -> [rms(first rank) * kv_gain | rotated last rot] -> cache row.  One CTA per token.
template <typename T>
__global__ void __launch_bounds__(NT) latent_prep_kernel(const T* __restrict__ y_q, const T* __restrict__ y_kv, int64_t ld, int q_rank, int rank, int rot,
                                                         const T* __restrict__ q_gain, const T* __restrict__ kv_gain, const float* __restrict__ freq,
                                                         float rot_gain, const int* __restrict__ positions, const int64_t* __restrict__ slots,
                                                         T* __restrict__ c, T* __restrict__ cache, float eps, int64_t n_slots,
                                                         int* __restrict__ status) {
  pdl_sync();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const bool is_q = blockIdx.y == 0;
  const T* src = (is_q ? y_q : y_kv) + t * ld;
  const T* gain = is_q ? q_gain : kv_gain;
  const int n = is_q ? q_rank : rank;
  T* dst = c + t * q_rank;
  if (!is_q) {
    const int64_t slot = slots[t];
    if (slot < 0 || slot >= n_slots) {           // a cache slot outside the cache: record it, skip the write
      if (threadIdx.x == 0) atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);
      return;
    }
    dst = cache + slot * (rank + rot);
    for (int i = threadIdx.x; i < rot / 2; i += NT) {
      float u = to_f<T>(src[rank + 2 * i]), v = to_f<T>(src[rank + 2 * i + 1]);
      turn(u, v, positions[t], freq[i], rot_gain);
      dst[rank + 2 * i] = from_f<T>(u);
      dst[rank + 2 * i + 1] = from_f<T>(v);
    }
  }
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += NT) { const float f = to_f<T>(src[i]); ss = fmaf(f, f, ss); }
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / n + eps);
  for (int i = threadIdx.x; i < n; i += NT) dst[i] = from_f<T>(to_f<T>(src[i]) * inv * to_f<T>(gain[i]));
}

// The last rot values of every head of src [T, H, src_w] rotated into dst [T, H, dst_w] from dst_off on (src itself allowed).
template <typename T>
__global__ void __launch_bounds__(NT) rotate_heads_kernel(const T* src, T* dst, const float* __restrict__ freq, float rot_gain,
                                                          const int* __restrict__ positions, int64_t n, int H, int src_w, int dst_w, int dst_off,
                                                          int rot) {
  pdl_sync();
  const int64_t i = (int64_t)blockIdx.x * NT + threadIdx.x;
  if (i >= n) return;
  const int half = rot / 2, p = (int)(i % half);
  const int64_t th = i / half;
  const T* s = src + th * src_w + (src_w - rot) + 2 * p;
  float u = to_f<T>(s[0]), v = to_f<T>(s[1]);
  turn(u, v, positions[th / H], freq[p], rot_gain);
  T* d = dst + th * dst_w + dst_off + 2 * p;
  d[0] = from_f<T>(u);
  d[1] = from_f<T>(v);
}

// Keys of an expanded prompt: the rotated part of cache row n behind the own dims of every head, k [n_rows, H, dim + rot].
template <typename T>
__global__ void __launch_bounds__(NT) fill_shared_part_kernel(const T* __restrict__ rows, int64_t ld, int rank, T* __restrict__ k, int64_t n, int H, int dim,
                                                              int rot) {
  pdl_sync();
  const int64_t i = (int64_t)blockIdx.x * NT + threadIdx.x;
  if (i >= n) return;
  const int d = (int)(i % rot);
  const int64_t nh = i / rot;
  k[nh * (dim + rot) + dim + d] = rows[(nh / H) * ld + rank + d];
}

}  // namespace

#define BY_TYPE(f32, ...)                                      \
  do {                                                         \
    if (f32) { using T = float; __VA_ARGS__; }                 \
    else { using T = __nv_bfloat16; __VA_ARGS__; }             \
  } while (0)

// y_q, y_kv: columns of projection rows with pitch ld; cache [n_slots, rank + rot].
MARY_API int mary_latent_prep(const void* y_q, const void* y_kv, int64_t ld, int q_rank, int rank, int rot, const void* q_gain, const void* kv_gain,
                              const float* freq, float rot_gain, const int* positions, const int64_t* slots, void* c, void* cache, float eps,
                              int n_tok, int64_t n_slots, int f32, cudaStream_t s) {
  if (n_tok <= 0) return MARY_OK;
  if (q_rank < 1 || rank < 1 || rot < 0 || rot % 2) return MARY_ERR_BAD_ARG;
  BY_TYPE(f32, MARY_LAUNCH((latent_prep_kernel<T>), dim3(n_tok, 2), NT, 0, s, (const T*)y_q, (const T*)y_kv, ld, q_rank, rank, rot, (const T*)q_gain,
                           (const T*)kv_gain, freq, rot_gain, positions, slots, (T*)c, (T*)cache, eps, n_slots, mary_status_ptr()));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_rotate_heads(const void* src, void* dst, const float* freq, float rot_gain, const int* positions, int n_tok, int H, int src_w,
                               int dst_w, int dst_off, int rot, int f32, cudaStream_t s) {
  if (n_tok <= 0 || rot == 0) return MARY_OK;
  if (H < 1 || rot < 0 || rot % 2 || rot > src_w || dst_off + rot > dst_w) return MARY_ERR_BAD_ARG;
  const int64_t n = (int64_t)n_tok * H * (rot / 2);
  BY_TYPE(f32, MARY_LAUNCH((rotate_heads_kernel<T>), (unsigned)((n + NT - 1) / NT), NT, 0, s, (const T*)src, (T*)dst, freq, rot_gain, positions, n, H, src_w,
                           dst_w, dst_off, rot));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_fill_shared_part(const void* rows, int64_t ld, int rank, void* k, int64_t n_rows, int H, int dim, int rot, int f32, cudaStream_t s) {
  if (n_rows <= 0 || rot == 0) return MARY_OK;
  if (H < 1 || rot < 0 || dim < 1) return MARY_ERR_BAD_ARG;
  const int64_t n = n_rows * H * rot;
  if ((n + NT - 1) / NT > 0x7fffffff) return MARY_ERR_BAD_ARG;
  BY_TYPE(f32, MARY_LAUNCH((fill_shared_part_kernel<T>), (unsigned)((n + NT - 1) / NT), NT, 0, s, (const T*)rows, ld, rank, (T*)k, n, H, dim, rot));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
