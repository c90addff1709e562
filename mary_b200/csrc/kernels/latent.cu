// Row kernels of latent attention with any widths, for bf16 and for 32-bit activations: norms of the query latent and of the key/value
// latent with rotation and cache append, rotation of the queries' rotated parts.  A pair of a rotation is (2i, 2i + 1); cosine and sine
// carry a common factor.  Norms, angles and rotations in exact 32-bit arithmetic.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int NT = 256, PREP = 128;

__device__ __forceinline__ void turn(float& u, float& v, int pos, float freq, float gain) {
  float s, c;
  sincosf((float)pos * freq, &s, &c);
  s *= gain; c *= gain;
  const float a = u * c - v * s, b = v * c + u * s;
  u = a; v = b;
}

// y_q [q_rank] -> rms * q_gain -> c;  y_kv [rank + rot] -> [rms(first rank) * kv_gain | rotated last rot] -> cache row.  One CTA per token
// and part; E values per access.
template <typename T, int E>
__global__ void __launch_bounds__(PREP) latent_prep_kernel(const T* __restrict__ y_q, const T* __restrict__ y_kv, int64_t ld, int q_rank, int rank, int rot,
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
    for (int i = threadIdx.x; i < rot / 2; i += PREP) {
      float u = to_f<T>(src[rank + 2 * i]), v = to_f<T>(src[rank + 2 * i + 1]);
      turn(u, v, positions[t], freq[i], rot_gain);
      dst[rank + 2 * i] = from_f<T>(u);
      dst[rank + 2 * i + 1] = from_f<T>(v);
    }
  }
  float ss = 0.f, f[E], g[E];
  for (int i = threadIdx.x * E; i < n; i += PREP * E) {
    load_e<T, E>(src + i, f);
#pragma unroll
    for (int j = 0; j < E; ++j) ss = fmaf(f[j], f[j], ss);
  }
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / n + eps);
  for (int i = threadIdx.x * E; i < n; i += PREP * E) {
    load_e<T, E>(src + i, f);
    load_e<T, E>(gain + i, g);
#pragma unroll
    for (int j = 0; j < E; ++j) f[j] *= inv * g[j];
    store_e<T, E>(dst + i, f);
  }
}

// The last rot values of every head of src [T, H, src_w] rotated into dst [T, H, dst_w] from dst_off on (src itself allowed).  A thread
// takes one pair of every `groups`-th head of a token: one sine and cosine for all of them.
template <typename T>
__global__ void __launch_bounds__(NT) rotate_heads_kernel(const T* src, T* dst, const float* __restrict__ freq, float rot_gain,
                                                          const int* __restrict__ positions, int64_t n, int H, int groups, int src_w, int dst_w,
                                                          int dst_off, int rot) {
  pdl_sync();
  const int64_t i = (int64_t)blockIdx.x * NT + threadIdx.x;
  if (i >= n) return;
  const int half = rot / 2, p = (int)(i % half), g = (int)(i / half % groups);
  const int64_t t = i / half / groups;
  float sn, cs;
  sincosf((float)positions[t] * freq[p], &sn, &cs);
  sn *= rot_gain; cs *= rot_gain;
  for (int h = g; h < H; h += groups) {
    const T* s = src + (t * H + h) * src_w + (src_w - rot) + 2 * p;
    T* d = dst + (t * H + h) * dst_w + dst_off + 2 * p;
    const float u = to_f<T>(s[0]), v = to_f<T>(s[1]);
    d[0] = from_f<T>(u * cs - v * sn);
    d[1] = from_f<T>(v * cs + u * sn);
  }
}

// Keys of an expanded prompt: the rotated part of cache row n behind the own dims of every head, k [n_rows, H, dim + rot]; V: what a thread
// copies.
template <typename V>
__global__ void __launch_bounds__(NT) fill_shared_part_kernel(const V* __restrict__ rows, int64_t ld, int rank, V* __restrict__ k, int64_t n, int H, int dim,
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
  BY_TYPE(f32, {
    const uintptr_t mask = 4 * sizeof(T) - 1;
    const bool vec = q_rank % 4 == 0 && rank % 4 == 0 && rot % 4 == 0 && ld % 4 == 0 &&
                     !(((uintptr_t)y_q | (uintptr_t)y_kv | (uintptr_t)q_gain | (uintptr_t)kv_gain | (uintptr_t)c | (uintptr_t)cache) & mask);
    auto fn = vec ? latent_prep_kernel<T, 4> : latent_prep_kernel<T, 1>;
    MARY_LAUNCH(fn, dim3(n_tok, 2), PREP, 0, s, (const T*)y_q, (const T*)y_kv, ld, q_rank, rank, rot, (const T*)q_gain, (const T*)kv_gain, freq, rot_gain,
                positions, slots, (T*)c, (T*)cache, eps, n_slots, mary_status_ptr());
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_rotate_heads(const void* src, void* dst, const float* freq, float rot_gain, const int* positions, int n_tok, int H, int src_w,
                               int dst_w, int dst_off, int rot, int f32, cudaStream_t s) {
  if (n_tok <= 0 || rot == 0) return MARY_OK;
  if (H < 1 || rot < 0 || rot % 2 || rot > src_w || dst_off + rot > dst_w) return MARY_ERR_BAD_ARG;
  const int groups = n_tok >= 512 && H >= 8 ? H / 8 : H;      // long batches: eight heads share one sine and cosine
  const int64_t n = (int64_t)n_tok * groups * (rot / 2);
  BY_TYPE(f32, MARY_LAUNCH((rotate_heads_kernel<T>), (unsigned)((n + NT - 1) / NT), NT, 0, s, (const T*)src, (T*)dst, freq, rot_gain, positions, n, H, groups,
                           src_w, dst_w, dst_off, rot));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_fill_shared_part(const void* rows, int64_t ld, int rank, void* k, int64_t n_rows, int H, int dim, int rot, int f32, cudaStream_t s) {
  if (n_rows <= 0 || rot == 0) return MARY_OK;
  if (H < 1 || rot < 0 || dim < 1) return MARY_ERR_BAD_ARG;
  // elements per 16 bytes; whole vectors where every boundary allows them
  const int E = f32 ? 4 : 8;
  const bool vec = ld % E == 0 && rank % E == 0 && dim % E == 0 && rot % E == 0 && !(((uintptr_t)rows | (uintptr_t)k) & 15);
  const int64_t n = n_rows * H * (vec ? rot / E : rot);
  if ((n + NT - 1) / NT > 0x7fffffff) return MARY_ERR_BAD_ARG;
  const unsigned grid = (unsigned)((n + NT - 1) / NT);
  if (vec) MARY_LAUNCH((fill_shared_part_kernel<uint4>), grid, NT, 0, s, (const uint4*)rows, ld / E, rank / E, (uint4*)k, n, H, dim / E, rot / E);
  else BY_TYPE(f32, MARY_LAUNCH((fill_shared_part_kernel<T>), grid, NT, 0, s, (const T*)rows, ld, rank, (T*)k, n, H, dim, rot));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
