// Row kernels of decoders that keep the residual stream in 32-bit floats, for bf16 and for 32-bit activations: embedding into the
// stream, norm of a sublayer's output added to the stream (with the following pre-norm or the stream's copy for the next
// projection), plain RMS norm, gated activation, per-head query / key norm with cache append for heads whose keys and values have
// widths of their own; dynamic tanh around the stream, and query / key norm over whole projection rows.  One CTA per row (or one warp per
// head); any width; norms, sums and activations in exact 32-bit arithmetic.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int NT = 256;

template <typename T>
__global__ void embed32_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ h, T* __restrict__ x, int H,
                               float scale, int vocab, int* __restrict__ status) {
  pdl_sync();
  int id = ids[blockIdx.x];
  if (id < 0 || id >= vocab) {                 // recorded, and redirected to row 0: no read outside the table
    if (threadIdx.x == 0) atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);
    id = 0;
  }
  const T* src = table + (int64_t)id * H;
  const int64_t o = (int64_t)blockIdx.x * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = to_f<T>(src[i]) * scale;
    h[o + i] = v;
    x[o + i] = from_f<T>(v);
  }
}

// h += rms(a) * w_post;  x = w_next ? rms(h) * w_next : h.  `a` is f32, rows of `lda`.  VEC: H % 8 == 0 and 16-byte aligned rows.
template <typename T, bool VEC>
__global__ void __launch_bounds__(NT) post_norm_add_kernel(const float* __restrict__ a, int64_t lda, const T* __restrict__ w_post,
                                                           float* __restrict__ h, const T* __restrict__ w_next, T* __restrict__ x, int H,
                                                           float eps) {
  pdl_sync();
  extern __shared__ float row[];
  __shared__ float red[32];
  const float* ar = a + (int64_t)blockIdx.x * lda;
  float* hr = h + (int64_t)blockIdx.x * H;
  T* xr = x + (int64_t)blockIdx.x * H;
  constexpr int E = VEC ? 8 : 1;
  float ss = 0.f;
  for (int i = threadIdx.x * E; i < H; i += NT * E) {
    float f[E];
    if constexpr (VEC) {
      *(float4*)f = *(const float4*)(ar + i);
      *(float4*)(f + 4) = *(const float4*)(ar + i + 4);
    } else {
      f[0] = ar[i];
    }
#pragma unroll
    for (int j = 0; j < E; ++j) { row[i + j] = f[j]; ss += f[j] * f[j]; }
  }
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / H + eps);
  float ss2 = 0.f;
  for (int i = threadIdx.x * E; i < H; i += NT * E) {
    float r[E], g[E];
    if constexpr (VEC) {
      *(float4*)r = *(const float4*)(hr + i);
      *(float4*)(r + 4) = *(const float4*)(hr + i + 4);
      if constexpr (sizeof(T) == 2) { unpack16(*(const uint4*)(w_post + i), g); }
      else { *(float4*)g = *(const float4*)(w_post + i); *(float4*)(g + 4) = *(const float4*)(w_post + i + 4); }
    } else {
      r[0] = hr[i]; g[0] = to_f<T>(w_post[i]);
    }
#pragma unroll
    for (int j = 0; j < E; ++j) {
      r[j] += row[i + j] * inv * g[j];
      row[i + j] = r[j];
      ss2 += r[j] * r[j];
    }
    if constexpr (VEC) {
      *(float4*)(hr + i) = *(float4*)r;
      *(float4*)(hr + i + 4) = *(float4*)(r + 4);
      if (!w_next) {
        if constexpr (sizeof(T) == 2) *(uint4*)(xr + i) = pack16(r);
        else { *(float4*)(xr + i) = *(float4*)r; *(float4*)(xr + i + 4) = *(float4*)(r + 4); }
      }
    } else {
      hr[i] = r[0];
      if (!w_next) xr[i] = from_f<T>(r[0]);
    }
  }
  if (!w_next) return;
  const float inv2 = 1.0f / sqrtf(block_sum_x(ss2, red) / H + eps);
  for (int i = threadIdx.x; i < H; i += NT) xr[i] = from_f<T>(row[i] * inv2 * to_f<T>(w_next[i]));
}

// y = rms(x) * w for f32 rows
template <typename T>
__global__ void rmsnorm32_kernel(const float* __restrict__ x, const T* __restrict__ w, T* __restrict__ y, int H, float eps) {
  pdl_sync();
  __shared__ float red[32];
  const float* xr = x + (int64_t)blockIdx.x * H;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) ss += xr[i] * xr[i];
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) y[(int64_t)blockIdx.x * H + i] = from_f<T>(xr[i] * inv * (w ? to_f<T>(w[i]) : 1.f));
}

template <typename T>
__global__ void glu_any_kernel(const T* __restrict__ gu, T* __restrict__ out, int F, int64_t n, int act, float limit) {
  pdl_sync();
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int64_t t = i / F, f = i % F;
  const float g = to_f<T>(gu[t * 2 * F + f]), u = to_f<T>(gu[t * 2 * F + F + f]);
  if (act == 3) {
    const float gl = fminf(g, limit), ul = fminf(fmaxf(u, -limit), limit);
    out[i] = from_f<T>(gl * sigmoid_x(1.702f * gl) * (ul + 1.0f));
    return;
  }
  const float k0 = 0.7978845608028654f, k1 = 0.044715f;
  const float a = act == 0 ? 0.5f * g * (1.0f + tanhf(k0 * (g + k1 * g * g * g))) : silu_x(g);
  out[i] = from_f<T>(a * u);
}

// y = act(y) in place on the first n columns of rows with pitch ld.  act: 0 = tanh-form GELU, 1 = SiLU
template <typename T>
__global__ void act_rows_kernel(T* __restrict__ y, int64_t ld, int n, int64_t total, int act) {
  pdl_sync();
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  T* p = y + i / n * ld + i % n;
  const float g = to_f<T>(*p), k0 = 0.7978845608028654f, k1 = 0.044715f;
  *p = from_f<T>(act == 0 ? 0.5f * g * (1.0f + tanhf(k0 * (g + k1 * g * g * g))) : silu_x(g));
}

__global__ void soft_cap_kernel(float* __restrict__ x, int64_t n, float cap) {
  pdl_sync();
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) x[i] = cap * tanhf(x[i] / cap);
}

// One warp per (token, head) of a projection row: RMS norm of query and key heads (gains optional), queries to qo, keys and values
// to their cache slots.  Keys are DK wide, values DV wide; q / k / v are row views of one projection with pitch ld.
template <typename T>
__global__ void qk_norm_append_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int64_t ld, int n_q, int n_kv,
                                      int DK, int DV, const T* __restrict__ q_gain, const T* __restrict__ k_gain,
                                      const int64_t* __restrict__ slots, T* __restrict__ qo, T* __restrict__ kc, T* __restrict__ vc, float eps,
                                      int n_tok, int64_t n_slots, int* __restrict__ status) {
  pdl_sync();
  const int heads = n_q + 2 * n_kv;
  const int64_t gw = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (gw >= (int64_t)n_tok * heads) return;
  const int t = (int)(gw / heads), hh = (int)(gw % heads), lane = threadIdx.x & 31;
  const bool is_q = hh < n_q, is_k = !is_q && hh < n_q + n_kv;
  if (!is_q && (slots[t] < 0 || slots[t] >= n_slots)) {       // a cache slot outside the cache: record it, skip the write
    if (lane == 0) atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);
    return;
  }
  if (!is_q && !is_k) {
    const int g = hh - n_q - n_kv;
    const T* src = v + (int64_t)t * ld + (int64_t)g * DV;
    T* dst = vc + (slots[t] * n_kv + g) * DV;
    for (int i = lane; i < DV; i += 32) dst[i] = src[i];
    return;
  }
  const T* src = is_q ? q + (int64_t)t * ld + (int64_t)hh * DK : k + (int64_t)t * ld + (int64_t)(hh - n_q) * DK;
  const T* gain = is_q ? q_gain : k_gain;
  T* dst = is_q ? qo + ((int64_t)t * n_q + hh) * DK : kc + (slots[t] * n_kv + (hh - n_q)) * DK;
  float inv = 1.f;
  if (gain) {
    float ss = 0.f;
    for (int i = lane; i < DK; i += 32) { const float f = to_f<T>(src[i]); ss += f * f; }
    inv = 1.0f / sqrtf(warp_sum(ss) / DK + eps);
  }
  for (int i = lane; i < DK; i += 32) dst[i] = from_f<T>(to_f<T>(src[i]) * inv * (gain ? to_f<T>(gain[i]) : 1.f));
}

// E values of storage type T, 16-byte aligned when E > 1 (E = 8, or 4 for f32).
template <typename T, int E> __device__ __forceinline__ void load_v(const T* p, float (&f)[E]) {
  if constexpr (E == 8 && sizeof(T) == 2) unpack16(*(const uint4*)p, f);
  else if constexpr (E == 8) {
    *(float4*)f = *(const float4*)p;
    *(float4*)(f + 4) = *(const float4*)(p + 4);
  } else load_e<T, E>(p, f);
}
template <typename T, int E> __device__ __forceinline__ void store_v(T* p, const float (&f)[E]) {
  if constexpr (E == 8 && sizeof(T) == 2) *(uint4*)p = pack16(f);
  else if constexpr (E == 8) {
    *(float4*)p = *(const float4*)f;
    *(float4*)(p + 4) = *(const float4*)(f + 4);
  } else store_e<T, E>(p, f);
}

template <typename T> struct Dyt {               // tanh(alpha x) * w + b
  const T* w; const T* b; const float* alpha;
};

// h[t] = table[ids[t]] * scale;  x = n(h)
template <typename T>
__global__ void embed_dyt_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ h, T* __restrict__ x, int H, float scale,
                                 Dyt<T> n, int vocab, int* __restrict__ status) {
  pdl_sync();
  int id = ids[blockIdx.x];
  if (id < 0 || id >= vocab) {                 // recorded, and redirected to row 0: no read outside the table
    if (threadIdx.x == 0) atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);
    id = 0;
  }
  const T* src = table + (int64_t)id * H;
  const int64_t o = (int64_t)blockIdx.x * H;
  const float alpha = *n.alpha;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = to_f<T>(src[i]) * scale;
    h[o + i] = v;
    x[o + i] = from_f<T>(fmaf(tanhf(alpha * v), to_f<T>(n.w[i]), to_f<T>(n.b[i])));
  }
}

// h += post(a);  x = next(h).  blockIdx.y: row.
template <typename T, int E>
__global__ void __launch_bounds__(NT) dyt_add_kernel(const float* __restrict__ a, int64_t lda, Dyt<T> post, float* __restrict__ h, Dyt<T> next,
                                                     T* __restrict__ x, int H) {
  pdl_sync();
  const int i = (blockIdx.x * NT + threadIdx.x) * E;
  if (i >= H) return;
  const int64_t row = blockIdx.y;
  const float al = *post.alpha, an = *next.alpha;
  float av[E], hv[E], w[E], b[E];
  load_v<float, E>(a + row * lda + i, av);
  load_v<float, E>(h + row * H + i, hv);
  load_v<T, E>(post.w + i, w);
  load_v<T, E>(post.b + i, b);
#pragma unroll
  for (int j = 0; j < E; ++j) hv[j] += fmaf(tanhf(al * av[j]), w[j], b[j]);
  store_v<float, E>(h + row * H + i, hv);
  load_v<T, E>(next.w + i, w);
  load_v<T, E>(next.b + i, b);
#pragma unroll
  for (int j = 0; j < E; ++j) hv[j] = fmaf(tanhf(an * hv[j]), w[j], b[j]);
  store_v<T, E>(x + row * H + i, hv);
}

// One CTA per token: RMS norm of the whole query row (nq values) and of the whole key row (nk), queries to qo, keys and values to their
// cache slot.  k null: queries only.
template <typename T, int E>
__global__ void __launch_bounds__(NT) row_norm_append_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int64_t ld, int nq,
                                                             int nk, int nv, const T* __restrict__ q_gain, const T* __restrict__ k_gain,
                                                             const int64_t* __restrict__ slots, T* __restrict__ qo, T* __restrict__ kc,
                                                             T* __restrict__ vc, float eps, int64_t n_slots, int* __restrict__ status) {
  pdl_sync();
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  auto norm = [&](const T* src, const T* gain, T* dst, int n) {
    float ss = 0.f, f[E], g[E];
    for (int i = threadIdx.x * E; i < n; i += NT * E) {
      load_v<T, E>(src + i, f);
#pragma unroll
      for (int j = 0; j < E; ++j) ss = fmaf(f[j], f[j], ss);
    }
    const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / n + eps);
    for (int i = threadIdx.x * E; i < n; i += NT * E) {
      load_v<T, E>(src + i, f);
      load_v<T, E>(gain + i, g);
#pragma unroll
      for (int j = 0; j < E; ++j) f[j] *= inv * g[j];
      store_v<T, E>(dst + i, f);
    }
  };
  if (blockIdx.y == 0) {
    norm(q + t * ld, q_gain, qo + t * nq, nq);
    return;
  }
  const int64_t slot = slots[t];
  if (slot < 0 || slot >= n_slots) {           // a cache slot outside the cache: record it, skip the write
    if (threadIdx.x == 0) atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);
    return;
  }
  for (int i = threadIdx.x * E; i < nv; i += NT * E) {
    float f[E];
    load_v<T, E>(v + t * ld + i, f);
    store_v<T, E>(vc + slot * nv + i, f);
  }
  norm(k + t * ld, k_gain, kc + slot * nk, nk);
}

}  // namespace

#define BY_TYPE(f32, ...)                                      \
  do {                                                         \
    if (f32) { using T = float; __VA_ARGS__; }                 \
    else { using T = __nv_bfloat16; __VA_ARGS__; }             \
  } while (0)

MARY_API int mary_embed32(const int* ids, const void* table, float* h, void* x, int T_, int H, float scale, int vocab, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  BY_TYPE(f32, MARY_LAUNCH((embed32_kernel<T>), T_, 128, 0, s, ids, (const T*)table, h, (T*)x, H, scale, vocab, mary_status_ptr()));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// h[T, H] (f32) += rms(a[T, H]) * w_post, then x[T, H] = rms(h) * w_next, or a copy of h when w_next is null.
MARY_API int mary_post_norm_add(const float* a, int64_t lda, const void* w_post, float* h, const void* w_next, void* x, int T_, int H, float eps,
                                int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  const size_t sm = (size_t)H * 4;
  if (sm > 200 * 1024) return MARY_ERR_BAD_ARG;
  const bool vec = H % 8 == 0 && lda % 4 == 0 && !(((uintptr_t)a | (uintptr_t)h | (uintptr_t)x | (uintptr_t)w_post) & 15);
  static MarySmemSlots slots[4] = {};
  BY_TYPE(f32, {
    auto fn = vec ? post_norm_add_kernel<T, true> : post_norm_add_kernel<T, false>;
    if (int rc = sm > 48 * 1024 ? mary_ensure_dyn_smem((const void*)fn, sm, &slots[(f32 ? 2 : 0) + (vec ? 1 : 0)]) : 0) return rc;
    MARY_LAUNCH(fn, T_, NT, sm, s, a, lda, (const T*)w_post, h, (const T*)w_next, (T*)x, H, eps);
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_rmsnorm32(const float* x, const void* w, void* y, int T_, int H, float eps, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  BY_TYPE(f32, MARY_LAUNCH((rmsnorm32_kernel<T>), T_, NT, 0, s, x, (const T*)w, (T*)y, H, eps));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// act: 0 = tanh-form GELU, 1 = SiLU, 3 = clamped by `limit`; any F
MARY_API int mary_glu_any(const void* gu, void* out, int T_, int F, int act, float limit, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (act < 0 || act > 3 || act == 2) return MARY_ERR_BAD_ARG;
  const int64_t n = (int64_t)T_ * F;
  BY_TYPE(f32, MARY_LAUNCH((glu_any_kernel<T>), (unsigned)((n + NT - 1) / NT), NT, 0, s, (const T*)gu, (T*)out, F, n, act, limit));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// act: 0 = tanh-form GELU, 1 = SiLU, in place on the first n columns of T rows with pitch ld
MARY_API int mary_act_rows(void* y, int64_t ld, int T_, int n, int act, int f32, cudaStream_t s) {
  if (T_ <= 0 || n <= 0) return MARY_OK;
  if (act < 0 || act > 1 || ld < n) return MARY_ERR_BAD_ARG;
  const int64_t total = (int64_t)T_ * n;
  BY_TYPE(f32, MARY_LAUNCH((act_rows_kernel<T>), (unsigned)((total + NT - 1) / NT), NT, 0, s, (T*)y, ld, n, total, act));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// x = cap * tanh(x / cap), n contiguous f32 values in place
MARY_API int mary_soft_cap(float* x, int64_t n, float cap, cudaStream_t s) {
  if (n <= 0) return MARY_OK;
  if (!(cap > 0.f)) return MARY_ERR_BAD_ARG;
  MARY_LAUNCH(soft_cap_kernel, (unsigned)((n + NT - 1) / NT), NT, 0, s, x, n, cap);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_qk_norm_append(const void* q, const void* k, const void* v, int64_t ld, int n_q, int n_kv, int DK, int DV, const void* q_gain,
                                 const void* k_gain, const int64_t* slots, void* qo, void* kc, void* vc, float eps, int n_tok, int64_t n_slots,
                                 int f32, cudaStream_t s) {
  if (n_tok <= 0) return MARY_OK;
  const int64_t warps = (int64_t)n_tok * (n_q + 2 * n_kv);
  BY_TYPE(f32, MARY_LAUNCH((qk_norm_append_kernel<T>), (unsigned)((warps + 7) / 8), 256, 0, s, (const T*)q, (const T*)k, (const T*)v, ld, n_q, n_kv, DK,
                           DV, (const T*)q_gain, (const T*)k_gain, slots, (T*)qo, (T*)kc, (T*)vc, eps, n_tok, n_slots, mary_status_ptr()));
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_embed_dyt(const int* ids, const void* table, float* h, void* x, int T_, int H, float scale, const void* w, const void* b,
                            const float* alpha, int vocab, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  BY_TYPE(f32, {
    const Dyt<T> n = {(const T*)w, (const T*)b, alpha};
    MARY_LAUNCH((embed_dyt_kernel<T>), T_, NT, 0, s, ids, (const T*)table, h, (T*)x, H, scale, n, vocab, mary_status_ptr());
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// h[T, H] (f32) += tanh(alpha a) w + b, then x[T, H] = tanh(alpha_n h) w_n + b_n.  `a` is f32, rows of `lda`.
MARY_API int mary_dyt_add(const float* a, int64_t lda, const void* w, const void* b, const float* alpha, float* h, const void* w_n, const void* b_n,
                          const float* alpha_n, void* x, int T_, int H, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (T_ > 65535 * 16) return MARY_ERR_BAD_ARG;
  const bool vec = H % 8 == 0 && lda % 4 == 0 &&
                   !(((uintptr_t)a | (uintptr_t)h | (uintptr_t)x | (uintptr_t)w | (uintptr_t)b | (uintptr_t)w_n | (uintptr_t)b_n) & 15);
  const int E = vec ? 8 : 1;
  BY_TYPE(f32, {
    const Dyt<T> post = {(const T*)w, (const T*)b, alpha}, next = {(const T*)w_n, (const T*)b_n, alpha_n};
    auto fn = vec ? dyt_add_kernel<T, 8> : dyt_add_kernel<T, 1>;
    for (int t = 0; t < T_; t += 65535)
      MARY_LAUNCH(fn, dim3((H + NT * E - 1) / (NT * E), T_ - t < 65535 ? T_ - t : 65535), NT, 0, s, a + (int64_t)t * lda, lda, post, h + (int64_t)t * H, next,
                  (T*)x + (int64_t)t * H, H);
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// q / k / v: columns of projection rows with pitch ld, nq / nk / nv values each; k null: queries only.
MARY_API int mary_row_norm_append(const void* q, const void* k, const void* v, int64_t ld, int nq, int nk, int nv, const void* q_gain,
                                  const void* k_gain, const int64_t* slots, void* qo, void* kc, void* vc, float eps, int n_tok, int64_t n_slots,
                                  int f32, cudaStream_t s) {
  if (n_tok <= 0) return MARY_OK;
  if (nq < 1 || (k && (nk < 1 || nv < 1))) return MARY_ERR_BAD_ARG;
  BY_TYPE(f32, {
    const bool vec = nq % 8 == 0 && nk % 8 == 0 && nv % 8 == 0 && ld % 8 == 0 &&
                     !(((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)q_gain | (uintptr_t)k_gain | (uintptr_t)qo | (uintptr_t)kc | (uintptr_t)vc) & 15);
    auto fn = vec ? row_norm_append_kernel<T, 8> : row_norm_append_kernel<T, 1>;
    MARY_LAUNCH(fn, dim3(n_tok, k ? 2 : 1), NT, 0, s, (const T*)q, (const T*)k, (const T*)v, ld, nq, nk, nv, (const T*)q_gain, (const T*)k_gain, slots,
                (T*)qo, (T*)kc, (T*)vc, eps, n_slots, mary_status_ptr());
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
