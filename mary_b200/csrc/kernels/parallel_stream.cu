// Row kernels of decoders with parallel sublayers around a 32-bit residual stream, for bf16 and for 32-bit activations: token plus
// token-pair embedding, rotation of queries and keys by split halves with cache append, rotation of queries, keys and values by neighbouring
// pairs with norms and cache append, and the residual step that adds the sublayers'
// outputs (the weighted rows of routed experts among them) and norms the new stream for whatever reads it next.  One CTA per token; any
// width; norms, sums and angles in exact 32-bit (angles: reduced in 64-bit) arithmetic.
#include "host_utils.h"
#include "routed.cuh"

using namespace mary;

namespace {

constexpr int NT = 256;

// h[t] = table[id] + pairs[(prev * mul_prev + id * mul_cur) mod buckets], the extra row `buckets` for the first token of a sequence; copies
// in the activation type to x0 and x1 (or null).  last[slot] keeps a sequence's newest token between steps: the CTA of a sequence's
// first row reads it and then replaces it, no other CTA touches it.
template <typename T, int E>
__global__ void __launch_bounds__(NT) embed_pairs_kernel(const int* __restrict__ ids, const T* __restrict__ table, const T* __restrict__ pairs,
                                                         int64_t mul_prev, int64_t mul_cur, int buckets, int* __restrict__ last,
                                                         const int* __restrict__ q_start, const int* __restrict__ seq_index,
                                                         const int* __restrict__ positions, const int* __restrict__ state_slots,
                                                         float* __restrict__ h, T* __restrict__ x0, T* __restrict__ x1, int64_t ldx, int H, int vocab,
                                                         int* __restrict__ status) {
  pdl_sync();
  __shared__ int rows[2];
  const int t = blockIdx.x;
  if (threadIdx.x == 0) {
    int id = ids[t];
    const int seq = seq_index[t], first = q_start[seq];
    const bool start = positions[t] == 0;
    int64_t prev = t > first ? ids[t - 1] : 0;
    if (t == first) {
      if (!start) prev = last[state_slots[seq]];
      last[state_slots[seq]] = ids[q_start[seq + 1] - 1];
    }
    int64_t r = (prev * mul_prev + (int64_t)id * mul_cur) % buckets;
    if (r < 0) r += buckets;
    if (id < 0 || id >= vocab) {               // recorded, and redirected to row 0: no read outside the table
      atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);
      id = 0;
    }
    rows[0] = id;
    rows[1] = start ? buckets : (int)r;
  }
  __syncthreads();
  const T *a = table + (int64_t)rows[0] * H, *b = pairs + (int64_t)rows[1] * H;
  for (int i = threadIdx.x * E; i < H; i += NT * E) {
    float u[E], v[E];
    load_v<T, E>(a + i, u);
    load_v<T, E>(b + i, v);
#pragma unroll
    for (int j = 0; j < E; ++j) u[j] += v[j];
    store_v<float, E>(h + (int64_t)t * H + i, u);
    if (x0) store_v<T, E>(x0 + t * ldx + i, u);
    if (x1) store_v<T, E>(x1 + t * ldx + i, u);
  }
}

// Queries rotated in place, keys rotated into the cache, values copied into the cache.  A row of nq query heads (nk key heads) of D values;
// dimensions i and i + n (i < n) of a head turn by position * freq[i], the others stay.  v: nv values per token.
template <typename T, int E>
__global__ void __launch_bounds__(NT) rotate_append_kernel(T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int64_t ld, int nq,
                                                           int nk, int D, int nv, int n, const double* __restrict__ freq,
                                                           const int* __restrict__ positions, const int64_t* __restrict__ slots, T* __restrict__ kc,
                                                           T* __restrict__ vc, int64_t n_slots, int* __restrict__ status) {
  pdl_sync();
  extern __shared__ float2 turn[];                             // cosine and sine per pair
  const int t = blockIdx.x;
  const int64_t slot = slots[t];
  const bool ok = slot >= 0 && slot < n_slots;
  if (!ok && threadIdx.x == 0) atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);       // a slot outside the cache: recorded, no write
  for (int i = threadIdx.x; i < n; i += NT) {
    const double a = positions[t] * freq[i], two_pi = 6.283185307179586;
    float s, c;
    sincosf((float)(a - rint(a / two_pi) * two_pi), &s, &c);
    turn[i] = make_float2(c, s);
  }
  __syncthreads();
  auto pair = [&](const T* src, T* dst, int i) {
    float u[E], w[E], x[E], y[E];
    load_v<T, E>(src + i, u);
    load_v<T, E>(src + n + i, w);
#pragma unroll
    for (int j = 0; j < E; ++j) {
      const float2 cs = turn[i + j];
      x[j] = u[j] * cs.x - w[j] * cs.y;
      y[j] = w[j] * cs.x + u[j] * cs.y;
    }
    store_v<T, E>(dst + i, x);
    store_v<T, E>(dst + n + i, y);
  };
  const int pv = n / E;
  if (q)
    for (int i = threadIdx.x; i < nq * pv; i += NT) {
      T* head = q + t * ld + (i / pv) * D;
      pair(head, head, i % pv * E);
    }
  if (!ok) return;
  const T* kr = k + t * ld;
  T* kd = kc + slot * nk * D;
  if (pv > 0)
    for (int i = threadIdx.x; i < nk * pv; i += NT) pair(kr + i / pv * D, kd + i / pv * D, i % pv * E);
  const int rest = (D - 2 * n) / E;
  for (int i = threadIdx.x; i < nk * rest; i += NT) {
    const int at = i / rest * D + 2 * n + i % rest * E;
    float f[E];
    load_v<T, E>(kr + at, f);
    store_v<T, E>(kd + at, f);
  }
  for (int i = threadIdx.x * E; i < nv; i += NT * E) {
    float f[E];
    load_v<T, E>(v + t * ld + i, f);
    store_v<T, E>(vc + slot * nv + i, f);
  }
}

// turn[t][i] = (cos, sin) of positions[t] * freq[i], times gain; angles reduced in 64 bits
__global__ void turn_table_kernel(const int* __restrict__ positions, const double* __restrict__ freq, int n, float gain, float2* __restrict__ turn,
                                  int64_t total) {
  pdl_sync();
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const double a = positions[i / n] * freq[i % n], two_pi = 6.283185307179586;
  float s, c;
  sincosf((float)(a - rint(a / two_pi) * two_pi), &s, &c);
  turn[i] = make_float2(c * gain, s * gain);
}

struct TurnIo {
  const float2* turn; int n;             // queries and keys: pairs 2 i, 2 i + 1 for i < n, the dimensions behind them stay
  const float2* vturn; int vn;           // values (vn = 0: not turned)
  const float* temp;                     // [nq] or null
  int nq, nk, D, DV;
  float eps;                             // < 0: no norm
};

// One warp per head in turn: query heads are turned, divided by their root mean square, multiplied by temp and written back; key heads the
// same without temp into the cache, value heads turned into the cache.  A lane holds NU units of 2 P neighbouring values.
template <typename T, int P, int NU>
__global__ void __launch_bounds__(NT) turn_norm_append_kernel(T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, int64_t ld, TurnIo io,
                                                              const int64_t* __restrict__ slots, T* __restrict__ kc, T* __restrict__ vc,
                                                              int64_t n_slots, int* __restrict__ status) {
  pdl_sync();
  constexpr int E = 2 * P;
  const int64_t t = blockIdx.x, slot = slots[t];
  const bool ok = slot >= 0 && slot < n_slots;
  if (!ok && threadIdx.x == 0) atomicCAS(status, 0, (int)MARY_ERR_BOUNDS);       // a slot outside the cache: recorded, no write
  const int lane = threadIdx.x & 31;
  for (int h = threadIdx.x >> 5; h < io.nq + 2 * io.nk; h += NT / 32) {
    const bool is_q = h < io.nq, is_v = h >= io.nq + io.nk;
    const int hk = h - io.nq - (is_v ? io.nk : 0), D = is_v ? io.DV : io.D, n = is_v ? io.vn : io.n;
    if (!is_q && !ok) continue;
    const T* src = is_q ? q + t * ld + h * D : (is_v ? v : k) + t * ld + hk * D;
    T* dst = is_q ? q + t * ld + h * D : (is_v ? vc : kc) + (slot * io.nk + hk) * D;
    const float2* turn = (is_v ? io.vturn : io.turn) + t * n;
    float f[NU][E], ss = 0.f;
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int c = (u * 32 + lane) * E;
      if constexpr (P > 1) {
        if (c < D) load_e<T, E>(src + c, f[u]);
      } else {
        f[u][0] = c < D ? to_f<T>(src[c]) : 0.f;
        f[u][1] = c + 1 < D ? to_f<T>(src[c + 1]) : 0.f;
      }
    }
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int c = (u * 32 + lane) * E;
      if (c >= D) break;
#pragma unroll
      for (int p = 0; p < P; ++p) {
        float &a = f[u][2 * p], &b = f[u][2 * p + 1];
        if (c / 2 + p < n) {
          const float2 cs = turn[c / 2 + p];
          const float x = a * cs.x - b * cs.y, y = b * cs.x + a * cs.y;
          a = x;
          b = y;
        }
        ss = fmaf(a, a, fmaf(b, b, ss));
      }
    }
    float m = 1.f;
    if (!is_v && io.eps >= 0.f) m = 1.0f / sqrtf(warp_sum(ss) / D + io.eps);
    if (is_q && io.temp) m *= io.temp[h];
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int c = (u * 32 + lane) * E;
      if (c >= D) break;
#pragma unroll
      for (int j = 0; j < E; ++j) f[u][j] *= m;
      if constexpr (P > 1) store_e<T, E>(dst + c, f[u]);
      else {
        dst[c] = from_f<T>(f[u][0]);
        if (c + 1 < D) dst[c + 1] = from_f<T>(f[u][1]);
      }
    }
  }
}

template <typename T> struct Follow {              // what reads the new stream: up to two norms of it, or a plain copy
  const T* w1; T* x1; const T* w2; T* x2;
  T* copy; int64_t ld;
};

// h = keep * h + m * (a + routed) + vec;  x1 = rms(h) * w1, x2 = rms(h) * w2, copy = h.
template <typename T, int E>
__global__ void __launch_bounds__(NT) stream_step_kernel(const float* __restrict__ a, int64_t lda, float m, Routed<T> r, const T* __restrict__ vec,
                                                         float* __restrict__ h, int keep, Follow<T> f, int H, float eps) {
  pdl_sync();
  extern __shared__ float row[];
  __shared__ float red[32];
  __shared__ RoutedRows list;
  const int64_t t = blockIdx.x;
  if (r.k > 0) {
    if (threadIdx.x == 0) list_routed(r, t, list);
    __syncthreads();
  }
  const float self = r.k > 0 ? list.self : 0.f;
  const int ns = r.k > 0 ? list.n : 0;
  float ss = 0.f;
  for (int i = threadIdx.x * E; i < H; i += NT * E) {
    float s[E], g[E];
#pragma unroll
    for (int j = 0; j < E; ++j) s[j] = 0.f;
    if (a) load_v<float, E>(a + t * lda + i, s);
    add_routed<T, E>(r, list, ns, self, t, i, H, s);
#pragma unroll
    for (int j = 0; j < E; ++j) s[j] *= m;
    if (keep) {
      load_v<float, E>(h + t * H + i, g);
#pragma unroll
      for (int j = 0; j < E; ++j) s[j] += g[j];
    }
    if (vec) {
      load_v<T, E>(vec + i, g);
#pragma unroll
      for (int j = 0; j < E; ++j) s[j] += g[j];
    }
    if (a || r.k > 0 || vec) store_v<float, E>(h + t * H + i, s);
    if (f.copy) store_v<T, E>(f.copy + t * f.ld + i, s);
#pragma unroll
    for (int j = 0; j < E; ++j) { row[i + j] = s[j]; ss = fmaf(s[j], s[j], ss); }
  }
  if (!f.x1) return;
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / H + eps);
  for (int i = threadIdx.x * E; i < H; i += NT * E) {          // the same elements this thread wrote above
    float g[E], y[E];
    load_v<T, E>(f.w1 + i, g);
#pragma unroll
    for (int j = 0; j < E; ++j) y[j] = row[i + j] * inv * g[j];
    store_v<T, E>(f.x1 + t * H + i, y);
    if (f.x2) {
      load_v<T, E>(f.w2 + i, g);
#pragma unroll
      for (int j = 0; j < E; ++j) y[j] = row[i + j] * inv * g[j];
      store_v<T, E>(f.x2 + t * H + i, y);
    }
  }
}

bool aligned16(std::initializer_list<const void*> ptrs) {
  uintptr_t u = 0;
  for (const void* p : ptrs) u |= (uintptr_t)p;
  return (u & 15) == 0;
}

}  // namespace

#define BY_TYPE(f32, ...)                                       \
  do {                                                          \
    if (f32) { using T = float; __VA_ARGS__; }                  \
    else { using T = __nv_bfloat16; __VA_ARGS__; }              \
  } while (0)

// h [T, H] f32, x0 / x1: rows of ldx elements or null.  pairs has buckets + 1 rows; last: one int per state slot.
MARY_API int mary_embed_pairs(const int* ids, const void* table, const void* pairs, int64_t mul_prev, int64_t mul_cur, int buckets, int* last,
                              const int* q_start, const int* seq_index, const int* positions, const int* state_slots, float* h, void* x0, void* x1,
                              int64_t ldx, int T_, int H, int vocab, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (buckets < 1 || !last || !state_slots) return MARY_ERR_BAD_ARG;
  const bool vec = H % 8 == 0 && ldx % 8 == 0 && aligned16({table, pairs, h, x0, x1});
  BY_TYPE(f32, {
    auto fn = vec ? embed_pairs_kernel<T, 8> : embed_pairs_kernel<T, 1>;
    MARY_LAUNCH(fn, T_, NT, 0, s, ids, (const T*)table, (const T*)pairs, mul_prev, mul_cur, buckets, last, q_start, seq_index, positions, state_slots, h,
                (T*)x0, (T*)x1, ldx, H, vocab, mary_status_ptr());
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// q (or null: nothing to rotate), k, v: columns of projection rows with pitch ld.  freq: n f64 rotation frequencies (n = 0: no rotation).
// kc [slots][nk][D], vc [slots][nv].
MARY_API int mary_rotate_append(void* q, const void* k, const void* v, int64_t ld, int nq, int nk, int D, int nv, int n, const double* freq,
                                const int* positions, const int64_t* slots, void* kc, void* vc, int T_, int64_t n_slots, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (nk < 1 || nv < 1 || n < 0 || 2 * n > D || n > 4096) return MARY_ERR_BAD_ARG;
  const bool vec = D % 8 == 0 && n % 8 == 0 && nv % 8 == 0 && ld % 8 == 0 && aligned16({q, k, v, kc, vc});
  BY_TYPE(f32, {
    auto fn = vec ? rotate_append_kernel<T, 8> : rotate_append_kernel<T, 1>;
    MARY_LAUNCH(fn, T_, NT, n * sizeof(float2), s, n > 0 ? (T*)q : nullptr, (const T*)k, (const T*)v, ld, nq, nk, D, nv, n, freq, positions, slots, (T*)kc,
                (T*)vc, n_slots, mary_status_ptr());
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// turn [T, n, 2] f32: cosine and sine of positions[t] * freq[i], times gain.
MARY_API int mary_turn_table(const int* positions, const double* freq, int n, float gain, float* turn, int T_, cudaStream_t s) {
  if (T_ <= 0 || n == 0) return MARY_OK;
  if (n < 0) return MARY_ERR_BAD_ARG;
  const int64_t total = (int64_t)T_ * n;
  MARY_LAUNCH(turn_table_kernel, (unsigned)((total + NT - 1) / NT), NT, 0, s, positions, freq, n, gain, (float2*)turn, total);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// q, k, v: columns of projection rows with pitch ld (q is replaced in place).  turn [T, n, 2], vturn [T, vn, 2]: tables as above (n or vn = 0: not
// turned); temp [nq] (or null): factors of the query heads; eps < 0: no norm of queries and keys.  kc [slots][nk][D], vc [slots][nk][DV].
MARY_API int mary_turn_norm_append(void* q, const void* k, const void* v, int64_t ld, int nq, int nk, int D, int DV, const float* turn, int n,
                                   const float* vturn, int vn, const float* temp, const int64_t* slots, void* kc, void* vc, float eps, int T_,
                                   int64_t n_slots, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (nq < 1 || nk < 1 || D < 1 || DV < 1 || D > 640 || DV > 640 || n < 0 || 2 * n > D || vn < 0 || 2 * vn > DV) return MARY_ERR_BAD_ARG;
  const TurnIo io = {(const float2*)turn, n, (const float2*)vturn, vn, temp, nq, nk, D, DV, eps};
  const bool vec = D % 4 == 0 && DV % 4 == 0 && ld % 4 == 0 && aligned16({q, k, v, kc, vc});
  const int widest = D > DV ? D : DV;
  BY_TYPE(f32, {
    auto fn = !vec ? turn_norm_append_kernel<T, 1, 10>
                   : (widest <= 128 ? turn_norm_append_kernel<T, 2, 1> : (widest <= 256 ? turn_norm_append_kernel<T, 2, 2> : turn_norm_append_kernel<T, 2, 5>));
    MARY_LAUNCH(fn, T_, NT, 0, s, (T*)q, (const T*)k, (const T*)v, ld, io, slots, (T*)kc, (T*)vc, n_slots, mary_status_ptr());
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

// a [T] rows of lda f32 (or null).  k > 0: routed experts, see routed.cuh (y with row_of, or sum [T, H], or neither when every entry stands for x).
// w1 / x1, w2 / x2: norm gains and [T, H] results (x1 null: no norm; x2 null: one norm); copy: rows of ldc elements or null.
MARY_API int mary_stream_step(const float* a, int64_t lda, float m, const void* y, int64_t ldy, const int* row_of, const float* sum, const int* idx,
                              const float* w, const void* x, int k, int n_experts, const void* vec, float* h, int keep, const void* w1, void* x1,
                              const void* w2, void* x2, void* copy, int64_t ldc, int T_, int H, float eps, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (k < 0 || k > ROUTED_MAX || (k > 0 && (!idx || !w || !x || (y && !row_of))) || (x1 && !w1) || (x2 && (!w2 || !x1))) return MARY_ERR_BAD_ARG;
  const bool wide = H % 8 == 0 && lda % 4 == 0 && ldy % 8 == 0 && ldc % 8 == 0 && aligned16({a, y, sum, x, vec, h, w1, x1, w2, x2, copy});
  const size_t sm = (size_t)H * 4;
  static MarySmemSlots smem_set[4] = {};
  BY_TYPE(f32, {
    const Routed<T> r = {(const T*)y, ldy, row_of, sum, idx, w, (const T*)x, k, n_experts};
    const Follow<T> f = {(const T*)w1, (T*)x1, (const T*)w2, (T*)x2, (T*)copy, ldc};
    auto fn = wide ? stream_step_kernel<T, 8> : stream_step_kernel<T, 1>;
    if (int rc = sm > 40 * 1024 ? mary_ensure_dyn_smem((const void*)fn, sm, &smem_set[(f32 ? 2 : 0) + (wide ? 1 : 0)]) : 0) return rc;
    MARY_LAUNCH(fn, T_, NT, sm, s, a, lda, m, r, (const T*)vec, h, keep, f, H, eps);
  });
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
