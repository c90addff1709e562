// Row kernels of decoders whose residual is several 32-bit streams side by side, for bf16 and for 32-bit activations.  A sublayer reads a weighted
// sum of the streams through a norm; its output is added to every stream with a weight of its own while the streams are mixed:
//   u = sum_s in[s] x_s,   x_t <- sum_s mix[s][t] x_s + out[t] y.
// One launch does the update after a sublayer (the weighted rows of routed experts and the logistic gate of a shared one among its inputs) and
// forms the next sublayer's normed input from the new streams while they are in registers; the first one takes the embedding for all streams.
// One CTA per token; any width; sums and norms in exact 32-bit arithmetic.
#include "host_utils.h"
#include "routed.cuh"

using namespace mary;

namespace {

constexpr int NT = 256, MAX_STREAMS = 16;

template <typename T> struct Update {              // the sublayer's output y = a * (gate ? sigmoid(gate[t]) : 1) + routed experts
  const float* a; int64_t lda;
  const float* gate; int64_t ldg;
  Routed<T> routed;
  const float* mix; const float* out;              // [S][S] (from, to), [S]
};
template <typename T> struct Source {              // what the streams start from: rows of an embedding table (ids null: xs itself)
  const int* ids; const T* table; int vocab; int* status;
};

// xs [T][S][H].  keep = 0: the new streams are not stored.  x = rms(sum_t in[t] x_t) * gain.
template <typename T, int E, int NS>
__global__ void __launch_bounds__(NT) mix_streams_kernel(Source<T> src, Update<T> up, float* __restrict__ xs, int S, int keep,
                                                         const float* __restrict__ in, const T* __restrict__ gain, T* __restrict__ x, int H, float eps) {
  pdl_sync();
  extern __shared__ float row[];
  __shared__ float red[32], s_mix[NS * NS], s_out[NS], s_in[NS];
  __shared__ RoutedRows list;
  __shared__ int s_id;
  const int64_t t = blockIdx.x;
  const Routed<T>& r = up.routed;
  for (int i = threadIdx.x; i < NS * NS; i += NT) {
    const int a = i / NS, b = i % NS;
    s_mix[i] = up.mix && a < S && b < S ? up.mix[a * S + b] : 0.f;
    if (a == 0) {
      s_out[b] = up.mix && b < S ? up.out[b] : 0.f;
      s_in[b] = b < S ? in[b] : 0.f;
    }
  }
  if (threadIdx.x == 0) {
    if (r.k > 0) list_routed(r, t, list);
    if (src.ids) {
      int id = src.ids[t];
      if (id < 0 || id >= src.vocab) {             // recorded, and redirected to row 0: no read outside the table
        atomicCAS(src.status, 0, (int)MARY_ERR_BOUNDS);
        id = 0;
      }
      s_id = id;
    }
  }
  __syncthreads();
  const float self = r.k > 0 ? list.self : 0.f;
  const int ns = r.k > 0 ? list.n : 0;
  float g = 1.f;
  if (up.gate) g = sigmoid_x(up.gate[t * up.ldg]);
  float* xt = xs + t * S * H;
  float ss = 0.f;
  for (int i = threadIdx.x * E; i < H; i += NT * E) {
    float u[E];
#pragma unroll
    for (int j = 0; j < E; ++j) u[j] = 0.f;
    if (src.ids) {
      float e[E];
      load_v<T, E>(src.table + (int64_t)s_id * H + i, e);
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        if (s >= S) break;
#pragma unroll
        for (int j = 0; j < E; ++j) u[j] = fmaf(s_in[s], e[j], u[j]);
        if (keep) store_v<float, E>(xt + s * H + i, e);
      }
    } else {
      float old[NS][E], y[E];
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        if (s < S) load_v<float, E>(xt + s * H + i, old[s]);
        else {
#pragma unroll
          for (int j = 0; j < E; ++j) old[s][j] = 0.f;
        }
      }
#pragma unroll
      for (int j = 0; j < E; ++j) y[j] = 0.f;
      if (up.a) {
        load_v<float, E>(up.a + t * up.lda + i, y);
#pragma unroll
        for (int j = 0; j < E; ++j) y[j] *= g;
      }
      add_routed<T, E>(r, list, ns, self, t, i, H, y);
#pragma unroll
      for (int b = 0; b < NS; ++b) {
        if (b >= S) break;
        float v[E];
#pragma unroll
        for (int j = 0; j < E; ++j) v[j] = s_out[b] * y[j];
#pragma unroll
        for (int a = 0; a < NS; ++a) {
          const float m = s_mix[a * NS + b];
#pragma unroll
          for (int j = 0; j < E; ++j) v[j] = fmaf(m, old[a][j], v[j]);
        }
        if (keep) store_v<float, E>(xt + b * H + i, v);
#pragma unroll
        for (int j = 0; j < E; ++j) u[j] = fmaf(s_in[b], v[j], u[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < E; ++j) { row[i + j] = u[j]; ss = fmaf(u[j], u[j], ss); }
  }
  const float inv = 1.0f / sqrtf(block_sum_x(ss, red) / H + eps);
  for (int i = threadIdx.x * E; i < H; i += NT * E) {          // the same elements this thread wrote above
    float w[E], y[E];
    load_v<T, E>(gain + i, w);
#pragma unroll
    for (int j = 0; j < E; ++j) y[j] = row[i + j] * inv * w[j];
    store_v<T, E>(x + t * H + i, y);
  }
}

template <typename T, int E, int NS>
int launch(const Source<T>& src, const Update<T>& up, float* xs, int S, int keep, const float* in, const T* gain, T* x, int n_tok, int H, float eps,
           cudaStream_t s) {
  static MarySmemSlots set = {};
  const size_t sm = (size_t)H * 4;
  if (int rc = sm > 40 * 1024 ? mary_ensure_dyn_smem((const void*)mix_streams_kernel<T, E, NS>, sm, &set) : 0) return rc;
  MARY_LAUNCH((mix_streams_kernel<T, E, NS>), n_tok, NT, sm, s, src, up, xs, S, keep, in, gain, x, H, eps);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

template <typename T>
int dispatch(const Source<T>& src, const Update<T>& up, float* xs, int S, int keep, const float* in, const T* gain, T* x, int n_tok, int H, float eps,
             bool vec, cudaStream_t s) {
#define BY_STREAMS(NS) (vec ? launch<T, 4, NS>(src, up, xs, S, keep, in, gain, x, n_tok, H, eps, s) \
                            : launch<T, 1, NS>(src, up, xs, S, keep, in, gain, x, n_tok, H, eps, s))
  if (S == 1) return BY_STREAMS(1);
  if (S == 2) return BY_STREAMS(2);
  if (S <= 4) return BY_STREAMS(4);
  if (S <= 8) return BY_STREAMS(8);
  return BY_STREAMS(16);
#undef BY_STREAMS
}

bool aligned16(std::initializer_list<const void*> ptrs) {
  uintptr_t u = 0;
  for (const void* p : ptrs) u |= (uintptr_t)p;
  return (u & 15) == 0;
}

template <typename T>
int run(const int* ids, const void* table, int vocab, const float* a, int64_t lda, const float* gate, int64_t ldg, const void* y, int64_t ldy,
        const int* row_of, const float* sum, const int* idx, const float* w, const void* rx, int k, int n_experts, const float* mix, const float* out,
        float* xs, int S, int keep, const float* in, const void* gain, void* x, int n_tok, int H, float eps, cudaStream_t s) {
  const bool vec = H % 8 == 0 && lda % 4 == 0 && ldy % 8 == 0 && aligned16({table, a, y, sum, rx, xs, gain, x});
  const Source<T> src = {ids, (const T*)table, vocab, mary_status_ptr()};
  const Update<T> up = {a, lda, gate, ldg, {(const T*)y, ldy, row_of, sum, idx, w, (const T*)rx, k, n_experts}, mix, out};
  return dispatch<T>(src, up, xs, S, keep, in, (const T*)gain, (T*)x, n_tok, H, eps, vec, s);
}

}  // namespace

// xs [T, S, H] f32, S <= 16.  ids (or null): every stream starts as the token's row of table.  Otherwise the streams are updated by what a sublayer
// gave: a [T] rows of lda f32 (or null), times the logistic function of gate[t * ldg] (or null); k > 0: routed experts, see routed.cuh; mix [S, S]
// (from, to), out [S].  x [T, H] = rms(sum_t in[t] xs_t) * gain in the activation type.  keep = 0: the updated streams are not stored.
MARY_API int mary_mix_streams(const int* ids, const void* table, int vocab, const float* a, int64_t lda, const float* gate, int64_t ldg, const void* y,
                              int64_t ldy, const int* row_of, const float* sum, const int* idx, const float* w, const void* rx, int k, int n_experts,
                              const float* mix, const float* out, float* xs, int S, int keep, const float* in, const void* gain, void* x, int T_, int H,
                              float eps, int f32, cudaStream_t s) {
  if (T_ <= 0) return MARY_OK;
  if (S < 1 || S > MAX_STREAMS || H < 1 || !xs || !in || !gain || !x || k < 0 || k > ROUTED_MAX || (k > 0 && (!idx || !w || !rx || (y && !row_of))))
    return MARY_ERR_BAD_ARG;
  if (ids ? (!table || a || k > 0) : (!mix || !out || (!a && k == 0))) return MARY_ERR_BAD_ARG;
  return f32 ? run<float>(ids, table, vocab, a, lda, gate, ldg, y, ldy, row_of, sum, idx, w, rx, k, n_experts, mix, out, xs, S, keep, in, gain, x, T_, H, eps, s)
             : run<__nv_bfloat16>(ids, table, vocab, a, lda, gate, ldg, y, ldy, row_of, sum, idx, w, rx, k, n_experts, mix, out, xs, S, keep, in, gain, x,
                                  T_, H, eps, s);
}
