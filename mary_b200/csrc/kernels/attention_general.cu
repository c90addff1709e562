// Causal paged attention for any head widths, group size and storage type (bf16 or 32-bit), with scores, softmax weights and sums in
// exact 32-bit arithmetic.  It is the path of 32-bit models and of head shapes that the specialised kernels (attention_fa.cu,
// attention_decode.cu) have no instantiation for.
//
// Work unit = (block of query tokens, kv head x chunk of its query heads, kv split): at most 16 (token, head) score rows.  Keys and
// values go through shared memory 32 at a time; warp w owns rows 4w .. 4w+3: in the score phase its lanes are the 32 keys, in the
// value phase its lanes cover the value dims.  Splits leave (m, l, o) partials that a second kernel merges.
#include "attention_form.cuh"
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int WARPS = 4, RPW = 4, ROWS = WARPS * RPW, KT = 32;

struct GenParams {
  const void* q; const void* kc; const void* vc; void* out;
  const int* page_table; const int* kv_len; const int* q_start; const int* blk_seq; const int* blk_q0;
  float* part_o; float* part_ml;
  int max_pages, page_size, Hq, Hkv, G, GC, gchunks, DK, DV, RQ, nsplit, window;
  int64_t k_tok, k_page, v_tok, v_page, out_ld;
  float scale;
  const float* bias;                     // [Hq][window], by distance, or null
  const void* gate; int64_t gate_ld;     // rows of gate_ld elements, head h at h * DV: the output times its logistic function; or null
  MaryAttnForm f;                        // two maps: Hq and Hkv count (head, map) pairs, the output is f32
};

// Query heads come in the order (kv head, head of its group, map), key heads as (kv head, map): the query head of member g of key head kvh.
__device__ __forceinline__ int query_head(const GenParams& p, int kvh, int g) { return ((kvh / p.f.maps) * p.G + g) * p.f.maps + kvh % p.f.maps; }

template <typename T>
__device__ __forceinline__ T gated(const GenParams& p, float v, int64_t row, int col) {
  if (p.gate) v *= sigmoid_x(to_f<T>(((const T*)p.gate)[row * p.gate_ld + col]));
  return from_f<T>(v);
}

// What turns a sum of weighted values into the result, given the maximum and the sum of the weights.
__device__ __forceinline__ float finish_scale(const GenParams& p, int head, float m, float l) {
  if (p.f.sink) {
    const float s = p.f.sink[head], top = fmaxf(m, s), c = expf(m - top);
    return c / (l * c + expf(s - top));
  }
  return l > 0.f ? 1.0f / l : 0.f;
}

template <typename T>
__device__ __forceinline__ void store_out(const GenParams& p, float v, int64_t row, int col) {
  if (p.f.maps == 2) ((float*)p.out)[row * p.out_ld + col] = v;
  else ((T*)p.out)[row * p.out_ld + col] = gated<T>(p, v, row, col);
}

template <typename T, int NV>      // NV: value dims per lane
__global__ void __launch_bounds__(WARPS * 32) attn_general_kernel(const GenParams p) {
  pdl_sync();
  extern __shared__ __align__(16) float sm[];
  const int nb = blockIdx.x, kvh = blockIdx.y / p.gchunks, g0 = (blockIdx.y % p.gchunks) * p.GC, split = blockIdx.z;
  const int gc = min(p.GC, p.G - g0);
  const int seq = p.blk_seq[nb], row0 = p.blk_q0[nb];
  const int q_end = p.q_start[seq + 1];
  const int nq = min(p.RQ, q_end - row0);
  const int R = nq * gc;
  const int qlen = q_end - p.q_start[seq];
  const int pos0 = p.kv_len[seq] - qlen + (row0 - p.q_start[seq]);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int DKP = p.DK + 1;
  float* sq = sm;                        // [ROWS][DK]
  float* sk = sq + ROWS * p.DK;          // [KT][DK + 1]
  float* sv = sk + KT * DKP;             // [KT][DV]
  const T* q = (const T*)p.q;
  const T* kc = (const T*)p.kc;
  const T* vc = (const T*)p.vc;
  for (int i = threadIdx.x; i < ROWS * p.DK; i += blockDim.x) {
    const int r = i / p.DK, d = i % p.DK;
    sq[i] = r < R ? to_f<T>(q[(int64_t)(row0 + r / gc) * p.f.q_ld + query_head(p, kvh, g0 + r % gc) * p.DK + d]) * query_temperature(p.f, pos0 + r / gc)
                  : 0.f;
  }
  const int k_hi = pos0 + nq, k_lo = max(p.window > 0 ? pos0 - p.window + 1 : 0, first_key(p.f, pos0));
  const int per = ((k_hi - k_lo + p.nsplit - 1) / p.nsplit + KT - 1) / KT * KT;
  const int s_lo = k_lo + split * per, s_hi = min(k_hi, s_lo + per);
  float m[RPW], l[RPW], o[RPW][NV];
#pragma unroll
  for (int r = 0; r < RPW; ++r) {
    m[r] = -INFINITY; l[r] = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v) o[r][v] = 0.f;
  }
  const int* pt = p.page_table + (int64_t)seq * p.max_pages;
  for (int kb = s_lo; kb < s_hi; kb += KT) {
    __syncthreads();
    const int nk = min(KT, s_hi - kb);
    for (int j = warp; j < KT; j += WARPS) {
      const bool in = j < nk;
      const int kp = kb + (in ? j : 0);
      const int page = pt[kp / p.page_size];
      const int64_t tok = kp % p.page_size;
      const T* kr = kc + (int64_t)page * p.k_page + tok * p.k_tok + (int64_t)kvh * p.DK;
      const T* vr = vc + (int64_t)page * p.v_page + tok * p.v_tok + (int64_t)(kvh / p.f.maps) * p.DV;
      for (int d = lane; d < p.DK; d += 32) sk[j * DKP + d] = in ? to_f<T>(kr[d]) : 0.f;
      for (int d = lane; d < p.DV; d += 32) sv[j * p.DV + d] = in ? to_f<T>(vr[d]) : 0.f;
    }
    __syncthreads();
    float s[RPW] = {};
    for (int d = 0; d < p.DK; ++d) {
      const float kd = sk[lane * DKP + d];
#pragma unroll
      for (int r = 0; r < RPW; ++r) s[r] = fmaf(sq[(warp * RPW + r) * p.DK + d], kd, s[r]);
    }
    const int kp = kb + lane;
    float pr[RPW];
#pragma unroll
    for (int r = 0; r < RPW; ++r) {
      const int rr = warp * RPW + r;
      const int qp = pos0 + rr / gc;
      const bool ok = rr < R && lane < nk && kp <= qp && (p.window <= 0 || qp - kp < p.window) && kp >= first_key(p.f, qp);
      float sv_ = -INFINITY;
      if (ok) {
        sv_ = s[r] * p.scale;
        if (p.f.cap > 0.f) sv_ = p.f.cap * tanhf(sv_ / p.f.cap);
        if (p.bias) sv_ += p.bias[(int64_t)(kvh * p.G + g0 + rr % gc) * p.window + (qp - kp)];
      }
      const float mx = fmaxf(m[r], warp_max(sv_));
      pr[r] = 0.f;
      if (mx == -INFINITY) continue;                // warp-uniform: nothing visible to this row yet
      const float corr = expf(m[r] - mx);
      pr[r] = ok ? expf(sv_ - mx) : 0.f;
      l[r] = l[r] * corr + warp_sum(pr[r]);
      m[r] = mx;
#pragma unroll
      for (int v = 0; v < NV; ++v) o[r][v] *= corr;
    }
    for (int j = 0; j < nk; ++j) {
      float vf[NV];
#pragma unroll
      for (int v = 0; v < NV; ++v) vf[v] = lane + 32 * v < p.DV ? sv[j * p.DV + lane + 32 * v] : 0.f;
#pragma unroll
      for (int r = 0; r < RPW; ++r) {
        const float pj = __shfl_sync(0xffffffffu, pr[r], j);
#pragma unroll
        for (int v = 0; v < NV; ++v) o[r][v] = fmaf(pj, vf[v], o[r][v]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < RPW; ++r) {
    const int rr = warp * RPW + r;
    if (rr >= R) continue;
    if (p.nsplit == 1) {
      const int64_t row = row0 + rr / gc;
      const int h = query_head(p, kvh, g0 + rr % gc), col = h * p.DV;
      const float inv = finish_scale(p, h, m[r], l[r]);
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const bool in = lane + 32 * v < p.DV;
        const float x = turned_back_lane(p.f, o[r][v] * inv, row, lane + 32 * v, p.DV, in);
        if (in) store_out<T>(p, x, row, col + lane + 32 * v);
      }
    } else {
      const int64_t pi = (((int64_t)nb * gridDim.y + blockIdx.y) * p.nsplit + split) * ROWS + rr;
#pragma unroll
      for (int v = 0; v < NV; ++v)
        if (lane + 32 * v < p.DV) p.part_o[pi * p.DV + lane + 32 * v] = o[r][v];
      if (lane == 0) { p.part_ml[pi * 2] = m[r]; p.part_ml[pi * 2 + 1] = l[r]; }
    }
  }
}

template <typename T>
__global__ void attn_general_combine_kernel(const GenParams p) {
  pdl_sync();
  const int nb = blockIdx.x, kvh = blockIdx.y / p.gchunks, g0 = (blockIdx.y % p.gchunks) * p.GC;
  const int gc = min(p.GC, p.G - g0);
  const int seq = p.blk_seq[nb], row0 = p.blk_q0[nb];
  const int R = min(p.RQ, p.q_start[seq + 1] - row0) * gc;
  for (int i0 = 0; i0 < R * p.DV; i0 += blockDim.x) {              // whole warps go through it together
    const bool in = i0 + (int)threadIdx.x < R * p.DV;
    const int i = in ? i0 + threadIdx.x : 0;
    const int r = i / p.DV, d = i % p.DV;
    const int64_t base = (((int64_t)nb * gridDim.y + blockIdx.y) * p.nsplit) * ROWS + r;
    float mm = -INFINITY;
    for (int s = 0; s < p.nsplit; ++s) mm = fmaxf(mm, p.part_ml[(base + (int64_t)s * ROWS) * 2]);
    float ll = 0.f, acc = 0.f;
    for (int s = 0; s < p.nsplit; ++s) {
      const int64_t pi = base + (int64_t)s * ROWS;
      const float ms = p.part_ml[pi * 2];
      const float c = ms == -INFINITY ? 0.f : expf(ms - mm);
      ll += p.part_ml[pi * 2 + 1] * c;
      acc += p.part_o[pi * p.DV + d] * c;
    }
    const int h = query_head(p, kvh, g0 + r % gc);
    const float x = turned_back_lane(p.f, acc * finish_scale(p, h, mm, ll), row0 + r / gc, d, p.DV, in);
    if (in) store_out<T>(p, x, row0 + r / gc, h * p.DV + d);
  }
}

// One warp per (token, head): out = rms(o[0] - mix * o[1]) * post over the DV values of o [T][H][2][DV].
template <typename T>
__global__ void map_difference_kernel(const float* __restrict__ o, T* __restrict__ out, int64_t out_ld, int n, int H, int DV, float mix, float post,
                                      float eps, const int* __restrict__ rows) {
  pdl_sync();
  const int w = (int)((blockIdx.x * (int64_t)blockDim.x + threadIdx.x) >> 5), lane = threadIdx.x & 31;
  if (w >= n * H) return;
  const int64_t t = rows ? rows[w / H] : w / H;
  const int h = w % H;
  const float* a = o + (t * H + h) * 2 * DV;
  float ss = 0.f;
  for (int d = lane; d < DV; d += 32) { const float v = fmaf(-mix, a[DV + d], a[d]); ss = fmaf(v, v, ss); }
  const float c = post / sqrtf(warp_sum(ss) / DV + eps);
  for (int d = lane; d < DV; d += 32) out[t * out_ld + h * DV + d] = from_f<T>(fmaf(-mix, a[DV + d], a[d]) * c);
}

template <typename T, int NV>
int launch(const GenParams& p, int NB, cudaStream_t s) {
  const size_t sm = ((size_t)ROWS * p.DK + (size_t)KT * (p.DK + 1 + p.DV)) * 4;
  static MarySmemSlots slots = {};
  if (sm > 48 * 1024)
    if (int rc = mary_ensure_dyn_smem((const void*)attn_general_kernel<T, NV>, sm, &slots)) return rc;
  MARY_LAUNCH((attn_general_kernel<T, NV>), dim3(NB, p.Hkv * p.gchunks, p.nsplit), WARPS * 32, sm, s, p);
  if (p.nsplit > 1) MARY_LAUNCH((attn_general_combine_kernel<T>), dim3(NB, p.Hkv * p.gchunks), 256, 0, s, p);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

template <typename T>
int dispatch(const GenParams& p, int NB, cudaStream_t s) {
  const int nv = (p.DV + 31) / 32;
  if (nv <= 1) return launch<T, 1>(p, NB, s);
  if (nv <= 2) return launch<T, 2>(p, NB, s);
  if (nv <= 4) return launch<T, 4>(p, NB, s);
  if (nv <= 8) return launch<T, 8>(p, NB, s);
  return launch<T, 16>(p, NB, s);
}

}  // namespace

// Query tokens of one sequence that a block may hold for a group of G query heads per kv head.
MARY_API int mary_attention_general_rows(int G) { return G >= ROWS ? 1 : ROWS / G; }
MARY_API int64_t mary_attention_general_scratch_floats(int NB, int Hq, int Hkv, int nsplit, int DV) {
  const int G = Hq / Hkv, gchunks = (G + ROWS - 1) / ROWS;
  return nsplit > 1 ? (int64_t)NB * Hkv * gchunks * nsplit * ROWS * (DV + 2) : 0;
}

// q [T, Hq, DK] contiguous; caches with element strides per token and per page, heads contiguous inside a token row; out rows of
// out_ld elements, head h at h * DV.  bias [Hq][window] (or null) is added to the scaled score by distance, gate (or null) multiplies the
// output by its logistic function.  form (or null): see attention_form.cuh; with two maps Hq and Hkv count (head, map) pairs, values have
// Hkv / 2 heads and out is f32 [T][Hq][DV], which mary_map_difference turns into the result.  blk_seq / blk_q0: NB blocks of at most RQ query tokens that never cross a sequence.
MARY_API int mary_attention_general(const void* q, const void* kc, const void* vc, void* out, const int* page_table, const int* kv_len,
                                    const int* q_start, const int* blk_seq, const int* blk_q0, int NB, int max_pages, int page_size, int64_t k_tok,
                                    int64_t k_page, int64_t v_tok, int64_t v_page, int64_t out_ld, int Hq, int Hkv, int DK, int DV, int RQ,
                                    int nsplit, int window, float scale, const float* bias, const void* gate, int64_t gate_ld,
                                    float* scratch, const MaryAttnForm* form, int f32, cudaStream_t s) {
  if (NB <= 0) return MARY_OK;
  if (Hkv < 1 || Hq % Hkv || DK < 1 || DV < 1 || DK > 640 || DV > 512 || nsplit < 1 || (bias && window < 1)) return MARY_ERR_BAD_ARG;
  GenParams p;
  p.q = q; p.kc = kc; p.vc = vc; p.out = out; p.page_table = page_table; p.kv_len = kv_len; p.q_start = q_start; p.blk_seq = blk_seq; p.blk_q0 = blk_q0;
  p.max_pages = max_pages; p.page_size = page_size; p.Hq = Hq; p.Hkv = Hkv; p.G = Hq / Hkv; p.DK = DK; p.DV = DV; p.RQ = RQ; p.nsplit = nsplit;
  p.window = window; p.k_tok = k_tok; p.k_page = k_page; p.v_tok = v_tok; p.v_page = v_page; p.out_ld = out_ld; p.scale = scale; p.bias = bias; p.gate = gate; p.gate_ld = gate_ld;
  p.f = form ? *form : MaryAttnForm{};
  if (p.f.maps < 1) p.f.maps = 1;
  if (p.f.q_ld <= 0) p.f.q_ld = (int64_t)Hq * DK;
  if (p.f.maps > 2 || Hkv % p.f.maps || (p.f.maps == 2 && (gate || bias || p.f.sink || p.f.turn)) || (p.f.turn && (DV & 1)) || (bias && p.f.chunk)) return MARY_ERR_BAD_ARG;
  p.GC = p.G < ROWS ? p.G : ROWS;
  p.gchunks = (p.G + p.GC - 1) / p.GC;
  if (RQ < 1 || RQ * p.GC > ROWS || (nsplit > 1 && !scratch)) return MARY_ERR_BAD_ARG;
  p.part_o = scratch;
  p.part_ml = scratch + (int64_t)NB * p.Hkv * p.gchunks * nsplit * ROWS * DV;
  return f32 ? dispatch<float>(p, NB, s) : dispatch<__nv_bfloat16>(p, NB, s);
}

// out[t, h] = rms(o[t, h, 0] - mix * o[t, h, 1]) * post for the listed token rows (rows null: all T); o f32 [T][H][2][DV].
MARY_API int mary_map_difference(const float* o, void* out, int64_t out_ld, const int* rows, int n, int H, int DV, float mix, float post, float eps,
                                 int f32, cudaStream_t s) {
  if (n <= 0) return MARY_OK;
  const int grid = (int)(((int64_t)n * H + 7) / 8);
  if (f32) MARY_LAUNCH((map_difference_kernel<float>), grid, 256, 0, s, o, (float*)out, out_ld, n, H, DV, mix, post, eps, rows);
  else MARY_LAUNCH((map_difference_kernel<__nv_bfloat16>), grid, 256, 0, s, o, (__nv_bfloat16*)out, out_ld, n, H, DV, mix, post, eps, rows);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}
