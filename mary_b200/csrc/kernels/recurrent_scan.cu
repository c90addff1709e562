// Linear recurrences over the tokens of a batch, with the state in 32-bit registers:
//
//   decayed linear attention   S_t = diag(a_t) S_{t-1} + k_t v_t^T                       o_t = S_t^T q_t    (a decay per key channel)
//   gated delta rule           S' = g_t S_{t-1};  u_t = b_t (v_t - S'^T k_t);  S_t = S' + k_t u_t^T;  o_t = S_t^T q_t   (a decay per head)
//
// The columns of S (one per value channel) are independent, so the grid is (column block, head, sequence) and every CTA walks the
// tokens of its sequence's portion: a column belongs to 8 lanes, each holding NR4 float4 of its rows.  The state is read from and
// returned to the sequence's slot, stored column by column, [slot][head][value channel][key channel padded to 4] (16-byte rows of
// consecutive key channels), and taken as zero when the portion starts at position 0.  Tokens are staged eight at a time in
// shared memory (next eight already in flight in registers).
//
// The delta rule's read S'^T k_t depends on the previous write, a chain of dot products over 8 lanes per token.  Four tokens at a
// time are therefore resolved against the state before them: with w_ij = g_{j+1} .. g_i and G_i = g_1 .. g_i,
//   u_i = b_i (v_i - G_i S_0^T k_i - sum_{j<i} w_ij (k_j . k_i) u_j),   o_i = G_i S_0^T q_i + sum_{j<=i} w_ij (k_j . q_i) u_j,
//   S_4 = G_4 S_0 + sum_j w_4j k_j u_j^T,
// which needs one round of reductions per four tokens; the k.k and k.q products are shared by all columns of the CTA.  The weights w
// are products of decays, never quotients, so a decay of zero is exact.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

constexpr int CT = 8;          // tokens per staged chunk

struct ScanParams {
  const void* q; const void* k; const void* v;      // token rows of ldq / ldk / ldv elements; q, k head h / rep, v head h
  const float* decay;                               // [T, H * DK] per channel, or [T, H] per head
  const float* beta;                                // [T, H] (delta rule)
  float* out;                                       // [T, H * DV]
  float* state;                                     // [slots][H][DV][DKS]
  const int* q_start; const int* kv_len; const int* slots;
  int64_t ldq, ldk, ldv;
  int H, rep, DK, DV, DKS;
  float q_scale;
};

// Sum V = 8 values over aligned groups of 8 lanes: lane l of the group ends with the total of value l.
__device__ __forceinline__ float sum8_scatter(float (&v)[8], int lane) {
#pragma unroll
  for (int o = 4; o >= 1; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float send = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  return v[0];
}

__device__ __forceinline__ float dot4(const float4& a, const float4& b, float c) {
  return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, c))));
}

template <typename TI, int E> struct Reg { uint4 v; };             // one 16-byte vector
template <typename TI> struct Reg<TI, 1> { TI v; };

template <typename TI, int NR4, bool DELTA, bool VEC, int NT>
__global__ void __launch_bounds__(NT) scan_kernel(const ScanParams p) {
  pdl_sync();
  constexpr int COLS = NT / 8, DKP = NR4 * 32;
  constexpr int E = VEC ? Pack<TI>::N : 1, NVQ = (CT * DKP / E + NT - 1) / NT;
  constexpr int EA = VEC ? 4 : 1, NVA = DELTA ? 1 : (CT * DKP / EA + NT - 1) / NT;
  typedef float Rows[CT][DKP];
  extern __shared__ __align__(16) float sm[];
  Rows *sq = (Rows*)sm, *sk = sq + 2, *sa = sk + 2;            // two buffers each; sa for channel decays only
  __shared__ float sv[2][CT][COLS], sg[2][CT], sb[2][CT], s_kk[2][4][4], s_kq[2][4][4];
  const int tid = threadIdx.x, lane8 = tid & 7, warp = tid >> 5, lane = tid & 31;
  const int seq = blockIdx.z, h = blockIdx.y, hk = h / p.rep;
  const int lcol = tid >> 3, col = blockIdx.x * COLS + lcol;
  const int row0 = p.q_start[seq], n = p.q_start[seq + 1] - row0;
  if (n <= 0) return;
  const bool fresh = p.kv_len[seq] == n;
  float* sp = p.state + (((int64_t)p.slots[seq] * p.H + h) * p.DV + col) * p.DKS;
  float4 st[NR4];
#pragma unroll
  for (int r = 0; r < NR4; ++r) {
    const int c = (r * 8 + lane8) * 4;
    st[r] = (!fresh && col < p.DV && c < p.DKS) ? *(const float4*)(sp + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (p.DK < DKP) {                       // channels beyond DK stay zero in both buffers
    for (int i = tid; i < (DELTA ? 4 : 6) * CT * DKP; i += NT) sm[i] = 0.f;
    __syncthreads();
  }
  const TI* qb = (const TI*)p.q + (int64_t)row0 * p.ldq + (int64_t)hk * p.DK;
  const TI* kb = (const TI*)p.k + (int64_t)row0 * p.ldk + (int64_t)hk * p.DK;
  const TI* vb = (const TI*)p.v + (int64_t)row0 * p.ldv + (int64_t)h * p.DV;
  const float* ab = DELTA ? p.decay + (int64_t)row0 * p.H + h : p.decay + ((int64_t)row0 * p.H + h) * p.DK;
  const float* bb = DELTA ? p.beta + (int64_t)row0 * p.H + h : nullptr;
  const int per_tok = p.DK / E, per_tok_a = p.DK / EA;

  Reg<TI, E> rq[NVQ], rk[NVQ];
  Reg<float, EA> ra[NVA];
  TI rv{};
  float rg = 1.f, rb = 0.f;
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < NVQ; ++i) {
      const int idx = tid + i * NT, t = t0 + idx / per_tok, c = (idx % per_tok) * E;
      rq[i] = {}; rk[i] = {};
      if (idx < CT * per_tok && t < n) {
        rq[i].v = *(const decltype(rq[i].v)*)(qb + (int64_t)t * p.ldq + c);
        rk[i].v = *(const decltype(rk[i].v)*)(kb + (int64_t)t * p.ldk + c);
      }
    }
    if constexpr (!DELTA) {
#pragma unroll
      for (int i = 0; i < NVA; ++i) {
        const int idx = tid + i * NT, t = t0 + idx / per_tok_a, c = (idx % per_tok_a) * EA;
        if (idx < CT * per_tok_a && t < n) ra[i].v = *(const decltype(ra[i].v)*)(ab + (int64_t)t * p.H * p.DK + c);
        else if constexpr (VEC) ra[i].v = make_uint4(0x3f800000u, 0x3f800000u, 0x3f800000u, 0x3f800000u);
        else ra[i].v = 1.f;
      }
    } else if (tid < CT) {
      const int t = t0 + tid;
      rg = t < n ? ab[(int64_t)t * p.H] : 1.f;
      rb = t < n ? bb[(int64_t)t * p.H] : 0.f;
    }
    const int t = t0 + tid / COLS, c = blockIdx.x * COLS + tid % COLS;
    rv = (t < n && c < p.DV) ? vb[(int64_t)t * p.ldv + c] : from_f<TI>(0.f);
  };
  auto stash = [&](int b) {
#pragma unroll
    for (int i = 0; i < NVQ; ++i) {
      const int idx = tid + i * NT, t = idx / per_tok, c = (idx % per_tok) * E;
      if (idx < CT * per_tok) {
        if constexpr (VEC) {
          float fq[E], fk[E];
          unpack16(rq[i].v, fq);
          unpack16(rk[i].v, fk);
#pragma unroll
          for (int j = 0; j < E; j += 4) {
            *(float4*)&sq[b][t][c + j] = make_float4(fq[j] * p.q_scale, fq[j + 1] * p.q_scale, fq[j + 2] * p.q_scale, fq[j + 3] * p.q_scale);
            *(float4*)&sk[b][t][c + j] = make_float4(fk[j], fk[j + 1], fk[j + 2], fk[j + 3]);
          }
        } else {
          sq[b][t][c] = to_f<TI>(rq[i].v) * p.q_scale;
          sk[b][t][c] = to_f<TI>(rk[i].v);
        }
      }
    }
    if constexpr (!DELTA) {
#pragma unroll
      for (int i = 0; i < NVA; ++i) {
        const int idx = tid + i * NT, t = idx / per_tok_a, c = (idx % per_tok_a) * EA;
        if (idx < CT * per_tok_a) {
          if constexpr (VEC) *(uint4*)&sa[b][t][c] = ra[i].v;
          else sa[b][t][c] = ra[i].v;
        }
      }
    } else if (tid < CT) {
      sg[b][tid] = rg;
      sb[b][tid] = rb;
    }
    sv[b][tid / COLS][tid % COLS] = to_f<TI>(rv);
  };

  fetch(0);
  stash(0);
  __syncthreads();
  for (int t0 = 0, b = 0; t0 < n; t0 += CT, b ^= 1) {
    const bool more = t0 + CT < n;
    if (more) fetch(t0 + CT);
    float o[CT];
    if constexpr (!DELTA) {
#pragma unroll
      for (int t = 0; t < CT; ++t) {
        const float vt = sv[b][t][lcol];
        float acc = 0.f;
#pragma unroll
        for (int r = 0; r < NR4; ++r) {
          const int c = (r * 8 + lane8) * 4;
          const float4 a4 = *(const float4*)&sa[b][t][c], k4 = *(const float4*)&sk[b][t][c], q4 = *(const float4*)&sq[b][t][c];
          st[r].x = fmaf(a4.x, st[r].x, k4.x * vt); st[r].y = fmaf(a4.y, st[r].y, k4.y * vt);
          st[r].z = fmaf(a4.z, st[r].z, k4.z * vt); st[r].w = fmaf(a4.w, st[r].w, k4.w * vt);
          acc = dot4(q4, st[r], acc);
        }
        o[t] = acc;
      }
      const float mine = sum8_scatter(o, lane);
      if (t0 + lane8 < n && col < p.DV) p.out[((int64_t)(row0 + t0 + lane8) * p.H + h) * p.DV + col] = mine;
    } else {
      // products of the chunk's keys with its keys and queries, weighted with the decays between them (two blocks of four tokens)
      for (int e = warp; e < 32; e += NT / 32) {
        const int blk = e >> 4, i = (e >> 2) & 3, j = e & 3;
        if (j > i) continue;
        const float* kj = sk[b][blk * 4 + j];
        const float* ki = sk[b][blk * 4 + i];
        const float* qi = sq[b][blk * 4 + i];
        float kk = 0.f, kq = 0.f;
        for (int c = lane * 4; c < DKP; c += 128) {
          const float4 a = *(const float4*)(kj + c);
          kk = dot4(a, *(const float4*)(ki + c), kk);
          kq = dot4(a, *(const float4*)(qi + c), kq);
        }
        kk = warp_sum(kk);
        kq = warp_sum(kq);
        if (lane == 0) {
          float w = 1.f;
          for (int l = j + 1; l <= i; ++l) w *= sg[b][blk * 4 + l];
          s_kk[blk][i][j] = w * kk;
          s_kq[blk][i][j] = w * kq;
        }
      }
      __syncthreads();
#pragma unroll
      for (int blk = 0; blk < 2; ++blk) {
        float d[8];                       // S_0^T k_0 .. k_3, S_0^T q_0 .. q_3
#pragma unroll
        for (int i = 0; i < 8; ++i) d[i] = 0.f;
#pragma unroll
        for (int r = 0; r < NR4; ++r) {
          const int c = (r * 8 + lane8) * 4;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            d[i] = dot4(*(const float4*)&sk[b][blk * 4 + i][c], st[r], d[i]);
            d[4 + i] = dot4(*(const float4*)&sq[b][blk * 4 + i][c], st[r], d[4 + i]);
          }
        }
        const float tot = sum8_scatter(d, lane);
#pragma unroll
        for (int i = 0; i < 8; ++i) d[i] = __shfl_sync(0xffffffffu, tot, (lane & ~7) | i);
        float u[4], G = 1.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          G *= sg[b][blk * 4 + i];
          float pred = G * d[i], oi = G * d[4 + i];
#pragma unroll
          for (int j = 0; j < i; ++j) pred = fmaf(s_kk[blk][i][j], u[j], pred);
          u[i] = sb[b][blk * 4 + i] * (sv[b][blk * 4 + i][lcol] - pred);
#pragma unroll
          for (int j = 0; j <= i; ++j) oi = fmaf(s_kq[blk][i][j], u[j], oi);
          o[blk * 4 + i] = oi;
        }
        float w = 1.f;
#pragma unroll
        for (int j = 3; j >= 0; --j) { u[j] *= w; w *= sg[b][blk * 4 + j]; }
#pragma unroll
        for (int r = 0; r < NR4; ++r) {
          const int c = (r * 8 + lane8) * 4;
          st[r].x *= G; st[r].y *= G; st[r].z *= G; st[r].w *= G;
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float4 k4 = *(const float4*)&sk[b][blk * 4 + j][c];
            st[r].x = fmaf(k4.x, u[j], st[r].x); st[r].y = fmaf(k4.y, u[j], st[r].y);
            st[r].z = fmaf(k4.z, u[j], st[r].z); st[r].w = fmaf(k4.w, u[j], st[r].w);
          }
        }
      }
      float mine = o[0];
#pragma unroll
      for (int t = 1; t < CT; ++t) mine = lane8 == t ? o[t] : mine;
      if (t0 + lane8 < n && col < p.DV) p.out[((int64_t)(row0 + t0 + lane8) * p.H + h) * p.DV + col] = mine;
    }
    if (more) stash(b ^ 1);
    __syncthreads();
  }
  if (col < p.DV) {
#pragma unroll
    for (int r = 0; r < NR4; ++r) {
      const int c = (r * 8 + lane8) * 4;
      if (c < p.DKS) *(float4*)(sp + c) = st[r];
    }
  }
}

template <typename TI, int NR4, bool DELTA, bool VEC>
int launch(const ScanParams& p, int S, cudaStream_t s) {
  constexpr int NT = DELTA ? 256 : 128, COLS = NT / 8;
  constexpr size_t SM = (size_t)(DELTA ? 4 : 6) * CT * NR4 * 32 * 4;
  static MarySmemSlots slots = {};
  if (int rc = mary_ensure_dyn_smem((const void*)scan_kernel<TI, NR4, DELTA, VEC, NT>, SM, &slots)) return rc;
  MARY_LAUNCH((scan_kernel<TI, NR4, DELTA, VEC, NT>), dim3((p.DV + COLS - 1) / COLS, p.H, S), NT, SM, s, p);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

template <typename TI, bool DELTA, bool VEC>
int dispatch(const ScanParams& p, int S, cudaStream_t s) {
  if (p.DK <= 32) return launch<TI, 1, DELTA, VEC>(p, S, s);
  if (p.DK <= 64) return launch<TI, 2, DELTA, VEC>(p, S, s);
  if (p.DK <= 128) return launch<TI, 4, DELTA, VEC>(p, S, s);
  return launch<TI, 8, DELTA, VEC>(p, S, s);
}

template <typename TI, bool DELTA>
int entry(const ScanParams& p, int S, cudaStream_t s) {
  constexpr int E = Pack<TI>::N;
  const bool vec = p.DK % E == 0 && p.DK % 4 == 0 && p.ldq % E == 0 && p.ldk % E == 0 && !(((uintptr_t)p.q | (uintptr_t)p.k | (uintptr_t)p.decay) & 15);
  return vec ? dispatch<TI, DELTA, true>(p, S, s) : dispatch<TI, DELTA, false>(p, S, s);
}

}  // namespace

// Pitch of a state column: the key width rounded up to whole 16-byte vectors.
MARY_API int mary_scan_state_pitch(int DK) { return (DK + 3) / 4 * 4; }

// q, k, v: bf16, or f32 when x_f32; the state [slots][H][DV][pitch] is updated in place.  S sequences, rows q_start[s] .. q_start[s+1].
MARY_API int mary_decay_scan(const void* q, const void* k, const void* v, const float* decay, float* out, float* state, const int* q_start,
                             const int* kv_len, const int* slots, int S, int64_t ldq, int64_t ldk, int64_t ldv, int H, int DK, int DV,
                             float q_scale, int x_f32, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (H < 1 || DK < 1 || DK > 256 || DV < 1 || S > 65535 || H > 65535) return MARY_ERR_BAD_ARG;
  ScanParams p = {q, k, v, decay, nullptr, out, state, q_start, kv_len, slots, ldq, ldk, ldv, H, 1, DK, DV, mary_scan_state_pitch(DK), q_scale};
  return x_f32 ? entry<float, false>(p, S, s) : entry<__nv_bfloat16, false>(p, S, s);
}

// f32 inputs; value head h reads query / key head h / (H / HK)
MARY_API int mary_delta_scan(const float* q, const float* k, const float* v, const float* decay, const float* beta, float* out, float* state,
                             const int* q_start, const int* kv_len, const int* slots, int S, int64_t ldq, int64_t ldk, int64_t ldv, int HK, int H,
                             int DK, int DV, float q_scale, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (HK < 1 || H < 1 || H % HK || DK < 1 || DK > 256 || DV < 1 || S > 65535 || H > 65535) return MARY_ERR_BAD_ARG;
  ScanParams p = {q, k, v, decay, beta, out, state, q_start, kv_len, slots, ldq, ldk, ldv, H, H / HK, DK, DV, mary_scan_state_pitch(DK), q_scale};
  return entry<float, true>(p, S, s);
}
