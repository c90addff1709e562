// Linear recurrences over the tokens of a batch, with the state in 32-bit registers:
//
//   decayed linear attention   S_t = diag(a_t) S_{t-1} + k_t v_t^T                       o_t = S_t^T q_t    (a decay per key channel)
//   decay per head             S_t = g_t S_{t-1} + b_t k_t v_t^T                         o_t = S_t^T q_t + skip v_t
//   gated delta rule           S' = g_t S_{t-1};  u_t = b_t (v_t - S'^T k_t);  S_t = S' + k_t u_t^T;  o_t = S_t^T q_t   (a decay per head)
//
// The columns of S (one per value channel) are independent, so the grid is (column block, head, sequence) and every CTA walks the
// tokens of its sequence's portion.  16 or 32 lanes share four columns: each lane holds NR4 float4 of key rows of all four, so a key or
// query value read from shared memory serves four columns (one read per multiply-add would saturate the shared-memory port), and the
// multiply-adds are issued in pairs (fma.rn.f32x2).  The state is read from and returned to the sequence's slot, stored column by
// column, [slot][head][value channel][key channel padded to 4], and taken as zero when the portion starts at position 0.  Tokens are
// staged eight at a time in shared memory, the next eight already in flight in registers; a thread always stages the same token of the
// eight and the same channels, through pointers that advance by eight rows.
//
// The delta rule's read S'^T k_t depends on the previous write, a chain of reductions over the lanes per token.  Four tokens at a
// time are therefore resolved against the state before them: with w_ij = g_{j+1} .. g_i and G_i = g_1 .. g_i,
//   u_i = b_i (v_i - G_i S_0^T k_i - sum_{j<i} w_ij (k_j . k_i) u_j),   o_i = G_i S_0^T q_i + sum_{j<=i} w_ij (k_j . q_i) u_j,
//   S_4 = G_4 S_0 + sum_j w_4j k_j u_j^T,
// which needs one round of reductions per four tokens; the products k.k and k.q do not depend on the column and are precomputed
// (mary_delta_prep).  A decay per head without the delta rule is the same with u_i = b_i v_i: half the reads, no chain.  The weights w are products of decays, never quotients, so a decay of zero is exact.
#include "host_utils.h"
#include "recurrent.cuh"

using namespace mary;

namespace {

constexpr int CT = 8;          // tokens per staged chunk
constexpr int CN = 4;          // columns per group of lanes

typedef unsigned long long f2;            // two packed f32
__device__ __forceinline__ f2 pack2(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float sum2(f2 v) {
  float a, b;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
  return a + b;
}
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

struct ScanParams {
  const void* q; const void* k; const void* v;      // token rows of ldq / ldk / ldv elements; q, k head h / rep, v head h
  const float* decay;                               // [T, H * DK] per channel (lda floats between tokens; 0: the same for all), or [T, H] per head
  const float* beta;                                // [T, H] (decay per head, delta rule)
  const float* pairs;                               // [T, HK, 8] (delta rule): k_j . k_i and k_j . q_i of the row's block of four;
                                                    // [T, HK, 4] (decay per head): k_j . q_i
  const float* skip;                                // [H] (decay per head)
  float* out;                                       // [T, H * DV]
  float* state;                                     // [slots][H][DV][DKS]
  const int* q_start; const int* kv_len; const int* slots;
  int64_t ldq, ldk, ldv, lda;
  int H, HK, rep, DK, DV, DKS;
  float q_scale;
};

template <typename TI, int E> struct Reg { uint4 v; };             // one 16-byte vector
template <typename TI> struct Reg<TI, 1> { TI v; };

// LN lanes share a group of CN columns: 16, or 32 when the grid is small.
template <typename TI, int NR4, int MODE, bool VEC, int NT, int LN>
__global__ void __launch_bounds__(NT) scan_kernel(const ScanParams p) {
  pdl_sync();
  constexpr bool BLOCKS = MODE != DECAY_CHANNEL, DELTA = MODE == DECAY_DELTA;
  constexpr int COLS = NT / LN * CN, DKP = NR4 * LN * 4;
  constexpr int TPT = NT / CT;                                     // staging threads per token
  constexpr int E = VEC ? Pack<TI>::N : 1, NVQ = (DKP / E + TPT - 1) / TPT;
  constexpr int EA = VEC ? 4 : 1, NVA = BLOCKS ? 1 : (DKP / EA + TPT - 1) / TPT;
  constexpr int NVV = COLS / TPT;
  typedef float Rows[CT][DKP];
  extern __shared__ __align__(16) float sm[];
  Rows *sq = (Rows*)sm, *sk = sq + 2, *sa = sk + 2;            // two buffers each; sa for channel decays only
  __shared__ __align__(16) float sv[2][CT][COLS];
  __shared__ __align__(16) float s_kk[2][CT][4], s_kq[2][CT][4], s_row[2][CT][4];      // weighted products; (G, suffix decay, beta, -) of a token
  const int tid = threadIdx.x, lane = tid & 31, ln = tid & (LN - 1);
  const int seq = blockIdx.z, h = blockIdx.y, hk = h / p.rep;
  const int gcol = tid / LN * CN, col0 = blockIdx.x * COLS + gcol;
  const int row0 = p.q_start[seq], n = p.q_start[seq + 1] - row0;
  if (n <= 0) return;
  const bool fresh = p.kv_len[seq] == n;
  float* sp = p.state + (((int64_t)p.slots[seq] * p.H + h) * p.DV + col0) * p.DKS;
  f2 st[CN][NR4][2];
#pragma unroll
  for (int c = 0; c < CN; ++c)
#pragma unroll
    for (int r = 0; r < NR4; ++r) {
      const int row = (r * LN + ln) * 4;
      ulonglong2 v = make_ulonglong2(0ull, 0ull);
      if (!fresh && col0 + c < p.DV && row < p.DKS) v = *(const ulonglong2*)(sp + (int64_t)c * p.DKS + row);
      st[c][r][0] = v.x; st[c][r][1] = v.y;
    }
  if (p.DK < DKP) {                       // channels beyond DK stay zero in both buffers
    for (int i = tid; i < (BLOCKS ? 4 : 6) * CT * DKP; i += NT) sm[i] = 0.f;
    __syncthreads();
  }
  // staging: this thread's token of a chunk and its channels
  const int my_t = tid / TPT, my_c = tid % TPT;
  const TI* qp = (const TI*)p.q + (int64_t)(row0 + my_t) * p.ldq + (int64_t)hk * p.DK + my_c * E;
  const TI* kp = (const TI*)p.k + (int64_t)(row0 + my_t) * p.ldk + (int64_t)hk * p.DK + my_c * E;
  const TI* vp = (const TI*)p.v + (int64_t)(row0 + my_t) * p.ldv + (int64_t)h * p.DV + blockIdx.x * COLS + my_c;
  const float* ap = BLOCKS ? p.decay + (int64_t)(row0 + lane) * p.H + h : p.decay + (int64_t)(row0 + my_t) * p.lda + (int64_t)h * p.DK + my_c * EA;
  const float* bp = BLOCKS ? p.beta + (int64_t)(row0 + lane) * p.H + h : nullptr;
  constexpr int NP = DELTA ? 2 : 1;
  const float4* pp = BLOCKS ? (const float4*)p.pairs + ((int64_t)(row0 + lane) * p.HK + hk) * NP : nullptr;
  const float skip = MODE == DECAY_HEAD ? p.skip[h] : 0.f;
  const int64_t step_q = CT * p.ldq, step_k = CT * p.ldk, step_v = CT * p.ldv, step_a = CT * (BLOCKS ? (int64_t)p.H : p.lda);
  const int ch_left = p.DK - my_c * E, ch_left_a = p.DK - my_c * EA, col_left = p.DV - blockIdx.x * COLS - my_c;

  Reg<TI, E> rq[NVQ], rk[NVQ];
  Reg<float, EA> ra[NVA];
  TI rv[NVV];
  float rg = 1.f, rb = 0.f;
  float4 rkk = make_float4(0.f, 0.f, 0.f, 0.f), rkq = rkk;
  auto fetch = [&](int t0) {             // the chunk at t0 (called for every chunk in order)
    const bool in = t0 + my_t < n;
#pragma unroll
    for (int i = 0; i < NVQ; ++i) {
      rq[i] = {}; rk[i] = {};
      if (in && i * TPT * E < ch_left) {
        rq[i].v = *(const decltype(rq[i].v)*)(qp + i * TPT * E);
        rk[i].v = *(const decltype(rk[i].v)*)(kp + i * TPT * E);
      }
    }
#pragma unroll
    for (int i = 0; i < NVV; ++i) rv[i] = (in && i * TPT < col_left) ? vp[i * TPT] : from_f<TI>(0.f);
    if constexpr (!BLOCKS) {
#pragma unroll
      for (int i = 0; i < NVA; ++i) {
        if (in && i * TPT * EA < ch_left_a) ra[i].v = *(const decltype(ra[i].v)*)(ap + i * TPT * EA);
        else if constexpr (VEC) ra[i].v = make_uint4(0x3f800000u, 0x3f800000u, 0x3f800000u, 0x3f800000u);
        else ra[i].v = 1.f;
      }
    } else if (tid < CT) {
      const bool mine = t0 + tid < n;
      rg = mine ? *ap : 1.f;
      rb = mine ? *bp : 0.f;
      if constexpr (DELTA) rkk = mine ? pp[0] : make_float4(0.f, 0.f, 0.f, 0.f);
      rkq = mine ? pp[NP - 1] : make_float4(0.f, 0.f, 0.f, 0.f);
      bp += step_a;
      pp += CT * p.HK * NP;
    }
    qp += step_q; kp += step_k; vp += step_v; ap += step_a;
  };
  auto stash = [&](int b) {
#pragma unroll
    for (int i = 0; i < NVQ; ++i) {
      if (i * TPT * E < ch_left) {
        const int c = (my_c + i * TPT) * E;
        if constexpr (VEC) {
          float fq[E], fk[E];
          unpack16(rq[i].v, fq);
          unpack16(rk[i].v, fk);
#pragma unroll
          for (int j = 0; j < E; j += 4) {
            *(float4*)&sq[b][my_t][c + j] = make_float4(fq[j] * p.q_scale, fq[j + 1] * p.q_scale, fq[j + 2] * p.q_scale, fq[j + 3] * p.q_scale);
            *(float4*)&sk[b][my_t][c + j] = make_float4(fk[j], fk[j + 1], fk[j + 2], fk[j + 3]);
          }
        } else {
          sq[b][my_t][c] = to_f<TI>(rq[i].v) * p.q_scale;
          sk[b][my_t][c] = to_f<TI>(rk[i].v);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NVV; ++i) sv[b][my_t][my_c + i * TPT] = to_f<TI>(rv[i]);
    if constexpr (!BLOCKS) {
#pragma unroll
      for (int i = 0; i < NVA; ++i) {
        if (i * TPT * EA < ch_left_a) {
          const int c = (my_c + i * TPT) * EA;
          if constexpr (VEC) *(uint4*)&sa[b][my_t][c] = ra[i].v;
          else sa[b][my_t][c] = ra[i].v;
        }
      }
    } else if (tid < 32) {
      // lane t < 8: row t % 4 of its block of four; decays of the block by shuffles
      float g[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) g[j] = __shfl_sync(0xffffffffu, rg, (lane & 4) | j);
      const int i = lane & 3;
      float w[4], G = 1.f, suffix = 1.f;            // w[j] = g_{j+1} .. g_i
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        w[j] = 1.f;
#pragma unroll
        for (int l = 0; l < 4; ++l)
          if (l > j && l <= i) w[j] *= g[l];
        if (j <= i) G *= g[j];
        else suffix *= g[j];
      }
      if (lane < CT) {
        if constexpr (DELTA) *(float4*)s_kk[b][lane] = make_float4(w[0] * rkk.x, w[1] * rkk.y, w[2] * rkk.z, w[3] * rkk.w);
        *(float4*)s_kq[b][lane] = make_float4(w[0] * rkq.x * p.q_scale, w[1] * rkq.y * p.q_scale, w[2] * rkq.z * p.q_scale, w[3] * rkq.w * p.q_scale);
        *(float4*)s_row[b][lane] = make_float4(G, suffix, rb, 0.f);
      }
    }
  };

  fetch(0);
  stash(0);
  __syncthreads();
  for (int t0 = 0, b = 0; t0 < n; t0 += CT, b ^= 1) {
    const bool more = t0 + CT < n;
    if (more) fetch(t0 + CT);
    if constexpr (!BLOCKS) {
      float o[CT * CN];                              // index token * 4 + column
#pragma unroll
      for (int t = 0; t < CT; ++t) {
        const float4 v4 = *(const float4*)&sv[b][t][gcol];
        const f2 vv[CN] = {pack2(v4.x, v4.x), pack2(v4.y, v4.y), pack2(v4.z, v4.z), pack2(v4.w, v4.w)};
        f2 acc[CN] = {0ull, 0ull, 0ull, 0ull};
#pragma unroll
        for (int r = 0; r < NR4; ++r) {
          const int row = (r * LN + ln) * 4;
          const ulonglong2 a = *(const ulonglong2*)&sa[b][t][row], k = *(const ulonglong2*)&sk[b][t][row], q = *(const ulonglong2*)&sq[b][t][row];
#pragma unroll
          for (int c = 0; c < CN; ++c) {
            st[c][r][0] = fma2(k.x, vv[c], mul2(a.x, st[c][r][0]));
            st[c][r][1] = fma2(k.y, vv[c], mul2(a.y, st[c][r][1]));
            acc[c] = fma2(q.x, st[c][r][0], acc[c]);
            acc[c] = fma2(q.y, st[c][r][1], acc[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < CN; ++c) o[t * CN + c] = sum2(acc[c]);
      }
      halve<32>(o, lane, LN / 2);
      halve<16>(o, lane, LN / 4);
      halve<8>(o, lane, LN / 8);
      halve<4>(o, lane, LN / 16);
      if constexpr (LN == 32) halve<2>(o, lane, 1);
      // LN = 16: the lane holds token l / 2, columns 2 (l % 2) and the next; LN = 32: token l / 4, column l % 4
      const int t = t0 + ln / (LN / 8), c = col0 + (LN == 32 ? ln & 3 : (ln & 1) * 2);
      if (t < n) {
        float* dst = p.out + ((int64_t)(row0 + t) * p.H + h) * p.DV + c;
        if (c < p.DV) dst[0] = o[0];
        if (LN == 16 && c + 1 < p.DV) dst[1] = o[1];
      }
    } else {
#pragma unroll
      for (int blk = 0; blk < 2; ++blk) {
        const int tb = blk * 4, my_col = ln / (LN / 4);
        constexpr int ND = DELTA ? 8 : 4;            // S_0^T k_0 .. k_3 (delta rule), S_0^T q_0 .. q_3
        float d[CN * ND];                            // index column * ND + product
        {
          f2 acc[CN][ND];
#pragma unroll
          for (int c = 0; c < CN; ++c)
#pragma unroll
            for (int i = 0; i < ND; ++i) acc[c][i] = 0ull;
#pragma unroll
          for (int r = 0; r < NR4; ++r) {
            const int row = (r * LN + ln) * 4;
#pragma unroll
            for (int i = 0; i < ND; ++i) {
              const ulonglong2 x = *(const ulonglong2*)(i < ND - 4 ? &sk[b][tb + i][row] : &sq[b][tb + i - (ND - 4)][row]);
#pragma unroll
              for (int c = 0; c < CN; ++c) acc[c][i] = fma2(x.y, st[c][r][1], fma2(x.x, st[c][r][0], acc[c][i]));
            }
          }
#pragma unroll
          for (int c = 0; c < CN; ++c)
#pragma unroll
            for (int i = 0; i < ND; ++i) d[c * ND + i] = sum2(acc[c][i]);
        }
        halve<CN * ND>(d, lane, LN / 2);
        halve<CN * ND / 2>(d, lane, LN / 4);         // the lane's column is my_col
#pragma unroll
        for (int bit = LN / 8; bit >= 1; bit >>= 1)
#pragma unroll
          for (int i = 0; i < ND; ++i) d[i] += __shfl_xor_sync(0xffffffffu, d[i], bit);
        float u[4], mine = 0.f, G4 = 1.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 row = *(const float4*)s_row[b][tb + i];
          const float4 kq = *(const float4*)s_kq[b][tb + i];
          const float kqv[4] = {kq.x, kq.y, kq.z, kq.w};
          const float vt = sv[b][tb + i][gcol + my_col];
          float oi = row.x * d[ND - 4 + i];
          if constexpr (DELTA) {
            const float4 kk = *(const float4*)s_kk[b][tb + i];
            const float kkv[4] = {kk.x, kk.y, kk.z, kk.w};
            float pred = row.x * d[i];
#pragma unroll
            for (int j = 0; j < i; ++j) pred = fmaf(kkv[j], u[j], pred);
            u[i] = row.z * (vt - pred);
          } else {
            u[i] = row.z * vt;
            oi = fmaf(skip, vt, oi);
          }
#pragma unroll
          for (int j = 0; j <= i; ++j) oi = fmaf(kqv[j], u[j], oi);
          if ((ln & 3) == i) mine = oi;
          if (i == 3) G4 = row.x;
        }
        const int t = t0 + tb + (ln & 3), c_mine = col0 + my_col;
        if (t < n && c_mine < p.DV && (LN == 16 || !(ln & 4))) p.out[((int64_t)(row0 + t) * p.H + h) * p.DV + c_mine] = mine;
#pragma unroll
        for (int j = 0; j < 3; ++j) u[j] *= s_row[b][tb + j][1];
        f2 uu[CN][4];
#pragma unroll
        for (int c = 0; c < CN; ++c)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float x = __shfl_sync(0xffffffffu, u[j], (lane & ~(LN - 1)) | (c * (LN / 4)) | (ln & (LN / 4 - 1)));
            uu[c][j] = pack2(x, x);
          }
        const f2 gg = pack2(G4, G4);
#pragma unroll
        for (int r = 0; r < NR4; ++r) {
          const int row = (r * LN + ln) * 4;
          ulonglong2 k[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) k[j] = *(const ulonglong2*)&sk[b][tb + j][row];
#pragma unroll
          for (int c = 0; c < CN; ++c) {
            st[c][r][0] = mul2(gg, st[c][r][0]);
            st[c][r][1] = mul2(gg, st[c][r][1]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              st[c][r][0] = fma2(k[j].x, uu[c][j], st[c][r][0]);
              st[c][r][1] = fma2(k[j].y, uu[c][j], st[c][r][1]);
            }
          }
        }
      }
    }
    if (more) stash(b ^ 1);
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < CN; ++c)
    if (col0 + c < p.DV) {
#pragma unroll
      for (int r = 0; r < NR4; ++r) {
        const int row = (r * LN + ln) * 4;
        if (row < p.DKS) *(ulonglong2*)(sp + (int64_t)c * p.DKS + row) = make_ulonglong2(st[c][r][0], st[c][r][1]);
      }
    }
}

template <typename TI, int NR4, int MODE, bool VEC, int LN>
int launch(const ScanParams& p, int S, cudaStream_t s) {
  constexpr int NT = (MODE == DECAY_CHANNEL ? 4 : 8) * LN, COLS = NT / LN * CN;
  constexpr size_t SM = (size_t)(MODE == DECAY_CHANNEL ? 6 : 4) * CT * NR4 * LN * 4 * 4;
  static MarySmemSlots slots = {};
  if (int rc = mary_ensure_dyn_smem((const void*)scan_kernel<TI, NR4, MODE, VEC, NT, LN>, SM, &slots)) return rc;
  MARY_LAUNCH((scan_kernel<TI, NR4, MODE, VEC, NT, LN>), dim3((p.DV + COLS - 1) / COLS, p.H, S), NT, SM, s, p);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

template <typename TI, int MODE, bool VEC>
int dispatch(const ScanParams& p, int S, cudaStream_t s) {
  if constexpr (MODE == DECAY_CHANNEL) {
    // twice the warps per column where 16 lanes would leave most of the machine without work (the delta rule loses more to the longer
    // reductions than it gains: 924 against 763 us for 4096 tokens of 32 heads)
    if (p.DK > 64 && (int64_t)((p.DV + 15) / 16) * p.H * S <= 3 * mary_num_sms())
      return p.DK <= 128 ? launch<TI, 1, MODE, VEC, 32>(p, S, s) : launch<TI, 2, MODE, VEC, 32>(p, S, s);
  }
  if (p.DK <= 64) return launch<TI, 1, MODE, VEC, 16>(p, S, s);
  if (p.DK <= 128) return launch<TI, 2, MODE, VEC, 16>(p, S, s);
  return launch<TI, 4, MODE, VEC, 16>(p, S, s);
}

template <typename TI, int MODE>
int entry(const ScanParams& p, int S, cudaStream_t s) {
  constexpr int E = Pack<TI>::N;
  const bool vec = p.DK % E == 0 && p.DK % 4 == 0 && p.ldq % E == 0 && p.ldk % E == 0 && p.lda % 4 == 0 && !(((uintptr_t)p.q | (uintptr_t)p.k | (uintptr_t)p.decay) & 15);
  return vec ? dispatch<TI, MODE, true>(p, S, s) : dispatch<TI, MODE, false>(p, S, s);
}

}  // namespace

// q, k, v: bf16, or f32 when x_f32; decay [T] rows of lda floats (0: one row for all tokens); the state [slots][H][DV][DK rounded up to 4] is updated in place.  S sequences, rows
// q_start[s] .. q_start[s+1].
MARY_API int mary_decay_scan(const void* q, const void* k, const void* v, const float* decay, int64_t lda, float* out, float* state, const int* q_start,
                             const int* kv_len, const int* slots, int S, int64_t ldq, int64_t ldk, int64_t ldv, int H, int DK, int DV,
                             float q_scale, int x_f32, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (H < 1 || DK < 1 || DK > 256 || DV < 1 || S > 65535 || H > 65535) return MARY_ERR_BAD_ARG;
  ScanParams p = {q, k, v, decay, nullptr, nullptr, nullptr, out, state, q_start, kv_len, slots, ldq, ldk, ldv, lda, H, H, 1, DK, DV, (DK + 3) / 4 * 4, q_scale};
  return x_f32 ? entry<float, DECAY_CHANNEL>(p, S, s) : entry<__nv_bfloat16, DECAY_CHANNEL>(p, S, s);
}

// f32 inputs; value head h reads query / key head h / (H / HK).  pairs [T, HK, 8]: for row i of a block of four tokens (counted from the
// first row of its sequence) k_j . k_i for j = 0 .. 3 (used for j < i) and k_j . q_i (used for j <= i).
MARY_API int mary_delta_scan(const float* q, const float* k, const float* v, const float* decay, const float* beta, const float* pairs, float* out,
                             float* state, const int* q_start, const int* kv_len, const int* slots, int S, int64_t ldq, int64_t ldk, int64_t ldv,
                             int HK, int H, int DK, int DV, float q_scale, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (HK < 1 || H < 1 || H % HK || DK < 1 || DK > 256 || DV < 1 || S > 65535 || H > 65535 || ((uintptr_t)pairs & 15)) return MARY_ERR_BAD_ARG;
  ScanParams p = {q, k, v, decay, beta, pairs, nullptr, out, state, q_start, kv_len, slots, ldq, ldk, ldv, 0, H, HK, H / HK, DK, DV, (DK + 3) / 4 * 4, q_scale};
  return entry<float, DECAY_DELTA>(p, S, s);
}

// f32 inputs; head h reads q / k of group h / (H / G).  pairs [T, G, 4]: k_j . q_i of the row's block of four tokens (used for j <= i);
// out = S^T q + skip v.
MARY_API int mary_head_decay_scan(const float* q, const float* k, const float* v, const float* decay, const float* beta, const float* pairs,
                                  const float* skip, float* out, float* state, const int* q_start, const int* kv_len, const int* slots, int S,
                                  int64_t ldq, int64_t ldk, int64_t ldv, int G, int H, int DK, int DV, cudaStream_t s) {
  if (S <= 0) return MARY_OK;
  if (G < 1 || H < 1 || H % G || DK < 1 || DK > 256 || DV < 1 || S > 65535 || H > 65535 || ((uintptr_t)pairs & 15)) return MARY_ERR_BAD_ARG;
  ScanParams p = {q, k, v, decay, beta, pairs, skip, out, state, q_start, kv_len, slots, ldq, ldk, ldv, 0, H, G, H / G, DK, DV, (DK + 3) / 4 * 4, 1.f};
  return entry<float, DECAY_HEAD>(p, S, s);
}
