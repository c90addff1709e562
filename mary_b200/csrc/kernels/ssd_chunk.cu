// The recurrence of a Mamba-2 layer over the prompt portions of a batch, 64 tokens at a time on the tensor cores:
//
//   S_t = g_t S_{t-1} + dt_t B_t x_t^T,   y_t = S_t^T C_t + skip x_t,   g_t = exp(-exp(a_log) dt_t) per head
//
// With c_i = log g_1 + .. + log g_i inside a chunk,
//   y_i = exp(c_i) S_0^T C_i + sum_{j<=i} exp(c_i - c_j) dt_j (C_i . B_j) x_j + skip x_i,
//   S_64 = exp(c_64) S_0 + sum_j exp(c_64 - c_j) dt_j B_j x_j^T.
//
// x, B and C are bf16 (outputs of the short convolutions); step sizes, decays and the state are 32-bit.  A 32-bit operand of a tensor-core
// product (the decayed products, the state, the weighted x) goes in as the sum of two bf16 values, rounded value and rounding error, so it
// keeps 16 significant bits; sums and the carried state are 32-bit.  The logarithms c are summed in 64 bits and kept as two floats: their
// differences stay exact however small the decays have become.
//
// One CTA = (32 value channels, head, sequence), four warps = (16 channels) x (half of the state's rows).  The state lives transposed in
// the accumulator registers of mma.m16n8k16, [channel][state row]; read that way an accumulator IS the second operand of the product that
// reads the state, so it never leaves the registers between chunks.  C, B and x of the next chunk are in flight while this one is worked on.
#include "host_utils.h"
#include "recurrent.cuh"

using namespace mary;

namespace {

typedef __nv_bfloat16 bf16;
constexpr int L = 64, PC = 32, NTH = 128;

struct ChunkParams {
  const bf16* xbc;                       // [T][C]: x [H P], B [G N], C [G N]
  const float* dt; const float* c_hi; const float* c_lo;      // [H][T]; c: log2 of the decay since the start of the token's chunk
  const float* skip; float* y; float* state;
  const int* q_start; const int* kv_len; const int* slots;
  int T, G, H, N, P, C;
};

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp4(uint32_t dst, const void* src, bool in) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(in ? 4 : 0) : "memory");
}
// (a, b) as two bf16 pairs: rounded values and rounding errors
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 back = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - back.x, b - back.y);
  hi = *(const uint32_t*)&h;
  lo = *(const uint32_t*)&l;
}
// byte offset of a 16-byte piece in a tile whose rows have CH of them; rows are permuted so that eight rows of a column hit all banks
template <int CH> __device__ __forceinline__ uint32_t at(int row, int piece) {
  if constexpr (CH >= 8) return (uint32_t)(row * CH + (piece ^ (row & 7))) * 16;
  else return (uint32_t)(row * CH + (piece ^ ((row >> 1) & 3))) * 16;
}

template <int NP> struct Lay {
  static constexpr int TILE = L * NP * 2, X = L * PC * 2, M = L * L * 2;
  static constexpr int SC = 2 * TILE + X, STAGE = SC + 3 * L * 4;       // C, B, x, (dt, c_hi, c_lo)
  static constexpr int M_AT = 2 * STAGE, XW_AT = M_AT + 2 * M, Y_AT = XW_AT + 2 * X, BYTES = Y_AT + L * PC * 4;
};

template <int NP>
__global__ void __launch_bounds__(NTH) ssd_chunk_kernel(const ChunkParams p) {
  pdl_sync();
  using S = Lay<NP>;
  constexpr int CN = NP / 8, NH = NP / 2, NT = NH / 8;      // 16-byte pieces per row of B / C; state rows and 8-row tiles of a warp
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sm = smem_u32(smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pw = warp & 1, nw = warp >> 1;
  const int seq = blockIdx.z, h = blockIdx.y, p0 = blockIdx.x * PC, g = h / (p.H / p.G), inner = p.H * p.P;
  const int row0 = p.q_start[seq], n = p.q_start[seq + 1] - row0;
  if (n <= 0) return;
  const bool fresh = p.kv_len[seq] == n;
  const int NS = (p.N + 3) / 4 * 4;
  float* state = p.state + ((int64_t)p.slots[seq] * p.H + h) * p.P * NS;
  const int lr = lane >> 2, lc = (lane & 3) * 2;            // row and first column of an accumulator tile held by this lane
  // S^T: tile t = state rows nw NH + 8 t .., channels p0 + 16 pw ..
  float st[NT][4];
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int ch = p0 + pw * 16 + lr + 8 * e, r = nw * NH + t * 8 + lc;
      float2 v = make_float2(0.f, 0.f);
      if (!fresh && ch < p.P && r < p.N) v = *(const float2*)(state + (int64_t)ch * NS + r);
      st[t][2 * e] = v.x;
      st[t][2 * e + 1] = v.y;
    }
  const float skip = p.skip[h];

  auto load = [&](int c) {                                  // chunk c -> stage c & 1
    const uint32_t s = sm + (c & 1) * S::STAGE;
    const int t0 = c * L;
    for (int i = tid; i < L * CN; i += NTH) {
      const int r = i / CN, k = i % CN;
      const bool in = t0 + r < n && k * 8 < p.N;
      const bf16* src = p.xbc + (int64_t)(row0 + (in ? t0 + r : 0)) * p.C + inner + g * p.N + (in ? k * 8 : 0);
      cp16(s + at<CN>(r, k), src + p.G * p.N, in);          // C
      cp16(s + S::TILE + at<CN>(r, k), src, in);            // B
    }
    for (int i = tid; i < L * (PC / 8); i += NTH) {
      const int r = i / (PC / 8), k = i % (PC / 8);
      const bool in = t0 + r < n && p0 + k * 8 < p.P;
      cp16(s + 2 * S::TILE + at<PC / 8>(r, k), p.xbc + (int64_t)(row0 + (in ? t0 + r : 0)) * p.C + h * p.P + (in ? p0 + k * 8 : 0), in);
    }
    if (tid < L) {                                          // tokens past the end: no step, the decay of the last one
      const int64_t o = (int64_t)h * p.T + row0 + min(t0 + tid, n - 1);
      const uint32_t d = s + S::SC + tid * 4;
      cp4(d, p.dt + o, t0 + tid < n);
      cp4(d + L * 4, p.c_hi + o, true);
      cp4(d + 2 * L * 4, p.c_lo + o, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  const int chunks = (n + L - 1) / L;
  load(0);
  for (int c = 0; c < chunks; ++c) {
    if (c + 1 < chunks) {
      load(c + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int stage = (c & 1) * S::STAGE;
    const uint32_t sC = sm + stage, sB = sC + S::TILE, sX = sB + S::TILE, sM = sm + S::M_AT, sW = sm + S::XW_AT;
    const float* dt = (const float*)(smem + stage + S::SC);
    const float *hi = dt + L, *lo = hi + L;
    const float hiL = hi[L - 1], loL = lo[L - 1];
    // x weighted for the state update
    for (int i = tid; i < L * (PC / 8); i += NTH) {
      const int r = i / (PC / 8);
      const uint32_t o = at<PC / 8>(r, i % (PC / 8));
      const float w = exp2f((hiL - hi[r]) + (loL - lo[r])) * dt[r];
      float f[8];
      unpack16(*(const uint4*)(smem + stage + 2 * S::TILE + o), f);
      uint4 a, b;
      split2(f[0] * w, f[1] * w, a.x, b.x);
      split2(f[2] * w, f[3] * w, a.y, b.y);
      split2(f[4] * w, f[5] * w, a.z, b.z);
      split2(f[6] * w, f[7] * w, a.w, b.w);
      *(uint4*)(smem + S::XW_AT + o) = a;
      *(uint4*)(smem + S::XW_AT + S::X + o) = b;
    }
    // decayed products of the chunk's tokens: the ten 16 x 16 blocks on and below the diagonal, shared out over the warps
    {
      constexpr int MT[10] = {3, 3, 2, 2, 3, 3, 2, 1, 0, 1}, JT[10] = {0, 2, 0, 2, 1, 3, 1, 1, 0, 0};
#pragma unroll
      for (int b = 0; b < 10; ++b) {
        if ((b & 3) != warp) continue;
        const int mt = MT[b], jt = JT[b];
        float gm[2][4] = {};
#pragma unroll
        for (int k = 0; k < NP / 16; ++k) {
          uint32_t a[4], q[4];
          ldsm4(a, sC + at<CN>(mt * 16 + (lane & 15), 2 * k + (lane >> 4)));
          ldsm4(q, sB + at<CN>(jt * 16 + (lane & 7) + ((lane >> 4) << 3), 2 * k + ((lane >> 3) & 1)));
          mma(gm[0], a, q[0], q[1]);
          mma(gm[1], a, q[2], q[3]);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = mt * 16 + lr + 8 * e;
          const float hii = hi[i], loi = lo[i];
#pragma unroll
          for (int t = 0; t < 2; ++t) {
            const int j = jt * 16 + t * 8 + lc;
            float w[2];
#pragma unroll
            for (int d = 0; d < 2; ++d)
              w[d] = j + d <= i ? gm[t][2 * e + d] * (exp2f((hii - hi[j + d]) + (loi - lo[j + d])) * dt[j + d]) : 0.f;
            uint32_t vh, vl;
            split2(w[0], w[1], vh, vl);
            const uint32_t o = at<L / 8>(i, jt * 2 + t) + (lane & 3) * 4;
            *(uint32_t*)(smem + S::M_AT + o) = vh;
            *(uint32_t*)(smem + S::M_AT + S::M + o) = vl;
          }
        }
      }
    }
    // what the state before the chunk gives (this warp's half of its rows)
    float y[4][2][4];
#pragma unroll
    for (int mt = 0; mt < 4; ++mt)
#pragma unroll
      for (int o = 0; o < 2; ++o)
#pragma unroll
        for (int e = 0; e < 4; ++e) y[mt][o][e] = 0.f;
#pragma unroll
    for (int k = 0; k < NH / 16; ++k) {
      uint32_t bh[2][2], bl[2][2];                          // [channel octet][half of the k rows]
#pragma unroll
      for (int o = 0; o < 2; ++o)
#pragma unroll
        for (int t = 0; t < 2; ++t) split2(st[2 * k + t][2 * o], st[2 * k + t][2 * o + 1], bh[o][t], bl[o][t]);
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) {
        uint32_t a[4];
        ldsm4(a, sC + at<CN>(mt * 16 + (lane & 15), (nw * NH + k * 16) / 8 + (lane >> 4)));
#pragma unroll
        for (int o = 0; o < 2; ++o) {
          mma(y[mt][o], a, bh[o][0], bh[o][1]);
          mma(y[mt][o], a, bl[o][0], bl[o][1]);
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < 4; ++mt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = mt * 16 + lr + 8 * e;
        const float w = exp2f(hi[i] + lo[i]);
#pragma unroll
        for (int o = 0; o < 2; ++o) {
          y[mt][o][2 * e] *= w;
          y[mt][o][2 * e + 1] *= w;
        }
      }
    __syncthreads();
    // tokens of the chunk among themselves: token blocks 0 and 3 on the first pair of warps, 1 and 2 on the second
#pragma unroll
    for (int mt = 0; mt < 4; ++mt) {
      if ((mt == 0 || mt == 3) != (nw == 0)) continue;
#pragma unroll
      for (int k = 0; k <= mt; ++k) {
        uint32_t a[4], b[4], q[4];
        const uint32_t o = at<L / 8>(mt * 16 + (lane & 15), 2 * k + (lane >> 4));
        ldsm4(a, sM + o);
        ldsm4(b, sM + S::M + o);
        ldsm4t(q, sX + at<PC / 8>(k * 16 + (lane & 15), pw * 2 + (lane >> 4)));
        mma(y[mt][0], a, q[0], q[1]);
        mma(y[mt][1], a, q[2], q[3]);
        mma(y[mt][0], b, q[0], q[1]);
        mma(y[mt][1], b, q[2], q[3]);
      }
    }
    // the other half's token blocks to shared memory
    auto y_at = [&](int i, int o) { return (float2*)(smem + S::Y_AT) + i * (PC / 2) + ((pw * 8 + o * 4 + (lane & 3)) ^ ((i & 3) << 2)); };
#pragma unroll
    for (int mt = 0; mt < 4; ++mt)
      if ((mt < 2) != (nw == 0)) {
#pragma unroll
        for (int o = 0; o < 2; ++o)
#pragma unroll
          for (int e = 0; e < 2; ++e) *y_at(mt * 16 + lr + 8 * e, o) = make_float2(y[mt][o][2 * e], y[mt][o][2 * e + 1]);
      }
    // state update
    const float decay = exp2f(hiL + loL);
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) st[t][e] *= decay;
#pragma unroll
    for (int k = 0; k < L / 16; ++k) {
      uint32_t a[4], b[4];
      const uint32_t o = at<PC / 8>(k * 16 + (lane & 7) + ((lane >> 4) << 3), pw * 2 + ((lane >> 3) & 1));
      ldsm4t(a, sW + o);
      ldsm4t(b, sW + S::X + o);
#pragma unroll
      for (int t = 0; t < NT; t += 2) {
        uint32_t q[4];
        ldsm4t(q, sB + at<CN>(k * 16 + (lane & 15), nw * NT + t + (lane >> 4)));
        mma(st[t], a, q[0], q[1]);
        mma(st[t + 1], a, q[2], q[3]);
        mma(st[t], b, q[0], q[1]);
        mma(st[t + 1], b, q[2], q[3]);
      }
    }
    float2 x[2][2][2];
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int o = 0; o < 2; ++o)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          x[m][o][e] = __bfloat1622float2(*(const __nv_bfloat162*)(smem + stage + 2 * S::TILE +
                                                                   at<PC / 8>((nw * 2 + m) * 16 + lr + 8 * e, pw * 2 + o) + (lane & 3) * 4));
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < 4; ++mt) {
      if ((mt < 2) != (nw == 0)) {
        continue;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int i = mt * 16 + lr + 8 * e;
        if (c * L + i >= n) continue;
        float* dst = p.y + (int64_t)(row0 + c * L + i) * inner + h * p.P + p0 + pw * 16 + lc;
#pragma unroll
        for (int o = 0; o < 2; ++o) {
          const float2 v = *y_at(i, o), xv = x[mt & 1][o][e];
          if (p0 + pw * 16 + o * 8 < p.P)
            *(float2*)(dst + o * 8) = make_float2(fmaf(skip, xv.x, y[mt][o][2 * e] + v.x), fmaf(skip, xv.y, y[mt][o][2 * e + 1] + v.y));
        }
      }
    }
  }
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int ch = p0 + pw * 16 + lr + 8 * e, r = nw * NH + t * 8 + lc;
      if (ch < p.P && r < p.N) *(float2*)(state + (int64_t)ch * NS + r) = make_float2(st[t][2 * e], st[t][2 * e + 1]);
    }
}

// silu(conv(xbc) + bias) in bf16: a thread takes four channels of four tokens
template <int TAPS>
__global__ void __launch_bounds__(256) ss_conv_kernel(const bf16* __restrict__ xbc, int64_t ldx, const bf16* __restrict__ w, const bf16* __restrict__ bias,
                                                      const bf16* __restrict__ ring_all, const int* __restrict__ q_start, const int* __restrict__ kv_len,
                                                      const int* __restrict__ slots, bf16* __restrict__ out, int taps, int C) {
  pdl_sync();
  const int seq = blockIdx.z, blk = blockIdx.y, ch = (blockIdx.x * 256 + threadIdx.x) * 4;
  const int first = q_start[seq], end = q_start[seq + 1], rb = first + blk * 4;
  if (rb >= end || ch >= C) return;
  const int pos = kv_len[seq] - (end - first) + blk * 4;
  float y[4][4];
  conv_block<bf16, TAPS, 4>(xbc, ldx, w, bias, ring_all + (int64_t)slots[seq] * taps * C, taps, C, ch, rb, first, end, pos, y);
#pragma unroll
  for (int t = 0; t < 4; ++t)
    if (rb + t < end) store_e<bf16, 4>(out + (int64_t)(rb + t) * C + ch, y[t]);
}

// One thread per (chunk, head): step sizes and the summed logarithms of the decays, [H][T]
__global__ void __launch_bounds__(128) ss_decay_kernel(const bf16* __restrict__ dt_in, int64_t ldx, const float* __restrict__ dt_bias,
                                                       const float* __restrict__ a_log, const int* __restrict__ q_start, float* __restrict__ dt,
                                                       float* __restrict__ c_hi, float* __restrict__ c_lo, int H, int T) {
  pdl_sync();
  const int h = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.z;
  const int t0 = q_start[seq] + blockIdx.y * L, t1 = min(t0 + L, q_start[seq + 1]);
  if (h >= H || t0 >= t1) return;
  const float bias = dt_bias[h], a = -expf(a_log[h]);
  const int64_t o = (int64_t)h * T;
  double c = 0.0;
  for (int t = t0; t < t1; t += 8) {
    float raw[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) raw[i] = t + i < t1 ? __bfloat162float(dt_in[(int64_t)(t + i) * ldx + h]) : 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (t + i >= t1) break;
      const float d = softplus_x(raw[i] + bias);
      c += (double)(a * d) * 1.4426950408889634;
      const float ch = (float)c;
      dt[o + t + i] = d;
      c_hi[o + t + i] = ch;
      c_lo[o + t + i] = (float)(c - (double)ch);
    }
  }
}

template <int NP>
int launch_chunk(const ChunkParams& p, int S, cudaStream_t s) {
  static MarySmemSlots slots = {};
  if (int rc = mary_ensure_dyn_smem((const void*)ssd_chunk_kernel<NP>, Lay<NP>::BYTES, &slots)) return rc;
  MARY_LAUNCH((ssd_chunk_kernel<NP>), dim3((p.P + PC - 1) / PC, p.H, S), NTH, Lay<NP>::BYTES, s, p);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

}  // namespace

// bf16 models: xbc, dt_in columns of projection rows with pitch ldx; results xbc_out [T, C] bf16 and dt, c_hi, c_lo [H, T] f32 as
// mary_ssd_chunk takes them.  S sequences of at most max_q rows each.
MARY_API int mary_ss_conv_decay(const void* xbc, int64_t ldx, const void* taps_w, const void* taps_b, const void* ring, const void* dt_in,
                                const float* dt_bias, const float* a_log, const int* q_start, const int* kv_len, const int* slots, void* xbc_out,
                                float* dt, float* c_hi, float* c_lo, int S, int max_q, int T, int H, int C, int taps, cudaStream_t s) {
  if (S <= 0 || max_q <= 0) return MARY_OK;
  if (H < 1 || C < 1 || C % 4 || ldx % 4 || taps < 1 || S > 65535 || (((uintptr_t)xbc | (uintptr_t)ring | (uintptr_t)taps_w | (uintptr_t)xbc_out) & 7))
    return MARY_ERR_BAD_ARG;
  if ((max_q + 3) / 4 > 65535) return MARY_ERR_BAD_ARG;
  const dim3 grid((C / 4 + 255) / 256, (max_q + 3) / 4, S);
  auto fn = taps == 4 ? ss_conv_kernel<4> : ss_conv_kernel<0>;
  MARY_LAUNCH(fn, grid, 256, 0, s, (const bf16*)xbc, ldx, (const bf16*)taps_w, (const bf16*)taps_b, (const bf16*)ring, q_start, kv_len, slots,
              (bf16*)xbc_out, taps, C);
  MARY_LAUNCH(ss_decay_kernel, dim3((H + 127) / 128, (max_q + L - 1) / L, S), 128, 0, s, (const bf16*)dt_in, ldx, dt_bias, a_log, q_start, dt, c_hi, c_lo,
              H, T);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_ssd_chunk_supported(int N, int P) { return N >= 8 && N <= 256 && N % 8 == 0 && P >= 8 && P % 8 == 0; }

// y [T, H P] f32; the state [slots][H][P][N] is read (zero for a portion that starts its sequence) and updated in place.
MARY_API int mary_ssd_chunk(const void* xbc, const float* dt, const float* c_hi, const float* c_lo, const float* skip, float* y, float* state,
                            const int* q_start, const int* kv_len, const int* slots, int S, int T, int G, int H, int N, int P, cudaStream_t s) {
  if (S <= 0 || T <= 0) return MARY_OK;
  if (G < 1 || H < 1 || H % G || H > 65535 || S > 65535 || !mary_ssd_chunk_supported(N, P) || ((uintptr_t)xbc & 15)) return MARY_ERR_BAD_ARG;
  const ChunkParams p = {(const bf16*)xbc, dt, c_hi, c_lo, skip, y, state, q_start, kv_len, slots, T, G, H, N, P, H * P + 2 * G * N};
  if (N <= 64) return launch_chunk<64>(p, S, s);
  if (N <= 128) return launch_chunk<128>(p, S, s);
  return launch_chunk<256>(p, S, s);
}
