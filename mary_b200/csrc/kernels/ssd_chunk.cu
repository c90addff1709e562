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
// The products C_i . B_j of a chunk are the same for every head of a group and come from a kernel of their own (gram).  One CTA of the
// recurrence = (32 value channels, head, sequence), eight warps = (16 channels) x (a quarter of the state's rows).  The state lives
// transposed in the accumulator registers of mma.m16n8k16, [channel][state row]; read that way an accumulator IS the second operand of the
// product that reads the state, so it never leaves the registers between chunks.  C, B and x of the next chunk are in flight while this
// one is worked on.  Rows in shared memory are padded by 16 bytes, so the eight rows of a fragment fall on different banks and every
// address of a loop is a base and a constant.
//
// Where heads and sequences leave most of the machine without work, a sequence is cut into segments of whole chunks: a first pass takes every
// segment but the last through the state update alone, from a state of zero, and the pass proper starts each segment from what the earlier
// ones left, S <- d S + E with a segment's end state E and its whole decay d.
#include "host_utils.h"
#include "typed.cuh"

using namespace mary;

namespace {

typedef __nv_bfloat16 bf16;
constexpr int L = 64, PC = 32, NTH = 256;

struct ChunkParams {
  const bf16* xbc;                       // [T][C]: x [H P], B [G N], C [G N]
  const float* dt; const float* c_hi; const float* c_lo;      // [H][T]; c: log2 of the decay since the start of the token's chunk
  const float* skip; float* y; float* state;
  float4* gram;                          // [chunk][G][10 blocks][2][32 lanes]: C_i . B_j as a lane's accumulators of two 16 x 8 tiles
  const int* q_start; const int* kv_len; const int* slots;
  int T, G, H, N, P;
  int64_t C;                             // elements between the rows of two tokens
  int segs;                              // segments per sequence
  float* seg_state;                      // segs > 1: [S][segs][H][P][NS]: the state before the portion, then the end states of segments 0 .. segs - 2
  float* seg_log;                        // [S][segs][H]: log2 of the decay over segment 0 .. segs - 2
  int per_head;                          // 1: decays that are the same for all tokens, dt, c_hi and c_lo [H][64] by place in the chunk
};

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t a) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mma_first(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {      // d = a b
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%10, %10, %10, %10};"
      : "=f"(d[0]), "=f"(d[1]), "=f"(d[2]), "=f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1), "f"(0.f));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp4(uint32_t dst, const void* src, bool in) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(in ? 4 : 0) : "memory");
}
__device__ __forceinline__ float pow2(float x) {            // x <= 0
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
// (a, b) as two bf16 pairs: rounded values and rounding errors
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 back = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - back.x, b - back.y);
  hi = *(const uint32_t*)&h;
  lo = *(const uint32_t*)&l;
}
// the ten 16 x 16 blocks on and below the diagonal of a chunk's 64 x 64 token pairs
__device__ __forceinline__ int blk_m(int b) { return b < 4 ? 3 : b < 7 ? 2 : b < 9 ? 1 : 0; }
__device__ __forceinline__ int blk_j(int b) { return b < 4 ? b : b < 7 ? b - 4 : b < 9 ? b - 7 : 0; }
// chunk c of a sequence whose rows start at row0: a place of its own among T / 64 + sequences places
__device__ __forceinline__ int64_t chunk_place(int row0, int seq, int c) { return row0 / L + seq + c; }

template <int NP> struct Lay {
  static constexpr int ROW = NP * 2 + 16, XROW = PC * 2 + 16, MROW = L * 2 + 16;        // bytes
  static constexpr int TILE = L * ROW, X = L * XROW, M = L * MROW;
  static constexpr int SC = 2 * TILE + X, STAGE = SC + 3 * L * 4;       // C, B, x, (dt, c_hi, c_lo)
  static constexpr int M_AT = 2 * STAGE, XW_AT = M_AT + 2 * M;
  static constexpr int Y_AT = M_AT, Y = L * PC * 4;                     // four partial results, over what the products have read by then
  static constexpr int BYTES = M_AT + 4 * Y;
  static_assert(2 * M + 2 * X <= 4 * Y, "the decayed products and the weighted x fit");
};

// 64 rows of B (and of C: WITH_C), THREADS threads; src: this thread's first piece of B.  Rows past `rows` and state rows past N are zero.
template <int NP, int THREADS, bool WITH_C = true>
__device__ __forceinline__ void load_bc(uint32_t dst_c, uint32_t dst_b, const bf16* src, int64_t ld, int c_off, bool col, int rows) {
  constexpr int CN = NP / 8, STEP = THREADS / CN;
  const int r0 = threadIdx.x / CN, k = threadIdx.x % CN;
  const uint32_t o = r0 * Lay<NP>::ROW + k * 16;
  const bf16* s = src;
#pragma unroll
  for (int i = 0; i < L / STEP; ++i) {
    const bool in = col && r0 + i * STEP < rows;
    if constexpr (WITH_C) cp16(dst_c + o + i * STEP * Lay<NP>::ROW, in ? s + c_off : src, in);
    cp16(dst_b + o + i * STEP * Lay<NP>::ROW, in ? s : src, in);
    s += STEP * ld;
  }
}
template <int NP, int THREADS> __device__ __forceinline__ const bf16* first_piece(const bf16* row, int64_t ld, int N) {
  constexpr int CN = NP / 8;
  const int k = threadIdx.x % CN;
  return row + (k * 8 < N ? (int64_t)(threadIdx.x / CN) * ld + k * 8 : 0);
}

template <int NP>
__global__ void __launch_bounds__(128) ssd_gram_kernel(const ChunkParams p) {
  pdl_sync();
  using S = Lay<NP>;
  extern __shared__ __align__(128) uint8_t smem[];
  const int seq = blockIdx.z, g = blockIdx.y, c = blockIdx.x, lane = threadIdx.x & 31;
  const int row0 = p.q_start[seq], n = p.q_start[seq + 1] - row0;
  if (c * L >= n) return;
  const uint32_t sC = smem_u32(smem), sB = sC + S::TILE;
  const bf16* row = p.xbc + (int64_t)(row0 + c * L) * p.C + p.H * p.P + g * p.N;
  const bool in = (int)(threadIdx.x / (NP / 8)) < n - c * L;
  load_bc<NP, 128>(sC, sB, in ? first_piece<NP, 128>(row, p.C, p.N) : row, p.C, p.G * p.N, (threadIdx.x % (NP / 8)) * 8 < p.N, n - c * L);
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  for (int b = threadIdx.x >> 5; b < 10; b += 4) {
    float gm[2][4] = {};
    const uint32_t ac = sC + (blk_m(b) * 16 + (lane & 15)) * S::ROW + (lane >> 4) * 16;
    const uint32_t bc = sB + (blk_j(b) * 16 + (lane & 7) + ((lane >> 4) << 3)) * S::ROW + ((lane >> 3) & 1) * 16;
#pragma unroll
    for (int k = 0; k < NP / 16; ++k) {
      uint32_t a[4], q[4];
      ldsm4(a, ac + k * 32);
      ldsm4(q, bc + k * 32);
      mma(gm[0], a, q[0], q[1]);
      mma(gm[1], a, q[2], q[3]);
    }
    float4* dst = p.gram + ((chunk_place(row0, seq, c) * p.G + g) * 10 + b) * 64 + lane;
#pragma unroll
    for (int t = 0; t < 2; ++t) dst[t * 32] = make_float4(gm[t][0], gm[t][1], gm[t][2], gm[t][3]);
  }
}

// STATE_ONLY: the first pass over segments.
template <int NP, bool STATE_ONLY>
__global__ void __launch_bounds__(NTH, NP <= 128 ? 2 : 1) ssd_chunk_kernel(const ChunkParams p) {
  pdl_sync();
  using S = Lay<NP>;
  constexpr int NH = NP / 4, NT = NH / 8;                   // state rows and 8-row tiles of a warp
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sm = smem_u32(smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pw = warp & 1, nw = warp >> 1;
  const int per_seq = STATE_ONLY ? p.segs - 1 : p.segs;
  const int seq = blockIdx.z / per_seq, seg = blockIdx.z % per_seq, h = blockIdx.y, p0 = blockIdx.x * PC, g = h / (p.H / p.G), inner = p.H * p.P;
  const int row0 = p.q_start[seq], n = p.q_start[seq + 1] - row0;
  if (n <= 0) return;
  const bool fresh = p.kv_len[seq] == n;
  const int NS = (p.N + 3) / 4 * 4;
  const int chunks = (n + L - 1) / L, seg_chunks = (chunks + p.segs - 1) / p.segs;
  const int c_lo = min(chunks, seg * seg_chunks), c_hi = min(chunks, c_lo + seg_chunks);
  if (!STATE_ONLY && c_lo >= c_hi) return;
  float* state = p.state + ((int64_t)p.slots[seq] * p.H + h) * p.P * NS;
  float* seg_at = p.segs > 1 ? p.seg_state + ((int64_t)seq * p.segs * p.H + h) * p.P * NS : nullptr;      // entry 0 of this head
  const int64_t seg_step = (int64_t)p.H * p.P * NS;
  const float* seg_log = p.segs > 1 ? p.seg_log + (int64_t)seq * p.segs * p.H + h : nullptr;
  const int lr = lane >> 2, lc = (lane & 3) * 2;            // row and first column of an accumulator tile held by this lane
  // S^T: tile t = state rows nw NH + 8 t .., channels p0 + 16 pw ..
  float st[NT][4];
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int ch = p0 + pw * 16 + lr + 8 * e, r = nw * NH + t * 8 + lc;
      float2 v = make_float2(0.f, 0.f);
      if (ch < p.P && r < p.N) {
        const int64_t at = (int64_t)ch * NS + r;
        if constexpr (STATE_ONLY) {
          if (seg == 0) *(float2*)(seg_at + at) = fresh ? v : *(const float2*)(state + at);
        } else if (p.segs > 1) {
          v = *(const float2*)(seg_at + at);
          for (int j = 0; j < seg; ++j) {
            const float d = pow2(seg_log[j * p.H]);
            const float2 end = *(const float2*)(seg_at + (j + 1) * seg_step + at);
            v = make_float2(fmaf(v.x, d, end.x), fmaf(v.y, d, end.y));
          }
        } else if (!fresh) {
          v = *(const float2*)(state + at);
        }
      }
      st[t][2 * e] = v.x;
      st[t][2 * e + 1] = v.y;
    }
  const float skip = p.skip[h];
  // what this thread copies of a chunk: pieces of B and C (rows bc_r, bc_r + STEP, ..), one piece of x, one token's step and decay
  constexpr int CN = NP / 8;
  const int bc_r = tid / CN;
  const bool bc_col = tid % CN * 8 < p.N;
  const bf16* bc_row = p.xbc + (int64_t)row0 * p.C + inner + g * p.N;
  const int xr = tid >> 2, xk = tid & 3;
  const bool x_col = p0 + xk * 8 < p.P;
  const bf16* x_row = p.xbc + (int64_t)row0 * p.C + h * p.P + (x_col ? p0 + xk * 8 : 0);
  const uint32_t x_at = xr * S::XROW + xk * 16;
  const int64_t dt_at = p.per_head ? (int64_t)h * L : (int64_t)h * p.T + row0;

  auto load = [&](int c) {                                  // chunk c -> stage c & 1
    const uint32_t s = sm + (c & 1) * S::STAGE;
    const int t0 = c * L, left = n - t0;
    const bf16* row = bc_row + (int64_t)t0 * p.C;
    load_bc<NP, NTH, !STATE_ONLY>(s, s + S::TILE, bc_r < left ? first_piece<NP, NTH>(row, p.C, p.N) : row, p.C, p.G * p.N, bc_col, left);
    const bool in = x_col && xr < left;
    cp16(s + 2 * S::TILE + x_at, x_row + (int64_t)(in ? t0 + xr : t0) * p.C, in);
    if (tid < L) {                                          // tokens past the end: no step, the decay of the last one
      const int64_t o = dt_at + (p.per_head ? min(tid, left - 1) : min(t0 + tid, n - 1));
      const uint32_t d = s + S::SC + tid * 4;
      cp4(d, p.dt + o, tid < left);
      cp4(d + L * 4, p.c_hi + o, true);
      cp4(d + 2 * L * 4, p.c_lo + o, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const float4* gram_at = p.gram + (chunk_place(row0, seq, 0) * p.G + g) * 640 + lane;
  float* y_at = p.y + (int64_t)(row0 + nw * 16 + lr) * inner + h * p.P + p0 + pw * 16 + lc;      // this lane's first result of a chunk
  // this lane's places in the fragments
  const uint32_t f_c = (lane & 15) * S::ROW + (nw * NH) * 2 + (lane >> 4) * 16;               // C, first operand
  const uint32_t f_m = (nw * 16 + (lane & 15)) * S::MROW + (lane >> 4) * 16;                  // decayed products, first operand
  const uint32_t f_x = (lane & 15) * S::XROW + (pw * 2 + (lane >> 4)) * 16;                   // x, second operand
  const uint32_t f_w = ((lane & 7) + ((lane >> 4) << 3)) * S::XROW + (pw * 2 + ((lane >> 3) & 1)) * 16;      // weighted x, first operand
  const uint32_t f_b = (lane & 15) * S::ROW + (nw * NH) * 2 + (lane >> 4) * 16;               // B, second operand

  double seg_sum = 0.0;
  if (c_lo < c_hi) load(c_lo);
  if constexpr (!STATE_ONLY) {
    gram_at += (int64_t)c_lo * p.G * 640;
    y_at += (int64_t)c_lo * L * inner;
  }
  for (int c = c_lo; c < c_hi; ++c) {
    float4 gm[2];
    if constexpr (!STATE_ONLY) { gm[0] = gram_at[warp * 64]; gm[1] = gram_at[warp * 64 + 32]; }
    if (c + 1 < c_hi) {
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
    {                                                       // x weighted for the state update
      const float w = pow2((hiL - hi[xr]) + (loL - lo[xr])) * dt[xr];
      float f[8];
      unpack16(*(const uint4*)(smem + stage + 2 * S::TILE + x_at), f);
      uint4 a, b;
      split2(f[0] * w, f[1] * w, a.x, b.x);
      split2(f[2] * w, f[3] * w, a.y, b.y);
      split2(f[4] * w, f[5] * w, a.z, b.z);
      split2(f[6] * w, f[7] * w, a.w, b.w);
      *(uint4*)(smem + S::XW_AT + x_at) = a;
      *(uint4*)(smem + S::XW_AT + S::X + x_at) = b;
    }
    if constexpr (!STATE_ONLY)
    for (int b = warp; b < 10; b += 8) {                    // decayed products
      const int mt = blk_m(b), jt = blk_j(b);
      const int i0 = mt * 16 + lr;
      const float hii[2] = {hi[i0], hi[i0 + 8]}, loi[2] = {lo[i0], lo[i0 + 8]};
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        const int j = jt * 16 + t * 8 + lc;
        const float2 hj = *(const float2*)(hi + j), lj = *(const float2*)(lo + j), dj = *(const float2*)(dt + j);
        const float gv[4] = {gm[t].x, gm[t].y, gm[t].z, gm[t].w};
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float w0 = gv[2 * e] * (pow2((hii[e] - hj.x) + (loi[e] - lj.x)) * dj.x);
          float w1 = gv[2 * e + 1] * (pow2((hii[e] - hj.y) + (loi[e] - lj.y)) * dj.y);
          if (mt == jt) {
            if (j > i0 + 8 * e) w0 = 0.f;
            if (j + 1 > i0 + 8 * e) w1 = 0.f;
          }
          uint32_t vh, vl;
          split2(w0, w1, vh, vl);
          uint8_t* d = smem + S::M_AT + (i0 + 8 * e) * S::MROW + j * 2;
          *(uint32_t*)d = vh;
          *(uint32_t*)(d + S::M) = vl;
        }
      }
      if (b + 8 < 10) { gm[0] = gram_at[(b + 8) * 64]; gm[1] = gram_at[(b + 8) * 64 + 32]; }
    }
    // what the state before the chunk gives (this warp's quarter of its rows), without the tokens' decay
    float y[4][2][4];
    if constexpr (!STATE_ONLY)
#pragma unroll
    for (int k = 0; k < NH / 16; ++k) {
      uint32_t bh[2][2], bl[2][2];                          // [channel octet][half of the k rows]
#pragma unroll
      for (int o = 0; o < 2; ++o)
#pragma unroll
        for (int t = 0; t < 2; ++t) split2(st[2 * k + t][2 * o], st[2 * k + t][2 * o + 1], bh[o][t], bl[o][t]);
      uint32_t a[4][4];
#pragma unroll
      for (int mt = 0; mt < 4; ++mt) ldsm4(a[mt], sC + f_c + mt * 16 * S::ROW + k * 32);
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int o = 0; o < 2; ++o) {
          if (k == 0) mma_first(y[mt][o], a[mt], bh[o][0], bh[o][1]);
          else mma(y[mt][o], a[mt], bh[o][0], bh[o][1]);
        }
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int o = 0; o < 2; ++o) mma(y[mt][o], a[mt], bl[o][0], bl[o][1]);
    }
    __syncthreads();
    // state update
    const float decay = pow2(hiL + loL);
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) st[t][e] *= decay;
#pragma unroll
    for (int k = 0; k < L / 16; ++k) {
      uint32_t a[4], b[4], q[NT / 2][4];
      ldsm4t(a, sW + f_w + k * 16 * S::XROW);
      ldsm4t(b, sW + S::X + f_w + k * 16 * S::XROW);
#pragma unroll
      for (int t = 0; t < NT / 2; ++t) ldsm4t(q[t], sB + f_b + k * 16 * S::ROW + t * 32);
#pragma unroll
      for (int t = 0; t < NT; ++t) mma(st[t], a, q[t / 2][2 * (t & 1)], q[t / 2][2 * (t & 1) + 1]);
#pragma unroll
      for (int t = 0; t < NT; ++t) mma(st[t], b, q[t / 2][2 * (t & 1)], q[t / 2][2 * (t & 1) + 1]);
    }
    if constexpr (STATE_ONLY) {
      seg_sum += (double)hiL + (double)loL;
      __syncthreads();
      continue;
    }
    // tokens of the chunk among themselves: token block nw, which this warp also finishes
    float z[2][4] = {};
    for (int k = 0; k <= nw; ++k) {
      uint32_t a[4], b[4], q[4];
      ldsm4(a, sM + f_m + k * 32);
      ldsm4(b, sM + S::M + f_m + k * 32);
      ldsm4t(q, sX + f_x + k * 16 * S::XROW);
      mma(z[0], a, q[0], q[1]);
      mma(z[1], a, q[2], q[3]);
      mma(z[0], b, q[0], q[1]);
      mma(z[1], b, q[2], q[3]);
    }
    const float own[2] = {pow2(hi[nw * 16 + lr] + lo[nw * 16 + lr]), pow2(hi[nw * 16 + lr + 8] + lo[nw * 16 + lr + 8])};
#pragma unroll
    for (int o = 0; o < 2; ++o)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float2 x = __bfloat1622float2(*(const __nv_bfloat162*)(smem + stage + 2 * S::TILE + (nw * 16 + lr + 8 * e) * S::XROW + (pw * 2 + o) * 16 + lc * 2));
        z[o][2 * e] = fmaf(skip, x.x, z[o][2 * e]);
        z[o][2 * e + 1] = fmaf(skip, x.y, z[o][2 * e + 1]);
      }
    __syncthreads();
    // partial results of the four quarters meet in shared memory: token i, channel pair c2 at place c2 ^ 4 (i & 3) of its row
    const int c2 = (pw * 8 + (lane & 3)) ^ ((lr & 3) << 2), c2_b = c2 ^ 4;
    float2* part = (float2*)(smem + S::Y_AT + nw * S::Y) + lr * (PC / 2);
#pragma unroll
    for (int mt = 0; mt < 4; ++mt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        part[(mt * 16 + 8 * e) * (PC / 2) + c2] = make_float2(y[mt][0][2 * e], y[mt][0][2 * e + 1]);
        part[(mt * 16 + 8 * e) * (PC / 2) + c2_b] = make_float2(y[mt][1][2 * e], y[mt][1][2 * e + 1]);
      }
    __syncthreads();
    const float2* sum = (const float2*)(smem + S::Y_AT) + (nw * 16 + lr) * (PC / 2);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      if (c * L + nw * 16 + lr + 8 * e >= n) continue;
#pragma unroll
      for (int o = 0; o < 2; ++o) {
        const int at = 8 * e * (PC / 2) + (o ? c2_b : c2);
        const float2 u = sum[at], v = sum[at + S::Y / 8], w = sum[at + 2 * (S::Y / 8)], x = sum[at + 3 * (S::Y / 8)];
        if (p0 + pw * 16 + o * 8 < p.P)
          *(float2*)(y_at + (e ? 8 * (int64_t)inner : 0) + o * 8) =
              make_float2(fmaf(own[e], (u.x + v.x) + (w.x + x.x), z[o][2 * e]), fmaf(own[e], (u.y + v.y) + (w.y + x.y), z[o][2 * e + 1]));
      }
    }
    gram_at += p.G * 640;
    y_at += L * (int64_t)inner;
  }
  if constexpr (STATE_ONLY) {
    state = seg_at + (seg + 1) * seg_step;
    if (p0 == 0 && tid == 0) p.seg_log[((int64_t)seq * p.segs + seg) * p.H + h] = (float)seg_sum;
  } else if (c_hi < chunks) {
    return;
  }
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int ch = p0 + pw * 16 + lr + 8 * e, r = nw * NH + t * 8 + lc;
      if (ch < p.P && r < p.N) *(float2*)(state + (int64_t)ch * NS + r) = make_float2(st[t][2 * e], st[t][2 * e + 1]);
    }
}

// silu(conv(xbc) + bias) in bf16: a thread takes four channels of CB tokens, the rows it reads all requested before the first is used
constexpr int CB = 8;
template <int TAPS>
__global__ void __launch_bounds__(128) ss_conv_kernel(const bf16* __restrict__ xbc, int64_t ldx, const bf16* __restrict__ w, const bf16* __restrict__ bias,
                                                      const bf16* __restrict__ ring_all, const int* __restrict__ q_start, const int* __restrict__ kv_len,
                                                      const int* __restrict__ slots, bf16* __restrict__ out, int n_taps, int C) {
  pdl_sync();
  const int taps = TAPS > 0 ? TAPS : n_taps;
  const int seq = blockIdx.z, ch = (blockIdx.x * 128 + threadIdx.x) * 4;
  const int first = q_start[seq], end = q_start[seq + 1], rb = first + blockIdx.y * CB;
  if (rb >= end || ch >= C) return;
  const int pos = kv_len[seq] - (end - first) + blockIdx.y * CB;
  const bf16* ring = ring_all + (int64_t)slots[seq] * taps * C;
  float b[4];
  load_e<bf16, 4>(bias + ch, b);
  if constexpr (TAPS > 0) {
    float v[TAPS + CB - 1][4];
#pragma unroll
    for (int r = 1 - TAPS; r < CB; ++r) {
      const bf16* src = rb + r >= first ? xbc + (int64_t)(rb + r) * ldx + ch : ring + (int64_t)((pos + r + TAPS) % TAPS) * C + ch;
      if (rb + r < end && pos + r >= 0) load_e<bf16, 4>(src, v[r + TAPS - 1]);
      else
#pragma unroll
        for (int e = 0; e < 4; ++e) v[r + TAPS - 1][e] = 0.f;
    }
    float wt[4][TAPS];
#pragma unroll
    for (int e = 0; e < 4; ++e)
      load_e<bf16, TAPS>(w + (int64_t)(ch + e) * TAPS, wt[e]);
#pragma unroll
    for (int t = 0; t < CB; ++t) {
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        y[e] = b[e];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) y[e] = fmaf(wt[e][j], v[t + j][e], y[e]);
        y[e] = silu_t<bf16>(y[e]);
      }
      if (rb + t < end) store_e<bf16, 4>(out + (int64_t)(rb + t) * C + ch, y);
    }
  } else {
    for (int t = 0; t < CB && rb + t < end; ++t) {
      float y[4] = {b[0], b[1], b[2], b[3]};
      for (int d = 0; d < taps; ++d) {                     // d tokens back
        const int r = t - d;
        float v[4];
        if (rb + r >= first) load_e<bf16, 4>(xbc + (int64_t)(rb + r) * ldx + ch, v);
        else if (pos + r >= 0) load_e<bf16, 4>(ring + (int64_t)((pos + r) % taps) * C + ch, v);
        else break;
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = fmaf(__bfloat162float(w[(int64_t)(ch + e) * taps + taps - 1 - d]), v[e], y[e]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = silu_t<bf16>(y[e]);
      store_e<bf16, 4>(out + (int64_t)(rb + t) * C + ch, y);
    }
  }
}

// One warp per (chunk, head): step sizes and the summed logarithms of the decays, [H][T]; a lane takes two tokens
__global__ void __launch_bounds__(256) ss_decay_kernel(const bf16* __restrict__ dt_in, int64_t ldx, const float* __restrict__ dt_bias,
                                                       const float* __restrict__ a_log, const int* __restrict__ q_start, float* __restrict__ dt,
                                                       float* __restrict__ c_hi, float* __restrict__ c_lo, int H, int T) {
  pdl_sync();
  const int h = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, seq = blockIdx.z;
  const int t0 = q_start[seq] + blockIdx.y * L, t1 = min(t0 + L, q_start[seq + 1]);
  if (h >= H || t0 >= t1) return;
  const float bias = dt_bias[h], a = -expf(a_log[h]);
  float d[2];
  double c[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int t = t0 + 2 * lane + i;
    d[i] = t < t1 ? softplus_x(__bfloat162float(dt_in[(int64_t)t * ldx + h]) + bias) : 0.f;
    c[i] = (double)(a * d[i]) * 1.4426950408889634;
  }
  c[1] += c[0];
  double before = c[1];                                // inclusive scan over the lanes, then what came before this lane
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= o) before += v;
  }
  before -= c[1];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int t = t0 + 2 * lane + i;
    if (t >= t1) continue;
    const double v = before + c[i];
    const float hi = (float)v;
    const int64_t o = (int64_t)h * T + t;
    dt[o] = d[i];
    c_hi[o] = hi;
    c_lo[o] = (float)(v - (double)hi);
  }
}

// Segments per sequence: as many as the machine has room for beside what heads and sequences fill, of eight chunks or more.
int chunk_segments(int S, int max_q, int H, int N, int P) {
  const int64_t blocks = (int64_t)((P + PC - 1) / PC) * H * S, room = (int64_t)mary_num_sms() * (N <= 128 ? 2 : 1);
  int segs = (int)(room / blocks);
  const int most = (max_q + L - 1) / L / 8;
  segs = segs < most ? segs : most;
  segs = segs < 16 ? segs : 16;
  return segs > 1 && (int64_t)S * segs <= 65535 ? segs : 1;
}
int64_t gram_floats(int T, int S, int G) { return ((int64_t)T / L + S + 1) * G * 10 * 64 * 4; }

template <int NP>
int launch_chunk(const ChunkParams& p, int S, int max_q, cudaStream_t s) {
  static MarySmemSlots slots[3] = {};
  if (int rc = mary_ensure_dyn_smem((const void*)ssd_gram_kernel<NP>, 2 * Lay<NP>::TILE, &slots[0])) return rc;
  if (int rc = mary_ensure_dyn_smem((const void*)ssd_chunk_kernel<NP, false>, Lay<NP>::BYTES, &slots[1])) return rc;
  if (int rc = mary_ensure_dyn_smem((const void*)ssd_chunk_kernel<NP, true>, Lay<NP>::BYTES, &slots[2])) return rc;
  const int cols = (p.P + PC - 1) / PC;
  MARY_LAUNCH((ssd_gram_kernel<NP>), dim3((max_q + L - 1) / L, p.G, S), 128, 2 * Lay<NP>::TILE, s, p);
  if (p.segs > 1) MARY_LAUNCH((ssd_chunk_kernel<NP, true>), dim3(cols, p.H, S * (p.segs - 1)), NTH, Lay<NP>::BYTES, s, p);
  MARY_LAUNCH((ssd_chunk_kernel<NP, false>), dim3(cols, p.H, S * p.segs), NTH, Lay<NP>::BYTES, s, p);
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
  if ((max_q + CB - 1) / CB > 65535 || ((uintptr_t)taps_b & 7)) return MARY_ERR_BAD_ARG;
  const dim3 grid((C / 4 + 127) / 128, (max_q + CB - 1) / CB, S);
  auto fn = taps == 4 ? ss_conv_kernel<4> : ss_conv_kernel<0>;
  MARY_LAUNCH(fn, grid, 128, 0, s, (const bf16*)xbc, ldx, (const bf16*)taps_w, (const bf16*)taps_b, (const bf16*)ring, q_start, kv_len, slots,
              (bf16*)xbc_out, taps, C);
  MARY_LAUNCH(ss_decay_kernel, dim3((H + 7) / 8, (max_q + L - 1) / L, S), 256, 0, s, (const bf16*)dt_in, ldx, dt_bias, a_log, q_start, dt, c_hi, c_lo,
              H, T);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

MARY_API int mary_ssd_chunk_supported(int N, int P) { return N >= 8 && N <= 256 && N % 8 == 0 && P >= 8 && P % 8 == 0; }

MARY_API int64_t mary_ssd_chunk_scratch_floats(int T, int S, int max_q, int G, int H, int N, int P) {
  const int segs = chunk_segments(S, max_q, H, N, P);
  return gram_floats(T, S, G) + (segs > 1 ? (int64_t)S * segs * H * ((int64_t)P * ((N + 3) / 4 * 4) + 1) : 0);
}

static int chunk_run(ChunkParams p, int S, int max_q, cudaStream_t s) {
  if (S <= 0 || p.T <= 0) return MARY_OK;
  p.segs = chunk_segments(S, max_q, p.H, p.N, p.P);
  p.seg_state = (float*)p.gram + gram_floats(p.T, S, p.G);
  p.seg_log = p.seg_state + (int64_t)S * p.segs * p.H * p.P * ((p.N + 3) / 4 * 4);
  if (p.G < 1 || p.H < 1 || p.H % p.G || p.H > 65535 || S > 65535 || !mary_ssd_chunk_supported(p.N, p.P) || p.C % 8 ||
      (((uintptr_t)p.xbc | (uintptr_t)p.gram) & 15))
    return MARY_ERR_BAD_ARG;
  if (p.N <= 64) return launch_chunk<64>(p, S, max_q, s);
  if (p.N <= 128) return launch_chunk<128>(p, S, max_q, s);
  return launch_chunk<256>(p, S, max_q, s);
}

// y [T, H P] f32; the state [slots][H][P][N] is read (zero for a portion that starts its sequence) and updated in place.  scratch:
// mary_ssd_chunk_scratch_floats(T, S, max_q, G, H, N, P) floats, 16-byte aligned.
MARY_API int mary_ssd_chunk(const void* xbc, const float* dt, const float* c_hi, const float* c_lo, const float* skip, float* y, float* state,
                            float* scratch, const int* q_start, const int* kv_len, const int* slots, int S, int max_q, int T, int G, int H, int N, int P,
                            cudaStream_t s) {
  return chunk_run({(const bf16*)xbc, dt, c_hi, c_lo, skip, y, state, (float4*)scratch, q_start, kv_len, slots, T, G, H, N, P, H * P + 2 * G * N, 1, nullptr, nullptr, 0}, S, max_q, s);
}

// Linear attention with one constant decay per head, S_t = d S_{t-1} + k_t v_t^T, y_t = S_t^T q_t: the same chunks with q, k, v for C, B, x.  vkq:
// rows of ld elements [v: H P | k: H N | q: H N]; one, c_hi, c_lo, zero [H][64]: step size 1, log2 of d^1 .. d^64 as two floats, no skip.
MARY_API int mary_lightning_chunk(const void* vkq, int64_t ld, const float* one, const float* c_hi, const float* c_lo, const float* zero, float* y,
                                  float* state, float* scratch, const int* q_start, const int* kv_len, const int* slots, int S, int max_q, int T, int H,
                                  int N, int P, cudaStream_t s) {
  if (ld < (int64_t)H * (P + 2 * N)) return MARY_ERR_BAD_ARG;
  return chunk_run({(const bf16*)vkq, one, c_hi, c_lo, zero, y, state, (float4*)scratch, q_start, kv_len, slots, T, H, H, N, P, ld, 1, nullptr, nullptr, 1}, S, max_q, s);
}
