// Causal (optionally sliding-window) attention for prefill over the paged KV cache, on tcgen05 tensor cores.
//
// The reference computes prefill attention with a SIMT kernel that gives one CTA to each (query, head) pair
// (src/models/inkling/banded.rs:109-299) or with materialised score blocks and library matmuls
// (src/models/inkling/burn.rs:550-797).  Here one CTA owns 128 query tokens of one head (MMA M = 128) and streams the
// keys and values of its KV head through shared memory 64 keys at a time, page by page:
//   warp 0    TMA for Q (once) and the K ring, a stage laid out [chunks][64 keys][64 dims] with the 128-byte swizzle.  With
//             64-token pages a stage is ONE 4-D operation (the tensor map orders the cache as dims-in-chunk, tokens,
//             chunks, pages, so the box [64, 64, chunks, 1] lands chunk-major); with 16-token pages it takes one
//             [16 tokens x 64 dims] operation per page and chunk, and the TMA unit's per-operation cost bounds the kernel;
//   warp 6    TMA for the V ring (same layout) — a ring of its own, so a K stage is refilled as soon as Q K^T has read
//             it and does not wait for the P V of that block;
//   warp 1    MMA: S[128 x 64] = Q K^T into one of two TMEM buffers (issued two blocks ahead), O[128 x DV] += P V with
//             V^T read from the V stage as an MN-major B operand and P from shared memory;
//   warps 2-5 (with attention forms also 7-10, two threads per row) softmax: thread r owns row r (TMEM lane r): tcgen05.ld of S, scale, causal / window mask, running maximum
//             with lazy rescale of O (only when the maximum grows by more than 2^8), P written to shared memory as bf16
//             in the un-swizzled K-major core-matrix layout, finally O / l to global memory.
// Blocks of keys that no row of the tile can see (beyond the causal diagonal, before the window) are never loaded.
// All waits are bounded; a wait that runs out sets the status word, frees TMEM and returns.
#include "attention_form.cuh"
#include "common.cuh"
#include "host_utils.h"

using namespace mary;

namespace {

constexpr int PAGE = 16, KB = 64, TR = 128, CHUNK = 64;
constexpr int NSBUF = 2;
constexpr int P_BYTES = TR * KB * 2;              // 16 KB
constexpr float RESCALE_THRESHOLD = 8.0f;

// SPLITP: P is handed to the tensor cores as the sum of two bf16 values (rounded value and rounding error), so that the softmax
// weights keep 16 significant bits; two P V products per block.
// BIAS: a bias by distance is added to the scaled score.  Every softmax warp copies the 95 values that its rows can meet in a block to
// shared memory, minus infinity outside the window and after the query, so the bias is the mask as well.
// MAPS = 1 or 2 makes the kernel honour FaParams::f (0: plain attention).  With two maps (query and key rows [map 0 | map 1], DK each) the
// tile walks its key blocks once per map, into accumulators of their own, and a row's thread forms the difference and its norm at the end.
template <int DK, int DV, bool SPLITP, bool BIAS, int MAPS>
struct FaCfg {
  static constexpr int NM = MAPS == 2 ? 2 : 1;
  static constexpr int NCK = DK / CHUNK, NCV = DV / CHUNK;
  static constexpr int Q_CHUNK_BYTES = TR * 128;
  static constexpr int Q_BYTES = NM * NCK * Q_CHUNK_BYTES;
  static constexpr int K_CHUNK_BYTES = KB * 128, V_CHUNK_BYTES = KB * 128;
  static constexpr int K_STAGE = NCK * K_CHUNK_BYTES, V_STAGE = NCV * V_CHUNK_BYTES;
  static constexpr int STAGES = (DK + DV > 384) ? 2 : 3;
  static constexpr int NPBUF = (SPLITP && DK + DV > 256) ? 1 : 2;
  // threads that share a query row, each with half of its scores (MAPS > 0, where shared memory has room for what they exchange): the row's
  // softmax is the longest chain of the kernel, and one warp per scheduler cannot hide its own latencies
  static constexpr int HW = (MAPS > 0 && NM * DK <= 128 && DV <= 128) ? 2 : 1;
  static constexpr int NTHREADS = 96 + 128 * HW;
  static constexpr int XCH_BYTES = HW == 2 ? 2 * 2 * TR * 4 : 0;
  static constexpr int BIAS_BYTES = BIAS ? 4 * 96 * 4 : 0;
  static constexpr int P_STAGE = SPLITP ? 2 * P_BYTES : P_BYTES;
  static constexpr int SMEM = Q_BYTES + STAGES * (K_STAGE + V_STAGE) + NPBUF * P_STAGE + BIAS_BYTES + XCH_BYTES + 1024 + 256;
  static constexpr int TMEM_COLS = 128 + NM * DV <= 256 ? 256 : 512;     // S: 2 x 64 columns at 0..127, O: DV columns per map at 128..
  static_assert(128 + NM * DV <= 512 && !(BIAS && MAPS), "accumulator columns");
  static_assert(DK % CHUNK == 0 && DV % CHUNK == 0 && DV <= 256 && DK <= 256, "head dims: multiples of 64 up to 256");
  static_assert(SMEM <= 232448, "shared memory budget");
};

struct FaParams {
  const int* page_table; const int* kv_len; const int* q_start; const int* blk_seq; const int* blk_tok0;
  __nv_bfloat16* out;      // rows of out_ld elements, head h at h * DV
  int64_t out_ld;          // elements between the output rows of two tokens
  int max_pages, Hq, Hkv, window, page;
  float scale_log2;
  const float* bias;       // BIAS: [Hq][window] by distance, added to the scaled score
  const __nv_bfloat16* gate;   // rows of gate_ld elements, head h at h * DV: the output times its logistic function; or null
  int64_t gate_ld;
  MaryAttnForm f;
  int* status;
};

__device__ __forceinline__ uint64_t fa_desc_kmajor_noswz(uint32_t addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  return (uint64_t)((addr >> 4) & 0x3FFF) | ((uint64_t)(lbo_bytes >> 4) << 16) | ((uint64_t)(sbo_bytes >> 4) << 32) | (1ull << 46);
}
__device__ __forceinline__ uint64_t fa_desc_mnmajor_sw128(uint32_t addr, uint32_t lbo_bytes, uint32_t sbo_bytes) {
  return (uint64_t)((addr >> 4) & 0x3FFF) | ((uint64_t)(lbo_bytes >> 4) << 16) | ((uint64_t)(sbo_bytes >> 4) << 32) | (1ull << 46) |
         (2ull << 61);
}

template <int DK, int DV, bool SPLITP, bool BIAS, int MAPS>
__global__ void __launch_bounds__((FaCfg<DK, DV, SPLITP, BIAS, MAPS>::NTHREADS), 1)
fa_prefill_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                  const __grid_constant__ CUtensorMap tm_v, const FaParams p) {
  using C = FaCfg<DK, DV, SPLITP, BIAS, MAPS>;
  constexpr int NM = C::NM, HW = C::HW;
  constexpr int STAGES = C::STAGES, NPBUF = C::NPBUF;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + C::Q_BYTES;
  uint8_t* sV = sK + STAGES * C::K_STAGE;
  uint8_t* sP = sV + STAGES * C::V_STAGE;
  uint64_t* bars = (uint64_t*)(sP + NPBUF * C::P_STAGE + C::BIAS_BYTES + C::XCH_BYTES);
  uint64_t* q_full = bars;                 // 1
  uint64_t* k_full = q_full + 1;           // [STAGES]
  uint64_t* k_empty = k_full + STAGES;
  uint64_t* v_full = k_empty + STAGES;
  uint64_t* v_empty = v_full + STAGES;
  uint64_t* s_full = v_empty + STAGES;     // [NSBUF]
  uint64_t* s_empty = s_full + NSBUF;
  uint64_t* p_full = s_empty + NSBUF;      // [NPBUF]
  uint64_t* pv_done = p_full + NPBUF;
  uint32_t* tmem_slot = (uint32_t*)(pv_done + NPBUF);
  volatile int* abort_flag = (volatile int*)(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // all heads of the last tiles of the batch first: they see the most keys, and short tiles are left to fill the end of the launch
  const int nb = gridDim.y - 1 - blockIdx.y, head = blockIdx.x;
  const int kvh = head / (p.Hq / p.Hkv);
  const int seq = p.blk_seq[nb], tok0 = p.blk_tok0[nb];          // tok0: index into the flattened token axis
  const int seq_tok0 = p.q_start[seq], seq_tok1 = p.q_start[seq + 1];
  const int nrows = min(TR, seq_tok1 - tok0);
  const int kvlen = p.kv_len[seq];
  const int pos_first = kvlen - (seq_tok1 - seq_tok0) + (tok0 - seq_tok0);   // position of the tile's first query token
  const int k_hi = pos_first + nrows;                                         // keys [0, k_hi) are visible to some row
  int k_lo = p.window > 0 ? max(0, pos_first - p.window + 1) : 0;
  if constexpr (MAPS > 0) k_lo = max(k_lo, first_key(p.f, pos_first));
  const int b_lo = k_lo / KB, b_hi = (k_hi + KB - 1) / KB;
  const int nblk = max(0, b_hi - b_lo);
  const int ntot = NM * nblk;                      // key blocks to go through, map after map

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < STAGES; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
    for (int b = 0; b < NSBUF; ++b) { mbar_init(&s_full[b], 1); mbar_init(&s_empty[b], 4 * HW); }
    for (int b = 0; b < NPBUF; ++b) { mbar_init(&p_full[b], 4 * HW); mbar_init(&pv_done[b], 1); }
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, C::TMEM_COLS); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_S = tmem_base;            // NSBUF x 64 columns
  const uint32_t tmem_O = tmem_base + 128;      // DV columns

  if (warp == 0 || warp == 6) {
    // ------------------------------------------------------------------ producers: warp 0 = Q + K ring, warp 6 = V ring
    if (nblk > 0) {
      const bool isK = warp == 0;
      if (isK && lane == 0) {
        mbar_expect_tx(q_full, C::Q_BYTES);
        for (int c = 0; c < NM * C::NCK; ++c) tma_load_2d(sQ + c * C::Q_CHUNK_BYTES, &tm_q, q_full, head * NM * DK + c * CHUNK, tok0);
      }
      const int* pt = p.page_table + (int64_t)seq * p.max_pages;
      uint64_t* full = isK ? k_full : v_full;
      uint64_t* empty = isK ? k_empty : v_empty;
      uint8_t* ring = isK ? sK : sV;
      const int stage_bytes = isK ? C::K_STAGE : C::V_STAGE;
      const int nchunk = isK ? C::NCK : C::NCV;
      const int hd = isK ? DK : DV;
      const CUtensorMap* tm = isK ? &tm_k : &tm_v;
      int stage = 0; uint32_t phase = 0;
      for (int i = 0; i < ntot; ++i) {
        const bool second = NM == 2 && i >= nblk;
        const int b = b_lo + (second ? i - nblk : i);
        const int row_head = isK ? kvh * NM + (second ? 1 : 0) : kvh;        // heads of hd values along a token's cache row
        int ok = 1;
        if (lane == 0) {
          ok = mbar_wait(&empty[stage], phase ^ 1, abort_flag, p.status, MARY_ERR_TIMEOUT_TMA) ? 1 : 0;
          if (ok) mbar_expect_tx(&full[stage], stage_bytes);
        }
        ok = __shfl_sync(0xffffffffu, ok, 0);
        if (!ok) goto done;
        if (p.page == KB) {
          if (lane == 0) {
            const int key0 = b * KB;
            const int page = (key0 < kvlen) ? pt[key0 / KB] : pt[0];
            tma_load_4d(ring + stage * stage_bytes, tm, &full[stage], 0, 0, row_head * nchunk, page);
          }
        } else
        // (KB / PAGE) pages x nchunk chunks operations of [16 tokens x 64 dims] (2 KB each), spread over the lanes
        for (int op = lane; op < (KB / PAGE) * nchunk; op += 32) {
          const int pg = op / nchunk, c = op % nchunk;
          const int key0 = b * KB + pg * PAGE;
          const int page = (key0 < kvlen) ? pt[key0 / PAGE] : pt[0];     // pages past the end: any valid page (masked)
          tma_load_3d(ring + stage * stage_bytes + c * (KB * 128) + pg * (PAGE * 128), tm, &full[stage], row_head * hd + c * CHUNK, 0, page);
        }
        __syncwarp();
        if (++stage == STAGES) { stage = 0; phase ^= 1; }
      }
    }
  } else if (warp == 1) {
    if (elect_one() && nblk > 0) {
      const uint32_t idesc_s = idesc_bf16(TR, KB);
      const uint32_t idesc_o = idesc_bf16(TR, DV) | (1u << 16);           // B operand MN-major
      if (!mbar_wait(q_full, 0, abort_flag, p.status, MARY_ERR_TIMEOUT_TMA)) goto done;
      const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP);
      auto issue_qk = [&](int i) -> bool {        // i = block index relative to b_lo
        const int stage = i % STAGES, sb = i % NSBUF;
        if (!mbar_wait(&s_empty[sb], ((i / NSBUF) & 1) ^ 1, abort_flag, p.status, MARY_ERR_TIMEOUT_MMA)) return false;
        if (!mbar_wait(&k_full[stage], (i / STAGES) & 1, abort_flag, p.status, MARY_ERR_TIMEOUT_TMA)) return false;
        tc_fence_after();
        const uint32_t kb_addr = smem_u32(sK + stage * C::K_STAGE);
        const uint32_t qm_addr = q_addr + (NM == 2 && i >= nblk ? C::NCK * C::Q_CHUNK_BYTES : 0);
#pragma unroll
        for (int c = 0; c < C::NCK; ++c) {
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            umma_f16(tmem_S + sb * KB, umma_desc_sw128(qm_addr + c * C::Q_CHUNK_BYTES + k * 32),
                     umma_desc_sw128(kb_addr + c * C::K_CHUNK_BYTES + k * 32), idesc_s, (c > 0 || k > 0) ? 1u : 0u);
          }
        }
        umma_commit(&k_empty[stage]);       // the K stage may be refilled once Q K^T has read it
        umma_commit(&s_full[sb]);
        return true;
      };
      if (!issue_qk(0)) goto done;
      if (ntot > 1 && !issue_qk(1)) goto done;
      for (int i = 0; i < ntot; ++i) {
        const int pb = i % NPBUF, stage = i % STAGES;
        if (!mbar_wait(&v_full[stage], (i / STAGES) & 1, abort_flag, p.status, MARY_ERR_TIMEOUT_TMA)) goto done;
        if (!mbar_wait(&p_full[pb], (i / NPBUF) & 1, abort_flag, p.status, MARY_ERR_TIMEOUT_MMA)) goto done;
        tc_fence_after();
        const uint32_t vb_addr = smem_u32(sV + stage * C::V_STAGE);
        const bool second = NM == 2 && i >= nblk;
        const uint32_t om = tmem_O + (second ? DV : 0);
        const int i0 = second ? nblk : 0;
#pragma unroll
        for (int kk = 0; kk < KB / 16; ++kk) {
          // A = P[:, 16 keys] (K-major, no swizzle: the two 16-byte key chunks of one MMA TR*16 bytes apart, 8-row groups
          // 128 bytes apart); B = V^T of those keys (MN-major, 128B swizzle: 64-dim groups one chunk apart, 8-key groups 1 KB apart)
          umma_f16(om, fa_desc_kmajor_noswz(p_addr + pb * C::P_STAGE + kk * 2 * (TR * 16), TR * 16, 128),
                   fa_desc_mnmajor_sw128(vb_addr + kk * 16 * 128, C::V_CHUNK_BYTES, 1024), idesc_o, (i > i0 || kk > 0) ? 1u : 0u);
        }
        if constexpr (SPLITP) {
#pragma unroll
          for (int kk = 0; kk < KB / 16; ++kk)
            umma_f16(om, fa_desc_kmajor_noswz(p_addr + pb * C::P_STAGE + P_BYTES + kk * 2 * (TR * 16), TR * 16, 128),
                     fa_desc_mnmajor_sw128(vb_addr + kk * 16 * 128, C::V_CHUNK_BYTES, 1024), idesc_o, 1u);
        }
        umma_commit(&v_empty[stage]);
        umma_commit(&pv_done[pb]);
        if (i + 2 < ntot && !issue_qk(i + 2)) goto done;
      }
    }
  } else if (nblk > 0) {
    // ------------------------------------------------------------------ softmax warps (2-5, and 7-10 when two threads share a row): thread = query row, or half of its scores
    const int q4 = warp & 3;                         // the TMEM lane group this warp may access
    const int r = q4 * 32 + lane;
    constexpr int KC = KB / HW;                      // scores of a block that a thread holds
    const int half = HW == 2 && warp > 6 ? 1 : 0, cb = half * KC;
    float* const xch = (float*)(sP + NPBUF * C::P_STAGE + C::BIAS_BYTES);       // [2][2][TR]
    // A wait that ran out must be seen by the whole warp, and a partner warp that stands at the pair's barrier must be let go: it finds
    // the abort flag raised and leaves as well.
    auto wait = [&](uint64_t* bar, uint32_t parity) -> bool {
      const bool ok = mbar_wait(bar, parity, abort_flag, p.status, MARY_ERR_TIMEOUT_MMA);
      if constexpr (HW == 2) {
        if (__all_sync(0xffffffffu, ok)) return true;
        asm volatile("bar.arrive %0, 64;" ::"r"(1 + q4) : "memory");
        return false;
      }
      return ok;
    };
    auto meet = [&]() -> bool {                      // the two warps of the pair
      asm volatile("bar.sync %0, 64;" ::"r"(1 + q4) : "memory");
      return !__any_sync(0xffffffffu, *abort_flag != 0);
    };
    const bool row_ok = r < nrows;
    const int qpos = pos_first + r;
    int lo_key = p.window > 0 ? qpos - p.window + 1 : 0;
    float sl2 = p.scale_log2;                        // this row's factor on the raw scores
    int full_from = p.window > 0 ? pos_first + TR - p.window : 0;      // blocks from this key on are inside every row's window and chunk
    if constexpr (MAPS > 0) {
      lo_key = max(lo_key, first_key(p.f, qpos));
      sl2 *= query_temperature(p.f, qpos);
      full_from = max(full_from, first_key(p.f, pos_first + TR - 1));
    }
    const uint32_t lane_off = (uint32_t)(q4 * 32) << 16;
    float m_ref = -INFINITY, l = 0.f, l_first = 0.f;
    float* const bias_row = (float*)(sP + NPBUF * C::P_STAGE) + q4 * 96;
    for (int i = 0; i < ntot; ++i) {
      const int sb = i % NSBUF, pb = i % NPBUF;
      const bool second = NM == 2 && i >= nblk;
      const int i0 = second ? nblk : 0;
      const uint32_t om = tmem_O + (second ? DV : 0);
      if (NM == 2 && i == nblk) { l_first = l; l = 0.f; m_ref = -INFINITY; }
      if constexpr (BIAS) {
        // bias_row[d]: rows q4 * 32 + lane and keys j of the block with distance base + d, d = 63 + lane - j
        const int base = pos_first + q4 * 32 - (b_lo + i) * KB - (KB - 1);
        const float* src = p.bias + (int64_t)head * p.window;
        __syncwarp();
#pragma unroll
        for (int k = 0; k < 3; ++k) {
          const int dist = base + k * 32 + lane;
          bias_row[k * 32 + lane] = dist >= 0 && dist < p.window ? src[dist] * 1.4426950408889634f : -INFINITY;
        }
        __syncwarp();
      }
      if (!wait(&s_full[sb], (i / NSBUF) & 1)) goto done;
      tc_fence_after();
      uint32_t sr[KC];
      tmem_ld_32x32b_x32(tmem_S + lane_off + sb * KB + cb, sr);
      if constexpr (HW == 1) tmem_ld_32x32b_x32(tmem_S + lane_off + sb * KB + 32, sr + 32);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_empty[sb]);
      const int key0 = (b_lo + i - i0) * KB;
      // A block that every row of the tile sees entirely (all blocks left of the diagonal band and inside the window) takes the
      // short path: no per-element mask, the maximum on the raw scores, one fused multiply-add and one exponential per element.
      // A thread owns one query row and walks its 64 scores in sequence, so this loop's instruction count bounds the block rate.
      const bool full_blk = key0 + KB - 1 <= pos_first && key0 >= full_from && (MAPS == 0 || sl2 > 0.f);
      float mx;
      if constexpr (MAPS > 0) {
        if (p.f.cap > 0.f) {
          float v[KC];
#pragma unroll
          for (int j = 0; j < KC; ++j) v[j] = __uint_as_float(sr[j]);
          cap_scores<KC>(v, sl2, p.f.cap);
#pragma unroll
          for (int j = 0; j < KC; ++j) sr[j] = __float_as_uint(v[j]);
        }
      }
      const float sc = MAPS > 0 && p.f.cap > 0.f ? 1.0f : sl2;               // factor on what `sr` now holds
      if constexpr (BIAS) {
        mx = -INFINITY;
#pragma unroll
        for (int j = 0; j < KB; ++j) {
          const float v = fmaf(__uint_as_float(sr[j]), p.scale_log2, bias_row[KB - 1 + lane - j]);
          sr[j] = __float_as_uint(v);
          mx = fmaxf(mx, v);
        }
      } else if (full_blk) {
        mx = __uint_as_float(sr[0]);
#pragma unroll
        for (int j = 1; j < KC; ++j) mx = fmaxf(mx, __uint_as_float(sr[j]));
        mx *= sc;
      } else {
        mx = -INFINITY;
#pragma unroll
        for (int j = 0; j < KC; ++j) {
          const int kj = key0 + cb + j;
          const bool ok = row_ok && kj <= qpos && kj >= lo_key;
          const float v = ok ? __uint_as_float(sr[j]) * sc : -INFINITY;
          sr[j] = __float_as_uint(v);
          mx = fmaxf(mx, v);
        }
      }
      if constexpr (HW == 2) {
        float* x = xch + (i & 1) * 2 * TR;
        x[half * TR + r] = mx;
        if (!meet()) goto done;
        mx = fmaxf(mx, x[(half ^ 1) * TR + r]);
      }
      const bool need = mx > m_ref + RESCALE_THRESHOLD;
      const bool first = (m_ref == -INFINITY);
      float corr = 1.f;
      if (need) { corr = first ? 0.f : exp2f(m_ref - mx); m_ref = mx; }
      uint32_t pw[KC / 2], pl[SPLITP ? KC / 2 : 1];
      float psum = 0.f;
      if (full_blk && !BIAS) {
        const float nm = -m_ref;
#pragma unroll
        for (int j = 0; j < KC / 2; ++j) {
          const float a = exp2f(fmaf(__uint_as_float(sr[2 * j]), sc, nm));
          const float b = exp2f(fmaf(__uint_as_float(sr[2 * j + 1]), sc, nm));
          __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
          pw[j] = *(uint32_t*)&h;
          if constexpr (SPLITP) {
            const float2 back = __bfloat1622float2(h);
            __nv_bfloat162 lo = __floats2bfloat162_rn(a - back.x, b - back.y);
            pl[j] = *(uint32_t*)&lo;
          }
          psum += a + b;
        }
      } else {
        const float nm = m_ref == -INFINITY ? 0.f : -m_ref;        // nothing visible yet: every score is minus infinity, every weight 0
#pragma unroll
        for (int j = 0; j < KC / 2; ++j) {
          const float a = exp2f(__uint_as_float(sr[2 * j]) + nm);
          const float b = exp2f(__uint_as_float(sr[2 * j + 1]) + nm);
          __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
          pw[j] = *(uint32_t*)&h;
          float2 back = __bfloat1622float2(h);
          if constexpr (SPLITP) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(a - back.x, b - back.y);
            pl[j] = *(uint32_t*)&lo;
            psum += a + b;
          } else {
            psum += back.x + back.y;
          }
        }
      }
      l = l * corr + psum;
      if (__any_sync(0xffffffffu, need && !first) && i > i0) {
        // O may only be touched once the previous P V has completed
        if (!wait(&pv_done[(i - 1) % NPBUF], ((i - 1) / NPBUF) & 1)) goto done;
        tc_fence_after();
#pragma unroll 1
        for (int c0 = half * (DV / HW); c0 < (half + 1) * (DV / HW); c0 += 32) {
          uint32_t o[32];
          tmem_ld_32x32b_x32(om + lane_off + c0, o);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * corr);
#pragma unroll
          for (int j = 0; j < 32; j += 8) tmem_st_32x32b_x8(om + lane_off + c0 + j, o + j);
        }
        tmem_st_wait();
      }
      if (i >= NPBUF) {
        // this P buffer was last read by the P V of block i - NPBUF
        if (!wait(&pv_done[pb], ((i - NPBUF) / NPBUF) & 1)) goto done;
      }
      // P (bf16) -> shared memory: chunk c holds keys 8c..8c+7 of every row, 16 bytes per row
#pragma unroll
      for (int c = 0; c < KC / 8; ++c)
        *(uint4*)(sP + pb * C::P_STAGE + (cb / 8 + c) * (TR * 16) + r * 16) = make_uint4(pw[4 * c], pw[4 * c + 1], pw[4 * c + 2], pw[4 * c + 3]);
      if constexpr (SPLITP) {
#pragma unroll
        for (int c = 0; c < KC / 8; ++c)
          *(uint4*)(sP + pb * C::P_STAGE + P_BYTES + (cb / 8 + c) * (TR * 16) + r * 16) = make_uint4(pl[4 * c], pl[4 * c + 1], pl[4 * c + 2], pl[4 * c + 3]);
      }
      fence_proxy_async();       // make the generic-proxy writes of P visible to the tensor core
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[pb]);
    }
    // ------------------------------------------------------------------ write out
    const int o_lo = half * (DV / HW), o_hi = o_lo + DV / HW;      // value columns of this thread
    const bool turned = MAPS == 1 && p.f.turn && row_ok;
    float4 cs[MAPS == 1 ? 8 : 1];                                  // angles of the next 32 columns, requested ahead of their use
    auto load_turn = [&](int c0) {
      if constexpr (MAPS == 1) {
        if (!turned) return;
        const float4* src = (const float4*)(p.f.turn + ((int64_t)(tok0 + r) * DV + c0) / 2);
#pragma unroll
        for (int j = 0; j < 8; ++j) cs[j] = __ldg(src + j);
      }
    };
    load_turn(o_lo);
    if (!wait(&pv_done[(ntot - 1) % NPBUF], ((ntot - 1) / NPBUF) & 1)) goto done;
    tc_fence_after();
    if constexpr (HW == 2) {
      // the other half's sums (buffers of the block loop that nobody reads any more after the first meeting)
      if (!meet()) goto done;
      xch[half * TR + r] = l;
      xch[(2 + half) * TR + r] = l_first;
      if (!meet()) goto done;
      l += xch[(half ^ 1) * TR + r];
      l_first += xch[(2 + (half ^ 1)) * TR + r];
    }
    if constexpr (MAPS == 1) {
      if (p.f.sink) l += exp2f(fmaf(p.f.sink[head], 1.4426950408889634f, -m_ref));
    }
    float inv_l = l > 0.f ? 1.f / l : 0.f;
    if constexpr (NM == 2) {
      // o = a0 - mix * a1 as w0 * O0 + w1 * O1, then the norm over the row's DV values
      float w0 = l_first > 0.f ? 1.f / l_first : 0.f, w1 = -p.f.mix * inv_l, ss = 0.f;
#pragma unroll 1
      for (int c0 = o_lo; c0 < o_hi; c0 += 32) {
        uint32_t a[32], b[32];
        tmem_ld_32x32b_x32(tmem_O + lane_off + c0, a);
        tmem_ld_32x32b_x32(tmem_O + lane_off + DV + c0, b);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          const float v = fmaf(w1, __uint_as_float(b[j]), w0 * __uint_as_float(a[j]));
          ss = fmaf(v, v, ss);
        }
      }
      if constexpr (HW == 2) {
        if (!meet()) goto done;
        xch[half * TR + r] = ss;
        if (!meet()) goto done;
        ss += xch[(half ^ 1) * TR + r];
      }
      const float c = p.f.post * rsqrtf(ss / DV + p.f.eps);
      w0 *= c;
      w1 *= c;
#pragma unroll 1
      for (int c0 = o_lo; c0 < o_hi; c0 += 32) {
        uint32_t a[32], b[32];
        tmem_ld_32x32b_x32(tmem_O + lane_off + c0, a);
        tmem_ld_32x32b_x32(tmem_O + lane_off + DV + c0, b);
        tmem_ld_wait();
        if (row_ok) {
          uint4 w[4];
          uint32_t* wp = (uint32_t*)w;
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            __nv_bfloat162 h = __floats2bfloat162_rn(fmaf(w1, __uint_as_float(b[2 * j]), w0 * __uint_as_float(a[2 * j])),
                                                     fmaf(w1, __uint_as_float(b[2 * j + 1]), w0 * __uint_as_float(a[2 * j + 1])));
            wp[j] = *(uint32_t*)&h;
          }
          uint4* dst = (uint4*)(p.out + (int64_t)(tok0 + r) * p.out_ld + head * DV + c0);
#pragma unroll
          for (int j = 0; j < 4; ++j) dst[j] = w[j];
        }
      }
    } else
#pragma unroll 1
    for (int c0 = o_lo; c0 < o_hi; c0 += 32) {
      uint32_t o[32];
      tmem_ld_32x32b_x32(tmem_O + lane_off + c0, o);
      tmem_ld_wait();
      if (row_ok) {
        __nv_bfloat16* dst = p.out + (int64_t)(tok0 + r) * p.out_ld + head * DV + c0;
        uint4 w[4];
        uint32_t* wp = (uint32_t*)w;
        if (p.gate) {
          const uint4* src = (const uint4*)(p.gate + (int64_t)(tok0 + r) * p.gate_ld + head * DV + c0);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const uint4 g = src[j];
            const __nv_bfloat162* gh = (const __nv_bfloat162*)&g;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const float2 f = __bfloat1622float2(gh[i]);
              float &a = *(float*)&o[8 * j + 2 * i], &b = *(float*)&o[8 * j + 2 * i + 1];
              a = __fdividef(a, 1.0f + __expf(-f.x));
              b = __fdividef(b, 1.0f + __expf(-f.y));
            }
          }
        }
        if constexpr (MAPS == 1) {
          if (turned) {
#pragma unroll
            for (int j = 0; j < 8; ++j) {
              float* x = (float*)o + 4 * j;
              const float2 a = turned_back(make_float2(cs[j].x, cs[j].y), x[0], x[1]), b = turned_back(make_float2(cs[j].z, cs[j].w), x[2], x[3]);
              x[0] = a.x; x[1] = a.y; x[2] = b.x; x[3] = b.y;
            }
            if (c0 + 32 < o_hi) load_turn(c0 + 32);
          }
        }
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          __nv_bfloat162 h = __floats2bfloat162_rn(__uint_as_float(o[2 * j]) * inv_l, __uint_as_float(o[2 * j + 1]) * inv_l);
          wp[j] = *(uint32_t*)&h;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) ((uint4*)dst)[j] = w[j];
      }
    }
  }
done:
  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, C::TMEM_COLS); }
}

int make_cache_map(CUtensorMap* m, const void* cache, int heads, int hd, int num_pages, int64_t tok_stride, int64_t page_stride, int page) {
  PFN_encodeTiled enc = mary_encode_fn();
  if (!enc) return MARY_ERR_CUDA;
  CUresult r;
  if (page == KB) {
    // dims: 64 elements of a chunk, 64 tokens of a page, chunks of a token row (all KV heads), pages; box = all chunks of one head
    cuuint64_t dims[4] = {CHUNK, KB, (cuuint64_t)(heads * hd / CHUNK), (cuuint64_t)num_pages};
    cuuint64_t strides[3] = {(cuuint64_t)tok_stride * 2, CHUNK * 2, (cuuint64_t)page_stride * 2};
    cuuint32_t box[4] = {CHUNK, KB, (cuuint32_t)(hd / CHUNK), 1};
    cuuint32_t estr[4] = {1, 1, 1, 1};
    r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(cache), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  } else {
    // dims: elements of one token row (all KV heads), 16 tokens of a page, pages; box = [64 dims x 16 tokens] of one page
    cuuint64_t dims[3] = {(cuuint64_t)(heads * hd), PAGE, (cuuint64_t)num_pages};
    cuuint64_t strides[2] = {(cuuint64_t)tok_stride * 2, (cuuint64_t)page_stride * 2};
    cuuint32_t box[3] = {CHUNK, PAGE, 1};
    cuuint32_t estr[3] = {1, 1, 1};
    r = enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(cache), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  }
  return r == CUDA_SUCCESS ? MARY_OK : MARY_ERR_CUDA;
}

template <int DK, int DV, bool SPLITP, bool BIAS, int MAPS = 0>
int launch_fa(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const FaParams& p, int NB, cudaStream_t s) {
  static MarySmemSlots smem_set = {};
  constexpr int SMEM = FaCfg<DK, DV, SPLITP, BIAS, MAPS>::SMEM;
  if (int rc = mary_ensure_dyn_smem((const void*)fa_prefill_kernel<DK, DV, SPLITP, BIAS, MAPS>, SMEM, &smem_set)) return rc;
  fa_prefill_kernel<DK, DV, SPLITP, BIAS, MAPS><<<dim3(p.Hq, NB), FaCfg<DK, DV, SPLITP, BIAS, MAPS>::NTHREADS, SMEM, s>>>(tq, tk, tv, p);
  MARY_CHECK_LAUNCH();
  return MARY_OK;
}

}  // namespace

MARY_API int mary_attention_prefill_tile_rows() { return TR; }

// 1 when the tensor-core prefill kernel exists for these head dims.
MARY_API int mary_attention_prefill_supported(int DK, int DV) {
  return (DK == 64 && DV == 64) || (DK == 128 && DV == 128) || (DK == 192 && DV == 128) || (DK == 256 && DV == 256);
}

// The same with an attention form of one map.
MARY_API int mary_attention_prefill_form_supported(int DK, int DV) {
  return (DK == 64 && DV == 64) || (DK == 128 && DV == 128) || (DK == 128 && DV == 64) || (DK == 256 && DV == 256);
}

// The same for two maps of DK values each.
MARY_API int mary_attention_prefill_maps_supported(int DK, int DV) {
  return (DK == 64 && DV == 64) || (DK == 64 && DV == 128) || (DK == 128 && DV == 128);
}

// q [T, Hq, DK] bf16 contiguous; kcache [pages, page_size (16 or 64), Hkv, DK] and vcache [.., Hkv, DV] bf16 with element strides per token
// and per page (heads contiguous inside a token row); out [T, Hq, DV] bf16.  blk_seq / blk_tok0: NB tiles of at most 128 query
// tokens that never cross a sequence.  Causal with the last query token of a sequence at position kv_len - 1; window > 0 keeps
// keys (pos - window, pos].  out_ld: elements between the output rows of two tokens (0: Hq * DV; a multiple of 8).  split_p: softmax
// weights with 16 significant bits.  bias [Hq][window] (or null; with split_p and equal widths only) is added to the scaled score by
// distance, gate (or null; 16-byte aligned rows) multiplies the output by its logistic function.  form (or null; with split_p, without bias): see attention_form.cuh; with two
// maps query and key rows have 2 DK values per head and T may exceed a row's pitch as form->q_ld says.  Returns MARY_ERR_BAD_ARG for head dims without an instantiation.
MARY_API int mary_attention_prefill(const void* q, const void* kcache, const void* vcache, void* out, const int* page_table,
                                    const int* kv_len, const int* q_start, const int* blk_seq, const int* blk_tok0, int NB, int T, int Hq,
                                    int Hkv, int DK, int DV, int num_pages, int max_pages, int64_t k_tok_stride, int64_t k_page_stride,
                                    int64_t v_tok_stride, int64_t v_page_stride, int window, float scale, int page_size,
                                    int64_t out_ld, int split_p, const float* bias, const void* gate, int64_t gate_ld, const MaryAttnForm* form, cudaStream_t s) {
  if (NB <= 0) return MARY_OK;
  if (NB > 65535) return MARY_ERR_BAD_ARG;
  const int maps = form && form->maps == 2 ? 2 : 1;
  if (form && (form->maps > 2 || !split_p || bias || (maps == 2 && (gate || form->sink || form->turn)) || (form->turn && (gate || ((uintptr_t)form->turn & 15))))) return MARY_ERR_BAD_ARG;
  const bool formed = form && maps == 1 && (form->chunk > 0 || form->sink || form->temp_every > 0 || form->cap > 0.f || form->turn);
  if (!(maps == 2 ? mary_attention_prefill_maps_supported(DK, DV)
                  : formed ? mary_attention_prefill_form_supported(DK, DV) : mary_attention_prefill_supported(DK, DV)) || Hkv < 1 || Hq % Hkv || (page_size != PAGE && page_size != KB)) return MARY_ERR_BAD_ARG;
  if ((k_tok_stride * 2) % 16 || (k_page_stride * 2) % 16 || (v_tok_stride * 2) % 16 || (v_page_stride * 2) % 16) return MARY_ERR_BAD_ARG;
  CUtensorMap tq, tk, tv;
  const uint64_t q_ld = form && form->q_ld > 0 ? (uint64_t)form->q_ld : (uint64_t)Hq * maps * DK;
  if (q_ld % 8 || ((uintptr_t)q & 15)) return MARY_ERR_BAD_ARG;
  int rc = mary_make_tmap_2d(&tq, q, 4, (uint64_t)T, (uint64_t)Hq * maps * DK, q_ld, TR, CHUNK, 1);
  if (rc) return rc;
  if ((rc = make_cache_map(&tk, kcache, Hkv * maps, DK, num_pages, k_tok_stride, k_page_stride, page_size))) return rc;
  if ((rc = make_cache_map(&tv, vcache, Hkv, DV, num_pages, v_tok_stride, v_page_stride, page_size))) return rc;
  FaParams p;
  p.page_table = page_table; p.kv_len = kv_len; p.q_start = q_start; p.blk_seq = blk_seq; p.blk_tok0 = blk_tok0;
  p.out = (__nv_bfloat16*)out; p.max_pages = max_pages; p.Hq = Hq; p.Hkv = Hkv; p.window = window; p.page = page_size;
  p.out_ld = out_ld > 0 ? out_ld : (int64_t)Hq * DV;
  p.bias = bias; p.gate = (const __nv_bfloat16*)gate; p.gate_ld = gate_ld;
  if (p.out_ld % 8 || ((uintptr_t)out & 15) || gate_ld % 8 || ((uintptr_t)gate & 15)) return MARY_ERR_BAD_ARG;
  if (bias && (!split_p || DK != DV || window < 1)) return MARY_ERR_BAD_ARG;
  p.scale_log2 = scale * 1.4426950408889634f; p.status = mary_status_ptr();
  p.f = form ? *form : MaryAttnForm{};
  if (maps == 2) {
    if (DV == 64) return launch_fa<64, 64, true, false, 2>(tq, tk, tv, p, NB, s);
    if (DK == 64) return launch_fa<64, 128, true, false, 2>(tq, tk, tv, p, NB, s);
    return launch_fa<128, 128, true, false, 2>(tq, tk, tv, p, NB, s);
  }
  if (formed) {
    if (DK == 128 && DV == 64) return launch_fa<128, 64, true, false, 1>(tq, tk, tv, p, NB, s);
    if (DK == 64) return launch_fa<64, 64, true, false, 1>(tq, tk, tv, p, NB, s);
    if (DK == 128) return launch_fa<128, 128, true, false, 1>(tq, tk, tv, p, NB, s);
    return launch_fa<256, 256, true, false, 1>(tq, tk, tv, p, NB, s);
  }
  if (bias) {
    if (DK == 64) return launch_fa<64, 64, true, true>(tq, tk, tv, p, NB, s);
    if (DK == 128) return launch_fa<128, 128, true, true>(tq, tk, tv, p, NB, s);
    return launch_fa<256, 256, true, true>(tq, tk, tv, p, NB, s);
  }
  if (split_p) {
    if (DK == 64) return launch_fa<64, 64, true, false>(tq, tk, tv, p, NB, s);
    if (DK == 128) return launch_fa<128, 128, true, false>(tq, tk, tv, p, NB, s);
    if (DK == 192) return launch_fa<192, 128, true, false>(tq, tk, tv, p, NB, s);
    return launch_fa<256, 256, true, false>(tq, tk, tv, p, NB, s);
  }
  if (DK == 64) return launch_fa<64, 64, false, false>(tq, tk, tv, p, NB, s);
  if (DK == 128) return launch_fa<128, 128, false, false>(tq, tk, tv, p, NB, s);
  if (DK == 192) return launch_fa<192, 128, false, false>(tq, tk, tv, p, NB, s);
  return launch_fa<256, 256, false, false>(tq, tk, tv, p, NB, s);
}
