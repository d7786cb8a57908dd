// Attention over all heads of a query at once (see csrc/joint_attention.cu) for sm_100a on tcgen05 / TMEM / TMA, with the keys on the
// 128-row side of the tensor core:
//
//   S^T[128 keys x columns] = K Q^T        O^T[128 value channels x columns] += V^T P^T
//
// A column is one (head, query) pair; the columns of a key/value head are adjacent and padded to 16.  So a thread owns a key and finds
// the scores of all heads for it in its own TMEM lane: mixing them is arithmetic on registers, and a few queries or heads leave no row
// of the tensor core idle.
//
//   warps 0-3 (0-15 for prompts)   scores -> probabilities, written as bf16 to shared memory (the B operand of P V)
//   then one warp each            MMA issuer; TMA producer of [128 keys x 64 channels] pieces in a ring of slots of one or two pieces
//   last two warps                row sums of the probabilities (mma.sync with a column of ones), so that numerator and denominator
//                                 hold the same rounded numbers
//
// Modes:
//   * mixed heads over prompts: a CTA takes up to 32 queries of all heads; its softmax warpgroups share them.
//   * mixed heads, one token per row: a slice of the keys.
//   * latent rows, one token per row: up to 64 heads read one row per key, its first channels are the value; the rows pass through the
//     ring twice, once for each product (the second time from L2).
//
// Mixed scores are bounded (the cap, or the product of unit queries and keys, times the row sums of the mix), so the softmax of the
// first two modes takes a fixed reference; the caller checks that the range fits fp32 exponents.  With r = 1 / (1 + exp2(k2 x)) a capped
// score is softcap (1 - 2 r), and in log2 units
//   score_h - reference_h = init_h + near_h[distance] + sum_g w[h, g] r_g.
// Latent scores take an online softmax whose reference moves only when a maximum grew by more than 2^8.
#include <string.h>

#include "mma_sync.cuh"

namespace tyr {

constexpr int KM_KEYS = 128;                   // keys of a tile
constexpr uint32_t KM_PIECE = KM_KEYS * 128;   // bytes of [128 keys x 64 channels]
constexpr int KM_SLOTS = 12;                   // most ring slots
constexpr int KM_COLS = 256;                   // most score columns

enum KmMode : int { KM_PROMPT = 0, KM_STEP = 1, KM_LATENT = 2 };

struct KmArgs {
  const __nv_bfloat16* q;                      // by (batch, token, head) strides
  __nv_bfloat16* out;
  const int* pos;                              // step: position of each row's token
  long long q_sb, q_ss, q_sh, out_sb, out_ss, out_sh;
  int S, H, G, rep, dk, dv;                    // S: tokens of a prompt
  int rn, nq, cols;                            // columns of a key/value head, queries, columns in all (G rn)
  int kp, vp, mb;                              // pieces of a key and of a value, 128-channel blocks of a value
  int pps, slots;                              // pieces of a ring slot, slots
  int lq;                                      // log2 of nq
  int hb;                                      // latent: heads of a CTA
  int cap, ring, window, splits;
  const float* near;                           // mixed heads: [H, reach + 1]
  int reach;
  uint16_t col[32];                            // first column of a head
  uint32_t prow[32];                           // and the byte offset of its row of probabilities
  float scale_log2;                            // latent
  float *part_acc, *part_ml;                   // [B, splits, H, dv], [B, splits, H, 2]: merged by a launch of its own
  int* err;
};

// Mixed heads: w [HT, HT], init and k2 [HT] of the scores above.  Kernel parameters, so that the arithmetic takes them as constants.
template <int HT>
struct KmTalk {
  float w[HT * HT], init[HT], k2[HT];
};

struct KmBars {
  uint64_t full[KM_SLOTS], empty[KM_SLOTS], q_ready, s_ready[2], s_free, p_ready, p_free, o_done, l_ready, wg[2];
  uint32_t tmem_base;
  int rescale_at;                              // latent: tile at which the sums and O were last scaled by `factor`
};

// Byte offsets from a 1024-byte aligned base.
struct KmLayout {
  uint32_t q, p, ring, bars, m, factor, wmax, total;
  __host__ __device__ KmLayout(int mode, int cols, int kp, int pps, int slots) {
    ring = 0;
    q = slots * pps * KM_PIECE;
    p = q + static_cast<uint32_t>(cols) * kp * 128;          // cols is a multiple of 16: both start on a swizzle atom
    bars = p + static_cast<uint32_t>(cols) * 256;
    m = bars + ((sizeof(KmBars) + 15) & ~15u);
    factor = m + (mode == KM_LATENT ? cols * 4 : 0);
    wmax = factor + (mode == KM_LATENT ? cols * 4 : 0);
    total = wmax + (mode == KM_LATENT ? cols * 16 : 0);
    // a value block of one piece: the MMA's upper 64 rows read whatever follows the slot (their results are not used)
    if (pps == 1 && total < q + KM_PIECE) total = q + KM_PIECE;
  }
};

template <bool V>
struct KmFlag {
  static constexpr bool value = V;
};

template <int N>
__device__ __forceinline__ void km_ld(uint32_t addr, uint32_t* r) {
  static_assert(N == 1 || N == 2 || N == 4 || N == 32, "");
  if constexpr (N == 1) asm volatile("tcgen05.ld.sync.aligned.32x32b.x1.b32 {%0}, [%1];" : "=r"(r[0]) : "r"(addr) : "memory");
  if constexpr (N == 2) asm volatile("tcgen05.ld.sync.aligned.32x32b.x2.b32 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
  if constexpr (N == 4)
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// HT: heads a thread handles (padded), QB: queries it takes at a time, WGS: softmax warpgroups.
template <int MODE, int HT, int QB, int WGS>
__global__ void __launch_bounds__((WGS * 4 + 4) * 32, 1)
joint_keymajor_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV, const __grid_constant__ KmArgs a,
                      const __grid_constant__ KmTalk<HT> tk) {
  constexpr int SB = MODE == KM_PROMPT ? 1 : 2;            // score buffers
  constexpr int SOFT = WGS * 4, THREADS = (SOFT + 4) * 32;
  pdl_trigger();
  extern __shared__ uint8_t km_raw[];
  uint8_t* const smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(km_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const KmLayout lay(MODE, a.cols, a.kp, a.pps, a.slots);
  KmBars& s = *reinterpret_cast<KmBars*>(smem + lay.bars);
  float* const sm_m = reinterpret_cast<float*>(smem + lay.m);
  float* const sm_f = reinterpret_cast<float*>(smem + lay.factor);
  float* const sm_w = reinterpret_cast<float*>(smem + lay.wmax);
  float* const sm_l = reinterpret_cast<float*>(smem + lay.q);          // 1 / row sums, over the queries once all products are done
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    for (int i = 0; i < a.slots; ++i) {
      mbar_init(&s.full[i], 1);
      mbar_init(&s.empty[i], 1);
    }
    mbar_init(&s.s_ready[0], 1);
    mbar_init(&s.s_ready[1], 1);
    mbar_init(&s.q_ready, SOFT + 2);
    mbar_init(&s.s_free, SOFT);
    mbar_init(&s.p_ready, SOFT);
    mbar_init(&s.p_free, 3);                               // P V retired, two summing warps
    mbar_init(&s.o_done, 1);
    mbar_init(&s.l_ready, 2);
    mbar_init(&s.wg[0], 4);
    mbar_init(&s.wg[1], 4);
    s.rescale_at = -1;
    mbar_fence_init();
  }
  if (warp == SOFT) {
    tmem_alloc(&s.tmem_base, 512);
    tmem_relinquish();
  }
  pdl_wait();
  // ---- what this CTA works on
  int b, h0 = 0, nh = a.H, i0 = 0, tiles, lo = 0, hi = 0, n_keys = 0, split = 0;
  bool valid = true;
  if constexpr (MODE == KM_PROMPT) {
    b = blockIdx.y;
    i0 = (gridDim.x - 1 - blockIdx.x) * a.nq;              // the longest rows first
    tiles = (min(i0 + a.nq, a.S) + KM_KEYS - 1) / KM_KEYS;
  } else {
    split = blockIdx.x;
    b = blockIdx.z;
    if (MODE == KM_LATENT) {
      h0 = blockIdx.y * a.hb;
      nh = min(a.hb, a.H - h0);
    }
    const int pos = a.pos[b];
    valid = pos >= 0 && (a.ring || pos < a.cap);
    if (!valid && tid == 0) report_error(a.err, ERR_BOUNDS, pos);
    // slots [lo, hi) of the store: a ring holds its last `cap` positions in an order that does not matter here
    n_keys = pos + 1;
    if (a.ring) n_keys = min(n_keys, a.cap);
    const int seen = a.window > 0 ? min(n_keys, a.window) : n_keys, first = n_keys - seen;
    int chunk = (seen + a.splits - 1) / a.splits;
    chunk = (chunk + KM_KEYS - 1) / KM_KEYS * KM_KEYS;
    lo = first + min(split * chunk, seen);
    hi = min(lo + chunk, n_keys);
    tiles = valid ? (hi - lo + KM_KEYS - 1) / KM_KEYS : 0;
  }
  if (MODE == KM_LATENT)
    for (int x = tid; x < a.cols; x += THREADS) { sm_m[x] = -INFINITY; sm_f[x] = 1.f; }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = s.tmem_base, o_base = tmem + SB * a.cols;
  const uint32_t slot_bytes = a.pps * KM_PIECE, ring = smem_u32(smem + lay.ring);
  const int ku = (a.kp + a.pps - 1) / a.pps;               // ring slots of one key
  const int vpb = min(2, a.vp);                            // pieces of a 128-channel value block (the last may have fewer)

  // ---- queries -> shared memory, K-major with the 128-byte swizzle: [key/value head][piece][column][64 channels]; by the softmax and
  // summing warps, while the first keys are on their way
  if (warp < SOFT || warp >= SOFT + 2) {
    constexpr int STAGERS = (SOFT + 2) * 32;
    const int me = warp < SOFT ? tid : tid - 64;
    const int chunks = a.kp * 8, n = a.cols * chunks;      // 16-byte chunks of a column
    constexpr int U = 4;                                   // loads in flight
    for (int x0 = me; x0 < n; x0 += U * STAGERS) {
      uint4 v[U];
      uint32_t at[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int x = x0 + u * STAGERS;
        const int col = x / chunks, c = x - col * chunks, g = col / a.rn, r = col - g * a.rn;
        int h, i = 0;
        bool live = x < n && valid && c * 8 < a.dk;
        if constexpr (MODE == KM_PROMPT) {
          h = g * a.rep + (r >> a.lq);
          i = i0 + (r & (a.nq - 1));
          live = live && (r >> a.lq) < a.rep && i < a.S;
        } else {
          h = MODE == KM_LATENT ? h0 + r : g * a.rep + r;
          live = live && r < (MODE == KM_LATENT ? nh : a.rep);
        }
        at[u] = lay.q + (static_cast<uint32_t>(g * a.kp + (c >> 3)) * a.rn + r) * 128 + (((c & 7) ^ (r & 7)) << 4);
        v[u] = live ? *reinterpret_cast<const uint4*>(a.q + b * a.q_sb + i * a.q_ss + h * a.q_sh + c * 8) : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (x0 + u * STAGERS < n) *reinterpret_cast<uint4*>(smem + at[u]) = v[u];
    }
    fence_proxy_async();
    __syncwarp();
    if (lane == 0) mbar_arrive(&s.q_ready);
  }

  if (warp == SOFT + 1) {
    // ------------------------------------------------------------------ TMA producer
    if (elect_one() && tiles > 0) {
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmV);
      uint32_t it = 0;
      bool ok = true;
      auto load = [&](const CUtensorMap* tm, int g, int piece, int count, int key) {
        const int st = it % a.slots;
        if (!mbar_wait(&s.empty[st], ((it / a.slots) & 1) ^ 1, a.err, 2500 + st)) { ok = false; return; }
        mbar_expect_tx(&s.full[st], count * KM_PIECE);
        for (int i = 0; i < count; ++i)
          tma_load_4d(smem + lay.ring + st * slot_bytes + i * KM_PIECE, tm, &s.full[st], (piece + i) * 64, g, key, b);
        ++it;
      };
      auto keys = [&](int j) {
        for (int g = 0; g < a.G && ok; ++g)
          for (int u = 0; u < ku && ok; ++u) load(&tmK, g, u * a.pps, min(a.pps, a.kp - u * a.pps), lo + j * KM_KEYS);
      };
      keys(0);
      for (int j = 0; j < tiles && ok; ++j) {
        if (j + 1 < tiles) keys(j + 1);
        for (int g = 0; g < a.G && ok; ++g)
          for (int m = 0; m < a.mb && ok; ++m) load(&tmV, g, m * 2, min(vpb, a.vp - m * 2), lo + j * KM_KEYS);
      }
      if (!ok)                                             // let the copies in flight land before the CTA unwinds
        for (uint32_t x = (it > static_cast<uint32_t>(a.slots) ? it - a.slots : 0); x < it; ++x)
          mbar_wait(&s.full[x % a.slots], (x / a.slots) & 1, nullptr, 0);
    }
  } else if (warp == SOFT) {
    // ------------------------------------------------------------------ MMA issuer
    if (elect_one() && tiles > 0) {
      const uint32_t id_s = make_idesc_f16(1, 128, a.rn, 0, 0), id_o = make_idesc_f16(1, 128, a.rn, 1, 0);
      // descriptors of the operands' first rows; the issuing thread only adds to their low words
      const uint64_t dq = make_smem_desc_sw128(smem_u32(smem + lay.q), 16, 1024), dp = make_smem_desc_sw128(smem_u32(smem + lay.p), 16, 1024);
      const uint64_t dk = make_smem_desc_sw128(ring, 16, 1024), dv = make_smem_desc_sw128(ring, KM_PIECE, 1024);
      const uint32_t piece_q = a.rn * 128;                 // bytes of 64 channels (or keys) of a key/value head's columns
      uint32_t st = 0, phase = 0;
      bool ok = mbar_wait(&s.q_ready, 0, a.err, 2590);
      auto wait_slot = [&]() {
        ok = ok && mbar_wait(&s.full[st], phase, a.err, 2600 + st);
        tc_fence_after();
        return st * slot_bytes;
      };
      auto free_slot = [&]() {
        umma_commit(&s.empty[st]);
        if (++st == static_cast<uint32_t>(a.slots)) { st = 0; phase ^= 1; }
      };
      auto scores = [&](int j) {
        const uint32_t s_col = tmem + (SB == 2 ? (j & 1) * a.cols : 0);
        for (int g = 0; g < a.G && ok; ++g)
          for (int u = 0; u < ku && ok; ++u) {
            const uint64_t ka = smem_desc_advance(dk, wait_slot());
            if (!ok) break;
            const int steps = min(a.pps * 4, (a.dk - u * a.pps * 64 + 15) / 16);
            const uint64_t qa = smem_desc_advance(dq, (g * a.kp + u * a.pps) * piece_q);
            const uint32_t d = s_col + g * a.rn;
#pragma unroll
            for (int k = 0; k < 8; ++k)
              if (k < steps)
                umma_f16_ss(d, smem_desc_advance(ka, (k >> 2) * KM_PIECE + (k & 3) * 32), smem_desc_advance(qa, (k >> 2) * piece_q + (k & 3) * 32), id_s,
                            u > 0 || k > 0 ? 1u : 0u);
            free_slot();
          }
        umma_commit(&s.s_ready[SB == 2 ? j & 1 : 0]);
      };
      if (ok) scores(0);
      for (int j = 0; j < tiles && ok; ++j) {
        // the next tile's scores: two buffers, of which the other went free when the probabilities of tile j - 1 were complete, or one,
        // free as soon as every thread has taken its scores
        if (j + 1 < tiles) {
          if (SB == 1) {
            ok = mbar_wait(&s.s_free, j & 1, a.err, 2610);
            tc_fence_after();
          }
          if (ok) scores(j + 1);
        }
        ok = ok && mbar_wait(&s.p_ready, j & 1, a.err, 2620);
        tc_fence_after();
        for (int g = 0; g < a.G && ok; ++g)
          for (int m = 0; m < a.mb && ok; ++m) {
            const uint64_t va = smem_desc_advance(dv, wait_slot()), pa = smem_desc_advance(dp, g * a.rn * 256);
            if (!ok) break;
            const uint32_t d = o_base + (g * a.mb + m) * a.rn;
#pragma unroll
            for (int k = 0; k < KM_KEYS / 16; ++k)
              umma_f16_ss(d, smem_desc_advance(va, k * 2048), smem_desc_advance(pa, (k >> 2) * piece_q + (k & 3) * 32), id_o, j > 0 || k > 0 ? 1u : 0u);
            free_slot();
          }
        umma_commit(&s.p_free);
      }
      umma_commit(&s.o_done);
    }
  } else if (warp >= SOFT + 2) {
    // ------------------------------------------------------------------ row sums of the probabilities
    const int w = warp - SOFT - 2, g8 = lane >> 2;
    float acc[KM_COLS / 32][4];
#pragma unroll
    for (int x = 0; x < KM_COLS / 32; ++x) acc[x][0] = acc[x][1] = acc[x][2] = acc[x][3] = 0.f;
    uint32_t row[KM_COLS / 32];                            // this lane's row of every 16-row block
#pragma unroll
    for (int x = 0; x < KM_COLS / 32; ++x) {
      const int n = (2 * x + w) * 16 + (lane & 15), gg = n / a.rn;
      row[x] = lay.p + static_cast<uint32_t>(gg) * a.rn * 256 + (n - gg * a.rn) * 128;
    }
    bool ok = true;
    for (int j = 0; j < tiles && ok; ++j) {
      ok = mbar_wait(&s.p_ready, j & 1, a.err, 2630 + w);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      if (MODE == KM_LATENT && *reinterpret_cast<volatile int*>(&s.rescale_at) == j) {
#pragma unroll
        for (int x = 0; x < KM_COLS / 32; ++x)
          if ((2 * x + w) * 16 < a.cols) {
            acc[x][0] *= sm_f[(2 * x + w) * 16 + g8];
            acc[x][2] *= sm_f[(2 * x + w) * 16 + g8 + 8];
          }
      }
#pragma unroll
      for (int k = 0; k < 8; ++k)
#pragma unroll
        for (int x = 0; x < KM_COLS / 32; ++x) {
          const int n0 = (2 * x + w) * 16;
          if (n0 >= a.cols) break;
          uint32_t f[4];
          ldsm4(f, smem + row[x] + (k >> 2) * a.rn * 128 + ((((k & 3) * 2 + (lane >> 4)) ^ (lane & 7)) << 4));
          mma_bf16(acc[x], f, 0x3f803f80u, 0x3f803f80u);
        }
      __syncwarp();
      if (lane == 0) mbar_arrive(&s.p_free);
    }
    // the queries' space is free once every product is done (an empty slice: once everybody has written to it)
    ok = ok && mbar_wait(tiles == 0 ? &s.q_ready : &s.o_done, 0, a.err, 2640 + w);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
#pragma unroll
      for (int x = 0; x < KM_COLS / 32; ++x) {
        const int n0 = (2 * x + w) * 16;
        if (n0 < a.cols && (lane & 3) == 0) {
          const bool part = MODE != KM_PROMPT && a.splits > 1;        // parts keep the sums, results their reciprocals
          sm_l[n0 + g8] = part ? acc[x][0] : 1.f / acc[x][0];
          sm_l[n0 + g8 + 8] = part ? acc[x][2] : 1.f / acc[x][2];
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&s.l_ready);
  } else {
    // ------------------------------------------------------------------ scores -> probabilities
    const int wg = warp >> 2, quarter = warp & 3, key = quarter * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quarter * 32) << 16;
    uint8_t* const p_row = smem + lay.p + (key >> 6) * (a.rn * 128);               // column n of head g: + g rn 256 + n 128 + swizzled p_off
    const uint32_t p_off = (key & 63) * 2;
    bool ok = true;
    for (int j = 0; j < tiles && ok; ++j) {
      ok = mbar_wait(&s.s_ready[SB == 2 ? j & 1 : 0], SB == 2 ? (j >> 1) & 1 : j & 1, a.err, 2700 + warp);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const uint32_t s_addr = tmem + lane_addr + (SB == 2 ? (j & 1) * a.cols : 0);
      const int kj = lo + j * KM_KEYS + key;                                        // this thread's key (slot of the store)
      auto p_writable = [&]() {
        if (j == 0) return true;
        const bool w = mbar_wait(&s.p_free, (j - 1) & 1, a.err, 2720 + warp);
        return static_cast<bool>(__all_sync(0xffffffffu, w));
      };
      if constexpr (MODE != KM_LATENT) {
        const int nqw = MODE == KM_PROMPT ? a.nq / WGS : 1, q_first = MODE == KM_PROMPT ? wg * nqw : 0;
        const int i_first = MODE == KM_PROMPT ? i0 + q_first : n_keys - 1;          // position of the first query
        const int tile_end = lo + j * KM_KEYS + KM_KEYS - 1;
        const bool edge = i_first - tile_end < a.reach || (MODE == KM_STEP && tile_end >= hi);
        for (int qb = 0; qb < nqw; qb += QB) {
          const int q0 = q_first + qb;
          float y[HT][QB];
          {
            uint32_t x[HT][QB];
#pragma unroll
            for (int h = 0; h < HT; ++h) km_ld<QB>(s_addr + a.col[h] + q0, x[h]);      // heads past the last: the last again
            tmem_wait_ld();
#pragma unroll
            for (int h = 0; h < HT; ++h)
#pragma unroll
              for (int e = 0; e < QB; ++e) y[h][e] = rcp(1.f + ex2(__uint_as_float(x[h][e]) * tk.k2[h]));
          }
          if (SB == 1 && qb + QB >= nqw) {                 // the last scores of the tile are in registers
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&s.s_free);
          }
          if (qb == 0 && !(ok = p_writable())) break;
          uint32_t off[QB];
#pragma unroll
          for (int e = 0; e < QB; ++e) off[e] = (q0 + e) * 128 + (p_off ^ (((q0 + e) & 7) << 4));
          // EDGE: some of the tile's pairs are masked or nearer than the last distance
          auto mix = [&](auto edge_t) {
            constexpr bool EDGE = decltype(edge_t)::value;
#pragma unroll
            for (int h = 0; h < HT; ++h) {
              if (h >= a.H) break;
              float c[QB];
#pragma unroll
              for (int e = 0; e < QB; ++e) c[e] = tk.init[h];
#pragma unroll
              for (int k = 0; k < HT; ++k)
#pragma unroll
                for (int e = 0; e < QB; ++e) c[e] = fmaf(y[k][e], tk.w[h * HT + k], c[e]);
              if constexpr (EDGE) {
                const float* nr = a.near + static_cast<long long>(h) * (a.reach + 1);
#pragma unroll
                for (int e = 0; e < QB; ++e) {
                  const int d = i_first + qb + e - kj;
                  c[e] += __ldg(nr + min(max(d, 0), a.reach));
                  if (MODE == KM_PROMPT ? d < 0 : kj >= hi) c[e] = -INFINITY;
                }
              }
              uint8_t* const dst = p_row + a.prow[h];
              // a single query: the swizzle follows the head's row
#pragma unroll
              for (int e = 0; e < QB; ++e)
                *reinterpret_cast<__nv_bfloat16*>(dst + (MODE == KM_STEP ? p_off ^ ((a.prow[h] >> 3) & 0x70) : off[e])) = __float2bfloat16(ex2(c[e]));
            }
          };
          if (edge) mix(KmFlag<true>{}); else mix(KmFlag<false>{});
        }
        if (!ok) break;
      } else {
        // online softmax over this warpgroup's share of the columns, 32 at a time; a warp's maxima meet in shared memory
        const bool live = kj < hi;
        const int half = WGS == 2 ? (a.cols / 16 + 1) / 2 * 16 : a.cols, c_lo = wg * half, c_hi = min(a.cols, c_lo + half);
        for (int c0 = c_lo; c0 < c_hi; c0 += 32) {
          uint32_t x[32];
          tmem_ld_32x32(s_addr + c0, x);                   // columns past the last may be read; they are not used
          tmem_wait_ld();
          float v[32];
#pragma unroll
          for (int e = 0; e < 32; ++e) v[e] = live ? __uint_as_float(x[e]) * a.scale_log2 : -INFINITY;
          // lane c ends with the maximum of column c over the warp's keys
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) {
            const bool up = lane & o;
#pragma unroll
            for (int e = 0; e < o; ++e) {
              const float send = up ? v[e] : v[e + o], keep = up ? v[e + o] : v[e];
              v[e] = fmaxf(keep, __shfl_xor_sync(0xffffffffu, send, o));
            }
          }
          if (c0 + lane < c_hi) sm_w[quarter * a.cols + c0 + lane] = v[0];
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(&s.wg[wg]);
        ok = mbar_wait(&s.wg[wg], 0, a.err, 2740);         // phases of this barrier: two to a tile
        ok = __all_sync(0xffffffffu, ok) && p_writable();  // also: the summing warps are done with the last factors
        if (!ok) break;
        // a thread owns a column: its reference, and the factor that a move of it asks for
        bool grow = false;
        if (c_lo + key < c_hi) {
          const int c = c_lo + key;
          const float mx = fmaxf(fmaxf(sm_w[c], sm_w[a.cols + c]), fmaxf(sm_w[2 * a.cols + c], sm_w[3 * a.cols + c]));
          const float m = sm_m[c];
          const bool up = mx > m + 8.f;                    // also the first tile: m is -inf
          sm_f[c] = up ? ex2(m - mx) : 1.f;
          if (up) sm_m[c] = mx;
          grow = up && j > 0;
        }
        if (__any_sync(0xffffffffu, grow) && lane == 0) *reinterpret_cast<volatile int*>(&s.rescale_at) = j;
        __syncwarp();
        if (lane == 0) mbar_arrive(&s.wg[wg]);
        ok = mbar_wait(&s.wg[wg], 1, a.err, 2741);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (*reinterpret_cast<volatile int*>(&s.rescale_at) == j) {    // P V of the tile before has retired: O is idle
          tc_fence_after();
          for (int mbk = 0; mbk < a.mb; ++mbk)
            for (int c0 = c_lo; c0 < c_hi; c0 += 16) {
              uint32_t o[16];
              tmem_ld_32x16(o_base + lane_addr + mbk * a.rn + c0, o);
              tmem_wait_ld();
#pragma unroll
              for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * sm_f[c0 + e]);
              tmem_st_32x16(o_base + lane_addr + mbk * a.rn + c0, o);
            }
          tmem_wait_st();
        }
        for (int c0 = c_lo; c0 < c_hi; c0 += 16) {
          uint32_t x[16];
          tmem_ld_32x16(s_addr + c0, x);
          tmem_wait_ld();
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const int n = c0 + e;
            const float p = live ? ex2(fmaf(__uint_as_float(x[e]), a.scale_log2, -sm_m[n])) : 0.f;
            *reinterpret_cast<__nv_bfloat16*>(p_row + n * 128 + (p_off ^ ((n & 7) << 4))) = __float2bfloat16(p);
          }
        }
      }
      tc_fence_before();
      fence_proxy_async();                                 // the probabilities are read by the tensor core
      __syncwarp();
      if (lane == 0) mbar_arrive(&s.p_ready);
    }
    // ---------------------------------------------------------------- O^T: lane = value channel, column = (head, query)
    if (ok && tiles > 0) ok = mbar_wait(&s.o_done, 0, a.err, 2760 + warp);
    if (ok) ok = mbar_wait(&s.l_ready, 0, a.err, 2780 + warp);
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    const long long part = static_cast<long long>(b) * a.splits + split;
    __nv_bfloat16* const sm_o = reinterpret_cast<__nv_bfloat16*>(smem + lay.p);
    const uint32_t o_row = a.H * a.dv;
    if (ok && valid) {
      for (int m = 0; m < a.mb; ++m) {
        const int d = m * 128 + key;
        for (int g = 0; g < a.G; ++g)
          for (int n0 = wg * 16; n0 < a.rn; n0 += 16 * WGS) {
            uint32_t o[16];
            if (tiles > 0) {
              tmem_ld_32x16(o_base + lane_addr + (g * a.mb + m) * a.rn + n0, o);
              tmem_wait_ld();
            } else {
#pragma unroll
              for (int e = 0; e < 16; ++e) o[e] = 0u;
            }
            if (d >= a.dv) continue;
            const float* l = sm_l + g * a.rn + n0;
#pragma unroll
            for (int e = 0; e < 16; ++e) {
              const int n = n0 + e;
              if constexpr (MODE == KM_PROMPT) {           // over the probabilities: [query][head][channel]
                const int r = n >> a.lq;
                if (r < a.rep) sm_o[static_cast<uint32_t>(n & (a.nq - 1)) * o_row + (g * a.rep + r) * a.dv + d] = __float2bfloat16(__uint_as_float(o[e]) * l[e]);
              } else {
                const int h = h0 + (MODE == KM_LATENT ? n : g * a.rep + n);
                if (n >= (MODE == KM_LATENT ? nh : a.rep)) break;
                if (a.splits == 1) a.out[b * a.out_sb + h * a.out_sh + d] = __float2bfloat16(__uint_as_float(o[e]) * l[e]);
                else a.part_acc[(part * a.H + h) * a.dv + d] = __uint_as_float(o[e]);
                if (a.splits > 1 && d == 0) {
                  a.part_ml[(part * a.H + h) * 2] = MODE == KM_LATENT ? sm_m[n] : 0.f;
                  a.part_ml[(part * a.H + h) * 2 + 1] = l[e];
                }
              }
            }
          }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == SOFT) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
  if constexpr (MODE == KM_PROMPT) {                       // rows of 8 channels
    const int chunks = a.H * a.dv / 8, per = a.dv / 8;
    for (int x = tid; x < a.nq * chunks; x += THREADS) {
      const int i = x / chunks, c = x - i * chunks, h = c / per, d = (c - h * per) * 8;
      if (i0 + i < a.S)
        *reinterpret_cast<uint4*>(a.out + b * a.out_sb + (i0 + i) * a.out_ss + h * a.out_sh + d) = *reinterpret_cast<const uint4*>(smem + lay.p + static_cast<uint32_t>(x) * 16);
    }
  }
}

// Slices of a step -> result: one CTA per (row, head), a thread per channel.
__global__ void __launch_bounds__(128) joint_merge_kernel(const float* __restrict__ acc, const float* __restrict__ ml, __nv_bfloat16* __restrict__ out, int H, int dv,
                                                          int splits, long long out_sb, long long out_sh) {
  __shared__ float w[32];
  pdl_entry();
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31;
  if (threadIdx.x < 32) {
    const float* src = ml + ((static_cast<long long>(b) * splits + lane) * H + h) * 2;
    const float mx = lane < splits ? src[0] : -INFINITY, lx = lane < splits ? src[1] : 0.f;
    const float M = warp_max(mx), f = ex2(mx - M), L = warp_sum(f * lx);
    w[lane] = f / L;
  }
  __syncthreads();
  for (int d = threadIdx.x; d < dv; d += 128) {
    const float* src = acc + (static_cast<long long>(b) * splits * H + h) * dv + d;
    float v = 0.f;
#pragma unroll 8
    for (int i = 0; i < splits; ++i) v += w[i] * src[static_cast<long long>(i) * H * dv];
    out[b * out_sb + h * out_sh + d] = __float2bfloat16(v);
  }
}

}  // namespace tyr

using namespace tyr;

namespace {
typedef CUresult (*KmEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                               const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
KmEncodeFn km_encode() {
  static KmEncodeFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<KmEncodeFn>(ptr);
  }
  return fn;
}
// bf16 (channel, head, key, batch) by element strides; a box is 64 channels of 128 keys.
int km_map(CUtensorMap* tm, const void* base, int D, int G, int T, int B, long long sg, long long st, long long sb) {
  KmEncodeFn fn = km_encode();
  if (!fn) return 1;
  cuuint64_t dims[4] = {(cuuint64_t)D, (cuuint64_t)G, (cuuint64_t)T, (cuuint64_t)B};
  cuuint64_t strides[3] = {(cuuint64_t)(G == 1 ? D : sg) * 2, (cuuint64_t)st * 2, (cuuint64_t)(B == 1 ? st * T : sb) * 2};
  cuuint32_t box[4] = {64, 1, KM_KEYS, 1}, es[4] = {1, 1, 1, 1};
  return fn(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : 2;
}

constexpr uint32_t kKmSmem = 227 * 1024 - 1024;            // less the room for alignment

// Fills in the sizes that follow from the shapes; false: the kernel does not take them.
bool km_plan(int mode, KmArgs& a) {
  if (a.H <= 0 || a.G <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || (a.dk & 15) || a.splits < 1 || a.splits > 32) return false;
  a.rep = a.H / a.G;
  a.kp = (a.dk + 63) / 64;
  a.vp = (a.dv + 63) / 64;
  a.mb = (a.vp + 1) / 2;
  a.pps = a.kp > 1 || a.vp > 1 ? 2 : 1;
  const int sb = mode == KM_PROMPT ? 1 : 2;
  auto fits = [&](int min_slots) {
    a.cols = a.G * a.rn;
    if (a.rn > 256 || a.cols > KM_COLS || sb * a.cols + a.cols * a.mb > 512) return false;
    for (a.slots = KM_SLOTS; a.slots >= min_slots; --a.slots)
      if (KmLayout(mode, a.cols, a.kp, a.pps, a.slots).total <= kKmSmem) return true;
    return false;
  };
  if (mode == KM_LATENT) {
    if (a.G != 1) return false;
    for (a.rn = a.H >= 64 ? 64 : (a.H + 15) / 16 * 16; a.rn >= 16; a.rn -= 16) {
      a.nq = 1;
      a.hb = a.rn;
      if (fits(3)) return true;
    }
    return false;
  }
  if (a.H > 32) return false;
  if (mode == KM_STEP) {
    a.nq = 1;
    a.rn = (a.rep + 15) / 16 * 16;
    return fits(2);
  }
  if ((a.dv & 7) || a.mb > 1) return false;                // results leave through the probabilities' space, in rows of 8 channels
  const int least = a.H <= 8 ? 16 : 8;                     // a warpgroup takes a quarter of the queries, 4 or 2 at a time
  for (a.nq = 32, a.lq = 5; a.nq >= least; a.nq /= 2, --a.lq) {
    a.rn = (a.rep * a.nq + 15) / 16 * 16;
    if (fits(2)) return true;
  }
  return false;
}

// `talk`: on the host, w [HT, HT], init [HT], k2 [HT] (null for latent rows).
template <int MODE, int HT, int QB, int WGS>
int km_launch(const CUtensorMap& tk, const CUtensorMap& tv, KmArgs& a, const float* talk, dim3 grid, void* stream) {
  KmTalk<HT> t{};
  if (talk != nullptr) memcpy(&t, talk, sizeof(t));
  for (int h = 0; h < HT && MODE != KM_LATENT; ++h) {
    const int x = h < a.H ? h : a.H - 1, g = x / a.rep, r = x % a.rep;
    a.col[h] = static_cast<uint16_t>(g * a.rn + r * a.nq);
    a.prow[h] = static_cast<uint32_t>(g) * a.rn * 256 + r * a.nq * 128;
  }
  auto kernel = joint_keymajor_kernel<MODE, HT, QB, WGS>;
  static bool configured[64] = {};               // the attribute is per device
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
  if (!configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kKmSmem + 1024);
    if (e != cudaSuccess) return 1000 + (int)e;
    configured[dev] = true;
  }
  const size_t smem = KmLayout(MODE, a.cols, a.kp, a.pps, a.slots).total + 1024;
  return (int)launch_dependent(kernel, grid, dim3((WGS * 4 + 4) * 32), smem, (cudaStream_t)stream, tk, tv, a, t);
}
}  // namespace

// Heads of a CTA for these sizes (0: the kernel does not take them).  mode 0 prompts, 1 steps of mixed heads, 2 steps over latent rows.
extern "C" TYR_EXPORT int tyr_keymajor_heads(int mode, int H, int G, int dk, int dv) {
  KmArgs a{};
  a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.splits = 1;
  if (mode < 0 || mode > 2 || !km_plan(mode, a)) return 0;
  return mode == KM_LATENT ? a.hb : H;
}

// Mixed heads over whole bf16 prompts.  strides: (batch, token, head) of q, k, v, out; dk multiple of 16, dv of 8, 16-byte aligned rows.
// `talk` lies on the host: w [HT, HT], init [HT], k2 [HT] with HT = 8, 16 or 32, the smallest that holds H; near [H, reach + 1] on the device.
extern "C" TYR_EXPORT int tyr_keymajor_prompt(const void* q, const void* k, const void* v, void* out, const float* talk, const float* near, int reach, const long long* st, int B, int S, int H, int G,
                                              int dk, int dv, int dvp, int* err, void* stream) {
  KmArgs a{};
  a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.splits = 1;
  if (B <= 0 || B > 65535 || S <= 0 || dv > dvp || (dvp & 7) || reach < 0 || !km_plan(KM_PROMPT, a)) return -1;
  for (int i = 0; i < 12; ++i)
    if (st[i] & 7) return -3;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(out)) & 15) return -4;
  a.q = (const __nv_bfloat16*)q; a.out = (__nv_bfloat16*)out; a.S = S; a.err = err;
  a.q_sb = st[0]; a.q_ss = st[1]; a.q_sh = st[2]; a.out_sb = st[9]; a.out_ss = st[10]; a.out_sh = st[11];
  a.near = near; a.reach = reach;
  CUtensorMap tk, tv;
  if (int r = km_map(&tk, k, dk, G, S, B, st[5], st[4], st[3])) return 3000 + r;
  if (int r = km_map(&tv, v, dvp, G, S, B, st[8], st[7], st[6])) return 4000 + r;
  const dim3 grid((S + a.nq - 1) / a.nq, B);
  return H <= 8 ? km_launch<KM_PROMPT, 8, 4, 4>(tk, tv, a, talk, grid, stream)
                : (H <= 16 ? km_launch<KM_PROMPT, 16, 2, 4>(tk, tv, a, talk, grid, stream) : km_launch<KM_PROMPT, 32, 2, 4>(tk, tv, a, talk, grid, stream));
}

// One token per row over bf16 stores that hold it.  talk null: latent rows [B, 1, cap, dk] whose first dv channels are the values of all
// heads (a ring must hold exactly the window), scale; else mixed heads over stores [B, G, cap, dk] and [B, G, cap, dvp].  strides:
// (batch, head) of q, then of out.  workspace: [B, splits, H, dv + 2] floats where splits > 1.
extern "C" TYR_EXPORT int tyr_keymajor_step(const void* q, const void* k, const void* v, void* out, const int* pos, const float* talk,
                                            const float* near, int reach, float scale, void* workspace,
                                            const long long* st, int B, int H, int G, int dk, int dv, int dvp, int cap, int ring, int window,
                                            int splits, int* err, void* stream) {
  KmArgs a{};
  const int mode = talk == nullptr ? KM_LATENT : KM_STEP;
  a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.splits = splits;
  if (B <= 0 || B > 65535 || cap <= 0 || window < 0 || reach < 0 || dv > dvp || (dvp & 7) || !km_plan(mode, a)) return -1;
  if ((mode == KM_STEP && (ring || window)) || (ring && window && window < cap) || (splits > 1 && workspace == nullptr)) return -2;
  if (((st[0] | st[1]) & 7) || ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15))
    return -3;
  a.q = (const __nv_bfloat16*)q; a.out = (__nv_bfloat16*)out; a.pos = pos; a.err = err;
  a.q_sb = st[0]; a.q_sh = st[1]; a.out_sb = st[2]; a.out_sh = st[3];
  a.near = near; a.reach = reach;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.cap = cap; a.ring = ring; a.window = window;
  a.part_acc = (float*)workspace;
  a.part_ml = a.part_acc + static_cast<long long>(B) * H * splits * dv;
  CUtensorMap tk, tv;
  if (int r = km_map(&tk, k, dk, G, cap, B, static_cast<long long>(cap) * dk, dk, static_cast<long long>(G) * cap * dk)) return 3000 + r;
  if (int r = km_map(&tv, v, dvp, G, cap, B, static_cast<long long>(cap) * dvp, dvp, static_cast<long long>(G) * cap * dvp)) return 4000 + r;
  int rc;
  if (mode == KM_LATENT) {
    const dim3 grid(splits, (H + a.hb - 1) / a.hb, B);
    rc = a.rn >= 32 ? km_launch<KM_LATENT, 8, 1, 2>(tk, tv, a, nullptr, grid, stream) : km_launch<KM_LATENT, 8, 1, 1>(tk, tv, a, nullptr, grid, stream);
  } else {
    const dim3 grid(splits, 1, B);
    rc = H <= 8 ? km_launch<KM_STEP, 8, 1, 1>(tk, tv, a, talk, grid, stream)
                : (H <= 16 ? km_launch<KM_STEP, 16, 1, 1>(tk, tv, a, talk, grid, stream) : km_launch<KM_STEP, 32, 1, 1>(tk, tv, a, talk, grid, stream));
  }
  if (rc != 0 || splits == 1) return rc;
  return (int)launch_dependent(joint_merge_kernel, dim3(H, B), dim3(128), 0, (cudaStream_t)stream, static_cast<const float*>(a.part_acc),
                               static_cast<const float*>(a.part_ml), a.out, H, dv, splits, a.out_sb, a.out_sh);
}
