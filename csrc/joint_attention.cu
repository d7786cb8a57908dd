// Attention in which all heads of a query are worked on together, because their scores are mixed or because they share one key:
//
//   s_g(i, j) = softcap tanh(scale temp_g q_g . k / softcap) + rel[bucket(i - j), g]
//   score_h   = sum_g talk[h, g] s_g                          (each step optional), j <= i, 0 <= i - j < window,
//
// softmax over the visible keys of every head.  Keys and values are separate rows, or the values are the first channels of the keys
// (one latent row for all heads).  csrc/joint_tcgen05.cu has the form for scores of bounded range; these take every score, and the sizes
// that one does not hold.
//
//   * prompt:  mixed heads over bf16 prompts.  One CTA owns 16 (or 8) queries with all their heads and walks the keys in tiles: Q K^T of all
//              heads, cap and bias on the way to shared memory; the mix as a product of `talk` with the scores of every (query, key) pair
//              on the tensor cores (a TF32 product of scores split in two, so that they keep 21 bits); online softmax by the warp that
//              owns the query; P V of all heads.  P V of a tile and Q K^T of the next share a phase.
//   * step:    one token per row over a bf16 store.  A CTA takes a slice of the keys and all heads (mixed) or a block of them (latent
//              rows: many heads read one row); tiles arrive through a cp.async ring; slices meet in the last CTA to finish.
//   * general: one CTA per (query, block of heads), fp32 arithmetic, any sizes, fp32 or bf16; keys of a prompt or of a store (plain or
//              ring).
//
// Compiled without fast math.
#include "mma_sync.cuh"

namespace tyr {

__device__ __forceinline__ float ja_load(const float* p) { return *p; }
__device__ __forceinline__ float ja_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ja_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void ja_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// What happens to the scores between the product and the softmax; null pointers and softcap 0 leave a step out.
struct ScoreArgs {
  const float* temp;           // [H]
  const float* rel;            // [rows, H]
  const int* bucket;           // [reach + 1]: row of a distance; distances past reach take the last entry
  const float* talk;           // [H, H]
  int reach;
  int rows;                    // rows of rel
  int talk_exact;              // the entries of talk are exact in TF32
  float scale, softcap;
};

struct JointArgs {
  const void *q, *k, *v;       // q: [B, S, H, .]; k / v: [B, ., G, .] by (batch, position or slot, head) element strides
  void* out;                   // [B * S, H, .] by row and head strides
  const int* pos;              // position of query 0 of each row (nullable: 0)
  long long q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh, out_ld, out_hs;
  int B, S, H, G, dk, dv, cap, ring, window, keys, hb;     // hb: heads of a CTA (all of them when they are mixed)
  ScoreArgs sc;
  int* err;
};

constexpr int JA_KEYS = 32;

template <typename T>
__global__ void __launch_bounds__(256) joint_general_kernel(JointArgs a) {
  extern __shared__ __align__(16) float ja_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h0 = blockIdx.y * a.hb, nh = min(a.hb, a.H - h0), rep = a.H / a.G;
  float* const sq = ja_smem;                              // [hb, dk]
  float* const acc = sq + a.hb * a.dk;                    // [hb, dv]
  float* const s = acc + a.hb * a.dv;                     // [hb, JA_KEYS] scores, then probabilities
  float* const s2 = s + a.hb * JA_KEYS;                   // [hb, JA_KEYS] mixed scores
  float* const m = s2 + a.hb * JA_KEYS;                   // [hb] running maximum, sum and this tile's factor
  float* const l = m + a.hb;
  float* const f = l + a.hb;
  pdl_entry();
  const long long row = blockIdx.x;
  const int b = static_cast<int>(row / a.S), i = static_cast<int>(row % a.S);
  const int p = (a.pos ? a.pos[b] : 0) + i;
  if (p < 0 || (!a.ring && p >= a.keys)) {                // a query without its own key in the store: report, leave the output
    if (tid == 0) report_error(a.err, ERR_BOUNDS, p);
    return;
  }
  const T* qp = static_cast<const T*>(a.q) + b * a.q_sb + i * a.q_ss + h0 * a.q_sh;
  for (int x = tid; x < nh * a.dk; x += 256) sq[x] = ja_load(qp + (x / a.dk) * a.q_sh + x % a.dk);
  for (int x = tid; x < nh * a.dv; x += 256) acc[x] = 0.f;
  for (int x = tid; x < nh; x += 256) { m[x] = -INFINITY; l[x] = 0.f; }
  __syncthreads();
  int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  if (a.ring) lo = max(lo, p - a.cap + 1);
  for (int base = lo; base <= p; base += JA_KEYS) {
    const int j = min(base + lane, p), slot = a.ring ? j % a.cap : j;      // keys past the query are masked below
    const T* kb = static_cast<const T*>(a.k) + b * a.k_sb + static_cast<long long>(slot) * a.k_ss;
    for (int h = warp; h < nh; h += 8) {
      const T* kr = kb + ((h0 + h) / rep) * a.k_sh;
      const float* qr = sq + h * a.dk;
      float dot = 0.f;
      for (int d = 0; d < a.dk; ++d) dot += qr[d] * ja_load(kr + d);
      dot *= a.sc.scale;
      if (a.sc.temp) dot *= a.sc.temp[h0 + h];
      if (a.sc.softcap > 0.f) dot = a.sc.softcap * tanhf(dot / a.sc.softcap);
      if (a.sc.rel) dot += a.sc.rel[static_cast<long long>(a.sc.bucket[min(p - j, a.sc.reach)]) * a.H + h0 + h];
      s[h * JA_KEYS + lane] = dot;
    }
    if (a.sc.talk) {
      __syncthreads();
      for (int h = warp; h < nh; h += 8) {
        float t = 0.f;
        for (int g = 0; g < a.H; ++g) t += a.sc.talk[h * a.H + g] * s[g * JA_KEYS + lane];
        s2[h * JA_KEYS + lane] = t;
      }
      __syncthreads();
    }
    const float* sc = a.sc.talk ? s2 : s;
    for (int h = warp; h < nh; h += 8) {
      const float x = base + lane <= p ? sc[h * JA_KEYS + lane] : -INFINITY;
      const float mo = m[h], mn = fmaxf(mo, warp_max(x)), w = expf(x - mn);
      const float sum = warp_sum(w);
      s[h * JA_KEYS + lane] = w;
      __syncwarp();
      if (lane == 0) {
        f[h] = expf(mo - mn);
        l[h] = l[h] * f[h] + sum;
        m[h] = mn;
      }
    }
    __syncthreads();
    const int nk = min(JA_KEYS, p - base + 1);
    const T* vb = static_cast<const T*>(a.v) + b * a.v_sb;
    for (int x = tid; x < nh * a.dv; x += 256) {
      const int h = x / a.dv;
      const T* vc = vb + ((h0 + h) / rep) * a.v_sh + x % a.dv;
      float o = acc[x] * f[h];
      for (int t = 0; t < nk; ++t) o += s[h * JA_KEYS + t] * ja_load(vc + static_cast<long long>(a.ring ? (base + t) % a.cap : base + t) * a.v_ss);
      acc[x] = o;
    }
    __syncthreads();
  }
  T* op = static_cast<T*>(a.out) + row * a.out_ld + h0 * a.out_hs;
  for (int x = tid; x < nh * a.dv; x += 256) ja_store(op + (x / a.dv) * a.out_hs + x % a.dv, acc[x] / l[x / a.dv]);
}


// ---- shared pieces of the tensor-core forms --------------------------------------------------------------------------
constexpr float kLog2e = 1.4426950408889634f;

// softcap tanh(x / softcap) by one exponential: k2 = 2 log2(e) (factors of the product) / softcap
__device__ __forceinline__ float ja_cap(float x, float k2, float softcap) { return softcap - 2.f * softcap * rcp(1.f + ex2(x * k2)); }

// talk[16 mt + (g, g + 8)][8 kk + (t, t + 4)] as the A operand, zeros outside; rows of ts floats
__device__ __forceinline__ void ja_talk_frag(uint32_t (&hi)[4], uint32_t (&lo)[4], const float* talk, int ts, int mt, int kk, int g, int t) {
#pragma unroll
  for (int e = 0; e < 4; ++e) split_tf32(talk[(mt * 16 + g + (e & 1) * 8) * ts + kk * 8 + t + (e >> 1) * 4], hi[e], lo[e]);
}

// One 8-pair tile of mixed scores: c[16 heads of mt x 8 pairs] = talk x s, s at s0[head * hs + pair].
__device__ __forceinline__ void ja_mix_step(float (&c)[4], const uint32_t (&hi)[4], const uint32_t (&lo)[4], bool exact, const float* s0, int hs, int kk,
                                            int g, int t) {
  uint32_t bh0, bl0, bh1, bl1;
  split_tf32(s0[(kk * 8 + t) * hs + g], bh0, bl0);
  split_tf32(s0[(kk * 8 + t + 4) * hs + g], bh1, bl1);
  mma_tf32(c, hi, bh0, bh1);
  mma_tf32(c, hi, bl0, bl1);
  if (!exact) mma_tf32(c, lo, bh0, bh1);
}

// ---- prompts with mixed heads ----------------------------------------------------------------------------------------
struct JointPromptArgs {
  const __nv_bfloat16 *q, *k, *v;        // heads of a token adjacent: rows of H dk, G dk, G dvp channels by (batch, token) strides
  __nv_bfloat16* out;                    // [B, S, H, dv]
  long long q_sb, q_ss, k_sb, k_ss, v_sb, v_ss;
  int S, H, G, dk, dv, dvp;              // dk and dvp multiples of 16
  ScoreArgs sc;
};
constexpr int JP_THREADS = 512, JP_WARPS = 16, JP_UNITS = 2, JP_BUCKETS = 2048;

// Byte offsets of the shared-memory parts; HPM heads share a 16-row tile, so a CTA has 16 / HPM queries.
struct JointPromptLayout {
  int q, k, v, s, p, talk, rel, alpha, bucket, total;
  int ts;                                // floats of a talk row
  __host__ __device__ JointPromptLayout(int hpm, int n, int H, int G, int dk, int dvp, int rows, int reach) {
    const int mq = 16 / hpm, h8 = (H + 7) / 8 * 8, h16 = (H + 15) / 16 * 16;
    auto up = [](int x) { return (x + 15) & ~15; };
    ts = h8 + 4;
    q = 0;
    k = up(q + mq * (H * dk + 8) * 2);
    v = up(k + n * (G * dk + 8) * 2);
    s = up(v + n * (G * dvp + 8) * 2 + 64);              // a column block of 32 may reach past the last row's end
    p = up(s + h8 * (mq * (n + 8) + 8) * 4);
    talk = up(p + H * (mq * (n + 8) + 8) * 2);
    rel = up(talk + h16 * ts * 4);
    alpha = up(rel + H * (rows | 1) * 4);
    bucket = up(alpha + H * mq * 4);
    total = up(bucket + (reach < JP_BUCKETS ? (reach + 1) * 2 : 0));
  }
};

// Work of one phase over 16-row tiles: a unit is up to two tiles of one key/value head and one block of columns (keys or channels).
template <int HPM>
struct JointTiles {
  int rep, tpg, ppg;                     // heads, tiles and pairs of tiles of a key/value head
  __device__ JointTiles(int H, int G) : rep(H / G), tpg((rep + HPM - 1) / HPM), ppg((tpg + 1) / 2) {}
  // head of a row half of tile s of group g; HPM 2: the halves are two heads (the second may be missing: the first again)
  __device__ int head(int g, int s, int half) const { return g * rep + (HPM == 1 ? s : min(2 * s + half, rep - 1)); }
  __device__ bool real(int s, int half) const { return HPM == 1 || 2 * s + half < rep; }
};

template <int HPM, int N>
__global__ void __launch_bounds__(JP_THREADS, 1) joint_prompt_kernel(JointPromptArgs a) {
  constexpr int MQ = 16 / HPM, NS = N + 8, HS = MQ * NS + 8, PS = N + 8, PH = MQ * PS + 8, MI = HPM == 1 ? 2 : 1;
  extern __shared__ __align__(16) uint8_t jp_smem[];
  const JointPromptLayout lay(HPM, N, a.H, a.G, a.dk, a.dvp, a.sc.rows, a.sc.reach);
  __nv_bfloat16* const sq = reinterpret_cast<__nv_bfloat16*>(jp_smem + lay.q);
  __nv_bfloat16* const sk = reinterpret_cast<__nv_bfloat16*>(jp_smem + lay.k);
  __nv_bfloat16* const sv = reinterpret_cast<__nv_bfloat16*>(jp_smem + lay.v);
  float* const ss = reinterpret_cast<float*>(jp_smem + lay.s);
  __nv_bfloat16* const sp = reinterpret_cast<__nv_bfloat16*>(jp_smem + lay.p);
  float* const talk = reinterpret_cast<float*>(jp_smem + lay.talk);
  float* const rel = reinterpret_cast<float*>(jp_smem + lay.rel);
  float* const alpha = reinterpret_cast<float*>(jp_smem + lay.alpha);
  uint16_t* const bucket = reinterpret_cast<uint16_t*>(jp_smem + lay.bucket);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int lr = lane & 15, lc = (lane >> 4) * 8, br = (lane & 7) + ((lane >> 4) << 3), bc = ((lane >> 3) & 1) * 8;
  const int H = a.H, G = a.G, dk = a.dk, dvp = a.dvp, reach = a.sc.reach, rrow = a.sc.rows | 1, h8 = (H + 7) / 8;
  const int qs = H * dk + 8, krow = G * dk + 8, vrow = G * dvp + 8;
  const int i0 = (gridDim.x - 1 - blockIdx.x) * MQ, b = blockIdx.y;      // the longest rows first
  const int tiles = (min(i0 + MQ, a.S) + N - 1) / N;
  const JointTiles<HPM> map(H, G);
  const bool small = reach < JP_BUCKETS, exact = a.sc.talk_exact != 0;
  pdl_entry();
  {
    const __nv_bfloat16* qp = a.q + b * a.q_sb;
    const int n = H * dk / 8;
    for (int x = tid; x < MQ * n; x += JP_THREADS) {
      const int r = x / n, d = (x - r * n) * 8;
      cp16_zfill(sq + r * qs + d, qp + min(i0 + r, a.S - 1) * a.q_ss + d, i0 + r < a.S);
    }
  }
  auto fetch_k = [&](int j) {
    const __nv_bfloat16* kp = a.k + b * a.k_sb;
    const int n = G * dk / 8;
    for (int x = tid; x < N * n; x += JP_THREADS) {
      const int r = x / n, d = (x - r * n) * 8, p = j * N + r;
      cp16_zfill(sk + r * krow + d, kp + min(p, a.S - 1) * a.k_ss + d, p < a.S);
    }
  };
  auto fetch_v = [&](int j) {
    const __nv_bfloat16* vp = a.v + b * a.v_sb;
    const int n = G * dvp / 8;
    for (int x = tid; x < N * n; x += JP_THREADS) {
      const int r = x / n, d = (x - r * n) * 8, p = j * N + r;
      cp16_zfill(sv + r * vrow + d, vp + min(p, a.S - 1) * a.v_ss + d, p < a.S);
    }
  };
  fetch_k(0);
  cp_commit();
  fetch_v(0);
  cp_commit();
  for (int x = tid; x < (H + 15) / 16 * 16 * lay.ts; x += JP_THREADS) {
    const int r = x / lay.ts, c = x % lay.ts;
    talk[x] = r < H && c < H ? a.sc.talk[r * H + c] : 0.f;
  }
  for (int x = tid; x < H * a.sc.rows; x += JP_THREADS) rel[(x % H) * rrow + x / H] = a.sc.rel[x];
  if (small)
    for (int x = tid; x <= reach; x += JP_THREADS) bucket[x] = static_cast<uint16_t>(a.sc.bucket[x]);
  for (int x = tid; x < (h8 * 8 - H) * HS; x += JP_THREADS) ss[H * HS + x] = 0.f;      // scores of heads that do not exist
  auto row_of = [&](int n) { n = min(max(n, 0), reach); return small ? static_cast<int>(bucket[n]) : a.sc.bucket[n]; };

  // ---- Q K^T of tile j, capped and with the distance bias -> ss
  auto products = [&](int j) {
    const int base = j * N;
    const bool far = i0 - (base + N - 1) >= reach;         // every pair of the tile is past the table's steps
    for (int u = warp; u < G * map.ppg * (N / 16); u += JP_WARPS) {
      const int kb = u % (N / 16), gp = u / (N / 16), kv = gp / map.ppg, s0 = gp % map.ppg * 2;
      const bool two = s0 + 1 < map.tpg;
      float c[2][2][4];
#pragma unroll
      for (int x = 0; x < 16; ++x) (&c[0][0][0])[x] = 0.f;
      const int lh = HPM == 1 ? 0 : lr >> 3, lq = HPM == 1 ? lr : lr & 7;
      const __nv_bfloat16* qa = sq + lq * qs + map.head(kv, s0, lh) * dk + lc;
      const __nv_bfloat16* qb = sq + lq * qs + map.head(kv, two ? s0 + 1 : s0, lh) * dk + lc;
      const __nv_bfloat16* kp = sk + (kb * 16 + br) * krow + kv * dk + bc;
#pragma unroll 4
      for (int x = 0; x < dk; x += 16) {
        uint32_t f[4], kf[4];
        ldsm4(kf, kp + x);
        ldsm4(f, qa + x);
        mma_bf16(c[0][0], f, kf[0], kf[1]);
        mma_bf16(c[0][1], f, kf[2], kf[3]);
        if (two) {
          ldsm4(f, qb + x);
          mma_bf16(c[1][0], f, kf[0], kf[1]);
          mma_bf16(c[1][1], f, kf[2], kf[3]);
        }
      }
      int rw[2][4];                                        // table rows of this lane's pairs
      if (!far) {
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int r = 0; r < (HPM == 1 ? 2 : 1); ++r) {
            const int n = i0 + g + 8 * r - (base + kb * 16 + 8 * e + 2 * t);
            rw[e][2 * r] = row_of(n);
            rw[e][2 * r + 1] = row_of(n - 1);
          }
      }
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        if (w == 1 && !two) break;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          if (!map.real(s0 + w, r)) continue;
          const int h = map.head(kv, s0 + w, r);
          const float k2 = 2.f * kLog2e * a.sc.scale * a.sc.temp[h] / a.sc.softcap;
          const float* rh = rel + h * rrow;
          const float last = rh[a.sc.rows - 1];
          float* dst = ss + h * HS + (HPM == 1 ? g + 8 * r : g) * NS + kb * 16 + 2 * t;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int ri = HPM == 1 ? 2 * r : 0;
            float2 y;
            y.x = ja_cap(c[w][e][2 * r], k2, a.sc.softcap) + (far ? last : rh[rw[e][ri]]);
            y.y = ja_cap(c[w][e][2 * r + 1], k2, a.sc.softcap) + (far ? last : rh[rw[e][ri + 1]]);
            *reinterpret_cast<float2*>(dst + 8 * e) = y;
          }
        }
      }
    }
  };

  float o[JP_UNITS][2][4][4];
#pragma unroll
  for (int x = 0; x < JP_UNITS * 32; ++x) (&o[0][0][0][0])[x] = 0.f;
  float m[MI][2], l[MI][2];
#pragma unroll
  for (int x = 0; x < MI; ++x) { m[x][0] = m[x][1] = -INFINITY; l[x][0] = l[x][1] = 0.f; }
  const int mq = HPM == 1 ? warp : warp & 7;               // this warp's query in the mix, and its tiles of 16 heads
  const int nc = (dvp + 31) / 32, units = G * map.ppg * nc;

  cp_wait<1>();
  __syncthreads();
  products(0);
  __syncthreads();
  if (tiles > 1) fetch_k(1);
  cp_commit();
  for (int j = 0; j < tiles; ++j) {
    const int base = j * N, i = i0 + mq;
    // ---- mix and softmax of this warp's query
#pragma unroll
    for (int x = 0; x < MI; ++x) {
      const int mt = HPM == 1 ? x : warp >> 3;
      if (mt * 16 >= H) break;
      float c[N / 8][4];
#pragma unroll
      for (int n = 0; n < N / 8; ++n) c[n][0] = c[n][1] = c[n][2] = c[n][3] = 0.f;
      for (int kk = 0; kk < h8; ++kk) {
        uint32_t hi[4], lo[4];
        ja_talk_frag(hi, lo, talk, lay.ts, mt, kk, g, t);
#pragma unroll
        for (int n = 0; n < N / 8; ++n) ja_mix_step(c[n], hi, lo, exact, ss + mq * NS + n * 8, HS, kk, g, t);
      }
      if (base + N - 1 > i) {
#pragma unroll
        for (int n = 0; n < N / 8; ++n)
#pragma unroll
          for (int e = 0; e < 2; ++e)
            if (base + n * 8 + 2 * t + e > i) c[n][e] = c[n][2 + e] = -INFINITY;
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float mx = -INFINITY;
#pragma unroll
        for (int n = 0; n < N / 8; ++n) mx = fmaxf(mx, fmaxf(c[n][2 * r], c[n][2 * r + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2)) * kLog2e;
        float f = 1.f;                                     // the reference moves only when the maximum has grown by more than 2^8
        if (mx > m[x][r] + 8.f) {
          f = ex2(m[x][r] - mx);
          l[x][r] *= f;
          m[x][r] = mx;
        }
        const int h = mt * 16 + g + 8 * r;
        const bool live = h < H;
        if (live && t == 0) alpha[h * MQ + mq] = f;
        __nv_bfloat16* dst = sp + h * PH + mq * PS + 2 * t;
#pragma unroll
        for (int n = 0; n < N / 8; ++n) {
          const float p0 = ex2(fmaf(c[n][2 * r], kLog2e, -m[x][r])), p1 = ex2(fmaf(c[n][2 * r + 1], kLog2e, -m[x][r]));
          l[x][r] += p0 + p1;
          if (live) *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16x2(p0, p1);
        }
      }
    }
    cp_wait<0>();
    __syncthreads();                                       // probabilities complete, scores read, values and the next keys there
    // ---- P V of this tile
#pragma unroll
    for (int y = 0; y < JP_UNITS; ++y) {
      const int u = warp + y * JP_WARPS;
      if (u >= units) break;
      const int cb = u % nc, gp = u / nc, kv = gp / map.ppg, s0 = gp % map.ppg * 2;
      const bool two = s0 + 1 < map.tpg;
      float f[2][2];
#pragma unroll
      for (int w = 0; w < 2; ++w)
#pragma unroll
        for (int r = 0; r < 2; ++r) f[w][r] = w == 1 && !two ? 1.f : alpha[map.head(kv, s0 + w, r) * MQ + (HPM == 1 ? g + 8 * r : g)];
      if (__any_sync(0xffffffffu, f[0][0] != 1.f || f[0][1] != 1.f || f[1][0] != 1.f || f[1][1] != 1.f)) {
#pragma unroll
        for (int w = 0; w < 2; ++w)
#pragma unroll
          for (int e = 0; e < 4; ++e) { o[y][w][e][0] *= f[w][0]; o[y][w][e][1] *= f[w][0]; o[y][w][e][2] *= f[w][1]; o[y][w][e][3] *= f[w][1]; }
      }
      const int lh = HPM == 1 ? 0 : lr >> 3, lq = HPM == 1 ? lr : lr & 7;
      const __nv_bfloat16* pa = sp + map.head(kv, s0, lh) * PH + lq * PS + lc;
      const __nv_bfloat16* pb = sp + map.head(kv, two ? s0 + 1 : s0, lh) * PH + lq * PS + lc;
      const __nv_bfloat16* vp = sv + lr * vrow + kv * dvp + cb * 32 + lc;
#pragma unroll
      for (int x = 0; x < N / 16; ++x) {
        uint32_t v0[4], v1[4], pf[4];
        ldsm4_t(v0, vp + x * 16 * vrow);
        ldsm4_t(v1, vp + x * 16 * vrow + 16);
        ldsm4(pf, pa + x * 16);
        mma_bf16(o[y][0][0], pf, v0[0], v0[1]);
        mma_bf16(o[y][0][1], pf, v0[2], v0[3]);
        mma_bf16(o[y][0][2], pf, v1[0], v1[1]);
        mma_bf16(o[y][0][3], pf, v1[2], v1[3]);
        if (two) {
          ldsm4(pf, pb + x * 16);
          mma_bf16(o[y][1][0], pf, v0[0], v0[1]);
          mma_bf16(o[y][1][1], pf, v0[2], v0[3]);
          mma_bf16(o[y][1][2], pf, v1[0], v1[1]);
          mma_bf16(o[y][1][3], pf, v1[2], v1[3]);
        }
      }
    }
    if (j + 1 < tiles) products(j + 1);
    __syncthreads();
    if (j + 1 < tiles) fetch_v(j + 1);
    if (j + 2 < tiles) fetch_k(j + 2);
    cp_commit();
  }
  cp_wait<0>();
#pragma unroll
  for (int x = 0; x < MI; ++x) {
    const int mt = HPM == 1 ? x : warp >> 3;
    if (mt * 16 >= H) break;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float sum = l[x][r];
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      const int h = mt * 16 + g + 8 * r;
      if (h < H && t == 0) alpha[h * MQ + mq] = 1.f / sum;
    }
  }
  __syncthreads();
#pragma unroll
  for (int y = 0; y < JP_UNITS; ++y) {
    const int u = warp + y * JP_WARPS;
    if (u >= units) break;
    const int cb = u % nc, gp = u / nc, kv = gp / map.ppg, s0 = gp % map.ppg * 2;
#pragma unroll
    for (int w = 0; w < 2; ++w) {
      if (w == 1 && s0 + 1 >= map.tpg) break;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int h = map.head(kv, s0 + w, r), qi = HPM == 1 ? g + 8 * r : g;
        if (!map.real(s0 + w, r) || i0 + qi >= a.S) continue;
        const float f = alpha[h * MQ + qi];
        __nv_bfloat16* dst = a.out + ((static_cast<long long>(b) * a.S + i0 + qi) * H + h) * a.dv;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = cb * 32 + e * 8 + 2 * t;
          const float x = o[y][w][e][2 * r] * f, z = o[y][w][e][2 * r + 1] * f;
          if (d + 1 < a.dv && (a.dv & 1) == 0) {
            *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16x2(x, z);
          } else {
            if (d < a.dv) dst[d] = __float2bfloat16(x);
            if (d + 1 < a.dv) dst[d + 1] = __float2bfloat16(z);
          }
        }
      }
    }
  }
}

// ---- one token per row -------------------------------------------------------------------------------------------------
struct JointStepArgs {
  const __nv_bfloat16* q;                // [B, H, dk] by (batch, head) strides
  const __nv_bfloat16 *k, *v;            // [B, G, cap, dk], [B, G, cap, dvp]; v null: values are the first channels of the keys (G == 1)
  __nv_bfloat16* out;                    // [B, H, dv] by (batch, head) strides
  const int* pos;                        // [B]
  float *part_acc, *part_ml;             // [B, splits, H, dv], [B, splits, H, 2]
  int* counters;                         // [B, blocks of heads]
  long long q_sb, q_sh, out_sb, out_sh;
  int B, H, G, dk, dv, dvp, cap, ring, window, splits, hb, stages;
  ScoreArgs sc;
  int* err;
};
constexpr int JS_THREADS = 256, JS_WARPS = 8;

struct JointStepLayout {
  int stage, k_bytes, q, s, s2, p, talk, rel, ml, total;
  int ts, mt;                            // floats of a talk row; 16-row tiles of heads
  __host__ __device__ JointStepLayout(bool mixed, int n, int hb, int G, int dk, int dvp, int vg, int rows, int stages) {
    const int rep = hb / G, h8 = (hb + 7) / 8 * 8, h16 = (hb + 15) / 16 * 16;
    auto up = [](int x) { return (x + 15) & ~15; };
    ts = h8 + 4;
    mt = mixed ? G * ((rep + 15) / 16) : (hb + 15) / 16;
    k_bytes = up(n * (G * dk + 8) * 2);
    stage = k_bytes + (vg ? up(n * (vg * dvp + 8) * 2) : 0);
    q = stages * stage + 64;                             // a column block of 32 may reach past the last row's end
    s = up(q + mt * 16 * (dk + 8) * 2);
    s2 = up(s + h16 * (n + 8) * 4);
    p = mixed ? up(s2 + h16 * (n + 8) * 4) : s2;
    talk = up(p + mt * 16 * (n + 8) * 2);
    rel = mixed ? up(talk + h16 * ts * 4) : talk;
    ml = mixed ? up(rel + hb * (rows | 1) * 4) : talk;
    total = up(ml + 3 * h16 * 4);
  }
};

// UNITS: blocks of (16 heads x 32 value channels) a warp accumulates.
template <bool MIXED, int N, int UNITS>
__global__ void __launch_bounds__(JS_THREADS, 1) joint_step_kernel(JointStepArgs a) {
  constexpr int NS = N + 8, KB = N / 16;
  extern __shared__ __align__(16) uint8_t js_smem[];
  __shared__ int s_last;
  const int split = blockIdx.x, hblk = blockIdx.y, b = blockIdx.z;
  const int h0 = hblk * a.hb, nh = min(a.hb, a.H - h0), G = a.G, rep = MIXED ? a.H / G : a.hb, dk = a.dk;
  const JointStepLayout lay(MIXED, N, a.hb, G, dk, a.dvp, a.v ? G : 0, a.sc.rows, a.stages);
  const int tpg = MIXED ? (rep + 15) / 16 : lay.mt;        // tiles of a key/value head
  __nv_bfloat16* const sq = reinterpret_cast<__nv_bfloat16*>(js_smem + lay.q);
  float* const ss = reinterpret_cast<float*>(js_smem + lay.s);
  float* const s2 = reinterpret_cast<float*>(js_smem + lay.s2);
  __nv_bfloat16* const sp = reinterpret_cast<__nv_bfloat16*>(js_smem + lay.p);
  float* const talk = reinterpret_cast<float*>(js_smem + lay.talk);
  float* const rel = reinterpret_cast<float*>(js_smem + lay.rel);
  const int h16 = (a.hb + 15) / 16 * 16, h8 = (a.hb + 7) / 8, rrow = a.sc.rows | 1;
  float* const ml = reinterpret_cast<float*>(js_smem + lay.ml);      // maximum, sum and this tile's factor of every head
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int lr = lane & 15, lc = (lane >> 4) * 8, br = (lane & 7) + ((lane >> 4) << 3), bc = ((lane >> 3) & 1) * 8;
  const int krow = G * dk + 8, vrow = a.v ? G * a.dvp + 8 : krow;
  // local head of row r of tile m (MIXED: tiles do not cross key/value heads); -1: none
  auto head_of = [&](int m, int r) {
    if (!MIXED) return m * 16 + r < nh ? m * 16 + r : -1;
    const int s = m % tpg * 16 + r;
    return s < rep ? m / tpg * rep + s : -1;
  };
  pdl_entry();
  const int pos = a.pos[b];
  if (pos < 0 || (!a.ring && pos >= a.cap)) {              // position outside the store: report, leave the output untouched
    if (tid == 0) report_error(a.err, ERR_BOUNDS, pos);
    return;
  }
  // key x of 0 .. n_keys - 1 is at distance n_keys - 1 - x from the token
  int n_keys = pos + 1;
  if (a.window > 0) n_keys = min(n_keys, a.window);
  if (a.ring) n_keys = min(n_keys, a.cap);
  const int start = pos + 1 - n_keys, slot0 = a.ring ? start % a.cap : start;
  int chunk = (n_keys + a.splits - 1) / a.splits;
  chunk = (chunk + N - 1) / N * N;
  const int lo = min(split * chunk, n_keys), hi = min(lo + chunk, n_keys), tiles = (hi - lo + N - 1) / N;
  auto fetch = [&](int j) {
    if (j < tiles) {
      uint8_t* const st = js_smem + j % a.stages * lay.stage;
      __nv_bfloat16* const sk = reinterpret_cast<__nv_bfloat16*>(st);
      __nv_bfloat16* const sv = reinterpret_cast<__nv_bfloat16*>(st + lay.k_bytes);
      auto rows = [&](const __nv_bfloat16* src, __nv_bfloat16* dst, int d, int row) {
        const int per = d / 8, n = G * per;
        for (int x = tid; x < N * n; x += JS_THREADS) {
          const int r = x / n, y = x - r * n, kv = y / per, c = (y - kv * per) * 8;
          int slot = slot0 + min(lo + j * N + r, hi - 1);  // rows past the slice are masked below
          if (slot >= a.cap) slot -= a.cap;
          cp16(dst + r * row + kv * d + c, src + ((static_cast<long long>(b) * G + kv) * a.cap + slot) * d + c);
        }
      };
      rows(a.k, sk, dk, krow);
      if (a.v) rows(a.v, sv, a.dvp, vrow);
    }
    cp_commit();
  };
  for (int j = 0; j + 1 < a.stages; ++j) fetch(j);
  for (int x = tid; x < lay.mt * 16 * (dk / 8); x += JS_THREADS) {
    const int r = x / (dk / 8), c = (x - r * (dk / 8)) * 8, h = head_of(r >> 4, r & 15);
    *reinterpret_cast<uint4*>(sq + r * (dk + 8) + c) =
        h >= 0 ? *reinterpret_cast<const uint4*>(a.q + b * a.q_sb + (h0 + h) * a.q_sh + c) : make_uint4(0u, 0u, 0u, 0u);
  }
  for (int x = tid; x < lay.mt * 16 * NS / 2; x += JS_THREADS) reinterpret_cast<uint32_t*>(sp)[x] = 0u;
  for (int x = tid; x < h16; x += JS_THREADS) { ml[x] = -INFINITY; ml[h16 + x] = 0.f; ml[2 * h16 + x] = 1.f; }
  if (MIXED) {
    for (int x = tid; x < h16 * lay.ts; x += JS_THREADS) {
      const int r = x / lay.ts, c = x % lay.ts;
      talk[x] = r < a.H && c < a.H ? a.sc.talk[r * a.H + c] : 0.f;
    }
    for (int x = tid; x < a.H * a.sc.rows; x += JS_THREADS) rel[(x % a.H) * rrow + x / a.H] = a.sc.rel[x];
    for (int x = tid; x < (h16 - a.H) * NS; x += JS_THREADS) ss[a.H * NS + x] = 0.f;
  }
  float o[UNITS][4][4];
#pragma unroll
  for (int x = 0; x < UNITS * 16; ++x) (&o[0][0][0])[x] = 0.f;
  const int nc = (a.dv + 31) / 32, units = lay.mt * nc, per_warp = (units + JS_WARPS - 1) / JS_WARPS;
  // unit u -> (key/value head, channel block, tile): the tiles of a head and block are adjacent, so that they share the value operand
  auto unit = [&](int u, int& kv, int& cb, int& m) {
    const int s = u % tpg, y = u / tpg;
    cb = y % nc;
    kv = y / nc;
    m = kv * tpg + s;
  };

  for (int j = 0; j < tiles; ++j) {
    if (a.stages == 3) cp_wait<1>(); else cp_wait<0>();
    __syncthreads();                                       // tile j is there and everyone is done with tile j - 1
    fetch(j + a.stages - 1);
    const uint8_t* const st = js_smem + j % a.stages * lay.stage;
    const __nv_bfloat16* const sk = reinterpret_cast<const __nv_bfloat16*>(st);
    const __nv_bfloat16* const sv = a.v ? reinterpret_cast<const __nv_bfloat16*>(st + lay.k_bytes) : sk;
    const int base = lo + j * N;
    // ---- Q K^T
    for (int u = warp; u < lay.mt * KB; u += JS_WARPS) {
      const int kb = u % KB, mt = u / KB, kv = mt / tpg;
      float c[2][2][4];                                    // even and odd channel steps apart: two chains in flight
#pragma unroll
      for (int x = 0; x < 16; ++x) (&c[0][0][0])[x] = 0.f;
      const __nv_bfloat16* qp = sq + (mt * 16 + lr) * (dk + 8) + lc;
      const __nv_bfloat16* kp = sk + (kb * 16 + br) * krow + kv * dk + bc;
      int x = 0;
#pragma unroll 2
      for (; x + 32 <= dk; x += 32) {
        uint32_t f[2][4], kf[2][4];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          ldsm4(f[e], qp + x + 16 * e);
          ldsm4(kf[e], kp + x + 16 * e);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma_bf16(c[e][0], f[e], kf[e][0], kf[e][1]);
          mma_bf16(c[e][1], f[e], kf[e][2], kf[e][3]);
        }
      }
      if (x < dk) {
        uint32_t f[4], kf[4];
        ldsm4(f, qp + x);
        ldsm4(kf, kp + x);
        mma_bf16(c[0][0], f, kf[0], kf[1]);
        mma_bf16(c[0][1], f, kf[2], kf[3]);
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int h = head_of(mt, g + 8 * r);
        if (h < 0) continue;
        const float k2 = MIXED ? 2.f * kLog2e * a.sc.scale * a.sc.temp[h] / a.sc.softcap : a.sc.scale * kLog2e;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int col = kb * 16 + 8 * e + 2 * t;
          float2 y = make_float2(c[0][e][2 * r] + c[1][e][2 * r], c[0][e][2 * r + 1] + c[1][e][2 * r + 1]);
          if (MIXED) {
            const int n = n_keys - 1 - (base + col);
            y.x = ja_cap(y.x, k2, a.sc.softcap) + rel[h * rrow + a.sc.bucket[min(max(n, 0), a.sc.reach)]];
            y.y = ja_cap(y.y, k2, a.sc.softcap) + rel[h * rrow + a.sc.bucket[min(max(n - 1, 0), a.sc.reach)]];
          } else {
            y.x *= k2;
            y.y *= k2;
          }
          *reinterpret_cast<float2*>(ss + h * NS + col) = y;
        }
      }
    }
    __syncthreads();
    if (MIXED) {
      for (int u = warp; u < h16 / 16 * (N / 8); u += JS_WARPS) {
        const int n = u % (N / 8), mt = u / (N / 8);
        float c[4] = {0.f, 0.f, 0.f, 0.f};
        for (int kk = 0; kk < h8; ++kk) {
          uint32_t th[4], tl[4];
          ja_talk_frag(th, tl, talk, lay.ts, mt, kk, g, t);
          ja_mix_step(c, th, tl, a.sc.talk_exact != 0, ss + n * 8, NS, kk, g, t);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<float2*>(s2 + (mt * 16 + g + 8 * r) * NS + n * 8 + 2 * t) = make_float2(c[2 * r] * kLog2e, c[2 * r + 1] * kLog2e);
      }
      __syncthreads();
    }
    // ---- softmax: a warp per head
    for (int m = 0; m < lay.mt * 16; m += JS_WARPS) {
      const int row = m + warp, h = head_of(row >> 4, row & 15);
      if (h < 0) continue;
      const float* x = (MIXED ? s2 : ss) + h * NS;
      float v[(N + 31) / 32], mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < (N + 31) / 32; ++e) {
        const int c = lane + 32 * e;
        v[e] = c < N && base + c < hi ? x[c] : -INFINITY;
        mx = fmaxf(mx, v[e]);
      }
      const float mo = ml[h], mn = fmaxf(mo, warp_max(mx));     // finite: the tile's first key is there
      float sum = 0.f;
#pragma unroll
      for (int e = 0; e < (N + 31) / 32; ++e) {
        const int c = lane + 32 * e;
        const float w = ex2(v[e] - mn);
        sum += w;
        if (c < N) sp[row * NS + c] = __float2bfloat16(w);
      }
      sum = warp_sum(sum);
      if (lane == 0) {
        const float f = ex2(mo - mn);
        ml[h16 + h] = ml[h16 + h] * f + sum;
        ml[2 * h16 + h] = f;
        ml[h] = mn;
      }
      __syncwarp();
    }
    __syncthreads();
    // ---- P V
    int last = -1;
    uint32_t vf[KB][2][4];
#pragma unroll
    for (int y = 0; y < UNITS; ++y) {
      const int u = warp * per_warp + y;
      if (y >= per_warp || u >= units) break;
      int kv, cb, mt;
      unit(u, kv, cb, mt);
      if (u / tpg != last) {
        last = u / tpg;
        const __nv_bfloat16* vp = sv + lr * vrow + kv * a.dvp + cb * 32 + lc;
#pragma unroll
        for (int x = 0; x < KB; ++x) {
          ldsm4_t(vf[x][0], vp + x * 16 * vrow);
          ldsm4_t(vf[x][1], vp + x * 16 * vrow + 16);
        }
      }
      const int ha = head_of(mt, g), hc = head_of(mt, g + 8);
      const float fa = ha < 0 ? 1.f : ml[2 * h16 + ha], fc = hc < 0 ? 1.f : ml[2 * h16 + hc];
      if (__any_sync(0xffffffffu, fa != 1.f || fc != 1.f)) {
#pragma unroll
        for (int e = 0; e < 4; ++e) { o[y][e][0] *= fa; o[y][e][1] *= fa; o[y][e][2] *= fc; o[y][e][3] *= fc; }
      }
#pragma unroll
      for (int x = 0; x < KB; ++x) {
        uint32_t pf[4];
        ldsm4(pf, sp + (mt * 16 + lr) * NS + x * 16 + lc);
        mma_bf16(o[y][0], pf, vf[x][0][0], vf[x][0][1]);
        mma_bf16(o[y][1], pf, vf[x][0][2], vf[x][0][3]);
        mma_bf16(o[y][2], pf, vf[x][1][0], vf[x][1][1]);
        mma_bf16(o[y][3], pf, vf[x][1][2], vf[x][1][3]);
      }
    }
  }
  cp_wait<0>();
  __syncthreads();
  // ---- this slice's part, or the result where there is only one slice
  const long long part = static_cast<long long>(b) * a.splits + split;
#pragma unroll
  for (int y = 0; y < UNITS; ++y) {
    const int u = warp * per_warp + y;
    if (y >= per_warp || u >= units) break;
    int kv, cb, mt;
    unit(u, kv, cb, mt);
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int h = head_of(mt, g + 8 * r);
      if (h < 0) continue;
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int z = 0; z < 2; ++z) {
          const int d = cb * 32 + e * 8 + 2 * t + z;
          if (d >= a.dv) continue;
          if (a.splits == 1) a.out[b * a.out_sb + (h0 + h) * a.out_sh + d] = __float2bfloat16(o[y][e][2 * r + z] / ml[h16 + h]);
          else a.part_acc[(part * a.H + h0 + h) * a.dv + d] = o[y][e][2 * r + z];
        }
    }
  }
  if (a.splits == 1) return;
  for (int h = tid; h < nh; h += JS_THREADS) {
    a.part_ml[(part * a.H + h0 + h) * 2] = ml[h];
    a.part_ml[(part * a.H + h0 + h) * 2 + 1] = ml[h16 + h];
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) s_last = atomicAdd(a.counters + b * gridDim.y + hblk, 1) == a.splits - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  float* const w = reinterpret_cast<float*>(js_smem);      // [nh, splits] weights of the slices
  for (int h = warp; h < nh; h += JS_WARPS) {
    const float* src = a.part_ml + (static_cast<long long>(b) * a.splits * a.H + h0 + h) * 2;
    const float mx = lane < a.splits ? __ldcg(src + static_cast<long long>(lane) * a.H * 2) : -INFINITY;
    const float lx = lane < a.splits ? __ldcg(src + static_cast<long long>(lane) * a.H * 2 + 1) : 0.f;
    const float M = warp_max(mx), f = ex2(mx - M), L = warp_sum(f * lx);
    if (lane < a.splits) w[h * a.splits + lane] = f / L;
  }
  __syncthreads();
  for (int x = tid; x < nh * a.dv; x += JS_THREADS) {
    const int h = x / a.dv, d = x - h * a.dv;
    const float* src = a.part_acc + (static_cast<long long>(b) * a.splits * a.H + h0 + h) * a.dv + d;
    float s = 0.f;
#pragma unroll 8
    for (int i = 0; i < a.splits; ++i) s += w[h * a.splits + i] * __ldcg(src + static_cast<long long>(i) * a.H * a.dv);
    a.out[b * a.out_sb + (h0 + h) * a.out_sh + d] = __float2bfloat16(s);
  }
  if (tid == 0) a.counters[b * gridDim.y + hblk] = 0;
}

}  // namespace tyr

using namespace tyr;

static int ja_check_scores(const ScoreArgs& sc) {
  if (sc.softcap < 0.f || (sc.rel != nullptr) != (sc.bucket != nullptr) || (sc.rel != nullptr && sc.reach < 0)) return -3;
  return 0;
}

// strides: (batch, position or slot, head) element strides of q, k, v, then row and head strides of out.  `keys`: positions a plain
// store or prompt holds.  dtype 0 = bf16, 1 = fp32.
extern "C" TYR_EXPORT int tyr_joint_attention(const void* q, const void* k, const void* v, void* out, const int* pos, const ScoreArgs* sc,
                                              const long long* strides, int B, int S, int H, int G, int dk, int dv, int cap, int ring,
                                              int window, int keys, int dtype, int* err, void* stream) {
  if (B <= 0 || S <= 0 || H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || window < 0 || (ring && cap <= 0)) return -1;
  if (const int r = ja_check_scores(*sc)) return r;
  JointArgs a{q, k, v, out, pos, strides[0], strides[1], strides[2], strides[3], strides[4], strides[5], strides[6], strides[7], strides[8], strides[9],
              strides[10], B, S, H, G, dk, dv, cap, ring, window, keys, H, *sc, err};
  const auto bytes = [&](int hb) { return static_cast<size_t>(hb) * (dk + dv + 2 * JA_KEYS + 3) * sizeof(float); };
  constexpr size_t kMax = 227 * 1024;
  if (sc->talk == nullptr)
    while (a.hb > 1 && bytes(a.hb) > 48 * 1024) a.hb = (a.hb + 1) / 2;
  if (bytes(a.hb) > kMax) return -2;
  auto kernel = dtype == 1 ? joint_general_kernel<float> : joint_general_kernel<__nv_bfloat16>;
  if (bytes(a.hb) > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kMax));
    if (e != cudaSuccess) return 1000 + (int)e;
  }
  const dim3 grid(static_cast<unsigned>(static_cast<long long>(B) * S), (H + a.hb - 1) / a.hb);
  return (int)launch_dependent(kernel, grid, dim3(256), bytes(a.hb), (cudaStream_t)stream, a);
}

constexpr int kJointSmem = 226 * 1024;       // what a CTA may hold, less its static part

template <typename F>
static int ja_allow_smem(F kernel) {
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kJointSmem);
}

// Form of the prompt kernel for these sizes: 100 * heads of a 16-row tile + keys of a tile; 0: none holds them.
extern "C" TYR_EXPORT int tyr_joint_prompt_form(int H, int G, int dk, int dvp, int rows, int reach) {
  if (H <= 0 || G <= 0 || H % G || H > 32 || dk <= 0 || dvp <= 0 || ((dk | dvp) & 15) || rows > 65535) return 0;
  for (int hpm = 1; hpm <= 2; ++hpm)
    for (int n = 32; n >= 16; n /= 2) {
      const int tpg = (H / G + hpm - 1) / hpm, units = G * ((tpg + 1) / 2) * ((dvp + 31) / 32);
      if (units <= JP_WARPS * JP_UNITS && JointPromptLayout(hpm, n, H, G, dk, dvp, rows, reach).total <= kJointSmem) return 100 * hpm + n;
    }
  return 0;
}

// Mixed heads over whole bf16 prompts.  strides: (batch, token) of q, k, v; the heads of a token are adjacent.  dk and dvp (the row of a
// value head, of which dv channels count) multiples of 16, 16-byte aligned rows.  out [B, S, H, dv].
extern "C" TYR_EXPORT int tyr_joint_prompt(const void* q, const void* k, const void* v, void* out, const ScoreArgs* sc, const long long* strides, int B,
                                           int S, int H, int G, int dk, int dv, int dvp, void* stream) {
  if (B <= 0 || B > 65535 || S <= 0 || dv <= 0 || dv > dvp || sc->talk == nullptr || sc->rel == nullptr || sc->temp == nullptr || sc->softcap <= 0.f) return -1;
  if (const int r = ja_check_scores(*sc)) return r;
  const int form = tyr_joint_prompt_form(H, G, dk, dvp, sc->rows, sc->reach);
  if (form == 0) return -2;
  for (int i = 0; i < 6; ++i)
    if (strides[i] & 7) return -3;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(out)) & 15) return -4;
  JointPromptArgs a{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, (__nv_bfloat16*)out, strides[0], strides[1], strides[2],
                    strides[3], strides[4], strides[5], S, H, G, dk, dv, dvp, *sc};
  const int hpm = form / 100, n = form % 100;
  const size_t smem = JointPromptLayout(hpm, n, H, G, dk, dvp, sc->rows, sc->reach).total;
  const dim3 grid((S + 16 / hpm - 1) / (16 / hpm), B);
  auto kernel = hpm == 1 ? (n == 32 ? joint_prompt_kernel<1, 32> : joint_prompt_kernel<1, 16>) : (n == 32 ? joint_prompt_kernel<2, 32> : joint_prompt_kernel<2, 16>);
  if (const int e = ja_allow_smem(kernel)) return 1000 + e;
  return (int)launch_dependent(kernel, grid, dim3(JP_THREADS), smem, (cudaStream_t)stream, a);
}

namespace {
struct JointStepForm { int n, hb, stages, units; };

// Largest tiles that fit: keys of a tile, heads of a CTA, stages of the ring, accumulator blocks of a warp.  n == 0: none.
JointStepForm joint_step_form(bool mixed, int H, int G, int dk, int dv, int dvp, int shared, int rows) {
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || ((dk | dvp) & 15) || (mixed && H > 64) || (!mixed && G != 1)) return {};
  const int nc = (dv + 31) / 32;
  for (int hb = mixed ? H : (H < 32 ? (H + 15) / 16 * 16 : 32); hb >= 1; hb = mixed ? 0 : (hb > 16 ? 16 : 0))
    for (int n = 64; n >= 16; n /= 2)
      for (int stages = 3; stages >= 2; --stages) {
        const JointStepLayout lay(mixed, n, hb, G, dk, dvp, shared ? 0 : G, rows, stages);
        const int units = (lay.mt * nc + JS_WARPS - 1) / JS_WARPS;
        if (units > 8 || lay.total > kJointSmem || (stages == 3 && lay.stage * 3 > 120 * 1024)) continue;
        return {n, hb, stages, units <= 2 ? 2 : (units <= 4 ? 4 : 8)};
      }
  return {};
}

template <bool MIXED, int N>
void (*joint_step_pick(int units))(JointStepArgs) {
  return units == 2 ? joint_step_kernel<MIXED, N, 2> : (units == 4 ? joint_step_kernel<MIXED, N, 4> : joint_step_kernel<MIXED, N, 8>);
}
}  // namespace

// Heads of a CTA of the step kernel (0: no form holds these sizes).  shared: values are the first dv channels of the keys.
extern "C" TYR_EXPORT int tyr_joint_step_heads(int mixed, int H, int G, int dk, int dv, int dvp, int shared, int rows) {
  const JointStepForm f = joint_step_form(mixed != 0, H, G, dk, dv, dvp, shared, rows);
  return f.n ? f.hb : 0;
}

// Floats of the split partials, then the ticket counters.
extern "C" TYR_EXPORT long long tyr_joint_step_workspace_bytes(int B, int H, int dv, int splits) {
  return static_cast<long long>(B) * H * splits * (dv + 2) * 4 + static_cast<long long>(B) * H * 4;
}

// One token per row over bf16 stores [B, G, cap, dk] and [B, G, cap, dvp] that hold it already; v null: latent rows (G == 1), whose first
// dv channels are the values of all heads.  strides: (batch, head) of q, then of out.  `workspace` must be zero-filled once after
// allocation (the kernel leaves the counters at zero); splits <= 32.
extern "C" TYR_EXPORT int tyr_joint_step(const void* q, const void* k, const void* v, void* out, const int* pos, const ScoreArgs* sc, void* workspace,
                                         const long long* strides, int B, int H, int G, int dk, int dv, int dvp, int cap, int ring, int window,
                                         int splits, int* err, void* stream) {
  if (B <= 0 || B > 65535 || cap <= 0 || window < 0 || splits < 1 || splits > 32 || (splits > 1 && workspace == nullptr)) return -1;
  if (const int r = ja_check_scores(*sc)) return r;
  const bool mixed = sc->talk != nullptr;
  if (mixed ? (v == nullptr || sc->rel == nullptr || sc->temp == nullptr || sc->softcap <= 0.f) : (v != nullptr || sc->rel != nullptr || sc->temp != nullptr)) return -1;
  const JointStepForm f = joint_step_form(mixed, H, G, dk, dv, dvp, v == nullptr, sc->rows);
  if (f.n == 0) return -2;
  if (((strides[0] | strides[1]) & 7) || ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15)) return -3;
  float* const acc = static_cast<float*>(workspace);
  float* const mlp = acc + static_cast<long long>(B) * H * splits * dv;
  JointStepArgs a{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, (__nv_bfloat16*)out, pos, acc, mlp,
                  (int*)(mlp + static_cast<long long>(B) * H * splits * 2), strides[0], strides[1], strides[2], strides[3], B, H, G, dk, dv, dvp, cap, ring,
                  window, splits, f.hb, f.stages, *sc, err};
  const size_t smem = JointStepLayout(mixed, f.n, f.hb, G, dk, dvp, v ? G : 0, sc->rows, f.stages).total;
  auto kernel = mixed ? (f.n == 64 ? joint_step_pick<true, 64>(f.units) : f.n == 32 ? joint_step_pick<true, 32>(f.units) : joint_step_pick<true, 16>(f.units))
                      : (f.n == 64 ? joint_step_pick<false, 64>(f.units) : f.n == 32 ? joint_step_pick<false, 32>(f.units) : joint_step_pick<false, 16>(f.units));
  if (const int e = ja_allow_smem(kernel)) return 1000 + e;
  const dim3 grid(splits, (H + f.hb - 1) / f.hb, B);
  return (int)launch_dependent(kernel, grid, dim3(JS_THREADS), smem, (cudaStream_t)stream, a);
}
