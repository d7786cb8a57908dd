// Attention in which all heads of a query are worked on together, because their scores are mixed or because they share one key:
//
//   s_g(i, j) = softcap tanh(scale temp_g q_g . k / softcap) + rel[bucket(i - j), g]
//   score_h   = sum_g talk[h, g] s_g                          (each step optional), j <= i, 0 <= i - j < window,
//
// softmax over the visible keys of every head.  Keys and values are separate rows, or the values are the first channels of the keys
// (one latent row for all heads).
//
//   * general: one CTA per (query, block of heads), fp32 arithmetic, any sizes, fp32 or bf16; keys of a prompt or of a store (plain or
//              ring).
//
// Compiled without fast math.
#include "common.cuh"

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
