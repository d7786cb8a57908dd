// Attention pieces for any head size, fp32 or bf16, with a logarithmic distance penalty on the scores:
//
//   score(i, j) = scale q_i . k_j - r1_h ln(1 + r2_h (i - j)),   0 <= i - j < window,
//
// a sink (the softmax denominator also holds exp(sink_h)), an output gate (element by element or one number per head, out_scale sigmoid(gate)),
// first positions that stay visible past the window, and an output whose channel pairs (m, m + dv / 2) are turned back by the query's angles.
//
//   * qk_norm_store: per-head RMSNorm of q and k (no rotation; weights and projection biases optional), v copied, rows of the padded batch written to the K/V store at
//                    their own positions (plain or ring).
//   * general:       one warp per (query, head), online softmax in fp32; reads keys from the prompt's own rows or from the store.
//
// The tensor-core forms are in attention_fwd.cu (prompts) and decode_attention.cu (one token); these kernels take the shapes and
// the precision those do not.  Compiled without fast math.
#include "common.cuh"

namespace tyr {

__device__ __forceinline__ float ag_load(const float* p) { return *p; }
__device__ __forceinline__ float ag_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ag_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void ag_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct QkNormArgs {
  const void* y;               // [B * S, ld]: q (H * dk) | k (G * dk) | v (G * dv); G = 0 when the layer has no keys of its own
  long long ld;
  const float *q_w, *k_w;      // [dk] (k_w unused when G == 0); null: ones
  const float* bias;           // [(H + G) dk + G dv] added to the columns of y (nullable)
  void* q_out;                 // [B * S, H, dkp]
  void* k_out;                 // [B * S, G, dkp]
  void* v_out;                 // [B * S, G, dvp] or null
  void *k_store, *v_store;     // [B, G, cap, dkp / dvp] or null
  const int* pos;              // position of token 0 of each row (nullable: 0)
  const int* lens;             // tokens of each row (nullable: S)
  int B, S, H, G, dk, dv, dkp, dvp, cap, ring;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(256) qk_norm_store_kernel(QkNormArgs a) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const int heads = a.H + 2 * a.G;
  const long long total = static_cast<long long>(a.B) * a.S * heads;
  const long long nw = static_cast<long long>(gridDim.x) * 8;
  for (long long i = blockIdx.x * 8LL + (threadIdx.x >> 5); i < total; i += nw) {
    const int hd = static_cast<int>(i % heads);
    const long long row = i / heads;
    const int b = static_cast<int>(row / a.S), s = static_cast<int>(row % a.S);
    const T* src = static_cast<const T*>(a.y) + row * a.ld;
    const bool is_q = hd < a.H, is_v = hd >= a.H + a.G;
    const int g = is_q ? hd : (is_v ? hd - a.H - a.G : hd - a.H);
    const int d_in = is_v ? a.dv : a.dk, d_out = is_v ? a.dvp : a.dkp;
    const int col = is_v ? (a.H + a.G) * a.dk + g * a.dv : hd * a.dk;
    src += col;
    const float* bias = a.bias ? a.bias + col : nullptr;
    T* dst = is_q ? static_cast<T*>(a.q_out) + (row * a.H + g) * d_out
                  : (is_v ? (a.v_out ? static_cast<T*>(a.v_out) + (row * a.G + g) * d_out : nullptr)
                          : static_cast<T*>(a.k_out) + (row * a.G + g) * d_out);
    T* slot = nullptr;
    if (!is_q && a.k_store != nullptr) {
      const int n = a.lens ? a.lens[b] : a.S;
      const int p0 = a.pos ? a.pos[b] : 0;
      const int p = p0 + s;
      const bool keep = s < n && p >= 0 && (a.ring ? p0 + n - p <= a.cap : p < a.cap);     // a ring store keeps the last cap positions
      if (keep)
        slot = static_cast<T*>(is_v ? a.v_store : a.k_store) + ((static_cast<long long>(b) * a.G + g) * a.cap + (a.ring ? p % a.cap : p)) * d_out;
    }
    float rstd = 1.f;
    if (!is_v) {
      float ss = 0.f;
      for (int d = lane; d < d_in; d += 32) {
        const float v = ag_load(src + d) + (bias ? bias[d] : 0.f);
        ss += v * v;
      }
      rstd = 1.f / sqrtf(warp_sum(ss) / d_in + a.eps);
    }
    const float* w = is_q ? a.q_w : a.k_w;
    for (int d = lane; d < d_out; d += 32) {
      float v = d < d_in ? ag_load(src + d) + (bias ? bias[d] : 0.f) : 0.f;
      if (!is_v && d < d_in) v = v * rstd * (w ? w[d] : 1.f);
      if (dst) ag_store(dst + d, v);
      if (slot) ag_store(slot + d, v);
    }
  }
}

// bf16 heads of up to 128 channels in 16-byte vectors: one CTA per token, half a warp per head.
__global__ void __launch_bounds__(256) qk_norm_store_vec_kernel(QkNormArgs a) {
  pdl_entry();
  const int sub = threadIdx.x >> 4, l8 = (threadIdx.x & 15) * 8;
  const long long row = blockIdx.x;
  const int b = static_cast<int>(row / a.S), s = static_cast<int>(row % a.S);
  const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.y) + row * a.ld;
  long long slot = -1;
  if (a.k_store != nullptr) {
    const int n = a.lens ? a.lens[b] : a.S, p0 = a.pos ? a.pos[b] : 0, p = p0 + s;
    if (s < n && p >= 0 && (a.ring ? p0 + n - p <= a.cap : p < a.cap)) slot = a.ring ? p % a.cap : p;
  }
  for (int hd0 = 0; hd0 < a.H + 2 * a.G; hd0 += 16) {
    const int hd = hd0 + sub;
    const bool on = hd < a.H + 2 * a.G, is_q = hd < a.H, is_v = hd >= a.H + a.G;
    const int g = is_q ? hd : (is_v ? hd - a.H - a.G : hd - a.H);
    const int d_in = is_v ? a.dv : a.dk, d_out = is_v ? a.dvp : a.dkp;
    const int col = (is_v ? (a.H + a.G) * a.dk + g * a.dv : hd * a.dk) + l8;
    float f[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = 0.f;
    if (on && l8 < d_in) {
      const uint4 u = *reinterpret_cast<const uint4*>(src + col);
      const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 t = unpack_bf16x2(w[e]);
        f[2 * e] = t.x; f[2 * e + 1] = t.y;
      }
      if (a.bias) {
        const float4 b0 = *reinterpret_cast<const float4*>(a.bias + col), b1 = *reinterpret_cast<const float4*>(a.bias + col + 4);
        f[0] += b0.x; f[1] += b0.y; f[2] += b0.z; f[3] += b0.w; f[4] += b1.x; f[5] += b1.y; f[6] += b1.z; f[7] += b1.w;
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!on || l8 >= d_out) continue;
    if (!is_v) {
      const float rstd = 1.f / sqrtf(ss / d_in + a.eps);
      const float* w = is_q ? a.q_w : a.k_w;
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= w && l8 < d_in ? rstd * w[l8 + e] : rstd;
    }
    const uint4 r = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
    void* dst = is_q ? a.q_out : (is_v ? a.v_out : a.k_out);
    if (dst) *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(dst) + (row * (is_q ? a.H : a.G) + g) * d_out + l8) = r;
    if (!is_q && slot >= 0)
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(is_v ? a.v_store : a.k_store) + ((static_cast<long long>(b) * a.G + g) * a.cap + slot) * d_out + l8) = r;
  }
}

struct GeneralAttnArgs {
  const void *q, *k, *v;       // q: [B, S, H, .]; k / v: [B, ., G, .] by (batch, position or slot, head) element strides
  void* out;                   // [B * S, .] rows of out_ld elements, channel h * dv + d
  const int* pos;              // position of query 0 of each row (nullable: 0)
  const float *r1, *r2;        // [H] distance penalty (nullable: none)
  const float* sink;           // [H] (nullable: none)
  const void* gate;            // [B * S, .] rows of gate_ld elements, channel h * dv + d (nullable: none)
  long long q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh, gate_ld, out_ld;
  int B, S, H, G, dk, dv, cap, ring, window, keys;
  float scale, out_scale;
  int* err;
  int keep;                    // positions 0 .. keep - 1 are visible past the window; a ring store holds them in its first slots
  int gate_head;               // the gate is one number per (row, head): channel h
  const float2* back;          // [back_rows, dv / 2] (cos, sin) (nullable)
  int back_rows;
};
constexpr int GA_WARPS = 4;
constexpr int GA_DMAX = 256;

template <typename T>
__global__ void __launch_bounds__(GA_WARPS * 32) general_attention_kernel(GeneralAttnArgs a) {
  __shared__ float sq[GA_WARPS][GA_DMAX];
  __shared__ float sp[GA_WARPS][32];
  pdl_entry();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long total = static_cast<long long>(a.B) * a.S * a.H;
  const long long i = blockIdx.x * static_cast<long long>(GA_WARPS) + warp;
  if (i >= total) return;
  const int h = static_cast<int>(i % a.H);
  const long long row = i / a.H;
  const int b = static_cast<int>(row / a.S), s = static_cast<int>(row % a.S);
  const int g = h / (a.H / a.G);
  const int p = (a.pos ? a.pos[b] : 0) + s;
  if (p < 0 || (!a.ring && p >= a.keys) || (a.back != nullptr && p >= a.back_rows)) {         // a query without its own key in the store or turns: report, leave the output
    if (lane == 0) report_error(a.err, ERR_BOUNDS, p);
    return;
  }
  const T* qp = static_cast<const T*>(a.q) + b * a.q_sb + s * a.q_ss + h * a.q_sh;
  const T* kb = static_cast<const T*>(a.k) + b * a.k_sb + g * a.k_sh;
  const T* vb = static_cast<const T*>(a.v) + b * a.v_sb + g * a.v_sh;
  for (int d = lane; d < a.dk; d += 32) sq[warp][d] = ag_load(qp + d);
  __syncwarp();
  const float r1 = a.r1 ? a.r1[h] : 0.f, r2 = a.r1 ? a.r2[h] : 0.f;
  const int ring_len = a.cap - a.keep;
  int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  if (a.ring) lo = max(lo, p - ring_len + 1);
  const int k0 = min(a.keep, lo), gap = lo - k0, n = p + 1 - gap;      // key i of n: position i, past the k0 kept ones i + gap
  auto slot_of = [&](int i) {
    const int j = i < k0 ? i : i + gap;
    return static_cast<long long>(a.ring && j >= a.keep ? a.keep + (j - a.keep) % ring_len : j);
  };
  float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f, acc[GA_DMAX / 32];
#pragma unroll
  for (int j = 0; j < GA_DMAX / 32; ++j) acc[j] = 0.f;
  for (int base = 0; base < n; base += 32) {
    const int i = base + lane, j = i < k0 ? i : i + gap;
    float sc = -INFINITY;
    if (i < n) {
      const T* kr = kb + slot_of(i) * a.k_ss;
      float dot = 0.f;
      for (int d = 0; d < a.dk; ++d) dot += sq[warp][d] * ag_load(kr + d);
      sc = dot * a.scale - r1 * log1pf(r2 * static_cast<float>(p - j));
    }
    const float mn = fmaxf(m, warp_max(sc));
    const float f = expf(m - mn), w = expf(sc - mn);
    l = l * f + warp_sum(w);
    m = mn;
    sp[warp][lane] = w;
    __syncwarp();
#pragma unroll
    for (int c = 0; c < GA_DMAX / 32; ++c) acc[c] *= f;
    const int nk = min(32, n - base);
    for (int t = 0; t < nk; ++t) {
      const float wt = sp[warp][t];
      const T* vr = vb + slot_of(base + t) * a.v_ss;
#pragma unroll
      for (int c = 0; c < GA_DMAX / 32; ++c)
        if (lane + 32 * c < a.dv) acc[c] += wt * ag_load(vr + lane + 32 * c);
    }
    __syncwarp();
  }
  T* op = static_cast<T*>(a.out) + row * a.out_ld + static_cast<long long>(h) * a.dv;
  const T* gp = a.gate ? static_cast<const T*>(a.gate) + row * a.gate_ld + static_cast<long long>(h) * (a.gate_head ? 1 : a.dv) : nullptr;
  if (a.back != nullptr) {                         // the queries are done with: a channel's partner is in another lane
#pragma unroll
    for (int c = 0; c < GA_DMAX / 32; ++c)
      if (lane + 32 * c < a.dv) sq[warp][lane + 32 * c] = acc[c];
    __syncwarp();
    const int half = a.dv / 2;
    const float2* cs = a.back + static_cast<long long>(p) * half;
#pragma unroll
    for (int c = 0; c < GA_DMAX / 32; ++c) {
      const int d = lane + 32 * c;
      if (d < half) acc[c] = sq[warp][d] * cs[d].x + sq[warp][d + half] * cs[d].y;
      else if (d < a.dv) acc[c] = sq[warp][d] * cs[d - half].x - sq[warp][d - half] * cs[d - half].y;
    }
  }
#pragma unroll
  for (int c = 0; c < GA_DMAX / 32; ++c)
    if (lane + 32 * c < a.dv) {
      const float g = gp ? a.out_scale / (1.f + expf(-ag_load(gp + (a.gate_head ? 0 : lane + 32 * c)))) : a.out_scale;
      ag_store(op + lane + 32 * c, acc[c] / l * g);
    }
}

}  // namespace tyr

using namespace tyr;

extern "C" TYR_EXPORT int tyr_qk_norm_store(const void* y, long long ld, const float* q_w, const float* k_w, const float* bias, void* q_out, void* k_out,
                                            void* v_out, void* k_store, void* v_store, const int* pos, const int* lens, int B, int S,
                                            int H, int G, int dk, int dv, int dkp, int dvp, int cap, int ring, float eps, int dtype,
                                            void* stream) {
  if (B <= 0 || S <= 0 || H <= 0 || G < 0 || dk <= 0 || dkp < dk || dvp < dv || (G > 0 && dv <= 0)) return -1;
  if ((k_store != nullptr) != (v_store != nullptr) || (k_store != nullptr && cap <= 0)) return -2;
  QkNormArgs a{y, ld, q_w, k_w, bias, q_out, k_out, v_out, k_store, v_store, pos, lens, B, S, H, G, dk, dv, dkp, dvp, cap, ring, eps};
  const uintptr_t al = reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(q_out) | reinterpret_cast<uintptr_t>(k_out) |
                       reinterpret_cast<uintptr_t>(v_out) | reinterpret_cast<uintptr_t>(k_store) | reinterpret_cast<uintptr_t>(v_store) |
                       reinterpret_cast<uintptr_t>(bias);
  if (dtype == 0 && ((ld | dk | dv | dkp | dvp) & 7) == 0 && dkp <= 128 && dvp <= 128 && (al & 15) == 0)
    return (int)launch_dependent(qk_norm_store_vec_kernel, dim3(static_cast<unsigned>(static_cast<long long>(B) * S)), dim3(256), 0, (cudaStream_t)stream, a);
  const long long want = (static_cast<long long>(B) * S * (H + 2 * G) + 7) / 8;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 32 ? want : 148LL * 32));
  return (int)(dtype == 1 ? launch_dependent(qk_norm_store_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, a)
                          : launch_dependent(qk_norm_store_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, a));
}

static int general_attention_launch(GeneralAttnArgs& a, const long long* strides, int dtype, void* stream) {
  if (a.B <= 0 || a.S <= 0 || a.H <= 0 || a.G <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || a.dk > GA_DMAX || a.dv > GA_DMAX) return -1;
  if ((a.ring && a.cap <= 0) || (a.r1 != nullptr) != (a.r2 != nullptr)) return -2;
  a.q_sb = strides[0]; a.q_ss = strides[1]; a.q_sh = strides[2];
  a.k_sb = strides[3]; a.k_ss = strides[4]; a.k_sh = strides[5];
  a.v_sb = strides[6]; a.v_ss = strides[7]; a.v_sh = strides[8];
  const dim3 grid(static_cast<unsigned>((static_cast<long long>(a.B) * a.S * a.H + GA_WARPS - 1) / GA_WARPS)), block(GA_WARPS * 32);
  return (int)(dtype == 1 ? launch_dependent(general_attention_kernel<float>, grid, block, 0, (cudaStream_t)stream, a)
                          : launch_dependent(general_attention_kernel<__nv_bfloat16>, grid, block, 0, (cudaStream_t)stream, a));
}

// strides: (batch, position or slot, head) element strides of q, k, v.  `keys`: positions the plain form may read (prompt length
// or capacity).  dk, dv <= 256.  out contiguous.
extern "C" TYR_EXPORT int tyr_general_attention(const void* q, const void* k, const void* v, void* out, const int* pos,
                                                const float* r1, const float* r2, const long long* strides, int B, int S, int H,
                                                int G, int dk, int dv, int cap, int ring, int window, int keys, float scale,
                                                int dtype, int* err, void* stream) {
  GeneralAttnArgs a{};
  a.q = q; a.k = k; a.v = v; a.out = out; a.pos = pos; a.r1 = r1; a.r2 = r2;
  a.B = B; a.S = S; a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.cap = cap; a.ring = ring; a.window = window; a.keys = keys;
  a.out_ld = static_cast<long long>(H) * dv;
  a.scale = scale; a.out_scale = 1.f; a.err = err;
  return general_attention_launch(a, strides, dtype, stream);
}

// The same over all earlier positions with a sink per head, an output gate and a factor (sink and gate nullable).  strides: as above,
// then the row strides of gate and out.
extern "C" TYR_EXPORT int tyr_general_attention_sink(const void* q, const void* k, const void* v, void* out, const int* pos, const float* sink,
                                                     const void* gate, const long long* strides, int B, int S, int H, int G, int dk, int dv,
                                                     int keys, float scale, float out_scale, int dtype, int* err, void* stream) {
  GeneralAttnArgs a{};
  a.q = q; a.k = k; a.v = v; a.out = out; a.pos = pos; a.sink = sink; a.gate = gate;
  a.B = B; a.S = S; a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.cap = keys; a.keys = keys;
  a.gate_ld = strides[9]; a.out_ld = strides[10];
  a.scale = scale; a.out_scale = out_scale; a.err = err;
  return general_attention_launch(a, strides, dtype, stream);
}

// A window (0: none) that leaves the first `keep` positions visible, in rows of a prompt, a plain store or one of `keep` slots followed by a
// ring; one gate per head (nullable: rows of strides[9] elements); `back` (nullable): [back_rows, dv / 2] pairs (cos, sin).  strides: as for
// the sink form.
extern "C" TYR_EXPORT int tyr_general_attention_kept(const void* q, const void* k, const void* v, void* out, const int* pos, const void* head_gate,
                                                     const void* back, int back_rows, const long long* strides, int B, int S, int H, int G, int dk, int dv, int cap,
                                                     int ring, int window, int keep, int keys, float scale, int dtype, int* err, void* stream) {
  if (keep < 0 || (ring && keep >= cap) || (back != nullptr && (dv & 1))) return -3;
  GeneralAttnArgs a{};
  a.q = q; a.k = k; a.v = v; a.out = out; a.pos = pos; a.gate = head_gate; a.gate_head = 1; a.back = static_cast<const float2*>(back); a.back_rows = back_rows;
  a.B = B; a.S = S; a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.cap = cap; a.ring = ring; a.window = window; a.keep = keep; a.keys = keys;
  a.gate_ld = strides[9]; a.out_ld = strides[10];
  a.scale = scale; a.out_scale = 1.f; a.err = err;
  return general_attention_launch(a, strides, dtype, stream);
}
