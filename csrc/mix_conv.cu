// What lies between a layer's input projection and its mixers, in one launch: the columns of the projection are cut into segments,
// and each segment takes an optional causal depthwise convolution over time (any number of taps, bias), an optional activation
// (SiLU or squared ReLU), an optional factor that depends on the position alone (query temperature
// 1 + coef ln(floor((p + 1) / every) + 1)), and a destination of its own: rows of heads that may be padded, and a K/V store.
//
//   * prompt: whole prompts [B, S, columns], rows of unequal length; leaves the last `taps` inputs of every row as the window.
//   * step:   one token per row; windows shifted in place.
//
// The vector form of the prompt kernel keeps the taps and a sliding window of 8 channels in registers, so that an input row is
// loaded once; the plain form takes any size, any number of taps and fp32.  Compiled without fast math.
#include "common.cuh"

namespace tyr {

constexpr int MC_SEGS = 6;
enum MixAct : int { MC_NONE = 0, MC_SILU = 1, MC_RELU2 = 2 };

struct MixSegment {
  int col, heads, d_in, d_out;   // source columns [col, col + heads * d_in); a head's d_in channels go to the first of d_out
  int taps, act;                 // taps 0: no convolution
  const float* w;                // [heads * d_in, taps]
  const float* bias;             // [heads * d_in] (nullable)
  void* window;                  // [B, heads * d_in, taps], the type of x (nullable)
  void* out;                     // rows of out_ld elements
  long long out_ld;
  void* store;                   // [B, heads, cap, store_d] by position (nullable; prompt only)
  int cap, store_d;
  float temp_coef, temp_every;   // temp_every 0: no factor
};

struct MixArgs {
  const void* x;                 // [B, S, .] by (batch, token) strides
  long long x_sb, x_ss;
  const int* lens;               // prompt: tokens of each row (nullable: S)
  const int* pos;                // step: position of the new token of each row
  int B, S, n_seg, groups;       // groups: channels (or vectors of 8) of all segments' outputs
  MixSegment seg[MC_SEGS];
};

__device__ __forceinline__ float mc_load(const float* p) { return *p; }
__device__ __forceinline__ float mc_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void mc_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void mc_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float mc_act(float v, int act) {
  if (act == MC_SILU) return v / (1.f + expf(-v));
  if (act == MC_RELU2) { const float r = fmaxf(v, 0.f); return r * r; }
  return v;
}
__device__ __forceinline__ float mc_temp(const MixSegment& s, int p) {
  return s.temp_every > 0.f ? 1.f + s.temp_coef * logf(floorf(static_cast<float>(p + 1) / s.temp_every) + 1.f) : 1.f;
}

// Output channel `o` of all segments -> its segment; `o` becomes the channel inside it.
__device__ __forceinline__ int mc_find(const MixArgs& a, int& o, int per) {
  int i = 0;
#pragma unroll
  for (int j = 0; j < MC_SEGS - 1; ++j) {
    const int n = a.seg[j].heads * a.seg[j].d_out / per;
    if (i == j && j + 1 < a.n_seg && o >= n) { o -= n; ++i; }
  }
  return i;
}

template <typename T, bool STEP>
__global__ void __launch_bounds__(256) mix_plain_kernel(const __grid_constant__ MixArgs a) {
  pdl_entry();
  const long long total = static_cast<long long>(a.B) * a.S * a.groups;
  for (long long i = blockIdx.x * 256LL + threadIdx.x; i < total; i += gridDim.x * 256LL) {
    int o = static_cast<int>(i % a.groups);
    const long long row = i / a.groups;
    const int b = static_cast<int>(row / a.S), t = static_cast<int>(row % a.S);
    const MixSegment& s = a.seg[mc_find(a, o, 1)];
    const int head = o / s.d_out, d = o % s.d_out;
    T* dst = static_cast<T*>(s.out) + row * s.out_ld + o;
    if (d >= s.d_in) {                                  // padded channel of a head
      mc_store(dst, 0.f);
      continue;
    }
    const int c = head * s.d_in + d, C = s.heads * s.d_in, K = s.taps;
    const T* xb = static_cast<const T*>(a.x) + b * a.x_sb + s.col + c;
    const int len = a.lens ? a.lens[b] : a.S;
    float acc;
    if (K == 0) {
      acc = mc_load(xb + t * a.x_ss);
    } else {
      acc = s.bias ? s.bias[c] : 0.f;
      const float* w = s.w + static_cast<long long>(c) * K;
      T* win = s.window ? static_cast<T*>(s.window) + (static_cast<long long>(b) * C + c) * K : nullptr;
      if constexpr (STEP) {
        for (int j = 0; j + 1 < K; ++j) {
          const T v = win[j + 1];
          win[j] = v;
          acc += mc_load(&v) * w[j];
        }
        const T v = *xb;
        win[K - 1] = v;
        acc += mc_load(&v) * w[K - 1];
      } else {
        for (int j = 0; j < K; ++j) {
          const int u = t - (K - 1) + j;
          if (u >= 0) acc += mc_load(xb + u * a.x_ss) * w[j];
        }
        if (win && t == len - 1)
          for (int j = 0; j < K; ++j) {
            const int u = t - (K - 1) + j;
            mc_store(win + j, u >= 0 ? mc_load(xb + u * a.x_ss) : 0.f);
          }
      }
    }
    acc = mc_act(acc, s.act) * mc_temp(s, STEP ? a.pos[b] : t);
    mc_store(dst, acc);
    if (!STEP && s.store && t < len && t < s.cap)
      mc_store(static_cast<T*>(s.store) + ((static_cast<long long>(b) * s.heads + head) * s.cap + t) * s.store_d + d, acc);
  }
}

// bf16, at most 4 taps, d_in a multiple of 8 and equal to d_out, 16-byte aligned rows.  A thread owns 8 channels x MC_TOK tokens.
constexpr int MC_TOK = 32;
__global__ void __launch_bounds__(256, 2) mix_vec_kernel(const __grid_constant__ MixArgs a) {
  pdl_entry();
  const int nblk = (a.S + MC_TOK - 1) / MC_TOK;
  const long long total = static_cast<long long>(a.B) * nblk * a.groups;
  const long long i = blockIdx.x * 256LL + threadIdx.x;
  if (i >= total) return;
  int o = static_cast<int>(i % a.groups);
  const long long bt = i / a.groups;
  const int t0 = static_cast<int>(bt % nblk) * MC_TOK, b = static_cast<int>(bt / nblk);
  const MixSegment& s = a.seg[mc_find(a, o, 8)];
  const int c = o * 8, K = s.taps, C = s.heads * s.d_in;
  const int head = c / s.d_in, d = c % s.d_in;
  const __nv_bfloat16* xb = static_cast<const __nv_bfloat16*>(a.x) + b * a.x_sb + s.col + c;
  const int len = a.lens ? a.lens[b] : a.S;
  float wt[8][4], bs[8];                           // fewer than 4 taps: leading zeros
#pragma unroll
  for (int e = 0; e < 8; ++e) {
    bs[e] = K > 0 && s.bias ? s.bias[c + e] : 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) wt[e][j] = K == 0 ? (j == 3 ? 1.f : 0.f) : (j >= 4 - K ? s.w[(c + e) * K + j - (4 - K)] : 0.f);
  }
  const int act = s.act, t1 = min(a.S, t0 + MC_TOK);
  const bool temps = s.temp_every > 0.f;
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(s.out) + (static_cast<long long>(b) * a.S + t0) * s.out_ld + c;
  __nv_bfloat16* slot = s.store ? static_cast<__nv_bfloat16*>(s.store) + ((static_cast<long long>(b) * s.heads + head) * s.cap + t0) * s.store_d + d : nullptr;
  const int keep = min(len, s.cap);                // tokens that go to the store
  auto load_row = [&](int t) {
    return t < 0 || t >= a.S ? make_uint4(0, 0, 0, 0) : *reinterpret_cast<const uint4*>(xb + t * a.x_ss);
  };
  auto unpack = [](const uint4& u, float (&f)[8]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 x = unpack_bf16x2(w[e]);
      f[2 * e] = x.x; f[2 * e + 1] = x.y;
    }
  };
  float win[4][8];                                 // x[t] in win[t % 4], counted from t0
#pragma unroll
  for (int j = 0; j < 3; ++j) unpack(load_row(t0 - 3 + j), win[j + 1]);
  uint4 next[4];
#pragma unroll
  for (int u = 0; u < 4; ++u) next[u] = load_row(t0 + u);
#pragma unroll 1
  for (int tb = t0; tb < t1; tb += 4) {
    uint4 row[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      row[u] = next[u];
      next[u] = load_row(tb + 4 + u < t1 ? tb + 4 + u : -1);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int t = tb + u;
      unpack(row[u], win[u]);
      if (t < t1) {
        float acc[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          acc[e] = bs[e];
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[e] += win[(u + 1 + j) & 3][e] * wt[e][j];
          if (act == MC_SILU) acc[e] = __fdividef(acc[e], 1.f + __expf(-acc[e]));
          if (act == MC_RELU2) acc[e] = fmaxf(acc[e], 0.f) * fmaxf(acc[e], 0.f);
        }
        if (temps) {
          const float f = mc_temp(s, t);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[e] *= f;
        }
        const uint4 r = make_uint4(pack_bf16x2(acc[0], acc[1]), pack_bf16x2(acc[2], acc[3]), pack_bf16x2(acc[4], acc[5]), pack_bf16x2(acc[6], acc[7]));
        *reinterpret_cast<uint4*>(dst + u * s.out_ld) = r;
        if (slot && t < keep) *reinterpret_cast<uint4*>(slot + u * s.store_d) = r;
      }
    }
    dst += 4 * s.out_ld;
    if (slot) slot += 4 * s.store_d;
  }
  if (K > 0 && s.window && len > t0 && len <= t0 + MC_TOK) {       // the row's last token lies here: its last K inputs
    __nv_bfloat16* w = static_cast<__nv_bfloat16*>(s.window) + (static_cast<long long>(b) * C + c) * K;
    for (int j = 0; j < K; ++j) {
      float f[8];
      unpack(load_row(len - K + j), f);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e * K + j] = __float2bfloat16(f[e]);
    }
  }
}

}  // namespace tyr

using namespace tyr;

// dtype: 0 = bf16, 1 = fp32 (x, windows, outputs and stores; taps and bias are fp32).  step: S must be 1, `pos` is required and
// every convolved segment needs its window.
extern "C" TYR_EXPORT int tyr_mix_conv(const MixArgs* args, int step, int dtype, void* stream) {
  MixArgs a = *args;
  if (a.B <= 0 || a.S <= 0 || a.n_seg <= 0 || a.n_seg > MC_SEGS || (step && (a.S != 1 || a.pos == nullptr))) return -1;
  bool vec = !step && dtype == 0 && (a.x_sb & 7) == 0 && (a.x_ss & 7) == 0 && (reinterpret_cast<uintptr_t>(a.x) & 15) == 0;
  long long channels = 0;
  for (int i = 0; i < a.n_seg; ++i) {
    const MixSegment& s = a.seg[i];
    if (s.heads <= 0 || s.d_in <= 0 || s.d_out < s.d_in || s.taps < 0 || s.out == nullptr || (s.taps > 0 && s.w == nullptr)) return -2;
    if (step && ((s.taps > 0 && s.window == nullptr) || s.store != nullptr)) return -3;
    if (s.store != nullptr && (s.cap <= 0 || s.store_d < s.d_in)) return -4;
    channels += static_cast<long long>(s.heads) * s.d_out;
    vec = vec && s.taps <= 4 && s.d_in == s.d_out && (s.d_in & 7) == 0 && (s.col & 7) == 0 && (s.out_ld & 7) == 0 && (s.store_d & 7) == 0 &&
          ((reinterpret_cast<uintptr_t>(s.out) | reinterpret_cast<uintptr_t>(s.store)) & 15) == 0;
  }
  if (channels > 0x7fffffffLL) return -1;
  a.groups = static_cast<int>(vec ? channels / 8 : channels);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (vec) {
    const long long total = static_cast<long long>(a.B) * ((a.S + MC_TOK - 1) / MC_TOK) * a.groups;
    return (int)launch_dependent(mix_vec_kernel, dim3(static_cast<unsigned>((total + 255) / 256)), dim3(256), 0, st, a);
  }
  const long long want = (static_cast<long long>(a.B) * a.S * a.groups + 255) / 256;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 64 ? want : 148LL * 64));
  if (step)
    return (int)(dtype == 1 ? launch_dependent(mix_plain_kernel<float, true>, grid, dim3(256), 0, st, a)
                            : launch_dependent(mix_plain_kernel<__nv_bfloat16, true>, grid, dim3(256), 0, st, a));
  return (int)(dtype == 1 ? launch_dependent(mix_plain_kernel<float, false>, grid, dim3(256), 0, st, a)
                          : launch_dependent(mix_plain_kernel<__nv_bfloat16, false>, grid, dim3(256), 0, st, a));
}
