// What lies between a layer's input projection and its mixers, in one launch: the columns of the projection are cut into segments,
// and each segment takes an optional causal depthwise convolution over time (any number of taps, bias), an optional activation
// (SiLU, squared ReLU or xIELU), an optional factor that depends on the position alone (query temperature
// 1 + coef ln(floor((p + 1) / every) + 1)), and a destination of its own: rows of heads that may be padded, and a K/V store.
//
//   * prompt: whole prompts [B, S, columns], rows of unequal length; leaves the last `taps` inputs of every row as the window.
//   * step:   one token per row; windows shifted in place.
//
// The vector form of the prompt kernel keeps the taps and a sliding window of 2 channels in registers, so that an input row is
// loaded once; the plain form takes any size, any number of taps and fp32.  Compiled without fast math.
#include "common.cuh"

namespace tyr {

constexpr int MC_SEGS = 6;
enum MixAct : int { MC_NONE = 0, MC_SILU = 1, MC_RELU2 = 2, MC_XIELU = 3 };

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
  float act_a, act_b;            // xIELU: a z^2 + z / 2 above zero, b (e^z - 1 - z) + z / 2 below
};

struct MixArgs {
  const void* x;                 // [B, S, .] by (batch, token) strides
  long long x_sb, x_ss;
  const int* lens;               // prompt: tokens of each row (nullable: S)
  const int* pos;                // step: position of the new token of each row
  int B, S, n_seg, groups;       // groups: channels (or pairs) of all segments' outputs
  MixSegment seg[MC_SEGS];
};

__device__ __forceinline__ float mc_load(const float* p) { return *p; }
__device__ __forceinline__ float mc_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void mc_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void mc_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float mc_xielu(float v, float a, float b) { return (v > 0.f ? a * v * v : b * (expm1f(v) - v)) + 0.5f * v; }
__device__ __forceinline__ float mc_act(float v, const MixSegment& s) {
  const int act = s.act;
  if (act == MC_SILU) return v / (1.f + expf(-v));
  if (act == MC_RELU2) { const float r = fmaxf(v, 0.f); return r * r; }
  if (act == MC_XIELU) return mc_xielu(v, s.act_a, s.act_b);
  return v;
}
__device__ __forceinline__ float mc_temp(const MixSegment& s, int p) {
  return s.temp_every > 0.f ? 1.f + s.temp_coef * logf(floorf(static_cast<float>(p + 1) / s.temp_every) + 1.f) : 1.f;
}
// the same for 16-bit results: approximate quotient, put right against its neighbours before the floor matters
__device__ __forceinline__ float mc_temp_fast(float coef, float every, int p) {
  const float n = static_cast<float>(p + 1);
  float q = floorf(__fdividef(n, every));
  if ((q + 1.f) * every <= n) q += 1.f;
  if (q * every > n) q -= 1.f;
  return 1.f + coef * __logf(q + 1.f);
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

// One thread per (token, output channel); blockIdx.y walks the tokens of the batch.
template <typename T, bool STEP>
__global__ void __launch_bounds__(256) mix_plain_kernel(const __grid_constant__ MixArgs a) {
  int o = static_cast<int>(blockIdx.x * 256 + threadIdx.x);
  const bool live = o < a.groups;
  const MixSegment& s = a.seg[mc_find(a, o, 1)];
  const int head = s.d_in == s.d_out ? 0 : o / s.d_out, d = s.d_in == s.d_out ? o : o % s.d_out;     // unpadded heads: one wide head
  pdl_entry();
  if (!live) return;
  for (long long row = blockIdx.y; row < static_cast<long long>(a.B) * a.S; row += gridDim.y) {
    const int b = STEP ? static_cast<int>(row) : static_cast<int>(row / a.S), t = STEP ? 0 : static_cast<int>(row % a.S);
    T* dst = static_cast<T*>(s.out) + row * s.out_ld + o;
    if (d >= s.d_in && s.d_in != s.d_out) {             // padded channel of a head
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
      if constexpr (STEP && sizeof(T) == 2) {
        if (K == 4) {                                   // the window in one access
          uint2 v = *reinterpret_cast<const uint2*>(win);
          v.x = __byte_perm(v.x, v.y, 0x5432);
          v.y = __byte_perm(v.y, __bfloat16_as_ushort(*xb), 0x5432);
          *reinterpret_cast<uint2*>(win) = v;
          const float2 u0 = unpack_bf16x2(v.x), u1 = unpack_bf16x2(v.y);
          acc += u0.x * w[0];
          acc += u0.y * w[1];
          acc += u1.x * w[2];
          acc += u1.y * w[3];
        } else {
          for (int j = 0; j + 1 < K; ++j) {
            const T v = win[j + 1];
            win[j] = v;
            acc += mc_load(&v) * w[j];
          }
          const T v = *xb;
          win[K - 1] = v;
          acc += mc_load(&v) * w[K - 1];
        }
      } else if constexpr (STEP) {
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
    acc = mc_act(acc, s) * mc_temp(s, STEP ? a.pos[b] : t);
    mc_store(dst, acc);
    if (!STEP && s.store && t < len && t < s.cap)
      mc_store(static_cast<T*>(s.store) + ((static_cast<long long>(b) * s.heads + c / s.d_in) * s.cap + t) * s.store_d + c % s.d_in, acc);
  }
}

// bf16, at most 4 taps, d_in even and equal to d_out, 4-byte aligned rows.  A thread owns 2 channels x MC_TOK tokens (few registers, so
// that many warps fit an SM: the kernel lives on loads in flight); the rows of its next eight tokens are on their way while it works
// on these.
constexpr int MC_TOK = 64, MC_VEC = 256;
__global__ void __launch_bounds__(MC_VEC, 4) mix_vec_kernel(const __grid_constant__ MixArgs a) {
  pdl_entry();
  const int nblk = (a.S + MC_TOK - 1) / MC_TOK;
  const long long total = static_cast<long long>(a.B) * nblk * a.groups;
  const long long i = blockIdx.x * static_cast<long long>(MC_VEC) + threadIdx.x;
  if (i >= total) return;
  int o = static_cast<int>(i % a.groups);
  const long long bt = i / a.groups;
  const int t0 = static_cast<int>(bt % nblk) * MC_TOK, b = static_cast<int>(bt / nblk);
  const MixSegment& s = a.seg[mc_find(a, o, 2)];
  const int c = o * 2, K = s.taps;
  const int len = a.lens ? a.lens[b] : a.S;
  float wt[2][4], bs[2];                           // fewer than 4 taps: leading zeros
  const bool quad = K == 4 && (reinterpret_cast<uintptr_t>(s.w) & 15) == 0;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    bs[e] = K > 0 && s.bias ? s.bias[c + e] : 0.f;
    if (quad) {
      const float4 w4 = *reinterpret_cast<const float4*>(s.w + (c + e) * 4);
      wt[e][0] = w4.x; wt[e][1] = w4.y; wt[e][2] = w4.z; wt[e][3] = w4.w;
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) wt[e][j] = K == 0 ? (j == 3 ? 1.f : 0.f) : (j >= 4 - K ? s.w[(c + e) * K + j - (4 - K)] : 0.f);
  }
  const int act = s.act;
  const float coef = s.temp_coef, every = s.temp_every, act_a = s.act_a, act_b = s.act_b;
  const long long x_ss = a.x_ss, out_ld = s.out_ld;
  const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.x) + b * a.x_sb + s.col + c + t0 * x_ss;
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(s.out) + (static_cast<long long>(b) * a.S + t0) * out_ld + c;
  __nv_bfloat16* slot = s.store ? static_cast<__nv_bfloat16*>(s.store) + ((static_cast<long long>(b) * s.heads + c / s.d_in) * s.cap + t0) * s.store_d + c % s.d_in : nullptr;
  const int store_d = s.store_d, keep = min(len, s.cap);      // keep: tokens that go to the store
  auto row = [&](int u) { return *reinterpret_cast<const uint32_t*>(src + u * x_ss); };
  float2 win[4];                                   // x[t] in win[(t - t0) % 4]
#pragma unroll
  for (int j = 0; j < 3; ++j) win[j + 1] = unpack_bf16x2(t0 > 0 ? row(j - 3) : 0u);      // before the start: zeros (MC_TOK >= 3)
  auto one = [&](int t, int u, uint32_t raw) {
    win[u] = unpack_bf16x2(raw);
    float a0 = bs[0], a1 = bs[1];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      a0 += win[(u + 1 + j) & 3].x * wt[0][j];
      a1 += win[(u + 1 + j) & 3].y * wt[1][j];
    }
    if (act == MC_SILU) {
      a0 = __fdividef(a0, 1.f + __expf(-a0));
      a1 = __fdividef(a1, 1.f + __expf(-a1));
    } else if (act == MC_RELU2) {
      a0 = fmaxf(a0, 0.f) * fmaxf(a0, 0.f);
      a1 = fmaxf(a1, 0.f) * fmaxf(a1, 0.f);
    } else if (act == MC_XIELU) {
      a0 = mc_xielu(a0, act_a, act_b);
      a1 = mc_xielu(a1, act_a, act_b);
    }
    if (every > 0.f) {
      const float f = mc_temp_fast(coef, every, t);
      a0 *= f; a1 *= f;
    }
    const uint32_t r = pack_bf16x2(a0, a1);
    *reinterpret_cast<uint32_t*>(dst) = r;
    dst += out_ld;
    if (slot) {
      if (t < keep) *reinterpret_cast<uint32_t*>(slot) = r;
      slot += store_d;
    }
  };
  if (t0 + MC_TOK <= a.S) {                        // a whole block
    uint32_t next[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) next[u] = row(u);
#pragma unroll 1
    for (int t = t0; t < t0 + MC_TOK; t += 8) {
      src += 8 * x_ss;
      const bool more = t + 8 < t0 + MC_TOK;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const uint32_t raw = next[u];
        if (more) next[u] = row(u);
        one(t + u, u & 3, raw);
      }
    }
  } else {
#pragma unroll 1
    for (int t = t0; t < a.S; t += 4) {
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (t + u < a.S) one(t + u, u, row(u));
      src += 4 * x_ss;
    }
  }
  if (K > 0 && s.window && len > t0 && len <= t0 + MC_TOK) {       // the row's last token lies here: its last K inputs
    const __nv_bfloat16* xb = static_cast<const __nv_bfloat16*>(a.x) + b * a.x_sb + s.col + c;
    __nv_bfloat16* w = static_cast<__nv_bfloat16*>(s.window) + (static_cast<long long>(b) * s.heads * s.d_in + c) * K;
    for (int j = 0; j < K; ++j) {
      const int t = len - K + j;
      w[j] = t < 0 ? __float2bfloat16(0.f) : xb[t * x_ss];
      w[K + j] = t < 0 ? __float2bfloat16(0.f) : xb[t * x_ss + 1];
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
  bool vec = !step && dtype == 0 && ((a.x_sb | a.x_ss) & 1) == 0 && (reinterpret_cast<uintptr_t>(a.x) & 3) == 0;
  long long channels = 0;
  for (int i = 0; i < a.n_seg; ++i) {
    const MixSegment& s = a.seg[i];
    if (s.heads <= 0 || s.d_in <= 0 || s.d_out < s.d_in || s.taps < 0 || s.out == nullptr || (s.taps > 0 && s.w == nullptr)) return -2;
    if (step && ((s.taps > 0 && s.window == nullptr) || s.store != nullptr)) return -3;
    if (reinterpret_cast<uintptr_t>(s.window) & 7) return -3;
    if (s.store != nullptr && (s.cap <= 0 || s.store_d < s.d_in)) return -4;
    channels += static_cast<long long>(s.heads) * s.d_out;
    vec = vec && s.taps <= 4 && s.d_in == s.d_out && ((s.d_in | s.col | s.out_ld | s.store_d) & 1) == 0 &&
          ((reinterpret_cast<uintptr_t>(s.out) | reinterpret_cast<uintptr_t>(s.store)) & 3) == 0;
  }
  if (channels > 0x7fffffffLL) return -1;
  a.groups = static_cast<int>(vec ? channels / 2 : channels);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (vec) {
    const long long total = static_cast<long long>(a.B) * ((a.S + MC_TOK - 1) / MC_TOK) * a.groups;
    return (int)launch_dependent(mix_vec_kernel, dim3(static_cast<unsigned>((total + MC_VEC - 1) / MC_VEC)), dim3(MC_VEC), 0, st, a);
  }
  const long long rows = static_cast<long long>(a.B) * a.S;
  const dim3 grid(static_cast<unsigned>((a.groups + 255) / 256), static_cast<unsigned>(rows < 65535 ? rows : 65535));
  if (step)
    return (int)(dtype == 1 ? launch_dependent(mix_plain_kernel<float, true>, grid, dim3(256), 0, st, a)
                            : launch_dependent(mix_plain_kernel<__nv_bfloat16, true>, grid, dim3(256), 0, st, a));
  return (int)(dtype == 1 ? launch_dependent(mix_plain_kernel<float, false>, grid, dim3(256), 0, st, a)
                          : launch_dependent(mix_plain_kernel<__nv_bfloat16, false>, grid, dim3(256), 0, st, a));
}
