// Queries, keys and values between their projection and attention: rotation of queries and keys by position (their first channels), values
// divided by their root mean square and turned by position as well, and the rows of keys and values in the store (plain, or `keep` slots
// for the first positions followed by a ring).
//
// Rotation pairs channel i with channel i + half of the rotated part; (cos, sin) come from tables [positions, half].
// Compiled without fast math.
#include "common.cuh"

namespace tyr {

__device__ __forceinline__ float rs_load(const float* p) { return *p; }
__device__ __forceinline__ float rs_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void rs_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void rs_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct RotaryStoreArgs {
  const void* y;               // [B * S, ld]: q (H * dk) | k (G * dk) | v (G * dv)
  long long ld;
  const float2 *key_turns, *value_turns;     // [positions, key_half], [positions, value_half] (null: no turns)
  void *q_out, *k_out, *v_out; // [B * S, H, q_row], [B * S, G, k_row], [B * S, G, v_row] (the last two nullable)
  void *k_store, *v_store;     // [B, G, cap, dkp], [B, G, cap, dvp] (nullable)
  const int* pos;              // position of token 0 of each row (nullable: 0)
  const int* lens;             // tokens of each row (nullable: S)
  int B, S, H, G, dk, dv, q_row, k_row, v_row, dkp, dvp, cap, ring, keep, key_half, value_half, positions, norm_v;
  float eps;
  int* err;
};

// slot of position p of a row with n tokens from p0 on, -1 when it is not kept
__device__ __forceinline__ int rs_slot(const RotaryStoreArgs& a, int p0, int n, int s) {
  const int p = p0 + s, len = a.cap - a.keep;
  if (a.k_store == nullptr || s >= n || p < 0) return -1;
  if (!a.ring) return p < a.cap ? p : -1;
  if (p < a.keep) return p;
  return p0 + n - p <= len ? a.keep + (p - a.keep) % len : -1;
}

// One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256) rotary_store_kernel(RotaryStoreArgs a) {
  pdl_entry();
  const int lane = threadIdx.x & 31, heads = a.H + 2 * a.G;
  const long long total = static_cast<long long>(a.B) * a.S * heads;
  for (long long i = blockIdx.x * 8LL + (threadIdx.x >> 5); i < total; i += gridDim.x * 8LL) {
    const int hd = static_cast<int>(i % heads);
    const long long row = i / heads;
    const int b = static_cast<int>(row / a.S), s = static_cast<int>(row % a.S);
    const int p0 = a.pos ? a.pos[b] : 0, p = p0 + s;
    if (p < 0 || p >= a.positions) {
      if (lane == 0 && hd == 0) report_error(a.err, ERR_BOUNDS, p);
      continue;
    }
    const bool is_q = hd < a.H, is_v = hd >= a.H + a.G;
    const int g = is_q ? hd : (is_v ? hd - a.H - a.G : hd - a.H);
    const int n_in = is_v ? a.dv : a.dk, n_out = is_q ? a.q_row : (is_v ? a.v_row : a.k_row), n_slot = is_v ? a.dvp : a.dkp;
    const T* src = static_cast<const T*>(a.y) + row * a.ld + (is_v ? (a.H + a.G) * a.dk + g * a.dv : hd * a.dk);
    T* dst = static_cast<T*>(is_q ? a.q_out : (is_v ? a.v_out : a.k_out));
    if (dst) dst += (row * (is_q ? a.H : a.G) + g) * n_out;
    const int at = is_q ? -1 : rs_slot(a, p0, a.lens ? a.lens[b] : a.S, s);
    T* slot = at < 0 ? nullptr : static_cast<T*>(is_v ? a.v_store : a.k_store) + ((static_cast<long long>(b) * a.G + g) * a.cap + at) * n_slot;
    float rstd = 1.f;
    if (is_v && a.norm_v) {
      float ss = 0.f;
      for (int d = lane; d < n_in; d += 32) {
        const float v = rs_load(src + d);
        ss += v * v;
      }
      rstd = 1.f / sqrtf(warp_sum(ss) / n_in + a.eps);
    }
    const float2* turns = is_v ? a.value_turns : a.key_turns;
    const int half = turns == nullptr ? 0 : (is_v ? a.value_half : a.key_half);
    turns += static_cast<long long>(p) * half;
    for (int d = lane; d < max(dst ? n_out : 0, slot ? n_slot : 0); d += 32) {
      float v = d < n_in ? rs_load(src + d) * rstd : 0.f;
      if (d < 2 * half) {
        const float2 cs = turns[d < half ? d : d - half];
        const float w = rs_load(src + (d < half ? d + half : d - half)) * rstd;
        v = d < half ? v * cs.x - w * cs.y : v * cs.x + w * cs.y;
      }
      if (dst && d < n_out) rs_store(dst + d, v);
      if (slot && d < n_slot) rs_store(slot + d, v);
    }
  }
}

__device__ __forceinline__ void rs_load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 t = unpack_bf16x2(w[e]);
    f[2 * e] = t.x; f[2 * e + 1] = t.y;
  }
}

// Turns of the eight channels from l8 on; whole vectors lie in one half of the rotated part.
struct Turns8 {
  float c[8], s[8];
  int partner;                 // channel offset of the pairs' other halves, 0: the channels do not turn
  __device__ __forceinline__ void load(const float2* turns, int p, int half, int l8) {
    partner = turns == nullptr || l8 >= 2 * half ? 0 : (l8 < half ? half : -half);
    if (partner == 0) return;
    const float4* t = reinterpret_cast<const float4*>(turns + static_cast<long long>(p) * half + (l8 < half ? l8 : l8 - half));
    const float sign = l8 < half ? -1.f : 1.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float4 x = t[e];
      c[2 * e] = x.x; s[2 * e] = sign * x.y; c[2 * e + 1] = x.z; s[2 * e + 1] = sign * x.w;
    }
  }
  __device__ __forceinline__ void apply(const __nv_bfloat16* src, float scale, float (&f)[8]) const {
    if (partner == 0) return;
    float w[8];
    rs_load8(src + partner, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = f[e] * c[e] + w[e] * scale * s[e];
  }
};

// bf16 heads of up to 128 channels in 16-byte vectors: one CTA per token, half a warp per head.
__global__ void __launch_bounds__(256, 5) rotary_store_vec_kernel(RotaryStoreArgs a) {
  pdl_entry();
  const int sub = threadIdx.x >> 4, l8 = (threadIdx.x & 15) * 8, subs = blockDim.x >> 4;
  const long long row = blockIdx.x;
  const int b = static_cast<int>(row / a.S), s = static_cast<int>(row % a.S);
  const int p0 = a.pos ? a.pos[b] : 0, p = p0 + s;
  if (p < 0 || p >= a.positions) {
    if (threadIdx.x == 0) report_error(a.err, ERR_BOUNDS, p);
    return;
  }
  const __nv_bfloat16* y = static_cast<const __nv_bfloat16*>(a.y) + row * a.ld;
  const int at = rs_slot(a, p0, a.lens ? a.lens[b] : a.S, s);
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  auto pack = [](const float (&f)[8]) { return make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7])); };
  Turns8 turn;
  turn.load(a.key_turns, p, a.key_half, l8);
#pragma unroll 2
  for (int hd = sub; hd < a.H + a.G; hd += subs) {
    const __nv_bfloat16* src = y + hd * a.dk + l8;
    uint4 r = zero;
    if (l8 < a.dk) {
      float f[8];
      rs_load8(src, f);
      turn.apply(src, 1.f, f);
      r = pack(f);
    }
    if (hd < a.H) {
      if (l8 < a.q_row) *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.q_out) + (row * a.H + hd) * a.q_row + l8) = r;
    } else {
      const int g = hd - a.H;
      if (a.k_out && l8 < a.k_row) *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.k_out) + (row * a.G + g) * a.k_row + l8) = r;
      if (at >= 0 && l8 < a.dkp)
        *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.k_store) + ((static_cast<long long>(b) * a.G + g) * a.cap + at) * a.dkp + l8) = r;
    }
  }
  turn.load(a.value_turns, p, a.value_half, l8);
  const int rounds = (a.G + subs - 1) / subs;
  // the subs that took no key in the last round begin with the values
  const int first = (sub + subs - (a.H + a.G) % subs) % subs;
  for (int i = 0; i < rounds; ++i) {                 // whole warps stay together for the sums
    const int g = first + i * subs;
    const __nv_bfloat16* src = y + (a.H + a.G) * a.dk + g * a.dv + l8;
    const bool on = g < a.G && l8 < a.dv;
    float f[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = 0.f;
    if (on) rs_load8(src, f);
    float rstd = 1.f;
    if (a.norm_v) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      rstd = 1.f / sqrtf(ss / a.dv + a.eps);
    }
    if (g >= a.G) continue;
    uint4 r = zero;
    if (on) {
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] *= rstd;
      turn.apply(src, rstd, f);
      r = pack(f);
    }
    if (a.v_out && l8 < a.v_row) *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.v_out) + (row * a.G + g) * a.v_row + l8) = r;
    if (at >= 0 && l8 < a.dvp)
      *reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.v_store) + ((static_cast<long long>(b) * a.G + g) * a.cap + at) * a.dvp + l8) = r;
  }
}

}  // namespace tyr

using namespace tyr;

// dtype: 0 = bf16, 1 = fp32 (rows, outputs and stores).  sizes: B, S, H, G, dk, dv, q_row, k_row, v_row, dkp, dvp, cap, ring, keep, key_half,
// value_half, positions, norm_v.
extern "C" TYR_EXPORT int tyr_rotary_store(const void* y, long long ld, const void* key_turns, const void* value_turns, void* q_out, void* k_out,
                                           void* v_out, void* k_store, void* v_store, const int* pos, const int* lens, const int* sizes, float eps,
                                           int dtype, int* err, void* stream) {
  RotaryStoreArgs a{y, ld, (const float2*)key_turns, (const float2*)value_turns, q_out, k_out, v_out, k_store, v_store, pos, lens,
                    sizes[0], sizes[1], sizes[2], sizes[3], sizes[4], sizes[5], sizes[6], sizes[7], sizes[8], sizes[9], sizes[10], sizes[11],
                    sizes[12], sizes[13], sizes[14], sizes[15], sizes[16], sizes[17], eps, err};
  if (a.B <= 0 || a.S <= 0 || a.H <= 0 || a.G <= 0 || a.dk <= 0 || a.dv <= 0 || a.q_row < a.dk || q_out == nullptr || a.positions <= 0) return -1;
  if ((k_store != nullptr) != (v_store != nullptr) || (k_store != nullptr && (a.cap <= 0 || a.dkp < a.dk || a.dvp < a.dv))) return -2;
  if (a.keep < 0 || (a.ring && a.keep >= a.cap)) return -3;
  if ((k_out && a.k_row < a.dk) || (v_out && a.v_row < a.dv) || 2 * a.key_half > a.dk || 2 * a.value_half > a.dv || a.key_half < 0 || a.value_half < 0) return -4;
  uintptr_t al = 0;
  for (const void* p : {y, key_turns, value_turns, (const void*)q_out, (const void*)k_out, (const void*)v_out, (const void*)k_store, (const void*)v_store})
    al |= reinterpret_cast<uintptr_t>(p);
  const int widest = max(max(max(a.q_row, a.k_row), max(a.v_row, a.dkp)), a.dvp);
  if (dtype == 0 && ((ld | a.dk | a.dv | a.q_row | a.k_row | a.v_row | a.dkp | a.dvp | a.key_half | a.value_half) & 7) == 0 && widest <= 128 && (al & 15) == 0) {
    const int heads = a.H + a.G;
    const unsigned threads = heads >= 12 ? 256 : (heads >= 6 ? 128 : 64);
    return (int)launch_dependent(rotary_store_vec_kernel, dim3(static_cast<unsigned>(static_cast<long long>(a.B) * a.S)), dim3(threads), 0, (cudaStream_t)stream, a);
  }
  const long long want = (static_cast<long long>(a.B) * a.S * (a.H + 2 * a.G) + 7) / 8;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 32 ? want : 148LL * 32));
  return (int)(dtype == 1 ? launch_dependent(rotary_store_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, a)
                          : launch_dependent(rotary_store_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, a));
}
