// The pieces of latent attention around its products:
//
//   * latent_norm_store: a row of the down projection holds the query latent, the key/value latent and one rotated key part.  Both latents
//                        are RMS-normed, the key part is rotated by its position, and (key/value latent | key part) is one row of the
//                        store (plain or ring) that serves every head as key and as value.
//   * rotate_heads:      the rotated channels of every query head, in place or into rows of their own.
//
// Rotation pairs channels 2i and 2i + 1; the angles are fractions of a turn reduced in double.  Compiled without fast math.
#include "common.cuh"

namespace tyr {

__device__ __forceinline__ float la_load(const float* p) { return *p; }
__device__ __forceinline__ float la_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void la_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void la_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// channel d of a part whose first `dims` channels turn
template <typename T>
__device__ __forceinline__ float la_rotated(const T* x, int d, int dims, int p, const double* turns) {
  if (d >= dims) return la_load(x + d);
  const double t = p * turns[d >> 1];
  float sn, cs;
  sincospif(2.f * static_cast<float>(t - rint(t)), &sn, &cs);
  const float u = la_load(x + (d & ~1)), v = la_load(x + (d | 1));
  return (d & 1) ? v * cs + u * sn : u * cs - v * sn;
}

struct LatentArgs {
  const void* y;               // [B * S, ld]: query latent (q_rank) | key/value latent (rank) | rotated part (rot)
  long long ld;
  const float *q_w, *kv_w;     // [q_rank], [rank]
  const double* turns;         // [dims / 2]
  void* cq;                    // [B * S, cq_ld]
  void* ck;                    // [B * S, width] rows of the store, zeros past rank + rot (nullable)
  long long cq_ld;
  void* store;                 // [B, cap, width] (nullable)
  const int* pos;              // position of token 0 of each row (nullable: 0)
  const int* lens;             // tokens of each row (nullable: S)
  int B, S, q_rank, rank, rot, dims, width, cap, ring;
  float eps;
};

// One warp per (row, latent).
template <typename T>
__global__ void __launch_bounds__(256) latent_norm_store_kernel(LatentArgs a) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const long long total = 2LL * a.B * a.S;
  for (long long i = blockIdx.x * 8LL + (threadIdx.x >> 5); i < total; i += gridDim.x * 8LL) {
    const bool is_q = (i & 1) == 0;
    const long long row = i >> 1;
    const int n = is_q ? a.q_rank : a.rank;
    const T* src = static_cast<const T*>(a.y) + row * a.ld + (is_q ? 0 : a.q_rank);
    const float* w = is_q ? a.q_w : a.kv_w;
    T *dst = nullptr, *slot = nullptr;
    int p = 0;
    if (is_q) {
      dst = static_cast<T*>(a.cq) + row * a.cq_ld;
    } else {
      const int b = static_cast<int>(row / a.S), s = static_cast<int>(row % a.S);
      const int len = a.lens ? a.lens[b] : a.S, p0 = a.pos ? a.pos[b] : 0;
      p = p0 + s;
      if (a.ck) dst = static_cast<T*>(a.ck) + row * a.width;
      if (a.store && s < len && p >= 0 && (a.ring ? p0 + len - p <= a.cap : p < a.cap))      // a ring store keeps the last cap positions
        slot = static_cast<T*>(a.store) + (static_cast<long long>(b) * a.cap + (a.ring ? p % a.cap : p)) * a.width;
    }
    auto put = [&](int d, float v) {
      if (dst) la_store(dst + d, v);
      if (slot) la_store(slot + d, v);
    };
    float ss = 0.f;
    bool vec = false;
    if constexpr (sizeof(T) == 2)
      vec = (n & 7) == 0 && ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(dst) | reinterpret_cast<uintptr_t>(slot) | reinterpret_cast<uintptr_t>(w)) & 15) == 0;
    if (vec) {
      auto load8 = [&](int d, float (&f)[8]) {
        const uint4 u = *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(src + d));
        const uint32_t r[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 t = unpack_bf16x2(r[e]);
          f[2 * e] = t.x; f[2 * e + 1] = t.y;
        }
      };
      for (int d = lane * 8; d < n; d += 256) {
        float f[8];
        load8(d, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
      }
      const float rstd = 1.f / sqrtf(warp_sum(ss) / n + a.eps);
      for (int d = lane * 8; d < n; d += 256) {
        float f[8];
        load8(d, f);
        uint32_t r[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) r[e] = pack_bf16x2(f[2 * e] * rstd * w[d + 2 * e], f[2 * e + 1] * rstd * w[d + 2 * e + 1]);
        const uint4 u = make_uint4(r[0], r[1], r[2], r[3]);
        if (dst) *reinterpret_cast<uint4*>(reinterpret_cast<char*>(dst + d)) = u;
        if (slot) *reinterpret_cast<uint4*>(reinterpret_cast<char*>(slot + d)) = u;
      }
    } else {
      for (int d = lane; d < n; d += 32) {
        const float v = la_load(src + d);
        ss += v * v;
      }
      const float rstd = 1.f / sqrtf(warp_sum(ss) / n + a.eps);
      for (int d = lane; d < n; d += 32) put(d, la_load(src + d) * rstd * w[d]);
    }
    if (!is_q)
      for (int d = lane; d < a.width - a.rank; d += 32) put(a.rank + d, d < a.rot ? la_rotated(src + a.rank, d, a.dims, p, a.turns) : 0.f);
  }
}

struct RotateArgs {
  const void* x;               // [B, S, H, .] by strides; the part to rotate starts at channel 0
  void* y;                     // the same with strides of its own; may be x
  const double* turns;
  const int* pos;              // position of token 0 of each row (nullable: 0)
  long long x_sb, x_ss, x_sh, y_sb, y_ss, y_sh;
  int B, S, H, rot, dims, width;      // channels [rot, width) of y are set to zero
};

constexpr int ROT_HEADS = 8;

// A thread per (token, channel pair, eight heads), which share the angle.
template <typename T>
__global__ void __launch_bounds__(256) rotate_heads_kernel(RotateArgs a) {
  pdl_entry();
  const int pairs = (a.width + 1) / 2, groups = (a.H + ROT_HEADS - 1) / ROT_HEADS;
  const long long total = static_cast<long long>(a.B) * a.S * groups * pairs;
  for (long long i = blockIdx.x * 256LL + threadIdx.x; i < total; i += gridDim.x * 256LL) {
    const int d = 2 * static_cast<int>(i % pairs), h0 = static_cast<int>(i / pairs % groups) * ROT_HEADS;
    const long long row = i / pairs / groups;
    const int b = static_cast<int>(row / a.S), s = static_cast<int>(row % a.S);
    const T* x = static_cast<const T*>(a.x) + b * a.x_sb + s * a.x_ss + h0 * a.x_sh + d;
    T* y = static_cast<T*>(a.y) + b * a.y_sb + s * a.y_ss + h0 * a.y_sh + d;
    float sn = 0.f, cs = 1.f;
    if (d + 1 < a.dims) {
      const double t = ((a.pos ? a.pos[b] : 0) + s) * a.turns[d >> 1];
      sincospif(2.f * static_cast<float>(t - rint(t)), &sn, &cs);
    }
    float u[ROT_HEADS], w[ROT_HEADS];
#pragma unroll
    for (int h = 0; h < ROT_HEADS; ++h) {
      u[h] = h0 + h < a.H && d < a.rot ? la_load(x + h * a.x_sh) : 0.f;
      w[h] = h0 + h < a.H && d + 1 < a.rot ? la_load(x + h * a.x_sh + 1) : 0.f;
    }
#pragma unroll
    for (int h = 0; h < ROT_HEADS; ++h) {
      if (h0 + h >= a.H) break;
      la_store(y + h * a.y_sh, u[h] * cs - w[h] * sn);
      if (d + 1 < a.width) la_store(y + h * a.y_sh + 1, w[h] * cs + u[h] * sn);
    }
  }
}

}  // namespace tyr

using namespace tyr;

// dtype: 0 = bf16, 1 = fp32 (activations and store; weights fp32, turns double).
extern "C" TYR_EXPORT int tyr_latent_norm_store(const void* y, long long ld, const float* q_w, const float* kv_w, const double* turns, void* cq,
                                                long long cq_ld, void* ck, void* store, const int* pos, const int* lens, int B, int S, int q_rank,
                                                int rank, int rot, int dims, int width, int cap, int ring, float eps, int dtype, void* stream) {
  if (B <= 0 || S <= 0 || q_rank <= 0 || rank <= 0 || rot < 0 || dims < 0 || dims > rot || (dims & 1) || width < rank + rot || cq == nullptr) return -1;
  if (store != nullptr && cap <= 0) return -2;
  LatentArgs a{y, ld, q_w, kv_w, turns, cq, ck, cq_ld, store, pos, lens, B, S, q_rank, rank, rot, dims, width, cap, ring, eps};
  const long long want = (2LL * B * S + 7) / 8;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 32 ? want : 148LL * 32));
  return (int)(dtype == 1 ? launch_dependent(latent_norm_store_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, a)
                          : launch_dependent(latent_norm_store_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, a));
}

// strides: (batch, token, head) element strides of x, then of y.
extern "C" TYR_EXPORT int tyr_rotate_heads(const void* x, void* y, const double* turns, const int* pos, const long long* strides, int B, int S, int H,
                                           int rot, int dims, int width, int dtype, void* stream) {
  if (B <= 0 || S <= 0 || H <= 0 || rot < 0 || dims < 0 || dims > rot || (dims & 1) || width < rot || width <= 0) return -1;
  RotateArgs a{x, y, turns, pos, strides[0], strides[1], strides[2], strides[3], strides[4], strides[5], B, S, H, rot, dims, width};
  const long long want = (static_cast<long long>(B) * S * ((H + ROT_HEADS - 1) / ROT_HEADS) * ((width + 1) / 2) + 255) / 256;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 32 ? want : 148LL * 32));
  return (int)(dtype == 1 ? launch_dependent(rotate_heads_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, a)
                          : launch_dependent(rotate_heads_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, a));
}
