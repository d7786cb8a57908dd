// RMSNorm family (memory-bound, one warp per row, fp32 accumulation).
//
//  * lincomb_rmsnorm: out = sum_i s_i * t_i (up to 4 bf16 inputs, fp32 device scalars) and
//    normed = out * rsqrt(mean(out^2) + eps) in ONE pass over the inputs.  This is the residual
//    stream update of the modded-nanogpt block (x = lam_x*x + lam_0*x0, x += lam*attn, ...)
//    fused with the pre-norm that follows it; the reference issues one broadcast-multiply, one
//    add and 5-7 norm kernels for the same thing (Examples/NanoChat/ModdedGPT.lean:449-452,
//    586-611; Tyr/Typed/Neural.lean:38-43).
//  * its backward: grads of every input and of every scalar from (d_out, d_normed).
//  * rmsnorm_weighted: y = x * rstd * w with w either plain, "(1 + w)" zero-centred (Qwen3.5) or
//    absent, optional SiLU(z) gate (GatedDeltaNet output norm) and optional residual add
//    (cc/src/tyr.cpp:3766-3772, Tyr/Model/Qwen35/Model.lean RMSNorm variants).
#include "common.cuh"

namespace tyr {

struct LincombArgs {
  const __nv_bfloat16* t[4];
  const float* scal;   // device pointer to n_in floats (nullptr = all ones)
  int n_in;
  int rows, D;
  float eps;
};

__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  uint4 u = *reinterpret_cast<const uint4*>(p);
  float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z),
         d = unpack_bf16x2(u.w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&f)[8]) {
  uint4 u;
  u.x = pack_bf16x2(f[0], f[1]); u.y = pack_bf16x2(f[2], f[3]);
  u.z = pack_bf16x2(f[4], f[5]); u.w = pack_bf16x2(f[6], f[7]);
  *reinterpret_cast<uint4*>(p) = u;
}

template <int NIN>
__global__ void __launch_bounds__(256)
lincomb_rmsnorm_fwd_kernel(LincombArgs a, __nv_bfloat16* __restrict__ out,
                           __nv_bfloat16* __restrict__ normed) {
  pdl_entry();
  const int warps = blockDim.x >> 5;
  const int lane = threadIdx.x & 31;
  float s[NIN];
#pragma unroll
  for (int i = 0; i < NIN; ++i) s[i] = a.scal ? a.scal[i] : 1.f;
  const int nvec = a.D >> 3;
  for (long long row = blockIdx.x * warps + (threadIdx.x >> 5); row < a.rows;
       row += static_cast<long long>(gridDim.x) * warps) {
    const long long base = row * a.D;
    float ss = 0.f;
    for (int v = lane; v < nvec; v += 32) {
      float acc[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] = 0.f;
#pragma unroll
      for (int i = 0; i < NIN; ++i) {
        float f[8];
        load8(a.t[i] + base + v * 8, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] += s[i] * f[j];
      }
      if (out) {
        store8(out + base + v * 8, acc);
        // normalise the value that is actually stored (bf16-rounded) so that the backward,
        // which only sees the stored tensor, recomputes the same statistics
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = __bfloat162float(__float2bfloat16(acc[j]));
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += acc[j] * acc[j];
    }
    if (normed == nullptr) continue;
    ss = warp_sum(ss);
    const float rstd = rsqrtf(ss / a.D + a.eps);
    for (int v = lane; v < nvec; v += 32) {
      float acc[8];
      if (out) {
        load8(out + base + v * 8, acc);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = 0.f;
#pragma unroll
        for (int i = 0; i < NIN; ++i) {
          float f[8];
          load8(a.t[i] + base + v * 8, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[j] += s[i] * f[j];
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] *= rstd;
      store8(normed + base + v * 8, acc);
    }
  }
}

struct LincombBwdArgs {
  const __nv_bfloat16* t[4];      // forward inputs (needed for the scalar gradients)
  __nv_bfloat16* dt[4];           // gradient outputs (nullable)
  const float* scal;
  float* dscal;                   // fp32[n_in], accumulated with atomics (nullable)
  const __nv_bfloat16* out;       // forward combined output (the tensor that was normalised)
  const __nv_bfloat16* d_out;     // nullable
  const __nv_bfloat16* d_normed;  // nullable
  int n_in, rows, D;
  float eps;
};

template <int NIN>
__global__ void __launch_bounds__(256)
lincomb_rmsnorm_bwd_kernel(LincombBwdArgs a) {
  pdl_entry();
  const int warps = blockDim.x >> 5;
  const int lane = threadIdx.x & 31;
  const int wid = threadIdx.x >> 5;
  float s[NIN], ds[NIN];
#pragma unroll
  for (int i = 0; i < NIN; ++i) {
    s[i] = a.scal ? a.scal[i] : 1.f;
    ds[i] = 0.f;
  }
  const int nvec = a.D >> 3;
  for (long long row = blockIdx.x * warps + wid; row < a.rows;
       row += static_cast<long long>(gridDim.x) * warps) {
    const long long base = row * a.D;
    float rstd = 0.f, coef = 0.f;
    if (a.d_normed) {
      float ss = 0.f, dot = 0.f;
      for (int v = lane; v < nvec; v += 32) {
        float o[8], dn[8];
        load8(a.out + base + v * 8, o);
        load8(a.d_normed + base + v * 8, dn);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          ss += o[j] * o[j];
          dot += o[j] * dn[j];
        }
      }
      ss = warp_sum(ss);
      dot = warp_sum(dot);
      rstd = rsqrtf(ss / a.D + a.eps);
      coef = rstd * rstd * rstd * dot / a.D;
    }
    for (int v = lane; v < nvec; v += 32) {
      float g[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] = 0.f;
      if (a.d_out) load8(a.d_out + base + v * 8, g);
      if (a.d_normed) {
        float o[8], dn[8];
        load8(a.out + base + v * 8, o);
        load8(a.d_normed + base + v * 8, dn);
#pragma unroll
        for (int j = 0; j < 8; ++j) g[j] += rstd * dn[j] - coef * o[j];
      }
#pragma unroll
      for (int i = 0; i < NIN; ++i) {
        if (a.dscal) {
          float f[8];
          load8(a.t[i] + base + v * 8, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) ds[i] += g[j] * f[j];
        }
        if (a.dt[i]) {
          float o[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) o[j] = s[i] * g[j];
          store8(a.dt[i] + base + v * 8, o);
        }
      }
    }
  }
  if (a.dscal) {
    __shared__ float red[4][8];
#pragma unroll
    for (int i = 0; i < NIN; ++i) {
      float v = warp_sum(ds[i]);
      if (lane == 0) red[i][wid] = v;
    }
    __syncthreads();
    if (threadIdx.x < NIN) {
      float v = 0.f;
      for (int w = 0; w < warps; ++w) v += red[threadIdx.x][w];
      atomicAdd(a.dscal + threadIdx.x, v);
    }
  }
}

// y = x * rstd * weight-ish (+ optional gate), used by the inference model families.
struct RmsWArgs {
  const __nv_bfloat16* x;
  const __nv_bfloat16* w;       // [D] (nullable)
  const __nv_bfloat16* gate;    // [rows, D] (nullable): y *= silu(gate)
  const __nv_bfloat16* resid;   // [rows, D] (nullable): x := x + resid before the norm
  __nv_bfloat16* resid_out;     // receives x + resid (nullable)
  __nv_bfloat16* y;
  int rows, D;
  float eps;
  int one_plus_w;               // weight = 1 + w
};

__global__ void __launch_bounds__(256) rmsnorm_weighted_kernel(RmsWArgs a) {
  pdl_entry();
  const int warps = blockDim.x >> 5;
  const int lane = threadIdx.x & 31;
  const int nvec = a.D >> 3;
  for (long long row = blockIdx.x * warps + (threadIdx.x >> 5); row < a.rows;
       row += static_cast<long long>(gridDim.x) * warps) {
    const long long base = row * a.D;
    float ss = 0.f;
    for (int v = lane; v < nvec; v += 32) {
      float f[8];
      load8(a.x + base + v * 8, f);
      if (a.resid) {
        float r[8];
        load8(a.resid + base + v * 8, r);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] += r[j];
        if (a.resid_out) {
          store8(a.resid_out + base + v * 8, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = __bfloat162float(__float2bfloat16(f[j]));
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += f[j] * f[j];
    }
    ss = warp_sum(ss);
    const float rstd = rsqrtf(ss / a.D + a.eps);
    for (int v = lane; v < nvec; v += 32) {
      float f[8];
      if (a.resid && a.resid_out) {
        load8(a.resid_out + base + v * 8, f);
      } else {
        load8(a.x + base + v * 8, f);
        if (a.resid) {
          float r[8];
          load8(a.resid + base + v * 8, r);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] += r[j];
        }
      }
      float w[8];
      if (a.w) {
        load8(a.w + v * 8, w);
        if (a.one_plus_w) {
#pragma unroll
          for (int j = 0; j < 8; ++j) w[j] += 1.f;
        }
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) w[j] = 1.f;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = f[j] * rstd * w[j];
      if (a.gate) {
        float g[8];
        load8(a.gate + base + v * 8, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= g[j] / (1.f + __expf(-g[j]));
      }
      store8(a.y + base + v * 8, f);
    }
  }
}

// Decode-sized inputs (a few dozen rows of a few thousand channels): one CTA per row, the row stays in registers between
// the sum of squares and the scaled write, so every operand is read once and the kernel is one load latency deep instead
// of two loops of eight dependent iterations per warp (8 - 9 us per launch with one warp per row, measured in a decode step).
constexpr int kRowVecs = 4;     // 16-byte vectors per thread: D <= 256 * 4 * 8

__global__ void __launch_bounds__(256) rmsnorm_weighted_row_kernel(RmsWArgs a) {
  pdl_entry();
  __shared__ float red[8];
  const int tid = threadIdx.x;
  const int nvec = a.D >> 3;
  const long long base = static_cast<long long>(blockIdx.x) * a.D;
  float f[kRowVecs][8];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kRowVecs; ++j) {
    const int v = tid + j * 256;
    if (v < nvec) {
      load8(a.x + base + v * 8, f[j]);
      if (a.resid) {
        float r[8];
        load8(a.resid + base + v * 8, r);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[j][e] += r[e];
        if (a.resid_out) {
          store8(a.resid_out + base + v * 8, f[j]);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[j][e] = __bfloat162float(__float2bfloat16(f[j][e]));
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += f[j][e] * f[j][e];
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) tot += (i < (blockDim.x >> 5)) ? red[i] : 0.f;
  const float rstd = rsqrtf(tot / a.D + a.eps);
#pragma unroll
  for (int j = 0; j < kRowVecs; ++j) {
    const int v = tid + j * 256;
    if (v < nvec) {
      float w[8];
      if (a.w) {
        load8(a.w + v * 8, w);
        if (a.one_plus_w) {
#pragma unroll
          for (int e = 0; e < 8; ++e) w[e] += 1.f;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] = 1.f;
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) f[j][e] = f[j][e] * rstd * w[e];
      if (a.gate) {
        float g[8];
        load8(a.gate + base + v * 8, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[j][e] *= g[e] / (1.f + __expf(-g[e]));
      }
      store8(a.y + base + v * 8, f[j]);
    }
  }
}

// Norm on a sublayer's output, added to an fp32 residual stream:
//   r = (resid ? resid : 0) + x / sqrt(mean(x^2) + eps) * gain,   resid_out = r,   y = r in the compute dtype.
// `gain` holds one number for all channels (n_gain == 1) or one per channel.  One CTA per row; a thread keeps up to kPnVecs
// vectors of 8 channels in registers between the reduction and the write.
struct PostNormArgs {
  const void* x;           // [rows, D] (TX)
  const float* gain;
  float* resid;            // [rows, D] in place (nullable: plain norm)
  void* y;                 // [rows, D] (TY), nullable
  long long x_stride;      // elements between rows of x
  int D, n_gain;
  float eps;
};
constexpr int kPnVecs = 4;

__device__ __forceinline__ void pn_load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 t = unpack_bf16x2(w[e]);
    f[2 * e] = t.x; f[2 * e + 1] = t.y;
  }
}
__device__ __forceinline__ void pn_load8(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void pn_store8(__nv_bfloat16* p, const float (&f)[8]) {
  uint4 u;
  u.x = pack_bf16x2(f[0], f[1]); u.y = pack_bf16x2(f[2], f[3]); u.z = pack_bf16x2(f[4], f[5]); u.w = pack_bf16x2(f[6], f[7]);
  *reinterpret_cast<uint4*>(p) = u;
}
__device__ __forceinline__ void pn_store8(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}
__device__ __forceinline__ float pn_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float pn_get(const float* p) { return *p; }
__device__ __forceinline__ void pn_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void pn_put(float* p, float v) { *p = v; }

template <typename TX, typename TY, bool VEC>
__global__ void __launch_bounds__(256) post_norm_residual_kernel(PostNormArgs a) {
  __shared__ float red[8];
  const long long row = blockIdx.x;
  const int tid = threadIdx.x, nw = blockDim.x >> 5;
  const TX* x = static_cast<const TX*>(a.x) + row * a.x_stride;
  float* resid = a.resid ? a.resid + row * a.D : nullptr;
  TY* y = a.y ? static_cast<TY*>(a.y) + row * a.D : nullptr;
  pdl_entry();
  float f[kPnVecs][8], ss = 0.f;
  if constexpr (VEC) {
#pragma unroll
    for (int j = 0; j < kPnVecs; ++j) {
      const int v = (tid + j * blockDim.x) * 8;
      if (v < a.D) {
        pn_load8(x + v, f[j]);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += f[j][e] * f[j][e];
      }
    }
  } else {
    for (int d = tid; d < a.D; d += blockDim.x) {
      const float t = pn_get(x + d);
      ss += t * t;
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nw; ++i) tot += red[i];
  const float rstd = rsqrtf(tot / a.D + a.eps);
  if constexpr (VEC) {
#pragma unroll
    for (int j = 0; j < kPnVecs; ++j) {
      const int v = (tid + j * blockDim.x) * 8;
      if (v >= a.D) continue;
      float w[8];
      if (a.n_gain == 1) {
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] = a.gain[0];
      } else {
        pn_load8(a.gain + v, w);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) f[j][e] *= rstd * w[e];
      if (resid) {
        float r[8];
        pn_load8(resid + v, r);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[j][e] += r[e];
        pn_store8(resid + v, f[j]);
      }
      if (y) pn_store8(y + v, f[j]);
    }
  } else {
    for (int d = tid; d < a.D; d += blockDim.x) {
      float t = pn_get(x + d) * rstd * a.gain[a.n_gain == 1 ? 0 : d];
      if (resid) {
        t += resid[d];
        resid[d] = t;
      }
      if (y) pn_put(y + d, t);
    }
  }
}

// A sublayer's output added to an fp32 residual stream, and the norm the next layer reads:
//   r = resid + x (x null: r = resid),   resid_out = r,   y = r / sqrt(mean(r^2) + eps) * gain.
struct AddNormArgs {
  const void* x;           // [rows, D] (TX), nullable
  const float* gain;       // [D]
  float* resid;            // [rows, D], in place
  void* y;                 // [rows, D] (TY)
  long long x_stride, r_stride;      // elements between rows
  int D;
  float eps;
};

template <typename TX, typename TY, bool VEC>
__global__ void __launch_bounds__(256) add_norm_kernel(AddNormArgs a) {
  __shared__ float red[8];
  const long long row = blockIdx.x;
  const int tid = threadIdx.x, nw = blockDim.x >> 5;
  const TX* x = a.x ? static_cast<const TX*>(a.x) + row * a.x_stride : nullptr;
  float* resid = a.resid + row * a.r_stride;
  TY* y = static_cast<TY*>(a.y) + row * a.D;
  pdl_entry();
  float f[kPnVecs][8], ss = 0.f;
  if constexpr (VEC) {
#pragma unroll
    for (int j = 0; j < kPnVecs; ++j) {
      const int v = (tid + j * blockDim.x) * 8;
      if (v < a.D) {
        pn_load8(resid + v, f[j]);
        if (x) {
          float t[8];
          pn_load8(x + v, t);
#pragma unroll
          for (int e = 0; e < 8; ++e) f[j][e] += t[e];
          pn_store8(resid + v, f[j]);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += f[j][e] * f[j][e];
      }
    }
  } else {
    for (int d = tid; d < a.D; d += blockDim.x) {
      float t = resid[d];
      if (x) {
        t += pn_get(x + d);
        resid[d] = t;
      }
      ss += t * t;
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nw; ++i) tot += red[i];
  const float rstd = rsqrtf(tot / a.D + a.eps);
  if constexpr (VEC) {
#pragma unroll
    for (int j = 0; j < kPnVecs; ++j) {
      const int v = (tid + j * blockDim.x) * 8;
      if (v >= a.D) continue;
      float w[8];
      pn_load8(a.gain + v, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[j][e] *= rstd * w[e];
      pn_store8(y + v, f[j]);
    }
  } else {
    for (int d = tid; d < a.D; d += blockDim.x) pn_put(y + d, resid[d] * rstd * a.gain[d]);
  }
}

// A sublayer with a norm on either side of it: its output joins an fp32 stream and the next sublayer reads the norm of the sum.
//   t = x + bias;   t <- norm(t) * post;   r = resid + t (replace: r = t);   resid_out = r;   y = norm(r) * gain (no gain: y = r).
struct SandwichNormArgs {
  const void* x;           // [rows, D] (TX)
  const float* bias;       // [D], nullable
  const float* post;       // [D], nullable: x joins as it is
  const float* gain;       // [D], nullable
  float* resid;            // [rows, D], in place
  void* y;                 // [rows, D] (TY)
  long long x_stride, y_stride;      // elements between rows
  int D, replace;
  float eps;
};

__device__ __forceinline__ float pn_block_sum(float v, float* red, int tid, int nw) {
  v = warp_sum(v);
  if ((tid & 31) == 0) red[tid >> 5] = v;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nw; ++i) tot += red[i];
  return tot;
}

// NV: vectors of 8 channels a thread holds (0: any size, element by element).  The weights are constants: they are on their way while the
// kernel in front of this one still runs.
template <typename TX, typename TY, int NV>
__global__ void __launch_bounds__(256) sandwich_norm_kernel(SandwichNormArgs a) {
  __shared__ float red[2][8];
  const long long row = blockIdx.x;
  const int tid = threadIdx.x, nw = blockDim.x >> 5;
  const TX* x = static_cast<const TX*>(a.x) + row * a.x_stride;
  float* resid = a.resid + row * a.D;
  TY* y = static_cast<TY*>(a.y) + row * a.y_stride;
  pdl_trigger();
  if constexpr (NV > 0) {
    constexpr bool EARLY = NV <= 2;                // registers for both gains
    float f[NV][8], r[NV][8], wp[EARLY ? NV : 1][8], wg[EARLY ? NV : 1][8], ss = 0.f;
    if constexpr (EARLY) {
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int v = (tid + j * blockDim.x) * 8;
        if (v >= a.D) continue;
        if (a.post) pn_load8(a.post + v, wp[j]);
        if (a.gain) pn_load8(a.gain + v, wg[j]);
      }
    }
    pdl_wait();
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int v = (tid + j * blockDim.x) * 8;
      if (v >= a.D) continue;
      pn_load8(x + v, f[j]);
      if (!a.replace) pn_load8(resid + v, r[j]);
      if (a.bias) {
        float b[8];
        pn_load8(a.bias + v, b);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[j][e] += b[e];
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += f[j][e] * f[j][e];
    }
    const float inner = a.post ? rsqrtf(pn_block_sum(ss, red[0], tid, nw) / a.D + a.eps) : 1.f;
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int v = (tid + j * blockDim.x) * 8;
      if (v >= a.D) continue;
      if (a.post) {
        float w[8];
        if constexpr (!EARLY) pn_load8(a.post + v, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[j][e] *= inner * (EARLY ? wp[EARLY ? j : 0][e] : w[e]);
      }
      if (!a.replace) {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[j][e] += r[j][e];
      }
      pn_store8(resid + v, f[j]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += f[j][e] * f[j][e];
    }
    const float outer = a.gain ? rsqrtf(pn_block_sum(ss, red[1], tid, nw) / a.D + a.eps) : 1.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int v = (tid + j * blockDim.x) * 8;
      if (v >= a.D) continue;
      if (a.gain) {
        float w[8];
        if constexpr (!EARLY) pn_load8(a.gain + v, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[j][e] *= outer * (EARLY ? wg[EARLY ? j : 0][e] : w[e]);
      }
      pn_store8(y + v, f[j]);
    }
  } else {
    pdl_wait();
    float ss = 0.f;
    for (int d = tid; d < a.D; d += blockDim.x) {
      const float t = pn_get(x + d) + (a.bias ? a.bias[d] : 0.f);
      ss += t * t;
    }
    const float inner = a.post ? rsqrtf(pn_block_sum(ss, red[0], tid, nw) / a.D + a.eps) : 1.f;
    ss = 0.f;
    for (int d = tid; d < a.D; d += blockDim.x) {
      float t = pn_get(x + d) + (a.bias ? a.bias[d] : 0.f);
      if (a.post) t *= inner * a.post[d];
      if (!a.replace) t += resid[d];
      resid[d] = t;
      ss += t * t;
    }
    const float outer = a.gain ? rsqrtf(pn_block_sum(ss, red[1], tid, nw) / a.D + a.eps) : 1.f;
    for (int d = tid; d < a.D; d += blockDim.x) pn_put(y + d, a.gain ? resid[d] * outer * a.gain[d] : resid[d]);
  }
}

static int grid_for_rows(long long rows, int warps_per_block) {
  long long blocks = (rows + warps_per_block - 1) / warps_per_block;
  const long long cap = 148LL * 16;
  return static_cast<int>(blocks < cap ? (blocks < 1 ? 1 : blocks) : cap);
}

}  // namespace tyr

using namespace tyr;

extern "C" TYR_EXPORT int tyr_lincomb_rmsnorm_fwd(const void* t0, const void* t1, const void* t2,
                                                  const void* t3, const float* scal, int n_in,
                                                  int rows, int D, void* out, void* normed,
                                                  float eps, void* stream) {
  if (n_in < 1 || n_in > 4 || (D & 7) || rows <= 0) return -1;
  LincombArgs a;
  a.t[0] = (const __nv_bfloat16*)t0; a.t[1] = (const __nv_bfloat16*)t1;
  a.t[2] = (const __nv_bfloat16*)t2; a.t[3] = (const __nv_bfloat16*)t3;
  a.scal = scal; a.n_in = n_in; a.rows = rows; a.D = D; a.eps = eps;
  const int grid = grid_for_rows(rows, 8);
  cudaStream_t st = (cudaStream_t)stream;
  auto o = (__nv_bfloat16*)out;
  auto n = (__nv_bfloat16*)normed;
  switch (n_in) {
    case 1: launch_dependent(lincomb_rmsnorm_fwd_kernel<1>, dim3(grid), dim3(256), 0, st, a, o, n); break;
    case 2: launch_dependent(lincomb_rmsnorm_fwd_kernel<2>, dim3(grid), dim3(256), 0, st, a, o, n); break;
    case 3: launch_dependent(lincomb_rmsnorm_fwd_kernel<3>, dim3(grid), dim3(256), 0, st, a, o, n); break;
    default: launch_dependent(lincomb_rmsnorm_fwd_kernel<4>, dim3(grid), dim3(256), 0, st, a, o, n); break;
  }
  return (int)cudaGetLastError();
}

extern "C" TYR_EXPORT int tyr_lincomb_rmsnorm_bwd(const void* const* t, void* const* dt,
                                                  const float* scal, float* dscal,
                                                  const void* out, const void* d_out,
                                                  const void* d_normed, int n_in, int rows, int D,
                                                  float eps, void* stream) {
  if (n_in < 1 || n_in > 4 || (D & 7) || rows <= 0) return -1;
  LincombBwdArgs a;
  for (int i = 0; i < 4; ++i) {
    a.t[i] = i < n_in ? (const __nv_bfloat16*)t[i] : nullptr;
    a.dt[i] = i < n_in ? (__nv_bfloat16*)dt[i] : nullptr;
  }
  a.scal = scal; a.dscal = dscal;
  a.out = (const __nv_bfloat16*)out;
  a.d_out = (const __nv_bfloat16*)d_out;
  a.d_normed = (const __nv_bfloat16*)d_normed;
  a.n_in = n_in; a.rows = rows; a.D = D; a.eps = eps;
  const int grid = grid_for_rows(rows, 8);
  cudaStream_t st = (cudaStream_t)stream;
  switch (n_in) {
    case 1: launch_dependent(lincomb_rmsnorm_bwd_kernel<1>, dim3(grid), dim3(256), 0, st, a); break;
    case 2: launch_dependent(lincomb_rmsnorm_bwd_kernel<2>, dim3(grid), dim3(256), 0, st, a); break;
    case 3: launch_dependent(lincomb_rmsnorm_bwd_kernel<3>, dim3(grid), dim3(256), 0, st, a); break;
    default: launch_dependent(lincomb_rmsnorm_bwd_kernel<4>, dim3(grid), dim3(256), 0, st, a); break;
  }
  return (int)cudaGetLastError();
}

extern "C" TYR_EXPORT int tyr_rmsnorm_weighted(const void* x, const void* w, const void* gate,
                                               const void* resid, void* resid_out, void* y,
                                               int rows, int D, float eps, int one_plus_w,
                                               void* stream) {
  if ((D & 7) || rows <= 0) return -1;
  RmsWArgs a;
  a.x = (const __nv_bfloat16*)x; a.w = (const __nv_bfloat16*)w;
  a.gate = (const __nv_bfloat16*)gate; a.resid = (const __nv_bfloat16*)resid;
  a.resid_out = (__nv_bfloat16*)resid_out; a.y = (__nv_bfloat16*)y;
  a.rows = rows; a.D = D; a.eps = eps; a.one_plus_w = one_plus_w;
  if (rows <= 2048 && D >= 1024 && D <= 256 * kRowVecs * 8)
    return (int)launch_dependent(rmsnorm_weighted_row_kernel, dim3(rows), dim3(256), 0, (cudaStream_t)stream, a);
  return (int)launch_dependent(rmsnorm_weighted_kernel, dim3(grid_for_rows(rows, 8)), dim3(256), 0, (cudaStream_t)stream, a);
}

// x_dtype / y_dtype: 0 = bf16, 1 = fp32; `gain` fp32 of one or D numbers; `resid` fp32 in place or null; `y` may be null.
extern "C" TYR_EXPORT int tyr_post_norm_residual(const void* x, long long x_stride, const float* gain, int n_gain, float* resid, void* y,
                                                 long long rows, int D, float eps, int x_dtype, int y_dtype, void* stream) {
  if (rows <= 0 || D <= 0 || (n_gain != 1 && n_gain != D) || (resid == nullptr && y == nullptr)) return -1;
  PostNormArgs a{x, gain, resid, y, x_stride, D, n_gain, eps};
  const uintptr_t al = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(resid) | reinterpret_cast<uintptr_t>(y) |
                       (n_gain == 1 ? 0 : reinterpret_cast<uintptr_t>(gain));
  const bool vec = (D & 7) == 0 && (x_stride & 7) == 0 && (al & 15) == 0 && D <= 256 * 8 * kPnVecs;
  int threads = 256;
  while (threads > 32 && threads * 4 >= D) threads >>= 1;       // narrow rows: no idle warps
  const dim3 grid(static_cast<unsigned>(rows)), block(threads);
  cudaStream_t st = (cudaStream_t)stream;
#define TYR_PN(TX, TY) (vec ? launch_dependent(post_norm_residual_kernel<TX, TY, true>, grid, block, 0, st, a) \
                            : launch_dependent(post_norm_residual_kernel<TX, TY, false>, grid, block, 0, st, a))
  if (x_dtype == 0) return (int)(y_dtype == 0 ? TYR_PN(__nv_bfloat16, __nv_bfloat16) : TYR_PN(__nv_bfloat16, float));
  return (int)(y_dtype == 0 ? TYR_PN(float, __nv_bfloat16) : TYR_PN(float, float));
#undef TYR_PN
}

extern "C" TYR_EXPORT int tyr_add_norm(const void* x, long long x_stride, const float* gain, float* resid, long long r_stride, void* y, long long rows,
                                       int D, float eps, int x_dtype, int y_dtype, void* stream) {
  if (rows <= 0 || D <= 0 || gain == nullptr || resid == nullptr || y == nullptr) return -1;
  AddNormArgs a{x, gain, resid, y, x_stride, r_stride, D, eps};
  const uintptr_t al = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(resid) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(gain);
  const bool vec = (D & 7) == 0 && (x_stride & 7) == 0 && (r_stride & 3) == 0 && (al & 15) == 0 && D <= 256 * 8 * kPnVecs;
  int threads = 256;
  while (threads > 32 && threads * 4 >= D) threads >>= 1;       // narrow rows: no idle warps
  const dim3 grid(static_cast<unsigned>(rows)), block(threads);
  cudaStream_t st = (cudaStream_t)stream;
#define TYR_AN(TX, TY) (vec ? launch_dependent(add_norm_kernel<TX, TY, true>, grid, block, 0, st, a) \
                            : launch_dependent(add_norm_kernel<TX, TY, false>, grid, block, 0, st, a))
  if (x_dtype == 0) return (int)(y_dtype == 0 ? TYR_AN(__nv_bfloat16, __nv_bfloat16) : TYR_AN(__nv_bfloat16, float));
  return (int)(y_dtype == 0 ? TYR_AN(float, __nv_bfloat16) : TYR_AN(float, float));
#undef TYR_AN
}

// bias, post, gain fp32 [D], each nullable; resid fp32 [rows, D] contiguous, in place; y rows of y_stride elements.
extern "C" TYR_EXPORT int tyr_sandwich_norm(const void* x, long long x_stride, const float* bias, const float* post, const float* gain, float* resid,
                                            void* y, long long y_stride, long long rows, int D, int replace, float eps, int x_dtype, int y_dtype,
                                            void* stream) {
  if (rows <= 0 || D <= 0 || x == nullptr || resid == nullptr || y == nullptr) return -1;
  SandwichNormArgs a{x, bias, post, gain, resid, y, x_stride, y_stride, D, replace, eps};
  const uintptr_t al = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(post) |
                       reinterpret_cast<uintptr_t>(gain) | reinterpret_cast<uintptr_t>(resid) | reinterpret_cast<uintptr_t>(y);
  const bool vec = (D & 7) == 0 && (x_stride & 7) == 0 && (y_stride & 7) == 0 && (al & 15) == 0 && D <= 256 * 8 * kPnVecs;
  int threads = 256;
  while (threads > 32 && threads * 4 >= D) threads >>= 1;       // narrow rows: no idle warps
  const dim3 grid(static_cast<unsigned>(rows)), block(threads);
  cudaStream_t st = (cudaStream_t)stream;
  const int nv = !vec ? 0 : D <= threads * 8 ? 1 : D <= threads * 16 ? 2 : 4;
#define TYR_SN(TX, TY)                                                                          \
  (nv == 0 ? launch_dependent(sandwich_norm_kernel<TX, TY, 0>, grid, block, 0, st, a)           \
           : nv == 1 ? launch_dependent(sandwich_norm_kernel<TX, TY, 1>, grid, block, 0, st, a) \
                     : nv == 2 ? launch_dependent(sandwich_norm_kernel<TX, TY, 2>, grid, block, 0, st, a) : launch_dependent(sandwich_norm_kernel<TX, TY, 4>, grid, block, 0, st, a))
  if (x_dtype == 0) return (int)(y_dtype == 0 ? TYR_SN(__nv_bfloat16, __nv_bfloat16) : TYR_SN(__nv_bfloat16, float));
  return (int)(y_dtype == 0 ? TYR_SN(float, __nv_bfloat16) : TYR_SN(float, float));
#undef TYR_SN
}
