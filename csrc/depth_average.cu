// The end of a layer whose successors average over depth, in one launch with the next norm:
//
//   X_n = x + norm(y) post,   x = sum_{j <= n} w_j X_j,   h = norm(x) gain
//
// y is the last sublayer's output (its norm optional), x the fp32 residual stream (updated in place), X_0 .. X_{n-1} the stored results of
// earlier layers (fp32, evenly spaced), X_n is stored beside them.  One CTA per row; the sum over the stored results does not wait for
// the norm of y.
#include "common.cuh"

namespace tyr {

struct DepthArgs {
  const void* y;               // [rows, D], row stride ld (nullable: X_n = x)
  long long ld;
  const float* post;           // [D]; null: y is added as it is
  float* x;                    // [rows, D]
  float* history;              // [n + 1, rows, D], `between` elements apart
  long long between;
  const float* weights;        // [n + 1]
  const float* gain;           // [D]
  void* h;                     // [rows, D]
  long long rows;
  int D, n, store;             // store: X_n goes to the history
  float eps;
};

__device__ __forceinline__ float4 dp_load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float4 dp_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void dp_store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ void dp_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ float dp_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float dp_load(const float* p) { return *p; }
__device__ __forceinline__ void dp_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void dp_store(float* p, float v) { *p = v; }

// The sum over the CTA, the same for all threads; `part` holds 32 floats and is not reused before the next barrier.
__device__ __forceinline__ float dp_block_sum(float v, float* part) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  return warp_sum(static_cast<int>(threadIdx.x & 31) < static_cast<int>(blockDim.x >> 5) ? part[threadIdx.x & 31] : 0.f);
}
__device__ __forceinline__ void dp_fma(float4& a, float w, const float4& v) {
  a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
}
__device__ __forceinline__ float dp_square(const float4& v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// NV vectors of four channels per thread, `blockDim.x` vectors apart.  FEW rows: no second CTA on an SM hides the loads, so more of them
// are on their way at a time.
template <typename TY, typename TH, int NV, bool FEW>
__global__ void __launch_bounds__(512, FEW ? 1 : NV == 1 ? 3 : NV == 2 ? 2 : 1) depth_average_kernel(DepthArgs a) {
  __shared__ float part[2][32];
  const int vecs = a.D / 4;
  float4 post[NV], gain[NV];
  pdl_trigger();
#pragma unroll
  for (int i = 0; i < NV; ++i) {                   // parameters: no kernel writes them
    const int c = threadIdx.x + i * blockDim.x;
    post[i] = gain[i] = make_float4(1.f, 1.f, 1.f, 1.f);
    if (c < vecs) {
      gain[i] = __ldg(reinterpret_cast<const float4*>(a.gain) + c);
      if (a.post) post[i] = __ldg(reinterpret_cast<const float4*>(a.post) + c);
    }
  }
  const float w_last = __ldg(a.weights + a.n);
  pdl_wait();
  for (long long row = blockIdx.x; row < a.rows; row += gridDim.x) {
    const long long base = row * a.D;
    float4 y[NV], x[NV], acc[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      y[i] = x[i] = acc[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < vecs) {
        if (a.y) y[i] = dp_load4(static_cast<const TY*>(a.y) + row * a.ld + 4 * c);
        x[i] = dp_load4(a.x + base + 4 * c);
      }
      ss += dp_square(y[i]);
    }
    constexpr int kUnroll = FEW ? 8 : 4;
#pragma unroll kUnroll
    for (int j = 0; j < a.n; ++j) {
      const float w = __ldg(a.weights + j);
      const float* src = a.history + j * a.between + base;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int c = threadIdx.x + i * blockDim.x;
        if (c < vecs) dp_fma(acc[i], w, dp_load4(src + 4 * c));
      }
    }
    const float mean = dp_block_sum(ss, part[0]) / a.D, r = a.post ? 1.f / sqrtf(mean + a.eps) : 1.f;     // always summed: its barrier parts the rows
    float* keep = a.history + a.n * a.between + base;
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      x[i].x = fmaf(y[i].x * r, post[i].x, x[i].x); x[i].y = fmaf(y[i].y * r, post[i].y, x[i].y);
      x[i].z = fmaf(y[i].z * r, post[i].z, x[i].z); x[i].w = fmaf(y[i].w * r, post[i].w, x[i].w);
      dp_fma(acc[i], w_last, x[i]);
      if (c < vecs) {
        if (a.store) dp_store4(keep + 4 * c, x[i]);
        dp_store4(a.x + base + 4 * c, acc[i]);
        ss += dp_square(acc[i]);
      }
    }
    const float q = 1.f / sqrtf(dp_block_sum(ss, part[1]) / a.D + a.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < vecs)
        dp_store4(static_cast<TH*>(a.h) + base + 4 * c,
                  make_float4(acc[i].x * q * gain[i].x, acc[i].y * q * gain[i].y, acc[i].z * q * gain[i].z, acc[i].w * q * gain[i].w));
    }
  }
}

// Any width: the row's sums are formed in the stream itself.
template <typename TY, typename TH>
__global__ void __launch_bounds__(256) depth_average_any_kernel(DepthArgs a) {
  __shared__ float part[2][32];
  pdl_entry();
  for (long long row = blockIdx.x; row < a.rows; row += gridDim.x) {
    const long long base = row * a.D;
    const TY* y = static_cast<const TY*>(a.y) + row * a.ld;
    float ss = 0.f;
    if (a.y)
      for (int c = threadIdx.x; c < a.D; c += blockDim.x) ss += dp_load(y + c) * dp_load(y + c);
    const float mean = dp_block_sum(ss, part[0]) / a.D, r = a.post ? 1.f / sqrtf(mean + a.eps) : 1.f;
    ss = 0.f;
    for (int c = threadIdx.x; c < a.D; c += blockDim.x) {
      float acc = 0.f, x = a.x[base + c];
      for (int j = 0; j < a.n; ++j) acc = fmaf(a.weights[j], a.history[j * a.between + base + c], acc);
      if (a.y) x = fmaf(dp_load(y + c) * r, a.post ? a.post[c] : 1.f, x);
      if (a.store) a.history[a.n * a.between + base + c] = x;
      acc = fmaf(a.weights[a.n], x, acc);
      a.x[base + c] = acc;
      ss += acc * acc;
    }
    const float q = 1.f / sqrtf(dp_block_sum(ss, part[1]) / a.D + a.eps);
    for (int c = threadIdx.x; c < a.D; c += blockDim.x) dp_store(static_cast<TH*>(a.h) + base + c, a.x[base + c] * q * a.gain[c]);
  }
}

}  // namespace tyr

using namespace tyr;

template <typename TY, typename TH>
static int depth_launch(const DepthArgs& a, bool vec, cudaStream_t st) {
  const unsigned rows = static_cast<unsigned>(a.rows < 148LL * 64 ? a.rows : 148LL * 64);
  const int vecs = a.D / 4;
  if (!vec || vecs > 4096) return (int)launch_dependent(depth_average_any_kernel<TY, TH>, dim3(rows), dim3(256), 0, st, a);
  const int nv = vecs <= 512 ? 1 : (vecs <= 1024 ? 2 : (vecs <= 2048 ? 4 : 8));
  const dim3 block(static_cast<unsigned>(((vecs + nv - 1) / nv + 31) / 32 * 32));
  const dim3 grid(rows);
  if (a.rows <= 148 && nv <= 2)
    return (int)(nv == 1 ? launch_dependent(depth_average_kernel<TY, TH, 1, true>, grid, block, 0, st, a)
                         : launch_dependent(depth_average_kernel<TY, TH, 2, true>, grid, block, 0, st, a));
  return (int)(nv == 1 ? launch_dependent(depth_average_kernel<TY, TH, 1, false>, grid, block, 0, st, a)
               : nv == 2 ? launch_dependent(depth_average_kernel<TY, TH, 2, false>, grid, block, 0, st, a)
               : nv == 4 ? launch_dependent(depth_average_kernel<TY, TH, 4, false>, grid, block, 0, st, a)
                         : launch_dependent(depth_average_kernel<TY, TH, 8, false>, grid, block, 0, st, a));
}

// dtypes: 0 = bf16, 1 = fp32 of y and of h.
extern "C" TYR_EXPORT int tyr_depth_average(const void* y, long long ld, const float* post, float* x, float* history, long long between,
                                            const float* weights, const float* gain, void* h, long long rows, int D, int n, int store, float eps,
                                            int y_dtype, int h_dtype, void* stream) {
  if (rows <= 0 || D <= 0 || n < 0 || x == nullptr || history == nullptr || weights == nullptr || gain == nullptr || h == nullptr) return -1;
  DepthArgs a{y, ld, post, x, history, between, weights, gain, h, rows, D, n, store, eps};
  uintptr_t al = 0;
  for (const void* p : {y, (const void*)post, (const void*)x, (const void*)history, (const void*)gain, (const void*)h}) al |= reinterpret_cast<uintptr_t>(p);
  const bool vec = (D & 3) == 0 && (ld & 3) == 0 && (between & 3) == 0 && (al & 15) == 0;
  cudaStream_t st = (cudaStream_t)stream;
  if (y_dtype == 0) return h_dtype == 0 ? depth_launch<__nv_bfloat16, __nv_bfloat16>(a, vec, st) : depth_launch<__nv_bfloat16, float>(a, vec, st);
  return h_dtype == 0 ? depth_launch<float, __nv_bfloat16>(a, vec, st) : depth_launch<float, float>(a, vec, st);
}
