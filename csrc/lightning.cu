// Linear attention with one decay per head (lightning attention):  S <- decay S + k v^T,  o = S^T q,  q, k and v after SiLU, state and
// read-out in fp32.
//
//   * recurrent: any sizes, fp32 or bf16 activations, token by token with the state in shared memory (prompts and single tokens).
//
// The decay comes as a double: fp32 carries it as a sum of two numbers, because a rounding of it would be applied anew at every token
// of a long memory.  Compiled without fast math.
#include "common.cuh"

namespace tyr {

__device__ __forceinline__ float lt_load(const float* p) { return *p; }
__device__ __forceinline__ float lt_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float lt_silu(float v) { return v / (1.f + expf(-v)); }
// SiLU in the activations' own type, as a projection with its activation leaves it
__device__ __forceinline__ float lt_act(float v, const float*) { return lt_silu(v); }
__device__ __forceinline__ float lt_act(float v, const __nv_bfloat16*) { return __bfloat162float(__float2bfloat16(lt_silu(v))); }

struct LightningArgs {
  const void *q, *k, *v;       // [B, S, H, .] by (batch, token, head) element strides, before SiLU
  const double* decay;         // [H]
  float* state;                // [B, H, dk, dv], in place
  float* out;                  // [B, S, H, dv]
  const int* lens;             // [B] tokens of each row (nullable: S)
  long long q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh;
  int S, H, dk, dv;
};

// One CTA per (row, head, 32 columns of the state); a warp owns every eighth state row, a lane one column.
template <typename T>
__global__ void __launch_bounds__(256) lightning_recurrent_kernel(LightningArgs a) {
  extern __shared__ __align__(16) float lt_smem[];
  float* const s = lt_smem;                       // [dk, 32]
  float* const sk = s + a.dk * 32;                // [dk]
  float* const sq = sk + a.dk;                    // [dk]
  float* const part = sq + a.dk;                  // [8, 32]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.x / a.H, h = blockIdx.x % a.H, col = blockIdx.y * 32 + lane;
  const bool live = col < a.dv;
  pdl_entry();
  const double decay = a.decay[h];
  const float hi = static_cast<float>(decay), lo = static_cast<float>(decay - hi);
  const int n = a.lens ? min(a.lens[b], a.S) : a.S;
  float* const st = a.state + static_cast<long long>(blockIdx.x) * a.dk * a.dv + col;
  for (int r = warp; r < a.dk; r += 8) s[r * 32 + lane] = live ? st[static_cast<long long>(r) * a.dv] : 0.f;
  const T* qp = static_cast<const T*>(a.q) + b * a.q_sb + h * a.q_sh;
  const T* kp = static_cast<const T*>(a.k) + b * a.k_sb + h * a.k_sh;
  const T* vp = static_cast<const T*>(a.v) + b * a.v_sb + h * a.v_sh + col;
  float* op = a.out + (static_cast<long long>(b) * a.S * a.H + h) * a.dv + col;
  for (int t = 0; t < n; ++t) {
    for (int d = tid; d < a.dk; d += 256) {
      sq[d] = lt_act(lt_load(qp + t * a.q_ss + d), qp);
      sk[d] = lt_act(lt_load(kp + t * a.k_ss + d), kp);
    }
    const float v = live ? lt_act(lt_load(vp + t * a.v_ss), vp) : 0.f;
    __syncthreads();
    float o = 0.f;
    for (int r = warp; r < a.dk; r += 8) {
      const float x = s[r * 32 + lane];
      const float y = fmaf(x, hi, fmaf(x, lo, sk[r] * v));
      s[r * 32 + lane] = y;
      o += y * sq[r];
    }
    part[warp * 32 + lane] = o;
    __syncthreads();
    if (warp == 0 && live) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += part[w * 32 + lane];
      op[static_cast<long long>(t) * a.H * a.dv] = sum;
    }
  }
  if (warp == 0 && live)
    for (int t = n; t < a.S; ++t) op[static_cast<long long>(t) * a.H * a.dv] = 0.f;
  for (int r = warp; r < a.dk; r += 8)
    if (live) st[static_cast<long long>(r) * a.dv] = s[r * 32 + lane];
}

}  // namespace tyr

using namespace tyr;

// strides: (batch, token, head) element strides of q, k, v.  dtype: 0 = bf16, 1 = fp32 activations.
extern "C" TYR_EXPORT int tyr_lightning_recurrent(const void* q, const void* k, const void* v, const double* decay, float* state, float* out,
                                                  const int* lens, const long long* strides, int B, int S, int H, int dk, int dv, int dtype,
                                                  void* stream) {
  if (B <= 0 || S <= 0 || H <= 0 || dk <= 0 || dv <= 0) return -1;
  LightningArgs a{q, k, v, decay, state, out, lens, strides[0], strides[1], strides[2], strides[3], strides[4], strides[5], strides[6], strides[7],
                  strides[8], S, H, dk, dv};
  const size_t smem = (static_cast<size_t>(dk) * 34 + 256) * sizeof(float);
  constexpr size_t kMax = 227 * 1024;
  if (smem > kMax) return -2;
  auto kernel = dtype == 1 ? lightning_recurrent_kernel<float> : lightning_recurrent_kernel<__nv_bfloat16>;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(kMax));
    if (e != cudaSuccess) return 1000 + (int)e;
  }
  const dim3 grid(static_cast<unsigned>(B * H), (dv + 31) / 32);
  return (int)launch_dependent(kernel, grid, dim3(256), smem, (cudaStream_t)stream, a);
}
