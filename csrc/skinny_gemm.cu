// y[M, N] = x[M, K] @ W[N, K]^T (+ bias) for decode-sized M (1..32 rows): a weight-streaming kernel.  The product is bound
// by reading W once from HBM, so a CTA owns 16 weight rows and its 8 warps split K; every lane streams 16 bytes of two
// weight rows per step straight into mma.sync m16n8k16 A fragments (W rows are the M dimension of the tile, the tokens the
// N dimension; the reduction over K is order-free, so a lane's 8 consecutive channels serve as the fragment's k-slots and
// the activations are loaded with the same addressing).  Tokens beyond M load nothing.  Warp partials meet in shared memory.
//
// The reference sends these products to the library GEMM (cc/src/tyr.cpp:1003-1036).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "common.cuh"
#include "gates.cuh"

namespace tyr {

constexpr int kSkWarps = 8;

struct SkinnyArgs {
  const __nv_bfloat16* x;      // [M, K], row stride ldx
  const __nv_bfloat16* w;      // [N, K], row stride ldw
  const __nv_bfloat16* w2;     // gated form only: the second matrix [N, K]; y = silu(x w^T) * (x w2^T)
  const __nv_bfloat16* bias;   // [N] or null
  __nv_bfloat16* y;            // [M, N], row stride ldy
  float* ws;                   // [M, N] fp32, zero on entry and exit; used when the reduction is split over gridDim.y CTAs
  long long ldx, ldw, ldy;
  int M, N, K;
  long long hx, hw, hy;        // per-head form: elements from head to head
  int act;                     // 6: xIELU with factors act_a, act_b, 9: tanh-GELU times aux, as in csrc/gemm_tcgen05.cu; 0: none
  float act_a, act_b;
  const __nv_bfloat16* aux;    // [M, N], row stride ldaux
  long long ldaux;
};

__device__ __forceinline__ float sk_act(float z, const SkinnyArgs& a, int tok, int row) {
  if (a.act == 9) return gelu_tanh(z) * __bfloat162float(a.aux[tok * a.ldaux + row]);
  return a.act == 6 ? fmaf(0.5f, z, z > 0.f ? a.act_a * z * z : a.act_b * (__expf(z) - 1.f - z)) : z;
}

__device__ __forceinline__ void mma_16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

constexpr long long kSkPrefetchBytes = 32LL << 20;   // L2 prefetch issued by one launch before its input is ready

template <int TILES, bool GATED>                   // token tiles of 8: M <= 8 * TILES; GATED: two matrices, SwiGLU epilogue
__global__ void __launch_bounds__(kSkWarps * 32) skinny_gemm_kernel(SkinnyArgs a) {
  __shared__ float part[GATED ? 2 : 1][kSkWarps][TILES][16][8];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int row0 = blockIdx.x * 16;
  // The weights are constants: while the kernel that produces `x` still runs (this one may already be resident, see
  // launch_dependent), pull the head of every weight row of this CTA into the L2.  The whole grid asks for at most
  // kSkPrefetchBytes, so what it brings in is still there when the loop below reads it.
  pdl_trigger();
  if (tid < (GATED ? 32 : 16) && (a.ldw & 7) == 0) {
    const int r = row0 + (tid & 15);
    const int chunks = a.K >> 5;
    const int c0 = static_cast<int>(static_cast<long long>(chunks) * blockIdx.y / gridDim.y);
    const int c1 = static_cast<int>(static_cast<long long>(chunks) * (blockIdx.y + 1) / gridDim.y);
    long long per_row = kSkPrefetchBytes / (static_cast<long long>(gridDim.x) * gridDim.y * (GATED ? 32 : 16));
    per_row = min(per_row & ~127LL, static_cast<long long>(c1 - c0) * 64);
    if (r < a.N && per_row >= 128)
      bulk_prefetch_l2((tid < 16 ? a.w : a.w2) + static_cast<long long>(r) * a.ldw + 32LL * c0, static_cast<uint32_t>(per_row));
  }
  pdl_wait();
  int r_lo = row0 + g, r_hi = row0 + g + 8;
  r_lo = r_lo < a.N ? r_lo : a.N - 1;            // clamped rows are not written
  r_hi = r_hi < a.N ? r_hi : a.N - 1;
  const __nv_bfloat16* w_lo = a.w + r_lo * a.ldw + 8 * t;
  const __nv_bfloat16* w_hi = a.w + r_hi * a.ldw + 8 * t;
  const __nv_bfloat16* v_lo = GATED ? a.w2 + r_lo * a.ldw + 8 * t : nullptr;
  const __nv_bfloat16* v_hi = GATED ? a.w2 + r_hi * a.ldw + 8 * t : nullptr;
  const __nv_bfloat16* xr[TILES];
  bool live[TILES];
#pragma unroll
  for (int i = 0; i < TILES; ++i) {
    const int tok = 8 * i + g;
    live[i] = tok < a.M;
    xr[i] = a.x + (live[i] ? tok : 0) * a.ldx + 8 * t;
  }
  float acc[TILES][4], acc2[TILES][4];
#pragma unroll
  for (int i = 0; i < TILES; ++i) {
    acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    acc2[i][0] = acc2[i][1] = acc2[i][2] = acc2[i][3] = 0.f;
  }

  const int chunks = a.K >> 5;                   // 32 channels per warp step
  const int c_lo = static_cast<int>(static_cast<long long>(chunks) * blockIdx.y / gridDim.y);
  const int c_hi = static_cast<int>(static_cast<long long>(chunks) * (blockIdx.y + 1) / gridDim.y);
#pragma unroll 4
  for (int c = c_lo + warp; c < c_hi; c += kSkWarps) {
    const uint4 lo = __ldcs(reinterpret_cast<const uint4*>(w_lo + 32 * c));    // streamed once: do not keep in cache
    const uint4 hi = __ldcs(reinterpret_cast<const uint4*>(w_hi + 32 * c));
    uint4 lo2 = make_uint4(0u, 0u, 0u, 0u), hi2 = lo2;
    if (GATED) {
      lo2 = __ldcs(reinterpret_cast<const uint4*>(v_lo + 32 * c));
      hi2 = __ldcs(reinterpret_cast<const uint4*>(v_hi + 32 * c));
    }
#pragma unroll
    for (int i = 0; i < TILES; ++i) {
      const uint4 xv = live[i] ? __ldg(reinterpret_cast<const uint4*>(xr[i] + 32 * c)) : make_uint4(0u, 0u, 0u, 0u);
      mma_16816(acc[i], lo.x, hi.x, lo.y, hi.y, xv.x, xv.y);
      mma_16816(acc[i], lo.z, hi.z, lo.w, hi.w, xv.z, xv.w);
      if (GATED) {
        mma_16816(acc2[i], lo2.x, hi2.x, lo2.y, hi2.y, xv.x, xv.y);
        mma_16816(acc2[i], lo2.z, hi2.z, lo2.w, hi2.w, xv.z, xv.w);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < TILES; ++i) {
    part[0][warp][i][g][2 * t] = acc[i][0];
    part[0][warp][i][g][2 * t + 1] = acc[i][1];
    part[0][warp][i][g + 8][2 * t] = acc[i][2];
    part[0][warp][i][g + 8][2 * t + 1] = acc[i][3];
    if (GATED) {
      part[1][warp][i][g][2 * t] = acc2[i][0];
      part[1][warp][i][g][2 * t + 1] = acc2[i][1];
      part[1][warp][i][g + 8][2 * t] = acc2[i][2];
      part[1][warp][i][g + 8][2 * t + 1] = acc2[i][3];
    }
  }
  __syncthreads();
  for (int idx = tid; idx < TILES * 8 * 16; idx += kSkWarps * 32) {
    const int tok = idx >> 4, r = idx & 15;        // consecutive threads write consecutive output columns
    const int row = row0 + r;
    if (tok < a.M && row < a.N) {
      float s = 0.f;
#pragma unroll
      for (int wp = 0; wp < kSkWarps; ++wp) s += part[0][wp][tok >> 3][r][tok & 7];
      if (GATED) {
        float u = 0.f;
#pragma unroll
        for (int wp = 0; wp < kSkWarps; ++wp) u += part[1][wp][tok >> 3][r][tok & 7];
        a.y[tok * a.ldy + row] = __float2bfloat16(s / (1.f + __expf(-s)) * u);
      } else if (gridDim.y == 1) {
        if (a.bias) s += __bfloat162float(a.bias[row]);
        a.y[tok * a.ldy + row] = __float2bfloat16(sk_act(s, a, tok, row));
      } else {
        atomicAdd(a.ws + static_cast<long long>(tok) * a.N + row, s);
      }
    }
  }
}

// A small matrix of its own for each head: gridDim.y heads, a warp owns 16 rows of the head's matrix and its whole contraction.
template <int TILES>
__global__ void __launch_bounds__(kSkWarps * 32) skinny_heads_kernel(SkinnyArgs a) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int row0 = (blockIdx.x * kSkWarps + warp) * 16;
  pdl_trigger();
  if (row0 >= a.N) return;
  const __nv_bfloat16* w = a.w + blockIdx.y * a.hw;
  const __nv_bfloat16* w_lo = w + min(row0 + g, a.N - 1) * a.ldw + 8 * t;        // clamped rows are not written
  const __nv_bfloat16* w_hi = w + min(row0 + g + 8, a.N - 1) * a.ldw + 8 * t;
  constexpr int U = 4;                             // the weights need nothing from the kernel in front of this one
  const int chunks = a.K >> 5;
  uint4 lo[U], hi[U];
#pragma unroll
  for (int u = 0; u < U; ++u)
    if (u < chunks) {
      lo[u] = __ldg(reinterpret_cast<const uint4*>(w_lo + 32 * u));
      hi[u] = __ldg(reinterpret_cast<const uint4*>(w_hi + 32 * u));
    }
  pdl_wait();
  const __nv_bfloat16* xr[TILES];
  bool live[TILES];
  float acc[TILES][4];
#pragma unroll
  for (int i = 0; i < TILES; ++i) {
    const int tok = 8 * i + g;
    live[i] = tok < a.M;
    xr[i] = a.x + blockIdx.y * a.hx + (live[i] ? tok : 0) * a.ldx + 8 * t;
    acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  }
  for (int c0 = 0; c0 < chunks; c0 += U) {
    uint4 xv[U][TILES];
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int i = 0; i < TILES; ++i) xv[u][i] = c0 + u < chunks && live[i] ? *reinterpret_cast<const uint4*>(xr[i] + 32 * (c0 + u)) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c0 + u >= chunks) break;
#pragma unroll
      for (int i = 0; i < TILES; ++i) {
        mma_16816(acc[i], lo[u].x, hi[u].x, lo[u].y, hi[u].y, xv[u][i].x, xv[u][i].y);
        mma_16816(acc[i], lo[u].z, hi[u].z, lo[u].w, hi[u].w, xv[u][i].z, xv[u][i].w);
      }
      if (c0 + u + U < chunks) {
        lo[u] = __ldg(reinterpret_cast<const uint4*>(w_lo + 32 * (c0 + u + U)));
        hi[u] = __ldg(reinterpret_cast<const uint4*>(w_hi + 32 * (c0 + u + U)));
      }
    }
  }
#pragma unroll
  for (int i = 0; i < TILES; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int tok = 8 * i + 2 * t + (e & 1), row = row0 + g + (e >> 1) * 8;
      if (tok < a.M && row < a.N) a.y[blockIdx.y * a.hy + tok * a.ldy + row] = __float2bfloat16(acc[i][e]);
    }
}

// Second pass of a split reduction: round the fp32 sums (+ bias) and leave the workspace zeroed for the next call.
__global__ void __launch_bounds__(256) skinny_finish_kernel(SkinnyArgs a) {
  pdl_entry();
  const long long n = static_cast<long long>(a.M) * a.N;
  for (long long i = blockIdx.x * 256LL + threadIdx.x; i < n; i += static_cast<long long>(gridDim.x) * 256) {
    const int tok = static_cast<int>(i / a.N), row = static_cast<int>(i - static_cast<long long>(tok) * a.N);
    float s = a.ws[i];
    a.ws[i] = 0.f;
    if (a.bias) s += __bfloat162float(a.bias[row]);
    a.y[tok * a.ldy + row] = __float2bfloat16(sk_act(s, a, tok, row));
  }
}

}  // namespace tyr

// The kernels above read the activations through the L1: the eight CTAs of an SM walk the same rows of x.  A kernel with a
// large shared-memory footprint earlier in the stream leaves the SMs split in favour of shared memory, and a kernel that
// states no preference inherits that split.  Ask for just the shared memory that the resident CTAs need (registers and
// threads bound their number); the rest is L1.
template <int TILES, bool GATED>
static void skinny_set_carveout() {
  const int per_cta = (GATED ? 2 : 1) * tyr::kSkWarps * TILES * 16 * 8 * 4 + 1024;
  int ctas = 0;
  if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&ctas, tyr::skinny_gemm_kernel<TILES, GATED>, tyr::kSkWarps * 32, 0) != cudaSuccess ||
      ctas < 1)
    return;
  int pct = (ctas * per_cta * 100 + 227 * 1024 - 1) / (227 * 1024);
  if (pct > 100) pct = 100;
  cudaFuncSetAttribute(tyr::skinny_gemm_kernel<TILES, GATED>, cudaFuncAttributePreferredSharedMemoryCarveout, pct);
}
static void skinny_prefer_l1() {
  static bool done[64] = {};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
  if (done[dev]) return;
  done[dev] = true;
  const char* v = getenv("TYR_SKINNY_CARVEOUT");
  if (v != nullptr && v[0] == '0') return;
  skinny_set_carveout<1, false>();
  skinny_set_carveout<2, false>();
  skinny_set_carveout<4, false>();
  skinny_set_carveout<1, true>();
  skinny_set_carveout<2, true>();
  skinny_set_carveout<4, true>();
}

// Number of CTAs the reduction should be split over for this shape (1 = no workspace needed): enough CTAs to cover the
// SMs about three times, at least 1024 channels per split.
extern "C" TYR_EXPORT int tyr_skinny_gemm_splits(int N, int K) {
  const int row_ctas = (N + 15) / 16;
  int splits = (3 * 148 + row_ctas - 1) / row_ctas;
  const int max_by_k = K / 1024 > 0 ? K / 1024 : 1;
  if (splits > max_by_k) splits = max_by_k;
  if (splits > 8) splits = 8;
  return splits < 1 ? 1 : splits;
}

static int skinny_launch(const void* x, const void* w, const void* bias, void* y, void* ws, long long ldx, long long ldw, long long ldy, int M,
                         int N, int K, int act, float act_a, float act_b, void* stream, const void* aux = nullptr, long long ldaux = 0) {
  using namespace tyr;
  if ((act != 0 && act != 6 && act != 9) || (act == 9) != (aux != nullptr)) return -4;
  if (M < 1 || M > 32 || N < 1 || K < 32 || (K & 31)) return -1;
  if ((ldx | ldw) & 7) return -2;                                    // 16-byte loads
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15) return -3;
  SkinnyArgs a{(const __nv_bfloat16*)x, (const __nv_bfloat16*)w, nullptr, (const __nv_bfloat16*)bias, (__nv_bfloat16*)y, (float*)ws, ldx, ldw, ldy, M, N, K,
               0, 0, 0, act, act_a, act_b, (const __nv_bfloat16*)aux, ldaux};
  const int splits = ws != nullptr ? tyr_skinny_gemm_splits(N, K) : 1;
  const dim3 grid((N + 15) / 16, splits);
  skinny_prefer_l1();
  if (M <= 8) launch_dependent(skinny_gemm_kernel<1, false>, dim3(grid), dim3(kSkWarps * 32), 0, (cudaStream_t)stream, a);
  else if (M <= 16) launch_dependent(skinny_gemm_kernel<2, false>, dim3(grid), dim3(kSkWarps * 32), 0, (cudaStream_t)stream, a);
  else launch_dependent(skinny_gemm_kernel<4, false>, dim3(grid), dim3(kSkWarps * 32), 0, (cudaStream_t)stream, a);
  if (splits > 1) {
    long long blocks = (static_cast<long long>(M) * N + 255) / 256;
    if (blocks > 592) blocks = 592;
    launch_dependent(skinny_finish_kernel, dim3((int)blocks), dim3(256), 0, (cudaStream_t)stream, a);
  }
  return (int)cudaGetLastError();
}

extern "C" TYR_EXPORT int tyr_skinny_gemm_bf16(const void* x, const void* w, const void* bias, void* y, void* ws, long long ldx,
                                               long long ldw, long long ldy, int M, int N, int K, void* stream) {
  return skinny_launch(x, w, bias, y, ws, ldx, ldw, ldy, M, N, K, 0, 0.f, 0.f, stream);
}

// The same with an activation in the epilogue (6: xIELU, factors act_a above zero and act_b below).
extern "C" TYR_EXPORT int tyr_skinny_gemm_act_bf16(const void* x, const void* w, const void* bias, void* y, void* ws, long long ldx, long long ldw,
                                                   long long ldy, int M, int N, int K, int act, float act_a, float act_b, void* stream) {
  return skinny_launch(x, w, bias, y, ws, ldx, ldw, ldy, M, N, K, act, act_a, act_b, stream);
}

// y[M, N] = gelu(x W^T) * aux (tanh form); aux [M, N] with row stride ldaux.
extern "C" TYR_EXPORT int tyr_skinny_gelu_mul_bf16(const void* x, const void* w, const void* aux, void* y, void* ws, long long ldx, long long ldw,
                                                   long long ldaux, long long ldy, int M, int N, int K, void* stream) {
  return skinny_launch(x, w, nullptr, y, ws, ldx, ldw, ldy, M, N, K, 9, 0.f, 0.f, stream, aux, ldaux);
}

// A product of its own for each head: y[m, h, :N] = x[m, h, :K] @ W[h]^T for `heads` heads, rows (ldx, ldy) and heads (hx, hw, hy) apart
// by element strides.
extern "C" TYR_EXPORT int tyr_skinny_heads_bf16(const void* x, const void* w, void* y, long long ldx, long long hx, long long hw, long long ldw,
                                                long long ldy, long long hy, int heads, int M, int N, int K, void* stream) {
  using namespace tyr;
  if (M < 1 || M > 32 || N < 1 || K < 32 || (K & 31) || heads < 1 || heads > 65535) return -1;
  if ((ldx | ldw | hx | hw) & 7) return -2;
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w)) & 15) return -3;
  SkinnyArgs a{(const __nv_bfloat16*)x, (const __nv_bfloat16*)w, nullptr, nullptr, (__nv_bfloat16*)y, nullptr, ldx, ldw, ldy, M, N, K, hx, hw, hy, 0, 0.f, 0.f};
  const dim3 grid((N + 16 * kSkWarps - 1) / (16 * kSkWarps), heads), block(kSkWarps * 32);
  const cudaStream_t st = (cudaStream_t)stream;
  return (int)(M <= 8 ? launch_dependent(skinny_heads_kernel<1>, grid, block, 0, st, a)
                      : M <= 16 ? launch_dependent(skinny_heads_kernel<2>, grid, block, 0, st, a) : launch_dependent(skinny_heads_kernel<4>, grid, block, 0, st, a));
}

// y[M, N] = silu(x wg^T) * (x wu^T): the gate and up projections of a SwiGLU MLP for decode-sized M in one pass over both
// matrices (same row stride ldw), no intermediate tensors.
extern "C" TYR_EXPORT int tyr_skinny_swiglu_bf16(const void* x, const void* wg, const void* wu, void* y, long long ldx,
                                                 long long ldw, long long ldy, int M, int N, int K, void* stream) {
  using namespace tyr;
  if (M < 1 || M > 32 || N < 1 || K < 32 || (K & 31)) return -1;
  if ((ldx | ldw) & 7) return -2;
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(wg) | reinterpret_cast<uintptr_t>(wu)) & 15) return -3;
  SkinnyArgs a{(const __nv_bfloat16*)x, (const __nv_bfloat16*)wg, (const __nv_bfloat16*)wu, nullptr, (__nv_bfloat16*)y, nullptr, ldx, ldw, ldy, M, N, K};
  const dim3 grid((N + 15) / 16, 1);
  skinny_prefer_l1();
  if (M <= 8) launch_dependent(skinny_gemm_kernel<1, true>, dim3(grid), dim3(kSkWarps * 32), 0, (cudaStream_t)stream, a);
  else if (M <= 16) launch_dependent(skinny_gemm_kernel<2, true>, dim3(grid), dim3(kSkWarps * 32), 0, (cudaStream_t)stream, a);
  else launch_dependent(skinny_gemm_kernel<4, true>, dim3(grid), dim3(kSkWarps * 32), 0, (cudaStream_t)stream, a);
  return (int)cudaGetLastError();
}
