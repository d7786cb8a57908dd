// bf16 expert products for a few tokens: a weight-streaming mixture of experts without a sorted layout.
//
//   moe_stream_up:   hid[pair] = clamped SwiGLU of (w * gate_e x, w * up_e x), e = ids[pair], w the pair's weight (a weighted input: the
//                    products are linear, so the weight goes onto their sums); the shared expert's rows (weight 1) follow those of the pairs
//   moe_stream_down: y[pair] = down_e hid[pair], the same rows
//
// The products are bound by reading each active expert's weights once.  As in csrc/skinny_gemm.cu a CTA owns 16 weight rows, its 8 warps
// split the contraction and stream 16 bytes per lane and row into mma.sync A fragments, with 8 pairs of one expert on the narrow side.
// A CTA finds the pairs of its expert in the token-major list of ids itself: with fewer pairs than experts, CTA row p stands for the
// expert of pair p and leaves when an earlier pair has the same one; otherwise CTA rows are experts, whose weights are on their way
// into L2 before the kernel in front of this one has ended.  The first CTA row is the shared expert.
//
// Gate and up rows come in the grouped GEMM's layout: per 256 rows, 128 gate rows, then the matching 128 up rows.
#include "common.cuh"
#include "gates.cuh"

namespace tyr {

constexpr int MS_WARPS = 8;
constexpr int MS_LIST = 2048;            // most (token, slot) pairs

struct MoeStreamArgs {
  const __nv_bfloat16* x;      // up: [T, K]; down: [pairs + T, ldx] rows of hidden channels
  const __nv_bfloat16* w;      // [E, rows, K] by strides
  const __nv_bfloat16* ws;     // the shared expert's (null: none)
  const int* ids;              // [T * k]
  const float* weights;        // [T * k]
  __nv_bfloat16* y;            // [pairs + T, ldy]
  long long ldx, ldw, ldws, w_expert, ldy;
  int T, k, E, N, Ns, K, Ks;   // output rows and contraction of an expert, of the shared one
  int by_pair;                 // CTA rows are pairs (else experts)
  float limit, limit_s, slope;
};

__device__ __forceinline__ void ms_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// 16 weight rows (32 with UP) times up to 8 * TILES listed pairs.
template <bool UP, int TILES>
__device__ __forceinline__ void ms_product(const MoeStreamArgs& a, const __nv_bfloat16* w, long long ldw, int row0, int K, bool shared, const int* list,
                                           int count, float (*part)[MS_WARPS][4][16][9]) {
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int pairs = a.T * a.k;
  const __nv_bfloat16* w_lo = w + g * ldw + 8 * t;
  const __nv_bfloat16* w_hi = w_lo + 8 * ldw;
  const long long up = 128 * ldw;                  // from a gate row to its up row
  const __nv_bfloat16* xr[TILES];
  bool live[TILES];
  float acc[UP ? 2 : 1][TILES][4];
#pragma unroll
  for (int i = 0; i < TILES; ++i) {
    const int n = 8 * i + g;
    live[i] = n < count;
    const int entry = live[i] ? (shared ? list[0] + n : list[n]) : 0;          // shared: consecutive tokens from list[0] on
    const long long row = UP ? (shared ? entry : entry / a.k) : (shared ? pairs + entry : entry);
    xr[i] = a.x + row * a.ldx + 8 * t;
#pragma unroll
    for (int m = 0; m < (UP ? 2 : 1); ++m) acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f;
  }
#pragma unroll 4
  for (int c = warp; c < (K >> 5); c += MS_WARPS) {
    const uint4 lo = __ldg(reinterpret_cast<const uint4*>(w_lo + 32 * c)), hi = __ldg(reinterpret_cast<const uint4*>(w_hi + 32 * c));
    uint4 lo2, hi2;
    if constexpr (UP) {
      lo2 = __ldg(reinterpret_cast<const uint4*>(w_lo + up + 32 * c));
      hi2 = __ldg(reinterpret_cast<const uint4*>(w_hi + up + 32 * c));
    }
#pragma unroll
    for (int i = 0; i < TILES; ++i) {
      const uint4 xv = live[i] ? *reinterpret_cast<const uint4*>(xr[i] + 32 * c) : make_uint4(0u, 0u, 0u, 0u);
      ms_mma(acc[0][i], lo.x, hi.x, lo.y, hi.y, xv.x, xv.y);
      ms_mma(acc[0][i], lo.z, hi.z, lo.w, hi.w, xv.z, xv.w);
      if constexpr (UP) {
        ms_mma(acc[1][i], lo2.x, hi2.x, lo2.y, hi2.y, xv.x, xv.y);
        ms_mma(acc[1][i], lo2.z, hi2.z, lo2.w, hi2.w, xv.z, xv.w);
      }
    }
  }
  __syncthreads();                                 // the previous pass has read its partial sums
#pragma unroll
  for (int m = 0; m < (UP ? 2 : 1); ++m)
#pragma unroll
    for (int i = 0; i < TILES; ++i) {
      part[m][warp][i][g][2 * t] = acc[m][i][0];
      part[m][warp][i][g][2 * t + 1] = acc[m][i][1];
      part[m][warp][i][g + 8][2 * t] = acc[m][i][2];
      part[m][warp][i][g + 8][2 * t + 1] = acc[m][i][3];
    }
  __syncthreads();
  for (int idx = tid; idx < count * 16; idx += MS_WARPS * 32) {
    const int n = idx >> 4, r = idx & 15;
    float s = 0.f, u = 0.f;
#pragma unroll
    for (int wp = 0; wp < MS_WARPS; ++wp) {
      s += part[0][wp][n >> 3][r][n & 7];
      if constexpr (UP) u += part[1][wp][n >> 3][r][n & 7];
    }
    const int entry = shared ? list[0] + n : list[n];
    if constexpr (UP) {
      const float f = shared ? 1.f : a.weights[entry];
      s = clamped_swiglu(f * s, f * u, shared ? a.limit_s : a.limit, a.slope);
    }
    a.y[(shared ? pairs + entry : entry) * a.ldy + row0 + r] = __float2bfloat16(s);
  }
}

template <bool UP>
__global__ void __launch_bounds__(MS_WARPS * 32, UP ? 2 : 3) moe_stream_kernel(MoeStreamArgs a) {
  extern __shared__ __align__(16) uint8_t ms_smem[];
  auto part = reinterpret_cast<float(*)[MS_WARPS][4][16][9]>(ms_smem);
  int* list = reinterpret_cast<int*>(ms_smem + sizeof(float) * (UP ? 2 : 1) * MS_WARPS * 4 * 16 * 9);
  __shared__ int s_count;
  const int tid = threadIdx.x, row0 = blockIdx.x * 16, pairs = a.T * a.k;
  const bool shared = a.ws != nullptr && blockIdx.y == 0;
  const int N = shared ? a.Ns : a.N, K = shared ? a.Ks : a.K;
  const long long ldw = shared ? a.ldws : a.ldw;
  pdl_trigger();
  if (row0 >= N) return;
  const int wrow = UP ? (row0 >> 7) * 256 + (row0 & 127) : row0;
  auto prefetch = [&](const __nv_bfloat16* w) {    // constants: on their way into L2 while the kernel in front of this one runs
    if (tid < (UP ? 32 : 16)) bulk_prefetch_l2(w + (tid < 16 ? tid : 112 + tid) * ldw, static_cast<uint32_t>(min(K, 4096)) * 2u);
  };
  if (shared) {
    const __nv_bfloat16* w = a.ws + wrow * ldw;
    prefetch(w);
    pdl_wait();
    for (int t0 = 0; t0 < a.T; t0 += 32) {
      __syncthreads();
      if (tid == 0) list[0] = t0;
      __syncthreads();
      const int n = min(32, a.T - t0);
      if (n <= 8) ms_product<UP, 1>(a, w, ldw, row0, K, true, list, n, part);
      else ms_product<UP, 4>(a, w, ldw, row0, K, true, list, n, part);
    }
    return;
  }
  const int unit = blockIdx.y - (a.ws != nullptr ? 1 : 0);
  if (!a.by_pair) prefetch(a.w + unit * a.w_expert + wrow * ldw);
  pdl_wait();
  const int e = a.by_pair ? a.ids[unit] : unit;
  int earlier = e < 0 || e >= a.E;
  if (tid == 0) s_count = 0;
  if (a.by_pair)
    for (int p = tid; p < unit; p += MS_WARPS * 32) earlier |= a.ids[p] == e;
  if (__syncthreads_or(earlier)) return;           // an earlier CTA row has this expert
  for (int p = tid; p < pairs; p += MS_WARPS * 32)
    if (a.ids[p] == e) list[atomicAdd(&s_count, 1)] = p;          // in any order: the pairs do not meet
  __syncthreads();
  const int count = s_count;
  const __nv_bfloat16* w = a.w + e * a.w_expert + wrow * ldw;
  for (int n0 = 0; n0 < count; n0 += 32) {
    const int n = min(32, count - n0);
    if (n <= 8) ms_product<UP, 1>(a, w, ldw, row0, K, false, list + n0, n, part);
    else if (n <= 16) ms_product<UP, 2>(a, w, ldw, row0, K, false, list + n0, n, part);
    else ms_product<UP, 4>(a, w, ldw, row0, K, false, list + n0, n, part);
  }
}

}  // namespace tyr

using namespace tyr;

template <bool UP>
static int moe_stream_launch(MoeStreamArgs a, cudaStream_t st) {
  const int pairs = a.T * a.k;
  if (a.T <= 0 || a.k <= 0 || a.E <= 0 || pairs > MS_LIST || a.N <= 0 || (a.N & 15) || a.K < 32 || (a.K & 31)) return -1;
  if (a.ws != nullptr && (a.Ns <= 0 || (a.Ns & 15) || a.Ks < 32 || (a.Ks & 31))) return -2;
  if ((a.ldx | a.ldw | a.ldws | a.w_expert) & 7) return -3;
  if ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(a.ws)) & 15) return -4;
  a.by_pair = pairs <= a.E ? 1 : 0;
  const int n = a.ws != nullptr && a.Ns > a.N ? a.Ns : a.N, rows = (a.by_pair ? pairs : a.E) + (a.ws != nullptr ? 1 : 0);
  if (rows > 65535) return -5;
  const dim3 grid(n / 16, rows);
  const size_t smem = sizeof(float) * (UP ? 2 : 1) * MS_WARPS * 4 * 16 * 9 + sizeof(int) * ((pairs + 3) & ~3);
  static bool configured[64] = {};                 // the attribute is per device
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
  if (!configured[dev]) {
    const int most = static_cast<int>(sizeof(float) * (UP ? 2 : 1) * MS_WARPS * 4 * 16 * 9 + sizeof(int) * MS_LIST);
    const cudaError_t e = cudaFuncSetAttribute(moe_stream_kernel<UP>, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e != cudaSuccess) return 1000 + static_cast<int>(e);
    configured[dev] = true;
  }
  return (int)launch_dependent(moe_stream_kernel<UP>, grid, dim3(MS_WARPS * 32), smem, st, a);
}

// x bf16 [T, K] (rows of ldx); gate_up [E, .., K] (experts w_expert elements apart), shared_gate_up [.., K] or null, both in blocks of 128 gate
// and 128 up rows; hid [T * k + T, ldh]: N hidden channels per pair, Ns per token for the shared expert (multiples of 16).
extern "C" TYR_EXPORT int tyr_moe_stream_up(const void* x, const void* gate_up, const void* shared_gate_up, const int* ids, const float* weights,
                                            void* hid, long long ldx, long long w_expert, long long ldh, int T, int k, int E, int N, int Ns, int K,
                                            float limit, float limit_shared, float slope, void* stream) {
  MoeStreamArgs a{(const __nv_bfloat16*)x, (const __nv_bfloat16*)gate_up, (const __nv_bfloat16*)shared_gate_up, ids, weights, (__nv_bfloat16*)hid,
                  ldx, K, K, w_expert, ldh, T, k, E, N, Ns, K, K, 0, limit, limit_shared, slope};
  return moe_stream_launch<true>(a, (cudaStream_t)stream);
}

// hid as above; down [E, N, .] with rows of ldw elements of which K count, shared_down [N, .] with rows of ldws of which Ks count;
// y [T * k + T, N].
extern "C" TYR_EXPORT int tyr_moe_stream_down(const void* hid, const void* down, const void* shared_down, const int* ids, void* y, long long ldh,
                                              long long ldw, long long ldws, long long w_expert, int T, int k, int E, int N, int K, int Ks,
                                              void* stream) {
  MoeStreamArgs a{(const __nv_bfloat16*)hid, (const __nv_bfloat16*)down, (const __nv_bfloat16*)shared_down, ids, nullptr, (__nv_bfloat16*)y,
                  ldh, ldw, ldws, w_expert, N, T, k, E, N, N, K, Ks, 0, 0.f, 0.f, 0.f};
  return moe_stream_launch<false>(a, (cudaStream_t)stream);
}
