// Embedding-table gradient: grad[id] += sum of the dy rows whose token is `id`, accumulated into an fp32 table.
//
// The token stream is Zipf-distributed: a handful of ids own thousands of rows each, and a plain scatter-add (one fp32
// atomic per element and occurrence, what `index_add_` does) serialises on those table rows.  Here the rows arrive SORTED
// by id (one sort per step serves the token table and every value-embedding table).  A CTA takes a run of consecutive
// sorted positions, keeps the running sum of equal ids in registers and touches the table once per id and run: the
// atomics drop from one per occurrence to one per (id, run), and dy is read exactly once, 16 bytes per thread and row.
//
// The reference differentiates `embedding` through autograd's dense scatter (Examples/NanoChat/ModdedGPT.lean:563-567,
// cc/src/tyr.cpp embedding op).
#include "common.cuh"

namespace tyr {

constexpr int kEmbedRun = 64;   // sorted positions per CTA

// dy [N, d] bf16 (row stride ld), order[p] = row of dy at sorted position p, sorted_ids[p] ascending, grad fp32 [V, d].
// blockDim.x * 8 >= d is not required: threads stride over the columns in 8-element vectors.
__global__ void __launch_bounds__(256)
embed_grad_sorted_kernel(const __nv_bfloat16* __restrict__ dy, const long long* __restrict__ order,
                         const long long* __restrict__ sorted_ids, float* __restrict__ grad, int N, int d, long long ld,
                         int V) {
  pdl_entry();
  __shared__ long long s_row[kEmbedRun];
  __shared__ long long s_id[kEmbedRun];
  const int p0 = blockIdx.x * kEmbedRun;
  const int n = min(kEmbedRun, N - p0);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    s_row[i] = order[p0 + i];
    s_id[i] = sorted_ids[p0 + i];
  }
  __syncthreads();
  for (int c = threadIdx.x * 8; c < d; c += blockDim.x * 8) {
    float acc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = 0.f;
    long long cur = s_id[0];
    for (int i = 0; i < n; ++i) {
      const long long id = s_id[i];
      if (id != cur) {
        if (cur >= 0 && cur < V) {
          float* g = grad + cur * d + c;
#pragma unroll
          for (int q = 0; q < 2; ++q)
            asm volatile("red.global.add.v4.f32 [%0], {%1, %2, %3, %4};" ::"l"(g + q * 4), "f"(acc[q * 4]), "f"(acc[q * 4 + 1]),
                         "f"(acc[q * 4 + 2]), "f"(acc[q * 4 + 3])
                         : "memory");
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = 0.f;
        cur = id;
      }
      const long long r = s_row[i];
      if (r < 0 || r >= N) continue;
      const uint4 u = *reinterpret_cast<const uint4*>(dy + r * ld + c);
      const float2 f0 = unpack_bf16x2(u.x), f1 = unpack_bf16x2(u.y), f2 = unpack_bf16x2(u.z), f3 = unpack_bf16x2(u.w);
      acc[0] += f0.x; acc[1] += f0.y; acc[2] += f1.x; acc[3] += f1.y;
      acc[4] += f2.x; acc[5] += f2.y; acc[6] += f3.x; acc[7] += f3.y;
    }
    if (cur >= 0 && cur < V) {
      float* g = grad + cur * d + c;
#pragma unroll
      for (int q = 0; q < 2; ++q)
        asm volatile("red.global.add.v4.f32 [%0], {%1, %2, %3, %4};" ::"l"(g + q * 4), "f"(acc[q * 4]), "f"(acc[q * 4 + 1]),
                     "f"(acc[q * 4 + 2]), "f"(acc[q * 4 + 3])
                     : "memory");
    }
  }
}

// Input rows of a decoder with sinusoidal positions: x[r, d] = table[ids[r], d] * scale + sin / cos(p * freq[d / 2]), fp32, channel 2i the
// sine and 2i + 1 the cosine.  `turns` holds the frequencies over 2 pi in double, so that the angle is reduced to a fraction of a turn
// before it is rounded and far positions keep their accuracy.  p = pos[r] (a decode step), else r % S.  Without `turns` nothing is added.
// A thread owns EP_PAIRS channel pairs of one position and walks the rows of the batch that share it (all of a prompt's; one of a step's).
constexpr int EP_PAIRS = 4;
__device__ __forceinline__ void ep_load(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 t = unpack_bf16x2(w[e]);
    f[2 * e] = t.x; f[2 * e + 1] = t.y;
  }
}
__device__ __forceinline__ void ep_load(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

template <typename T>
__global__ void __launch_bounds__(256) embed_positions_kernel(const long long* __restrict__ ids, const T* __restrict__ table, const double* __restrict__ turns,
                                                              const int* __restrict__ pos, float* __restrict__ x, int B, int S, int D,
                                                              int vocab, float scale, int vec, int* err) {
  pdl_entry();
  const int half = (D + 1) / 2, parts = (half + EP_PAIRS - 1) / EP_PAIRS;
  const long long units = static_cast<long long>(pos ? B : S) * parts;
  for (long long i = blockIdx.x * 256LL + threadIdx.x; i < units; i += gridDim.x * 256LL) {
    const int u = static_cast<int>(i / parts), k0 = static_cast<int>(i % parts) * EP_PAIRS;
    const int p = pos ? pos[u] : u;
    float add[2 * EP_PAIRS];
#pragma unroll
    for (int j = 0; j < EP_PAIRS; ++j) {
      if (turns == nullptr) {
        add[2 * j] = add[2 * j + 1] = 0.f;
        continue;
      }
      const double t = k0 + j < half ? p * turns[k0 + j] : 0.0;
      sincospif(2.f * static_cast<float>(t - rint(t)), &add[2 * j], &add[2 * j + 1]);
    }
    const long long stride = pos ? 1 : S;
    for (int b = 0; b < (pos ? 1 : B); ++b) {
      const long long r = u + b * stride;
      const long long id = ids[r];
      if (id < 0 || id >= vocab) {
        if (k0 == 0) report_error(err, ERR_BOUNDS, static_cast<int>(id));
        continue;
      }
      const T* e = table + id * D + 2 * k0;
      float* o = x + r * D + 2 * k0;
      if (vec) {
        float f[8];
        ep_load(e, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = f[j] * scale + add[j];
        reinterpret_cast<float4*>(o)[0] = make_float4(f[0], f[1], f[2], f[3]);
        reinterpret_cast<float4*>(o)[1] = make_float4(f[4], f[5], f[6], f[7]);
      } else {
#pragma unroll
        for (int j = 0; j < 2 * EP_PAIRS; ++j)
          if (2 * k0 + j < D) o[j] = static_cast<float>(e[j]) * scale + add[j];
      }
    }
  }
}

}  // namespace tyr

// Returns 0 on success, -1 on a bad shape / alignment.
extern "C" TYR_EXPORT int tyr_embed_grad_sorted(const void* dy, const long long* order, const long long* sorted_ids, float* grad,
                                                int N, int d, long long ld, int V, void* stream) {
  if (N <= 0 || d <= 0 || (d & 7) || (ld & 7) || V <= 0) return -1;
  if ((reinterpret_cast<uintptr_t>(dy) | reinterpret_cast<uintptr_t>(grad)) & 15) return -1;
  const int blocks = (N + tyr::kEmbedRun - 1) / tyr::kEmbedRun;
  const int threads = d / 8 >= 256 ? 256 : ((d / 8 + 31) / 32) * 32;
  tyr::launch_dependent(tyr::embed_grad_sorted_kernel, dim3(blocks), dim3(threads), 0, reinterpret_cast<cudaStream_t>(stream),
      reinterpret_cast<const __nv_bfloat16*>(dy), order, sorted_ids, grad, N, d, ld, V);
  return static_cast<int>(cudaGetLastError());
}

// ids int64 [B, S]; table [vocab, D] (dtype 0 = bf16, 1 = fp32); turns double [(D + 1) / 2] or null; pos int32 [B] (S == 1) or null; x fp32 [B, S, D].
// An id outside the table is recorded in `err` and its row left alone.
extern "C" TYR_EXPORT int tyr_embed_positions(const void* ids, const void* table, const double* turns, const int* pos, float* x, int B,
                                              int S, int D, int vocab, float scale, int dtype, int* err, void* stream) {
  using namespace tyr;
  if (B <= 0 || S <= 0 || D <= 0 || vocab <= 0 || (pos != nullptr && S != 1)) return -1;
  const long long want = ((pos ? B : S) * static_cast<long long>(((D + 1) / 2 + EP_PAIRS - 1) / EP_PAIRS) + 255) / 256;
  const int vec = (D & 7) == 0 && ((reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(x)) & 15) == 0;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 32 ? want : 148LL * 32));
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto* id = static_cast<const long long*>(ids);
  if (dtype == 1)
    return (int)launch_dependent(embed_positions_kernel<float>, grid, dim3(256), 0, st, id, static_cast<const float*>(table), turns, pos, x, B, S, D,
                                 vocab, scale, vec, err);
  return (int)launch_dependent(embed_positions_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, id, static_cast<const __nv_bfloat16*>(table), turns, pos,
                               x, B, S, D, vocab, scale, vec, err);
}
