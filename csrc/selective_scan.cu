// Selective scan (Mamba): per channel c and state n of a sequence
//
//   delta = softplus(dt + dt_bias[c]),   S[c, n] <- exp(delta A[c, n]) S[c, n] + delta x B[n],   y = sum_n S[c, n] C[n] + D[c] x,
//   out = scale * y * silu(z),
//
// with the state and everything that enters it in fp32.  A thread keeps SPT states of one channel in registers and LPC adjacent
// lanes share a channel, so the recurrence itself needs no communication; the sums over n are finished for LPC tokens at a time by
// a transposing butterfly (LPC - 1 shuffles for LPC tokens).
//
//   * prompt: a CTA walks the tokens of 128 / LPC channels in tiles of 32, four warps on the recurrence and four on everything around it.
//   * step: one token per row; bound by one read and one write of the state.
//
// EXACT (the fp32 mode): library exponentials and, close to 1, 1 + expm1: a one-ulp bias of exp, applied at every token, would add
// up over the memory of a slowly decaying state.  Otherwise the decay is one ex2.approx.  Compiled without fast math.
#include "common.cuh"

namespace tyr {

__device__ __forceinline__ float ss_load(const float* p) { return *p; }
__device__ __forceinline__ float ss_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ss_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void ss_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
template <bool EXACT>
__device__ __forceinline__ float ss_softplus(float v) {
  if constexpr (EXACT) return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v)));
  const float e = __expf(-fabsf(v));             // ln(1 + e): the logarithm, or its series where 1 + e would lose digits of e
  return fmaxf(v, 0.f) + (e > 0.0625f ? __logf(1.f + e) : e * (1.f - e * (0.5f - e * (0.33333333f - e * 0.25f))));
}
template <bool EXACT>
__device__ __forceinline__ float ss_silu(float v) {
  if constexpr (EXACT) return v / (1.f + expf(-v));
  return __fdividef(v, 1.f + __expf(-v));        // far below 0 the divisor is huge or infinite, and the quotient 0
}

// exp(delta a): `a` comes premultiplied by log2(e) unless EXACT
template <bool EXACT>
__device__ __forceinline__ float ss_decay(float delta, float a) {
  if constexpr (EXACT) {
    const float g = delta * a;
    return g > -0.5f ? 1.f + expm1f(g) : expf(g);
  } else {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(delta * a));
    return r;
  }
}

struct ScanArgs {
  const void *x, *dt, *z, *bm, *cm;      // rows of (token) with contiguous channels / states; element strides below
  long long x_ld, dt_ld, z_ld, bc_ld, out_ld;
  const float *a, *d, *dt_bias;          // [C, N] (= -exp(A_log)), [C], [C]
  float* state;                          // [B, C, N]
  void* out;
  const int* lens;                       // tokens of each row (nullable: S)
  int B, S, C, N, fresh;                 // fresh: the state starts at zero
  float scale;
};

constexpr int SS_THREADS = 128;

// eight consecutive elements at p (those at index >= n are zero), kept raw so that the loads stay in flight until they are used
template <typename T>
struct Raw8;
template <>
struct Raw8<__nv_bfloat16> {
  uint4 u;
  __device__ __forceinline__ void load(const __nv_bfloat16* p, int n, bool vec) {
    u = make_uint4(0, 0, 0, 0);
    if (vec) {
      if (n >= 8) u = *reinterpret_cast<const uint4*>(p);
    } else {
      uint32_t w[4] = {0, 0, 0, 0};
#pragma unroll
      for (int e = 0; e < 8; ++e)
        if (e < n) w[e >> 1] |= static_cast<uint32_t>(__bfloat16_as_ushort(p[e])) << (16 * (e & 1));
      u = make_uint4(w[0], w[1], w[2], w[3]);
    }
  }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 t = unpack_bf16x2(w[e]);
      f[2 * e] = t.x; f[2 * e + 1] = t.y;
    }
  }
};
template <>
struct Raw8<float> {
  float v[8];
  __device__ __forceinline__ void load(const float* p, int n, bool vec) {
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = e < n ? p[e] : 0.f;
  }
  __device__ __forceinline__ void get(float (&f)[8]) const {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = v[e];
  }
};
__device__ __forceinline__ void ss_store8(__nv_bfloat16* p, int n, bool vec, const float (&f)[8]) {
  if (vec) {
    if (n >= 8)
      *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (e < n) p[e] = __float2bfloat16(f[e]);
  }
}
__device__ __forceinline__ void ss_store8(float* p, int n, bool vec, const float (&f)[8]) {
#pragma unroll
  for (int e = 0; e < 8; ++e)
    if (e < n) p[e] = f[e];
}

template <int SPT, int LPC>
struct ScanShape {
  static constexpr int CH = SS_THREADS / LPC;            // channels of a CTA
  static constexpr int NP = SPT * LPC;                   // states, padded
  static constexpr int TOK = NP >= 128 ? 16 : 32;        // tokens of a tile
  static constexpr int CL = CH + 1;                      // row length that spreads the banks
};
template <int SPT, int LPC>
struct __align__(16) ScanTile {
  using H = ScanShape<SPT, LPC>;
  float b[H::TOK][H::NP], c[H::TOK][H::NP];
  float2 d[H::TOK][H::CL];                               // {delta, delta x}
  float y[H::TOK][H::CL];                                // sum_n S C
};

// 256 threads: warps 0 - 3 run the recurrence of tile i, warps 4 - 7 meanwhile prepare tile i + 1 (softplus, delta x), finish and write
// tile i - 1 (skip, gate) and keep the loads of tile i + 2 in flight.  One barrier per tile; the tiles alternate between two buffers.
template <typename T, int SPT, int LPC>
__global__ void __launch_bounds__(2 * SS_THREADS, (sizeof(T) == 2 && SPT == 4 && LPC == 4) ? 4 : (SPT == 16 ? 1 : 2)) scan_prompt_kernel(ScanArgs a, int vec) {
  using H = ScanShape<SPT, LPC>;
  constexpr bool EXACT = sizeof(T) == 4;
  constexpr int CH = H::CH, NP = H::NP, TOK = H::TOK;
  constexpr int V8 = (CH + 7) / 8;                       // vectors of 8 channels per token
  constexpr int PER = (TOK * V8 + SS_THREADS - 1) / SS_THREADS;      // vectors per helper thread and tile
  constexpr int BPT = (TOK * NP + SS_THREADS - 1) / SS_THREADS;      // B (and C) values per helper thread and tile
  extern __shared__ __align__(16) uint8_t ss_smem[];
  ScanTile<SPT, LPC>* const tile = reinterpret_cast<ScanTile<SPT, LPC>*>(ss_smem);
  pdl_entry();
  const int b = blockIdx.y, c0 = blockIdx.x * CH;
  const int n = a.lens ? min(a.lens[b], a.S) : a.S;
  const int tiles = (n + TOK - 1) / TOK;
  const long long row0 = static_cast<long long>(b) * a.S;
  if (threadIdx.x >= SS_THREADS) {
    // ------------------------------------------------------------------ helpers
    const int tid = threadIdx.x - SS_THREADS;
    const T *xp = static_cast<const T*>(a.x) + row0 * a.x_ld + c0, *dtp = static_cast<const T*>(a.dt) + row0 * a.dt_ld + c0;
    const T *zp = static_cast<const T*>(a.z) + row0 * a.z_ld + c0;
    const T *bp = static_cast<const T*>(a.bm) + row0 * a.bc_ld, *cp = static_cast<const T*>(a.cm) + row0 * a.bc_ld;
    T* op = static_cast<T*>(a.out) + row0 * a.out_ld + c0;
    const int live = min(a.C - c0, CH);
    // vector j of this thread: token i / V8, channels 8 (i % V8) .. of the tile, i = tid + j SS_THREADS
    auto left = [&](int j, int t0, int& t, int& k) {
      const int i = tid + j * SS_THREADS;
      t = i / V8; k = (i % V8) * 8;
      return (i < TOK * V8 && t0 + t < n) ? live - k : 0;
    };
    Raw8<T> rx[PER], rd[PER], px[PER], pz[PER];
    T rb[BPT], rc[BPT];
    auto fetch = [&](int t0) {
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        int t, k;
        const int m = left(j, t0, t, k);
        rx[j].load(xp + (t0 + t) * a.x_ld + k, m, vec);
        rd[j].load(dtp + (t0 + t) * a.dt_ld + k, m, vec);
      }
#pragma unroll
      for (int j = 0; j < BPT; ++j) {
        const int i = tid + j * SS_THREADS, t = t0 + i / NP, k = i % NP;
        const bool ok = i < TOK * NP && t < n && k < a.N;
        rb[j] = ok ? bp[t * a.bc_ld + k] : T(0.f);
        rc[j] = ok ? cp[t * a.bc_ld + k] : T(0.f);
      }
    };
    auto prepare = [&](int t0, ScanTile<SPT, LPC>& o) {
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        int t, k;
        const int m = left(j, t0, t, k);
        if (tid + j * SS_THREADS >= TOK * V8) continue;
        float fx[8], fd[8];
        rx[j].get(fx);
        rd[j].get(fd);
#pragma unroll
        for (int e = 0; e < 8; ++e)
          if (k + e < CH) {
            const float delta = e < m ? ss_softplus<EXACT>(fd[e] + a.dt_bias[c0 + k + e]) : 0.f;      // 0: the state stays
            o.d[t][k + e] = make_float2(delta, delta * fx[e]);
          }
      }
#pragma unroll
      for (int j = 0; j < BPT; ++j) {
        const int i = tid + j * SS_THREADS;
        if (i < TOK * NP) {
          o.b[i / NP][i % NP] = ss_load(&rb[j]);
          o.c[i / NP][i % NP] = ss_load(&rc[j]);
        }
      }
    };
    auto finish = [&](int t0, const ScanTile<SPT, LPC>& o) {
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        int t, k;
        const int m = left(j, t0, t, k);
        if (m <= 0) continue;
        float fx[8], fz[8], r[8];
        px[j].get(fx);
        pz[j].get(fz);
#pragma unroll
        for (int e = 0; e < 8; ++e) r[e] = e < m && k + e < CH ? a.scale * ((o.y[t][k + e] + a.d[c0 + k + e] * fx[e]) * ss_silu<EXACT>(fz[e])) : 0.f;
        ss_store8(op + (t0 + t) * a.out_ld + k, m, vec, r);
      }
    };
    if (tiles > 0) {
      fetch(0);
      prepare(0, tile[0]);
      fetch(TOK);
    }
    __syncthreads();
    for (int i = 0; i <= tiles; ++i) {
      if (i > 0) finish((i - 1) * TOK, tile[(i - 1) & 1]);
      if (i < tiles) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
          int t, k;
          const int m = left(j, i * TOK, t, k);
          px[j].load(xp + (i * TOK + t) * a.x_ld + k, m, vec);
          pz[j].load(zp + (i * TOK + t) * a.z_ld + k, m, vec);
        }
        prepare((i + 1) * TOK, tile[(i + 1) & 1]);
        fetch((i + 2) * TOK);
        __syncthreads();
      }
    }
    // rows of a padded batch: nothing reads them, but they must hold numbers
    for (int i = tid; i < (a.S - n) * CH; i += SS_THREADS)
      if (c0 + i % CH < a.C) ss_store(op + (n + i / CH) * a.out_ld + i % CH, 0.f);
    return;
  }
  // -------------------------------------------------------------------- recurrence
  const int ch = threadIdx.x / LPC, l = threadIdx.x % LPC, c = c0 + ch;
  float A[SPT], S[SPT];
  float* st = a.state + (static_cast<long long>(b) * a.C + c) * a.N;
#pragma unroll
  for (int i = 0; i < SPT; ++i) {
    const int k = l * SPT + i;
    const bool ok = c < a.C && k < a.N;
    A[i] = ok ? a.a[static_cast<long long>(c) * a.N + k] * (EXACT ? 1.f : 1.4426950408889634f) : 0.f;
    S[i] = ok && !a.fresh ? st[k] : 0.f;
  }
  __syncthreads();
  constexpr int G = LPC < 4 ? 4 : LPC;                   // tokens whose sums are finished together
  for (int ti = 0; ti < tiles; ++ti) {
    ScanTile<SPT, LPC>& o = tile[ti & 1];
#pragma unroll 2
    for (int tg = 0; tg < TOK; tg += G) {
      float y[G];
#pragma unroll
      for (int u = 0; u < G; ++u) {
        const int t = tg + u;
        const float2 dd = o.d[t][ch];
        float bv[SPT], cv[SPT];
        if constexpr (SPT % 4 == 0) {
#pragma unroll
          for (int i = 0; i < SPT; i += 4) {
            const float4 b4 = *reinterpret_cast<const float4*>(&o.b[t][l * SPT + i]), c4 = *reinterpret_cast<const float4*>(&o.c[t][l * SPT + i]);
            bv[i] = b4.x; bv[i + 1] = b4.y; bv[i + 2] = b4.z; bv[i + 3] = b4.w;
            cv[i] = c4.x; cv[i + 1] = c4.y; cv[i + 2] = c4.z; cv[i + 3] = c4.w;
          }
        } else {
#pragma unroll
          for (int i = 0; i < SPT; i += 2) {
            const float2 b2 = *reinterpret_cast<const float2*>(&o.b[t][l * SPT + i]), c2 = *reinterpret_cast<const float2*>(&o.c[t][l * SPT + i]);
            bv[i] = b2.x; bv[i + 1] = b2.y;
            cv[i] = c2.x; cv[i + 1] = c2.y;
          }
        }
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < SPT; ++i) {
          S[i] = ss_decay<EXACT>(dd.x, A[i]) * S[i] + dd.y * bv[i];
          acc += S[i] * cv[i];
        }
        y[u] = acc;
      }
      if constexpr (LPC <= 2) {
#pragma unroll
        for (int u = 0; u < G; ++u) {
          if constexpr (LPC == 2) y[u] += __shfl_xor_sync(0xffffffffu, y[u], 1);
          if (l == 0) o.y[tg + u][ch] = y[u];
        }
      } else {
        // butterfly: after the round over bit h, a lane keeps the tokens whose bit h equals its own
#pragma unroll
        for (int h = LPC / 2; h >= 1; h >>= 1) {
          const bool up = (l & h) != 0;
#pragma unroll
          for (int u = 0; u < h; ++u) {
            const float keep = up ? y[u + h] : y[u], give = up ? y[u] : y[u + h];
            y[u] = keep + __shfl_xor_sync(0xffffffffu, give, h);
          }
        }
        o.y[tg + l][ch] = y[0];
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < SPT; ++i) {
    const int k = l * SPT + i;
    if (c < a.C && k < a.N) st[k] = S[i];
  }
}

// vec: elements of a state vector access (4, 2 or 1), which divide SPT and N
template <typename T, int SPT, int LPC>
__global__ void __launch_bounds__(SS_THREADS) scan_step_kernel(ScanArgs a, int vec) {
  constexpr bool EXACT = sizeof(T) == 4;
  pdl_trigger();
  const int b = blockIdx.y, l = threadIdx.x % LPC, c = blockIdx.x * (SS_THREADS / LPC) + threadIdx.x / LPC;
  const bool live = c < a.C;
  float* st = a.state + (static_cast<long long>(b) * a.C + (live ? c : 0)) * a.N + l * SPT;
  const float* ap = a.a + static_cast<long long>(live ? c : 0) * a.N + l * SPT;
  if (live && l * SPT < a.N) asm volatile("prefetch.global.L2 [%0];" ::"l"(st));      // written a whole step earlier
  float A[SPT], S[SPT];
#pragma unroll
  for (int i = 0; i < SPT; ++i) A[i] = live && l * SPT + i < a.N ? ap[i] * (EXACT ? 1.f : 1.4426950408889634f) : 0.f;
  const float dskip = live ? a.d[c] : 0.f, bias = live ? a.dt_bias[c] : 0.f;
  pdl_wait();
  if (SPT % 4 == 0 && vec == 4) {
#pragma unroll
    for (int i = 0; i + 3 < SPT; i += 4) {
      const float4 v = live && l * SPT + i < a.N ? *reinterpret_cast<const float4*>(st + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
    }
  } else if (vec >= 2) {
#pragma unroll
    for (int i = 0; i < SPT; i += 2) {
      const float2 v = live && l * SPT + i < a.N ? *reinterpret_cast<const float2*>(st + i) : make_float2(0.f, 0.f);
      S[i] = v.x; S[i + 1] = v.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < SPT; ++i) S[i] = live && l * SPT + i < a.N ? st[i] : 0.f;
  }
  const T *bp = static_cast<const T*>(a.bm) + b * a.bc_ld + l * SPT, *cp = static_cast<const T*>(a.cm) + b * a.bc_ld + l * SPT;
  const float x = live ? ss_load(static_cast<const T*>(a.x) + b * a.x_ld + c) : 0.f;
  const float z = live ? ss_load(static_cast<const T*>(a.z) + b * a.z_ld + c) : 0.f;
  const float delta = live ? ss_softplus<EXACT>(ss_load(static_cast<const T*>(a.dt) + b * a.dt_ld + c) + bias) : 0.f;
  float acc = 0.f;
#pragma unroll
  for (int i = 0; i < SPT; ++i) {
    const bool ok = l * SPT + i < a.N;
    S[i] = ss_decay<EXACT>(delta, A[i]) * S[i] + delta * x * (ok ? ss_load(bp + i) : 0.f);
    acc += S[i] * (ok ? ss_load(cp + i) : 0.f);
  }
#pragma unroll
  for (int h = LPC / 2; h >= 1; h >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, h);
  if (!live) return;
  if (l == 0) ss_store(static_cast<T*>(a.out) + b * a.out_ld + c, a.scale * ((acc + dskip * x) * ss_silu<EXACT>(z)));
  if (SPT % 4 == 0 && vec == 4) {
#pragma unroll
    for (int i = 0; i + 3 < SPT; i += 4)
      if (l * SPT + i < a.N) *reinterpret_cast<float4*>(st + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
  } else if (vec >= 2) {
#pragma unroll
    for (int i = 0; i < SPT; i += 2)
      if (l * SPT + i < a.N) *reinterpret_cast<float2*>(st + i) = make_float2(S[i], S[i + 1]);
  } else {
#pragma unroll
    for (int i = 0; i < SPT; ++i)
      if (l * SPT + i < a.N) st[i] = S[i];
  }
}

template <typename T, int SPT, int LPC>
static int scan_launch(const ScanArgs& a, int step, int vec, cudaStream_t st) {
  const dim3 grid((a.C + SS_THREADS / LPC - 1) / (SS_THREADS / LPC), a.B);
  if (step) return (int)launch_dependent(scan_step_kernel<T, SPT, LPC>, grid, dim3(SS_THREADS), 0, st, a, vec);
  constexpr size_t smem = 2 * sizeof(ScanTile<SPT, LPC>);
  if (smem > 48 * 1024) {
    static bool configured[64] = {};            // the attribute is per device
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
    if (!configured[dev]) {
      const cudaError_t e = cudaFuncSetAttribute(scan_prompt_kernel<T, SPT, LPC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return 1000 + (int)e;
      configured[dev] = true;
    }
  }
  return (int)launch_dependent(scan_prompt_kernel<T, SPT, LPC>, grid, dim3(2 * SS_THREADS), smem, st, a, vec);
}

}  // namespace tyr

using namespace tyr;

// Row strides in elements (rows of a batch evenly spaced): x, dt, z [B, S, C], B / C [B, S, N], out [B, S, C].  state fp32 [B, C, N]
// contiguous, in place.  dtype: 0 = bf16, 1 = fp32.  At most 256 states.  step: S == 1 and a state that goes on.
extern "C" TYR_EXPORT int tyr_selective_scan(const void* x, const void* dt, const void* z, const void* bm, const void* cm, const long long* ld,
                                             const float* A, const float* D, const float* dt_bias, float* state, void* out,
                                             const int* lens, int B, int S, int C, int N, int fresh, int step, float scale, int dtype,
                                             void* stream) {
  if (B <= 0 || B > 65535 || S <= 0 || C <= 0 || N <= 0 || N > 256 || (step && (S != 1 || fresh || lens != nullptr))) return -1;
  ScanArgs a;
  a.x = x; a.dt = dt; a.z = z; a.bm = bm; a.cm = cm;
  a.x_ld = ld[0]; a.dt_ld = ld[1]; a.z_ld = ld[2]; a.bc_ld = ld[3]; a.out_ld = ld[4];
  a.a = A; a.d = D; a.dt_bias = dt_bias; a.state = state; a.out = out; a.lens = lens;
  a.B = B; a.S = S; a.C = C; a.N = N; a.fresh = fresh; a.scale = scale;
  const uintptr_t al = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(dt) | reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out);
  const int vec = step ? ((reinterpret_cast<uintptr_t>(state) & 15) || (N & 1) ? 1 : (N & 3) ? 2 : 4)
                       : ((al & 15) == 0 && ((ld[0] | ld[1] | ld[2] | ld[4] | C) & 7) == 0);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define TYR_SS(SPT_, LPC_) return dtype == 1 ? scan_launch<float, SPT_, LPC_>(a, step, vec, st) : scan_launch<__nv_bfloat16, SPT_, LPC_>(a, step, vec, st);
  if (N <= 8) TYR_SS(4, 2)
  if (N <= 16) TYR_SS(4, 4)
  if (N <= 24) TYR_SS(6, 4)
  if (N <= 32) TYR_SS(8, 4)
  if (N <= 64) TYR_SS(8, 8)
  if (N <= 128) TYR_SS(8, 16)
  TYR_SS(16, 16)
#undef TYR_SS
}
