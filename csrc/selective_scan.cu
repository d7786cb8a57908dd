// Selective scan (Mamba): per channel c and state n of a sequence
//
//   delta = softplus(dt + dt_bias[c]),   S[c, n] <- exp(delta A[c, n]) S[c, n] + delta x B[n],   y = sum_n S[c, n] C[n] + D[c] x,
//   out = scale * y * silu(z),
//
// with the state and everything that enters it in fp32.  A thread keeps SPT states of one channel in registers and LPC adjacent
// lanes share a channel, so the recurrence itself needs no communication; the sums over n are finished for LPC tokens at a time by
// a transposing butterfly (LPC - 1 shuffles for LPC tokens).
//
//   * prompt: a CTA of 128 threads walks the tokens of 128 / LPC channels in tiles of 32; the inputs of the next tile are loaded into
//     registers while this one runs, softplus and delta x are computed once per (token, channel) and kept in shared memory.
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
__device__ __forceinline__ float ss_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float ss_silu(float v) { return v / (1.f + expf(-v)); }

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

// eight consecutive elements at p (those at index >= n are zero)
__device__ __forceinline__ void ss_load8(const __nv_bfloat16* p, int n, bool vec, float (&f)[8]) {
  if (vec && n >= 8) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 t = unpack_bf16x2(w[e]);
      f[2 * e] = t.x; f[2 * e + 1] = t.y;
    }
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = e < n ? __bfloat162float(p[e]) : 0.f;
  }
}
__device__ __forceinline__ void ss_load8(const float* p, int n, bool vec, float (&f)[8]) {
  if (vec && n >= 8) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = e < n ? p[e] : 0.f;
  }
}
__device__ __forceinline__ void ss_store8(__nv_bfloat16* p, int n, bool vec, const float (&f)[8]) {
  if (vec && n >= 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (e < n) p[e] = __float2bfloat16(f[e]);
  }
}
__device__ __forceinline__ void ss_store8(float* p, int n, bool vec, const float (&f)[8]) {
  if (vec && n >= 8) {
    reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (e < n) p[e] = f[e];
  }
}

template <typename T, int SPT, int LPC>
__global__ void __launch_bounds__(SS_THREADS) scan_prompt_kernel(ScanArgs a, int vec) {
  constexpr bool EXACT = sizeof(T) == 4;
  constexpr int CH = SS_THREADS / LPC;                  // channels of the CTA
  constexpr int NP = SPT * LPC;                         // states, padded
  constexpr int SS_TOK = NP > 128 ? 16 : 32;            // tokens of a tile
  constexpr int CL = CH + 1;                            // row lengths that spread the banks
  constexpr int V8 = (CH + 7) / 8;                      // vectors of 8 channels per token
  constexpr int PER = (SS_TOK * V8 + SS_THREADS - 1) / SS_THREADS;      // vectors per thread and tile
  constexpr int BPT = (SS_TOK * NP + SS_THREADS - 1) / SS_THREADS;      // B (and C) values per thread and tile
  __shared__ float2 s_d[SS_TOK][CL];                    // {delta, delta x}
  __shared__ float s_y[SS_TOK][CL];
  __shared__ __align__(16) float s_b[SS_TOK][NP], s_c[SS_TOK][NP];
  pdl_entry();
  const int b = blockIdx.y, c0 = blockIdx.x * CH, tid = threadIdx.x;
  const int ch = tid / LPC, l = tid % LPC, c = c0 + ch;
  const int n = a.lens ? min(a.lens[b], a.S) : a.S;
  const long long row0 = static_cast<long long>(b) * a.S;
  const T *xp = static_cast<const T*>(a.x) + row0 * a.x_ld + c0, *dtp = static_cast<const T*>(a.dt) + row0 * a.dt_ld + c0;
  const T *zp = static_cast<const T*>(a.z) + row0 * a.z_ld + c0;
  const T *bp = static_cast<const T*>(a.bm) + row0 * a.bc_ld, *cp = static_cast<const T*>(a.cm) + row0 * a.bc_ld;
  T* op = static_cast<T*>(a.out) + row0 * a.out_ld + c0;
  float A[SPT], S[SPT];
  float* st = a.state + (static_cast<long long>(b) * a.C + c) * a.N;
#pragma unroll
  for (int i = 0; i < SPT; ++i) {
    const int k = l * SPT + i;
    const bool ok = c < a.C && k < a.N;
    A[i] = ok ? a.a[static_cast<long long>(c) * a.N + k] * (EXACT ? 1.f : 1.4426950408889634f) : 0.f;
    S[i] = ok && !a.fresh ? st[k] : 0.f;
  }
  // the inputs of a tile: PER vectors of 8 channels (token i / V8, channels 8 (i % V8)) and BPT values of B and C
  float fx[PER][8], fd[PER][8];
  T rb[BPT], rc[BPT];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int i = tid + j * SS_THREADS, t = t0 + i / V8, k = (i % V8) * 8;
      const int left = (i < SS_TOK * V8 && t < n) ? min(a.C - c0, CH) - k : 0;
      ss_load8(xp + t * a.x_ld + k, left, vec, fx[j]);
      ss_load8(dtp + t * a.dt_ld + k, left, vec, fd[j]);
    }
#pragma unroll
    for (int j = 0; j < BPT; ++j) {
      const int i = tid + j * SS_THREADS, t = t0 + i / NP, k = i % NP;
      const bool ok = i < SS_TOK * NP && t < n && k < a.N;
      rb[j] = ok ? bp[t * a.bc_ld + k] : T(0.f);
      rc[j] = ok ? cp[t * a.bc_ld + k] : T(0.f);
    }
  };
  if (n > 0) fetch(0);
  for (int t0 = 0; t0 < n; t0 += SS_TOK) {
    float hx[PER][8];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int i = tid + j * SS_THREADS, t = i / V8, k = (i % V8) * 8;
#pragma unroll
      for (int e = 0; e < 8; ++e) hx[j][e] = fx[j][e];
      if (i < SS_TOK * V8) {
#pragma unroll
        for (int e = 0; e < 8; ++e)
          if (k + e < CH) {
            const bool ok = t0 + t < n && c0 + k + e < a.C;
            const float delta = ok ? ss_softplus(fd[j][e] + a.dt_bias[c0 + k + e]) : 0.f;      // 0: the state stays
            s_d[t][k + e] = make_float2(delta, delta * fx[j][e]);
          }
      }
    }
#pragma unroll
    for (int j = 0; j < BPT; ++j) {
      const int i = tid + j * SS_THREADS;
      if (i < SS_TOK * NP) {
        s_b[i / NP][i % NP] = ss_load(&rb[j]);
        s_c[i / NP][i % NP] = ss_load(&rc[j]);
      }
    }
    __syncthreads();
    float fz[PER][8];
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int i = tid + j * SS_THREADS, t = t0 + i / V8, k = (i % V8) * 8;
      ss_load8(zp + t * a.z_ld + k, (i < SS_TOK * V8 && t < n) ? min(a.C - c0, CH) - k : 0, vec, fz[j]);
    }
    if (t0 + SS_TOK < n) fetch(t0 + SS_TOK);
    // ---- the recurrence, G tokens at a time
    constexpr int G = LPC < 4 ? 4 : LPC;
#pragma unroll 1
    for (int tg = 0; tg < SS_TOK; tg += G) {
      float y[G];
#pragma unroll
      for (int u = 0; u < G; ++u) {
        const int t = tg + u;
        const float2 dd = s_d[t][ch];
        float acc = 0.f;
#pragma unroll
        for (int i = 0; i < SPT; i += 2) {
          const float2 bv = *reinterpret_cast<const float2*>(&s_b[t][l * SPT + i]), cv = *reinterpret_cast<const float2*>(&s_c[t][l * SPT + i]);
          S[i] = ss_decay<EXACT>(dd.x, A[i]) * S[i] + dd.y * bv.x;
          S[i + 1] = ss_decay<EXACT>(dd.x, A[i + 1]) * S[i + 1] + dd.y * bv.y;
          acc += S[i] * cv.x;
          acc += S[i + 1] * cv.y;
        }
        y[u] = acc;
      }
      if constexpr (LPC <= 2) {
#pragma unroll
        for (int u = 0; u < G; ++u) {
          if constexpr (LPC == 2) y[u] += __shfl_xor_sync(0xffffffffu, y[u], 1);
          if (l == 0) s_y[tg + u][ch] = y[u];
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
        s_y[tg + l][ch] = y[0];
      }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int i = tid + j * SS_THREADS, t = i / V8, k = (i % V8) * 8;
      if (i < SS_TOK * V8 && t0 + t < n) {
        float r[8];
#pragma unroll
        for (int e = 0; e < 8; ++e)
          r[e] = (k + e < CH && c0 + k + e < a.C) ? a.scale * ((s_y[t][k + e] + a.d[c0 + k + e] * hx[j][e]) * ss_silu(fz[j][e])) : 0.f;
        ss_store8(op + (t0 + t) * a.out_ld + k, min(a.C - c0, CH) - k, vec, r);
      }
    }
    // the next tile writes s_d / s_b / s_c, which every thread has finished reading before the barrier above; s_y is written again
    // only after the next tile's first barrier
  }
  // rows of a padded batch: nothing reads them, but they must hold numbers
  for (int i = tid; i < (a.S - n) * CH; i += SS_THREADS)
    if (c0 + i % CH < a.C) ss_store(op + (n + i / CH) * a.out_ld + i % CH, 0.f);
#pragma unroll
  for (int i = 0; i < SPT; ++i) {
    const int k = l * SPT + i;
    if (c < a.C && k < a.N) st[k] = S[i];
  }
}

template <typename T, int SPT, int LPC>
__global__ void __launch_bounds__(SS_THREADS) scan_step_kernel(ScanArgs a, int vec) {
  constexpr bool EXACT = sizeof(T) == 4;
  pdl_trigger();
  const int b = blockIdx.y, l = threadIdx.x % LPC, c = blockIdx.x * (SS_THREADS / LPC) + threadIdx.x / LPC;
  const bool live = c < a.C;
  float* st = a.state + (static_cast<long long>(b) * a.C + (live ? c : 0)) * a.N + l * SPT;
  const float* ap = a.a + static_cast<long long>(live ? c : 0) * a.N + l * SPT;
  float A[SPT], S[SPT];
  // constants, and the state, which was last written a whole step earlier
#pragma unroll
  for (int i = 0; i < SPT; ++i) A[i] = live && l * SPT + i < a.N ? ap[i] * (EXACT ? 1.f : 1.4426950408889634f) : 0.f;
  const float dskip = live ? a.d[c] : 0.f, bias = live ? a.dt_bias[c] : 0.f;
  pdl_wait();
  if (vec) {
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
  const float delta = live ? ss_softplus(ss_load(static_cast<const T*>(a.dt) + b * a.dt_ld + c) + bias) : 0.f;
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
  if (l == 0) ss_store(static_cast<T*>(a.out) + b * a.out_ld + c, a.scale * ((acc + dskip * x) * ss_silu(z)));
  if (vec) {
#pragma unroll
    for (int i = 0; i < SPT; i += 2)
      if (l * SPT + i < a.N) *reinterpret_cast<float2*>(st + i) = make_float2(S[i], S[i + 1]);
  } else {
#pragma unroll
    for (int i = 0; i < SPT; ++i)
      if (l * SPT + i < a.N) st[i] = S[i];
  }
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
  const int vec = step ? ((N & 1) == 0 && (reinterpret_cast<uintptr_t>(state) & 7) == 0)
                       : ((al & 15) == 0 && ((ld[0] | ld[1] | ld[2] | ld[4] | C) & 7) == 0);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define TYR_SS(SPT_, LPC_)                                                                                                        \
  {                                                                                                                               \
    const dim3 grid((C + SS_THREADS / LPC_ - 1) / (SS_THREADS / LPC_), B), block(SS_THREADS);                                     \
    if (dtype == 1)                                                                                                               \
      return (int)(step ? launch_dependent(scan_step_kernel<float, SPT_, LPC_>, grid, block, 0, st, a, vec)                       \
                        : launch_dependent(scan_prompt_kernel<float, SPT_, LPC_>, grid, block, 0, st, a, vec));                   \
    return (int)(step ? launch_dependent(scan_step_kernel<__nv_bfloat16, SPT_, LPC_>, grid, block, 0, st, a, vec)                 \
                      : launch_dependent(scan_prompt_kernel<__nv_bfloat16, SPT_, LPC_>, grid, block, 0, st, a, vec));             \
  }
  if (N <= 8) TYR_SS(4, 2)
  if (N <= 16) TYR_SS(4, 4)
  if (N <= 24) TYR_SS(6, 4)
  if (N <= 32) TYR_SS(8, 4)
  if (N <= 64) TYR_SS(8, 8)
  if (N <= 128) TYR_SS(8, 16)
  TYR_SS(16, 16)
#undef TYR_SS
}
