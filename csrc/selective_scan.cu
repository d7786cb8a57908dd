// Selective scan (Mamba): per channel c and state n of a sequence
//
//   delta = softplus(dt + dt_bias[c]),   S[c, n] <- exp(delta A[c, n]) S[c, n] + delta x B[n],   y = sum_n S[c, n] C[n] + D[c] x,
//   out = scale * y * silu(z),
//
// with the state and everything that enters it in fp32.  A thread keeps SPT states of one channel in registers and LPC adjacent
// lanes share a channel, so the recurrence itself needs no communication; the sums over n are finished for LPC tokens at a time by a
// transposing butterfly.  With SPT = 8 the reads of B and C are nearly warp-wide broadcasts, and the kernel is bound by one ex2 per
// (token, channel, state); pairs of states share packed fp32 instructions.
//
//   * prompt: a CTA walks the tokens of its channels in tiles of 32, two warps on the recurrence and four on everything around it.
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

// The decay exp(delta a).  EXACT: of a; otherwise of the product delta a log2(e).
template <bool EXACT>
__device__ __forceinline__ float ss_decay(float delta, float a) {
  if constexpr (EXACT) {
    const float g = delta * a;
    return g > -0.5f ? 1.f + expm1f(g) : expf(g);
  } else {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(a));
    return r;
  }
}

// packed pairs of fp32
__device__ __forceinline__ uint64_t pack2(float x, float y) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ void unpack2(uint64_t v, float& x, float& y) { asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v)); }
__device__ __forceinline__ uint64_t mul2(uint64_t x, uint64_t y) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(x), "l"(y));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t x, uint64_t y, uint64_t z) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(x), "l"(y), "l"(z));
  return r;
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

constexpr int SS_REC = 64;             // threads of a prompt CTA on the recurrence
constexpr int SS_HELP = 128;           // ... and on the rest
constexpr int SS_STEP = 128;           // threads of a step CTA

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
  static constexpr int CH = SS_REC / LPC;                // channels of a CTA
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
template <int SPT, int LPC>
struct __align__(16) ScanSmem {
  ScanTile<SPT, LPC> tile[2];
  float bias[ScanShape<SPT, LPC>::CH], skip[ScanShape<SPT, LPC>::CH];
};

// SS_REC threads run the recurrence of tile i; the helpers meanwhile prepare tile i + 1 (softplus, delta x), finish and write tile
// i - 1 (skip, gate) and keep the loads of tile i + 2 in flight.  One barrier per tile; the tiles alternate between two buffers.
template <typename T, int SPT, int LPC>
__global__ void __launch_bounds__(SS_REC + SS_HELP, (sizeof(T) == 2 && SPT <= 8) ? 4 : 2) scan_prompt_kernel(ScanArgs a, int vec) {
  using H = ScanShape<SPT, LPC>;
  constexpr bool EXACT = sizeof(T) == 4;
  constexpr int CH = H::CH, NP = H::NP, TOK = H::TOK;
  constexpr int V8 = (CH + 7) / 8;                       // vectors of 8 channels per token
  constexpr int PER = (TOK * V8 + SS_HELP - 1) / SS_HELP;      // vectors per helper thread and tile
  constexpr int BPT = (TOK * NP + SS_HELP - 1) / SS_HELP;      // B (and C) values per helper thread and tile
  extern __shared__ __align__(16) uint8_t ss_smem[];
  if (CH % 8 != 0) vec = 0;
  ScanSmem<SPT, LPC>& sm = *reinterpret_cast<ScanSmem<SPT, LPC>*>(ss_smem);
  ScanTile<SPT, LPC>* const tile = sm.tile;
  pdl_entry();
  const int b = blockIdx.y, c0 = blockIdx.x * CH;
  const int n = a.lens ? min(a.lens[b], a.S) : a.S;
  const int tiles = (n + TOK - 1) / TOK;
  const long long row0 = static_cast<long long>(b) * a.S;
  if (threadIdx.x >= SS_REC) {
    // ------------------------------------------------------------------ helpers
    const int tid = threadIdx.x - SS_REC;
    const T *xp = static_cast<const T*>(a.x) + row0 * a.x_ld + c0, *dtp = static_cast<const T*>(a.dt) + row0 * a.dt_ld + c0;
    const T *zp = static_cast<const T*>(a.z) + row0 * a.z_ld + c0;
    const T *bp = static_cast<const T*>(a.bm) + row0 * a.bc_ld, *cp = static_cast<const T*>(a.cm) + row0 * a.bc_ld;
    T* op = static_cast<T*>(a.out) + row0 * a.out_ld + c0;
    const int live = min(a.C - c0, CH);
    for (int i = tid; i < CH; i += SS_HELP) {
      sm.bias[i] = i < live ? a.dt_bias[c0 + i] : 0.f;
      sm.skip[i] = i < live ? a.d[c0 + i] : 0.f;
    }
    asm volatile("bar.sync 1, %0;" ::"n"(SS_HELP) : "memory");      // the helpers alone
    // vector j of this thread: token i / V8, channels 8 (i % V8) .. of the tile, i = tid + j SS_HELP.  FULL: the tile lies inside the
    // sequence and the channels, and vectors are aligned.
    const bool full_ch = vec && live == CH && CH % 8 == 0 && a.N == NP;
    auto full = [&](int t0) { return full_ch && t0 + TOK <= n; };
    auto left = [&](int j, int t0) {
      const int i = tid + j * SS_HELP;
      return (i < TOK * V8 && t0 + i / V8 < n) ? live - (i % V8) * 8 : 0;
    };
    const int tv = tid / V8, kv = (tid % V8) * 8;                        // vector 0; the others are SS_HELP / V8 tokens further each
    constexpr int DT = SS_HELP / V8;
    static_assert(SS_HELP % V8 == 0, "vectors of a token belong to one round");
    const T *x0 = xp + static_cast<long long>(tv) * a.x_ld + kv, *d0 = dtp + static_cast<long long>(tv) * a.dt_ld + kv, *z0 = zp + static_cast<long long>(tv) * a.z_ld + kv;
    T* o0 = op + static_cast<long long>(tv) * a.out_ld + kv;
    const T *b0 = bp + static_cast<long long>(tid / NP) * a.bc_ld + tid % NP, *cc0 = cp + static_cast<long long>(tid / NP) * a.bc_ld + tid % NP;
    Raw8<T> rx[PER], rd[PER], px[PER], pz[PER];
    T rb[BPT], rc[BPT];
    auto fetch = [&](int t0) {
      const bool f = full(t0);
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        const int m = f && TOK * V8 % SS_HELP == 0 ? 8 : left(j, t0);
        rx[j].load(x0 + (t0 + j * DT) * a.x_ld, m, vec);
        rd[j].load(d0 + (t0 + j * DT) * a.dt_ld, m, vec);
      }
      if constexpr (NP <= SS_HELP && SS_HELP % NP == 0) {
#pragma unroll
        for (int j = 0; j < BPT; ++j) {
          const int dt = j * (SS_HELP / NP);
          const bool ok = f || (tid / NP + dt < TOK && t0 + tid / NP + dt < n && tid % NP < a.N);
          rb[j] = ok ? b0[(t0 + dt) * a.bc_ld] : T(0.f);
          rc[j] = ok ? cc0[(t0 + dt) * a.bc_ld] : T(0.f);
        }
      } else {
#pragma unroll
        for (int j = 0; j < BPT; ++j) {
          const int i = tid + j * SS_HELP, t = t0 + i / NP, k = i % NP;
          const bool ok = i < TOK * NP && t < n && k < a.N;
          rb[j] = ok ? bp[t * a.bc_ld + k] : T(0.f);
          rc[j] = ok ? cp[t * a.bc_ld + k] : T(0.f);
        }
      }
    };
    auto prepare = [&](int t0, ScanTile<SPT, LPC>& o) {
      const bool f = full(t0);
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        if (TOK * V8 % SS_HELP != 0 && tid + j * SS_HELP >= TOK * V8) continue;
        float fx[8], fd[8];
        rx[j].get(fx);
        rd[j].get(fd);
        float2* row = &o.d[tv + j * DT][kv];
        if (f) {
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const float delta = ss_softplus<EXACT>(fd[e] + sm.bias[kv + e]);
            row[e] = make_float2(delta, delta * fx[e]);
          }
        } else {
          const int m = left(j, t0);
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (kv + e < CH) {
              const float delta = e < m ? ss_softplus<EXACT>(fd[e] + sm.bias[kv + e]) : 0.f;      // 0: the state stays
              row[e] = make_float2(delta, delta * fx[e]);
            }
        }
      }
#pragma unroll
      for (int j = 0; j < BPT; ++j) {
        const int i = tid + j * SS_HELP;
        if (TOK * NP % SS_HELP == 0 || i < TOK * NP) {
          (&o.b[0][0])[i] = ss_load(&rb[j]);
          (&o.c[0][0])[i] = ss_load(&rc[j]);
        }
      }
    };
    auto finish = [&](int t0, const ScanTile<SPT, LPC>& o) {
      const bool f = full(t0);
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        const int m = left(j, t0);
        if (m <= 0) continue;
        float fx[8], fz[8], r[8];
        px[j].get(fx);
        pz[j].get(fz);
        const float* row = &o.y[tv + j * DT][kv];
        if (f) {
#pragma unroll
          for (int e = 0; e < 8; ++e) r[e] = (row[e] + sm.skip[kv + e] * fx[e]) * (a.scale * ss_silu<EXACT>(fz[e]));
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) r[e] = e < m && kv + e < CH ? (row[e] + sm.skip[kv + e] * fx[e]) * (a.scale * ss_silu<EXACT>(fz[e])) : 0.f;
        }
        ss_store8(o0 + (t0 + j * DT) * a.out_ld, m, vec, r);
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
          const int m = left(j, i * TOK);
          px[j].load(x0 + (i * TOK + j * DT) * a.x_ld, m, vec);
          pz[j].load(z0 + (i * TOK + j * DT) * a.z_ld, m, vec);
        }
        prepare((i + 1) * TOK, tile[(i + 1) & 1]);
        fetch((i + 2) * TOK);
        __syncthreads();
      }
    }
    // rows of a padded batch: nothing reads them, but they must hold numbers
    for (int i = tid; i < (a.S - n) * CH; i += SS_HELP)
      if (c0 + i % CH < a.C) ss_store(op + (n + i / CH) * a.out_ld + i % CH, 0.f);
    return;
  }
  // -------------------------------------------------------------------- recurrence
  const int ch = threadIdx.x / LPC, l = threadIdx.x % LPC, c = c0 + ch;
  float* st = a.state + (static_cast<long long>(b) * a.C + c) * a.N;
  uint64_t A[SPT / 2], S[SPT / 2];                       // pairs of states
#pragma unroll
  for (int i = 0; i < SPT; i += 2) {
    float av[2], sv[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = l * SPT + i + e;
      const bool ok = c < a.C && k < a.N;
      av[e] = ok ? a.a[static_cast<long long>(c) * a.N + k] * (EXACT ? 1.f : 1.4426950408889634f) : 0.f;
      sv[e] = ok && !a.fresh ? st[k] : 0.f;
    }
    A[i / 2] = pack2(av[0], av[1]);
    S[i / 2] = pack2(sv[0], sv[1]);
  }
  __syncthreads();
  constexpr int G = LPC < 2 ? 2 : LPC;                   // tokens whose sums are finished together
  constexpr int U = SPT > 8 ? 1 : 2;                     // tokens whose operands are loaded together
  uint64_t bv[U][SPT / 2], cv[U][SPT / 2];
  float2 dd[U];                                          // {delta, delta x}
  auto load = [&](const ScanTile<SPT, LPC>& o, int t0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = t0 + u;
      dd[u] = o.d[t][ch];
#pragma unroll
      for (int i = 0; i < SPT / 2; i += SPT % 4 == 0 ? 2 : 1) {
        if constexpr (SPT % 4 == 0) {
          const ulonglong2 b4 = *reinterpret_cast<const ulonglong2*>(&o.b[t][l * SPT + 2 * i]), c4 = *reinterpret_cast<const ulonglong2*>(&o.c[t][l * SPT + 2 * i]);
          bv[u][i] = b4.x; bv[u][i + 1] = b4.y;
          cv[u][i] = c4.x; cv[u][i + 1] = c4.y;
        } else {
          bv[u][i] = *reinterpret_cast<const uint64_t*>(&o.b[t][l * SPT + 2 * i]);
          cv[u][i] = *reinterpret_cast<const uint64_t*>(&o.c[t][l * SPT + 2 * i]);
        }
      }
    }
  };
  for (int ti = 0; ti < tiles; ++ti) {
    ScanTile<SPT, LPC>& o = tile[ti & 1];
    load(o, 0);
#pragma unroll 2
    for (int tg = 0; tg < TOK; tg += G) {
      float y[G];
#pragma unroll
      for (int g0 = 0; g0 < G; g0 += U) {
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const uint64_t delta = pack2(dd[u].x, dd[u].x), dx = pack2(dd[u].y, dd[u].y);
          uint64_t acc = 0;
#pragma unroll
          for (int i = 0; i < SPT / 2; ++i) {
            float a0, a1;
            unpack2(EXACT ? A[i] : mul2(delta, A[i]), a0, a1);
            a0 = ss_decay<EXACT>(dd[u].x, a0);
            a1 = ss_decay<EXACT>(dd[u].x, a1);
            S[i] = fma2(pack2(a0, a1), S[i], mul2(dx, bv[u][i]));
            acc = fma2(S[i], cv[u][i], acc);
          }
          float y0, y1;
          unpack2(acc, y0, y1);
          y[g0 + u] = y0 + y1;
        }
        // the next operands are on their way while the sums below are finished (past the tile's end: its last tokens again, unused)
        load(o, min(tg + g0 + U, TOK - U));
      }
      if constexpr (LPC == 1) {
#pragma unroll
        for (int u = 0; u < G; ++u) o.y[tg + u][ch] = y[u];
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
  for (int i = 0; i < SPT; i += 2) {
    float sv[2];
    unpack2(S[i / 2], sv[0], sv[1]);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = l * SPT + i + e;
      if (c < a.C && k < a.N) st[k] = sv[e];
    }
  }
}

// vec: elements of a state vector access (4, 2 or 1), which divide SPT and N
template <typename T, int SPT, int LPC>
__global__ void __launch_bounds__(SS_STEP) scan_step_kernel(ScanArgs a, int vec) {
  constexpr bool EXACT = sizeof(T) == 4;
  pdl_trigger();
  const int b = blockIdx.y, l = threadIdx.x % LPC, c = blockIdx.x * (SS_STEP / LPC) + threadIdx.x / LPC;
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
    S[i] = ss_decay<EXACT>(delta, EXACT ? A[i] : delta * A[i]) * S[i] + delta * x * (ok ? ss_load(bp + i) : 0.f);
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
static int step_launch(const ScanArgs& a, int vec, cudaStream_t st) {
  const dim3 grid((a.C + SS_STEP / LPC - 1) / (SS_STEP / LPC), a.B);
  return (int)launch_dependent(scan_step_kernel<T, SPT, LPC>, grid, dim3(SS_STEP), 0, st, a, vec);
}

template <typename T, int SPT, int LPC>
static int prompt_launch(const ScanArgs& a, int vec, cudaStream_t st) {
  constexpr int CH = ScanShape<SPT, LPC>::CH;
  const dim3 grid((a.C + CH - 1) / CH, a.B);
  constexpr size_t smem = sizeof(ScanSmem<SPT, LPC>);
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
  return (int)launch_dependent(scan_prompt_kernel<T, SPT, LPC>, grid, dim3(SS_REC + SS_HELP), smem, st, a, vec);
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
#define TYR_SS(kind, SPT_, LPC_) return dtype == 1 ? kind##_launch<float, SPT_, LPC_>(a, vec, st) : kind##_launch<__nv_bfloat16, SPT_, LPC_>(a, vec, st);
  if (step) {                                   // few states per thread: enough threads to keep the memory busy
    if (N <= 8) TYR_SS(step, 4, 2)
    if (N <= 16) TYR_SS(step, 4, 4)
    if (N <= 32) TYR_SS(step, 4, 8)
    if (N <= 64) TYR_SS(step, 8, 8)
    if (N <= 128) TYR_SS(step, 8, 16)
    TYR_SS(step, 16, 16)
  }
  if (N <= 8) TYR_SS(prompt, 8, 1)
  if (N <= 16) TYR_SS(prompt, 8, 2)
  if (N <= 24) TYR_SS(prompt, 6, 4)
  if (N <= 32) TYR_SS(prompt, 8, 4)
  if (N <= 64) TYR_SS(prompt, 8, 8)
  if (N <= 128) TYR_SS(prompt, 8, 16)
  TYR_SS(prompt, 16, 16)
#undef TYR_SS
}
