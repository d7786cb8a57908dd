// Gated delta rule for any head size and for fp32 as well as bf16 activations: the pieces around the tensor-core chunk form
// and the 128-wide decode tile of delta_rule.cu.
//
//   * conv_silu:     causal depthwise convolution + SiLU with any number of taps, over whole prompts.
//   * conv_gates:    one decode token: convolution window shifted in place, SiLU, and the per-head gates.
//   * gates:         log decay -exp(A_log) softplus(a + dt_bias) and write strength sigmoid(b) for whole prompts.
//   * recurrent:     the recurrence itself, token by token, the state in registers (one token for decode, any number for
//                    prompts; rows of a batch may be shorter than the padded length).  The decay is one number per token and
//                    value head, or (CHANNEL) one per key channel, computed here from its projection together with the write strength.
//   * gated_norm:    o / rms(o) * w * silu(z) or sigmoid(z) per head on the fp32 read-out.
//
// This unit is compiled without fast math: a decay close to 1 is applied thousands of times, and the few-ulp bias of the
// approximate exponential would grow with the sequence.
#include "common.cuh"

namespace tyr {

__device__ __forceinline__ float dg_load(const float* p) { return *p; }
__device__ __forceinline__ float dg_load(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void dg_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void dg_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float dg_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }
__device__ __forceinline__ float dg_log_decay(float a, float dt_bias, float a_log) {
  const float v = a + dt_bias;
  const float sp = fmaxf(v, 0.f) + log1pf(expf(-fabsf(v)));
  return -expf(a_log) * sp;
}

// exp(g) for a log decay g <= 0.  Close to 1 the result is 1 + expm1(g), rounded once: a one-ulp bias of exp itself, applied at
// every token, would add up over the memory of a slowly decaying head.
__device__ __forceinline__ float dg_decay(float g) { return g > -0.5f ? 1.f + expm1f(g) : expf(g); }

// y[b, s, c] = silu(sum_j w[c, j] x[b, s - (K - 1) + j, c]); x rows strided, y contiguous
template <typename T>
__global__ void __launch_bounds__(256) conv_silu_kernel(const T* __restrict__ x, const float* __restrict__ w, T* __restrict__ y,
                                                        long long total, int S, int C, int K, long long x_sb, long long x_ss) {
  pdl_entry();
  for (long long i = blockIdx.x * 256LL + threadIdx.x; i < total; i += gridDim.x * 256LL) {
    const int c = static_cast<int>(i % C);
    const long long bs = i / C;
    const int s = static_cast<int>(bs % S);
    const T* xb = x + (bs / S) * x_sb + c;
    float acc = 0.f;
    for (int j = 0; j < K; ++j) {
      const int t = s - (K - 1) + j;
      if (t >= 0) acc += dg_load(xb + t * x_ss) * w[static_cast<long long>(c) * K + j];
    }
    dg_store(y + i, acc * dg_sigmoid(acc));
  }
}

// One token per row.  conv_state: [B, C, K] last K inputs, shifted in place.  a / b rows strided.
template <typename T>
__global__ void __launch_bounds__(256) conv_gates_kernel(const T* __restrict__ x, const T* __restrict__ b_in, const T* __restrict__ a_in,
                                                         long long ld_x, long long ld_b, long long ld_a, T* __restrict__ conv_state,
                                                         const float* __restrict__ w, const float* __restrict__ dt_bias,
                                                         const float* __restrict__ a_log, T* __restrict__ y, float* __restrict__ g,
                                                         float* __restrict__ beta, int B, int C, int K, int Hv) {
  pdl_entry();
  const long long idx = blockIdx.x * 256LL + threadIdx.x;
  const long long n_conv = static_cast<long long>(B) * C;
  if (idx < n_conv) {
    const int b = static_cast<int>(idx / C), c = static_cast<int>(idx % C);
    T* st = conv_state + idx * K;
    const float* wc = w + static_cast<long long>(c) * K;
    const T x_new = x[b * ld_x + c];
    float acc = 0.f;
    for (int j = 0; j + 1 < K; ++j) {
      const T t = st[j + 1];
      st[j] = t;
      acc += dg_load(&t) * wc[j];
    }
    st[K - 1] = x_new;
    acc += dg_load(&x_new) * wc[K - 1];
    dg_store(y + idx, acc * dg_sigmoid(acc));
  } else if (idx < n_conv + static_cast<long long>(B) * Hv) {
    const long long j = idx - n_conv;
    const int b = static_cast<int>(j / Hv), h = static_cast<int>(j % Hv);
    beta[j] = dg_sigmoid(dg_load(b_in + b * ld_b + h));
    g[j] = dg_log_decay(dg_load(a_in + b * ld_a + h), dt_bias[h], a_log[h]);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) delta_gates_kernel(const T* __restrict__ b_in, const T* __restrict__ a_in, long long ld_b,
                                                          long long ld_a, const float* __restrict__ dt_bias,
                                                          const float* __restrict__ a_log, float* __restrict__ g,
                                                          float* __restrict__ beta, long long rows, int Hv) {
  pdl_entry();
  const long long i = blockIdx.x * 256LL + threadIdx.x;
  if (i >= rows * Hv) return;
  const long long r = i / Hv;
  const int h = static_cast<int>(i % Hv);
  beta[i] = dg_sigmoid(dg_load(b_in + r * ld_b + h));
  g[i] = dg_log_decay(dg_load(a_in + r * ld_a + h), dt_bias[h], a_log[h]);
}

// The recurrence.  A warp owns 8 columns of the [dk, dv] state of one (batch, value head); a lane keeps RPL rows (4 i + rg) of
// one column in registers, so both column sums are finished with two shuffles and no warp waits for another.  The token's q
// and k pass through the warp's own shared-memory row; the next token's loads are issued before this token's arithmetic.
struct RecurrentArgs {
  const void *q, *k, *v;                 // [B, S, H, d] by (batch, token, head) element strides
  const float *g, *beta;                 // [B, S, Hv]
  const void *a_raw, *b_raw;             // CHANNEL: projections of decay [B * S, .] (channel hv * dk + d) and write strength (channel hv)
  const float *dt_bias, *a_log;          // CHANNEL: [Hv * dk], [Hv]
  long long a_ld, b_ld;                  // CHANNEL: row strides
  float* state;                          // [B, Hv, dk, dv], in place
  float* out;                            // [B, S, Hv, dv]
  const int* lens;                       // [B] tokens of each row (nullable: S)
  long long q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh;
  int S, Hk, Hv, dk, dv;
};
constexpr int REC_WARPS = 4;

template <typename T, int RPL, bool CHANNEL>
__global__ void __launch_bounds__(REC_WARPS * 32) gdr_recurrent_kernel(RecurrentArgs a) {
  constexpr int DKM = 4 * RPL;           // largest dk of this instance
  constexpr int EPL = (DKM + 31) / 32;   // q / k elements a lane loads per token
  __shared__ float sk[REC_WARPS][DKM], sq[REC_WARPS][DKM], sd[REC_WARPS][CHANNEL ? DKM : 1];
  const int bh = blockIdx.x, b = bh / a.Hv, hv = bh % a.Hv, hk = hv / (a.Hv / a.Hk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int col = (blockIdx.y * REC_WARPS + warp) * 8 + (lane & 7), rg = lane >> 3;
  const bool col_ok = col < a.dv;
  pdl_entry();
  const int n = a.lens ? min(a.lens[b], a.S) : a.S;
  const T* qp = static_cast<const T*>(a.q) + b * a.q_sb + hk * a.q_sh;
  const T* kp = static_cast<const T*>(a.k) + b * a.k_sb + hk * a.k_sh;
  const T* vp = static_cast<const T*>(a.v) + b * a.v_sb + hv * a.v_sh + col;
  const float* gp = a.g + static_cast<long long>(b) * a.S * a.Hv + hv;
  const float* bp = a.beta + static_cast<long long>(b) * a.S * a.Hv + hv;
  float* op = a.out + (static_cast<long long>(b) * a.S * a.Hv + hv) * a.dv + col;
  float* sp = a.state + static_cast<long long>(bh) * a.dk * a.dv + col;
  float s[RPL];
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = 4 * i + rg;
    s[i] = (col_ok && r < a.dk) ? sp[static_cast<long long>(r) * a.dv] : 0.f;
  }
  const float q_scale = 1.f / sqrtf(static_cast<float>(a.dk));
  const T* ap = static_cast<const T*>(a.a_raw) + static_cast<long long>(b) * a.S * a.a_ld + static_cast<long long>(hv) * a.dk;
  const T* brp = static_cast<const T*>(a.b_raw) + static_cast<long long>(b) * a.S * a.b_ld + hv;
  float bias[CHANNEL ? EPL : 1], a_log = 0.f;
  if constexpr (CHANNEL) {
    a_log = a.a_log[hv];
#pragma unroll
    for (int e = 0; e < EPL; ++e) bias[e] = lane + 32 * e < a.dk ? a.dt_bias[static_cast<long long>(hv) * a.dk + lane + 32 * e] : 0.f;
  }
  float nq[EPL], nk[EPL], na[CHANNEL ? EPL : 1], nv = 0.f, ng = 0.f, nb = 0.f;
  auto fetch = [&](int t) {
#pragma unroll
    for (int e = 0; e < EPL; ++e) {
      const int d = lane + 32 * e;
      nq[e] = d < a.dk ? dg_load(qp + t * a.q_ss + d) : 0.f;
      nk[e] = d < a.dk ? dg_load(kp + t * a.k_ss + d) : 0.f;
      if constexpr (CHANNEL) na[e] = d < a.dk ? dg_load(ap + t * a.a_ld + d) : 0.f;
    }
    nv = col_ok ? dg_load(vp + t * a.v_ss) : 0.f;
    if constexpr (CHANNEL) {
      nb = dg_sigmoid(dg_load(brp + t * a.b_ld));
    } else {
      ng = gp[static_cast<long long>(t) * a.Hv];
      nb = bp[static_cast<long long>(t) * a.Hv];
    }
  };
  if (n > 0) fetch(0);
  for (int t = 0; t < n; ++t) {
    float qs = 0.f, ks = 0.f;
#pragma unroll
    for (int e = 0; e < EPL; ++e) { qs += nq[e] * nq[e]; ks += nk[e] * nk[e]; }
    qs = warp_sum(qs); ks = warp_sum(ks);
    const float qn = q_scale / sqrtf(qs + 1e-6f), kn = 1.f / sqrtf(ks + 1e-6f);
#pragma unroll
    for (int e = 0; e < EPL; ++e) {
      const int d = lane + 32 * e;
      if (d < DKM) { sq[warp][d] = nq[e] * qn; sk[warp][d] = nk[e] * kn; }
      if constexpr (CHANNEL)
        if (d < DKM) sd[warp][d] = dg_decay(dg_log_decay(na[e], bias[e], a_log));
    }
    const float v = nv, decay = CHANNEL ? 1.f : dg_decay(ng), beta = nb;
    __syncwarp();
    if (t + 1 < n) fetch(t + 1);
    float kv = 0.f;
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
      s[i] *= CHANNEL ? sd[warp][4 * i + rg] : decay;
      kv += s[i] * sk[warp][4 * i + rg];
    }
    kv += __shfl_xor_sync(0xffffffffu, kv, 8);
    kv += __shfl_xor_sync(0xffffffffu, kv, 16);
    const float u = beta * (v - kv);
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
      s[i] += sk[warp][4 * i + rg] * u;
      o += s[i] * sq[warp][4 * i + rg];
    }
    o += __shfl_xor_sync(0xffffffffu, o, 8);
    o += __shfl_xor_sync(0xffffffffu, o, 16);
    if (rg == 0 && col_ok) op[static_cast<long long>(t) * a.Hv * a.dv] = o;
    __syncwarp();
  }
  if (rg == 0 && col_ok)
    for (int t = n; t < a.S; ++t) op[static_cast<long long>(t) * a.Hv * a.dv] = 0.f;
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    const int r = 4 * i + rg;
    if (col_ok && r < a.dk) sp[static_cast<long long>(r) * a.dv] = s[i];
  }
}

// the gate of gated_norm: SiLU, or the sigmoid alone (act 1)
__device__ __forceinline__ float dg_gate(float z, int act) { return act == 1 ? dg_sigmoid(z) : z * dg_sigmoid(z); }

// o: fp32 [rows, Hv, dv]; z and y: rows of stride ld_z / ld_y, channel h * dv + d; w: fp32 [dv].  One warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) gated_norm_kernel(const float* __restrict__ o, const T* __restrict__ z, long long ld_z,
                                                         const float* __restrict__ w, T* __restrict__ y, long long ld_y, long long rows,
                                                         int Hv, int dv, float eps, int act) {
  pdl_entry();
  const int lane = threadIdx.x & 31;
  const long long nw = static_cast<long long>(gridDim.x) * 8;
  for (long long i = blockIdx.x * 8LL + (threadIdx.x >> 5); i < rows * Hv; i += nw) {
    const float* op = o + i * dv;
    const T* zp = z + (i / Hv) * ld_z + (i % Hv) * dv;
    T* yp = y + (i / Hv) * ld_y + (i % Hv) * dv;
    if ((dv & 3) == 0 && dv <= 256 && sizeof(T) == 2 && ((ld_z | ld_y) & 3) == 0 && ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(y)) & 7) == 0) {
      float4 v[2];
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int d = 4 * lane + 128 * j;
        v[j] = d < dv ? *reinterpret_cast<const float4*>(op + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
      }
      const float rstd = 1.f / sqrtf(warp_sum(ss) / dv + eps);
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int d = 4 * lane + 128 * j;
        if (d < dv) {
          const uint2 zu = *reinterpret_cast<const uint2*>(reinterpret_cast<const char*>(zp + d));
          const float2 z0 = unpack_bf16x2(zu.x), z1 = unpack_bf16x2(zu.y);
          const float4 wv = *reinterpret_cast<const float4*>(w + d);
          uint2 r;
          r.x = pack_bf16x2(v[j].x * rstd * wv.x * dg_gate(z0.x, act), v[j].y * rstd * wv.y * dg_gate(z0.y, act));
          r.y = pack_bf16x2(v[j].z * rstd * wv.z * dg_gate(z1.x, act), v[j].w * rstd * wv.w * dg_gate(z1.y, act));
          *reinterpret_cast<uint2*>(reinterpret_cast<char*>(yp + d)) = r;
        }
      }
    } else {
      float ss = 0.f;
      for (int d = lane; d < dv; d += 32) ss += op[d] * op[d];
      const float rstd = 1.f / sqrtf(warp_sum(ss) / dv + eps);
      for (int d = lane; d < dv; d += 32) {
        const float zz = dg_load(zp + d);
        dg_store(yp + d, op[d] * rstd * w[d] * dg_gate(zz, act));
      }
    }
  }
}

// The same for wide heads (all of a layer's channels normed together): one CTA per (row, head).
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) gated_norm_wide_kernel(const float* __restrict__ o, const T* __restrict__ z, long long ld_z,
                                                              const float* __restrict__ w, T* __restrict__ y, long long ld_y, int Hv, int dv,
                                                              float eps, int act) {
  __shared__ float red[8];
  pdl_entry();
  const int tid = threadIdx.x;
  const long long i = blockIdx.x;
  const float* op = o + i * dv;
  const T* zp = z + (i / Hv) * ld_z + (i % Hv) * dv;
  T* yp = y + (i / Hv) * ld_y + (i % Hv) * dv;
  constexpr int NV = 4;                  // float4 vectors of a thread kept between the reduction and the write
  float4 v[NV];
  float ss = 0.f;
  if constexpr (VEC) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int d = 4 * (tid + 256 * j);
      v[j] = d < dv ? *reinterpret_cast<const float4*>(op + d) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
  } else {
    for (int d = tid; d < dv; d += 256) ss += op[d] * op[d];
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int k = 0; k < 8; ++k) tot += red[k];
  const float rstd = 1.f / sqrtf(tot / dv + eps);
  if constexpr (VEC) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int d = 4 * (tid + 256 * j);
      if (d >= dv) continue;
      const uint2 zu = *reinterpret_cast<const uint2*>(reinterpret_cast<const char*>(zp + d));
      const float2 z0 = unpack_bf16x2(zu.x), z1 = unpack_bf16x2(zu.y);
      const float4 wv = *reinterpret_cast<const float4*>(w + d);
      uint2 r;
      r.x = pack_bf16x2(v[j].x * rstd * wv.x * dg_gate(z0.x, act), v[j].y * rstd * wv.y * dg_gate(z0.y, act));
      r.y = pack_bf16x2(v[j].z * rstd * wv.z * dg_gate(z1.x, act), v[j].w * rstd * wv.w * dg_gate(z1.y, act));
      *reinterpret_cast<uint2*>(reinterpret_cast<char*>(yp + d)) = r;
    }
  } else {
    for (int d = tid; d < dv; d += 256) dg_store(yp + d, op[d] * rstd * w[d] * dg_gate(dg_load(zp + d), act));
  }
}

}  // namespace tyr

using namespace tyr;

// dtype: 0 = bf16, 1 = fp32 (activations; weights, gates, state and read-out are fp32 in every case)
extern "C" TYR_EXPORT int tyr_conv_silu(const void* x, const float* w, void* y, int B, int S, int C, int K, long long x_sb,
                                        long long x_ss, int dtype, void* stream) {
  if (B <= 0 || S <= 0 || C <= 0 || K <= 0) return -1;
  const long long total = static_cast<long long>(B) * S * C;
  const long long want = (total + 255) / 256;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 64 ? want : 148LL * 64));
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == 1)
    return (int)launch_dependent(conv_silu_kernel<float>, grid, dim3(256), 0, st, (const float*)x, w, (float*)y, total, S, C, K, x_sb, x_ss);
  return (int)launch_dependent(conv_silu_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, (const __nv_bfloat16*)x, w, (__nv_bfloat16*)y, total,
                               S, C, K, x_sb, x_ss);
}

extern "C" TYR_EXPORT int tyr_delta_conv_gates(const void* x, const void* b_in, const void* a_in, long long ld_x, long long ld_b,
                                               long long ld_a, void* conv_state, const float* w, const float* dt_bias,
                                               const float* a_log, void* y, float* g, float* beta, int B, int C, int K, int Hv,
                                               int dtype, void* stream) {
  if (B <= 0 || C <= 0 || K <= 0 || Hv <= 0) return -1;
  const long long n = static_cast<long long>(B) * (C + Hv);
  const dim3 grid(static_cast<unsigned>((n + 255) / 256));
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == 1)
    return (int)launch_dependent(conv_gates_kernel<float>, grid, dim3(256), 0, st, (const float*)x, (const float*)b_in, (const float*)a_in, ld_x,
                                 ld_b, ld_a, (float*)conv_state, w, dt_bias, a_log, (float*)y, g, beta, B, C, K, Hv);
  return (int)launch_dependent(conv_gates_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, (const __nv_bfloat16*)x, (const __nv_bfloat16*)b_in,
                               (const __nv_bfloat16*)a_in, ld_x, ld_b, ld_a, (__nv_bfloat16*)conv_state, w, dt_bias, a_log,
                               (__nv_bfloat16*)y, g, beta, B, C, K, Hv);
}

extern "C" TYR_EXPORT int tyr_delta_gates(const void* b_in, const void* a_in, long long ld_b, long long ld_a, const float* dt_bias,
                                          const float* a_log, float* g, float* beta, long long rows, int Hv, int dtype, void* stream) {
  if (rows <= 0 || Hv <= 0) return -1;
  const dim3 grid(static_cast<unsigned>((rows * Hv + 255) / 256));
  cudaStream_t st = (cudaStream_t)stream;
  if (dtype == 1)
    return (int)launch_dependent(delta_gates_kernel<float>, grid, dim3(256), 0, st, (const float*)b_in, (const float*)a_in, ld_b, ld_a, dt_bias,
                                 a_log, g, beta, rows, Hv);
  return (int)launch_dependent(delta_gates_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, (const __nv_bfloat16*)b_in, (const __nv_bfloat16*)a_in,
                               ld_b, ld_a, dt_bias, a_log, g, beta, rows, Hv);
}

// strides: (batch, token, head) element strides of q, k, v.  dk <= 256.
static int recurrent_launch(RecurrentArgs& a, const long long* strides, int B, int dtype, bool channel, void* stream) {
  if (B <= 0 || a.S <= 0 || a.Hk <= 0 || a.Hv <= 0 || a.Hv % a.Hk || a.dk <= 0 || a.dk > 256 || a.dv <= 0) return -1;
  a.q_sb = strides[0]; a.q_ss = strides[1]; a.q_sh = strides[2];
  a.k_sb = strides[3]; a.k_ss = strides[4]; a.k_sh = strides[5];
  a.v_sb = strides[6]; a.v_ss = strides[7]; a.v_sh = strides[8];
  const int dk = a.dk;
  const dim3 grid(B * a.Hv, (a.dv + 8 * REC_WARPS - 1) / (8 * REC_WARPS)), block(REC_WARPS * 32);
  cudaStream_t st = (cudaStream_t)stream;
#define TYR_REC(T, CH)                                                                                      \
  (dk <= 32 ? launch_dependent(gdr_recurrent_kernel<T, 8, CH>, grid, block, 0, st, a)                       \
            : dk <= 64 ? launch_dependent(gdr_recurrent_kernel<T, 16, CH>, grid, block, 0, st, a)           \
                       : dk <= 128 ? launch_dependent(gdr_recurrent_kernel<T, 32, CH>, grid, block, 0, st, a) \
                                   : launch_dependent(gdr_recurrent_kernel<T, 64, CH>, grid, block, 0, st, a))
  if (channel) return (int)(dtype == 1 ? TYR_REC(float, true) : TYR_REC(__nv_bfloat16, true));
  return (int)(dtype == 1 ? TYR_REC(float, false) : TYR_REC(__nv_bfloat16, false));
#undef TYR_REC
}

extern "C" TYR_EXPORT int tyr_gdr_recurrent(const void* q, const void* k, const void* v, const float* g, const float* beta,
                                            float* state, float* out, const int* lens, const long long* strides, int B, int S,
                                            int Hk, int Hv, int dk, int dv, int dtype, void* stream) {
  RecurrentArgs a{};
  a.q = q; a.k = k; a.v = v; a.g = g; a.beta = beta; a.state = state; a.out = out; a.lens = lens;
  a.S = S; a.Hk = Hk; a.Hv = Hv; a.dk = dk; a.dv = dv;
  return recurrent_launch(a, strides, B, dtype, false, stream);
}

// A decay per key channel: a_raw [B * S, .] (channel hv * dk + d) and b_raw (channel hv) in the activations' type, strides[9] and
// strides[10] their row strides; log decay -exp(a_log[hv]) softplus(a_raw + dt_bias), write strength sigmoid(b_raw).
extern "C" TYR_EXPORT int tyr_gdr_recurrent_channel(const void* q, const void* k, const void* v, const void* a_raw, const void* b_raw,
                                                    const float* dt_bias, const float* a_log, float* state, float* out, const int* lens,
                                                    const long long* strides, int B, int S, int Hk, int Hv, int dk, int dv, int dtype,
                                                    void* stream) {
  RecurrentArgs a{};
  a.q = q; a.k = k; a.v = v; a.a_raw = a_raw; a.b_raw = b_raw; a.dt_bias = dt_bias; a.a_log = a_log;
  a.a_ld = strides[9]; a.b_ld = strides[10];
  a.state = state; a.out = out; a.lens = lens;
  a.S = S; a.Hk = Hk; a.Hv = Hv; a.dk = dk; a.dv = dv;
  return recurrent_launch(a, strides, B, dtype, true, stream);
}

// act: 0 = SiLU gate, 1 = sigmoid gate
extern "C" TYR_EXPORT int tyr_gated_norm(const float* o, const void* z, long long ld_z, const float* w, void* y, long long ld_y, long long rows,
                                         int Hv, int dv, float eps, int act, int dtype, void* stream) {
  if (rows <= 0 || Hv <= 0 || dv <= 0 || act < 0 || act > 1) return -1;
  if ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(w)) & 15) return -2;
  const long long want = (rows * Hv + 7) / 8;
  const dim3 grid(static_cast<unsigned>(want < 148LL * 32 ? want : 148LL * 32));
  cudaStream_t st = (cudaStream_t)stream;
  if (dv > 256) {
    const dim3 wide(static_cast<unsigned>(rows * Hv));
    if (dtype == 1)
      return (int)launch_dependent(gated_norm_wide_kernel<float, false>, wide, dim3(256), 0, st, o, (const float*)z, ld_z, w, (float*)y, ld_y, Hv, dv, eps, act);
    const bool vec = (dv & 3) == 0 && dv <= 4096 && ((ld_z | ld_y) & 3) == 0 && ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(y)) & 7) == 0;
    return (int)(vec ? launch_dependent(gated_norm_wide_kernel<__nv_bfloat16, true>, wide, dim3(256), 0, st, o, (const __nv_bfloat16*)z, ld_z, w,
                                        (__nv_bfloat16*)y, ld_y, Hv, dv, eps, act)
                     : launch_dependent(gated_norm_wide_kernel<__nv_bfloat16, false>, wide, dim3(256), 0, st, o, (const __nv_bfloat16*)z, ld_z, w,
                                        (__nv_bfloat16*)y, ld_y, Hv, dv, eps, act));
  }
  if (dtype == 1)
    return (int)launch_dependent(gated_norm_kernel<float>, grid, dim3(256), 0, st, o, (const float*)z, ld_z, w, (float*)y, ld_y, rows, Hv, dv, eps, act);
  return (int)launch_dependent(gated_norm_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, o, (const __nv_bfloat16*)z, ld_z, w, (__nv_bfloat16*)y, ld_y,
                               rows, Hv, dv, eps, act);
}
