// Linear attention with one decay per head (lightning attention):  S <- decay S + k v^T,  o = S^T q,  state and read-out in fp32.
//
//   * chunk:     bf16 prompts, 64 tokens at a time on the tensor cores:
//                  o_i = decay^(i + 1) S^T q_i + sum_{j <= i} decay^(i - j) (q_i . k_j) v_j,   S <- decay^m S + sum_j decay^(m - 1 - j) k_j v_j^T.
//                The bf16 operands are exact; every fp32 operand (state, decayed products, decayed values) is the sum of three bf16
//                numbers, so that the products are those of fp32 numbers, accumulated in fp32.
//   * step:      one token per row, SiLU inside; bound by one read and one write of the state.
//   * recurrent: any sizes, fp32 or bf16 activations, token by token with the state in shared memory.
//
// The decay comes as a double: fp32 carries it as a sum of two numbers, because a rounding of it would be applied anew at every token
// of a long memory.  Compiled without fast math.
#include "mma_sync.cuh"

namespace tyr {

__device__ __forceinline__ float lt_silu(float v) { return v / (1.f + expf(-v)); }
// SiLU in the activations' own type, as a projection with its activation leaves it
__device__ __forceinline__ float lt_act(const float* p, int silu) { return silu ? lt_silu(*p) : *p; }
__device__ __forceinline__ float lt_act(const __nv_bfloat16* p, int silu) {
  const float v = __bfloat162float(*p);
  return silu ? __bfloat162float(__float2bfloat16(lt_silu(v))) : v;
}

struct LightningArgs {
  const void *q, *k, *v;       // [B, S, H, .] by (batch, token, head) element strides
  const double* decay;         // [H]
  float* state;                // [B, H, dk, dv], in place
  float* out;                  // [B, S, H, dv]
  const int* lens;             // [B] tokens of each row (nullable: S)
  long long q_sb, q_ss, q_sh, k_sb, k_ss, k_sh, v_sb, v_ss, v_sh;
  int S, H, dk, dv, silu;      // silu: q, k and v come before their activation
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
      sq[d] = lt_act(qp + t * a.q_ss + d, a.silu);
      sk[d] = lt_act(kp + t * a.k_ss + d, a.silu);
    }
    const float v = live ? lt_act(vp + t * a.v_ss, a.silu) : 0.f;
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

// ---- prompts in chunks ----------------------------------------------------------------------------------------------
constexpr int LC_C = 64, LC_DK = 128, LC_DV = 64;          // tokens of a chunk, largest key size, value columns of a CTA
constexpr int LC_LDK = LC_DK + 8, LC_LDV = LC_DV + 8;      // padded rows: 8 rows start on 8 different 16-byte banks

struct __align__(16) ChunkSmem {
  __nv_bfloat16 q[2][LC_C * LC_LDK], k[2][LC_C * LC_LDK], v[2][LC_C * LC_LDV];
  __nv_bfloat16 dv[3][LC_C * LC_LDV];                      // decayed values, three terms
  __nv_bfloat16 s[3][LC_DK * LC_LDV];                      // state, three terms
  float pw[LC_C + 4];                                      // powers of the decay, 0 .. LC_C
};

// x and y as sums of three bf16 numbers each, packed in pairs
__device__ __forceinline__ void lc_split(float x, float y, uint32_t (&r)[3]) {
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    r[i] = pack_bf16x2(x, y);
    const float2 h = unpack_bf16x2(r[i]);
    x -= h.x;
    y -= h.y;
  }
}

// One CTA per (64 value columns, row and head).  Read-out: warp w takes 16 tokens (w / 2) and 32 of the columns (w % 2).  State: warp w
// keeps rows [16 w, 16 w + 16) x 64 columns in registers and mirrors them in shared memory for the next chunk's read-out.
__global__ void __launch_bounds__(256, 1) lightning_chunk_kernel(LightningArgs a) {
  extern __shared__ __align__(16) uint8_t lc_smem[];
  ChunkSmem& sm = *reinterpret_cast<ChunkSmem*>(lc_smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int b = blockIdx.y / a.H, h = blockIdx.y % a.H, col0 = blockIdx.x * LC_DV, cols = min(LC_DV, a.dv - col0);
  const int ks = (a.dk + 15) / 16;                         // 16-channel steps of the keys
  for (int i = tid; i < static_cast<int>(sizeof(ChunkSmem) / 16); i += 256) reinterpret_cast<uint4*>(lc_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
  pdl_entry();
  __syncthreads();
  if (tid <= LC_C) sm.pw[tid] = static_cast<float>(pow(a.decay[h], static_cast<double>(tid)));
  const int n = a.lens ? min(a.lens[b], a.S) : a.S, chunks = (n + LC_C - 1) / LC_C;
  const __nv_bfloat16* qp = static_cast<const __nv_bfloat16*>(a.q) + b * a.q_sb + h * a.q_sh;
  const __nv_bfloat16* kp = static_cast<const __nv_bfloat16*>(a.k) + b * a.k_sb + h * a.k_sh;
  const __nv_bfloat16* vp = static_cast<const __nv_bfloat16*>(a.v) + b * a.v_sb + h * a.v_sh + col0;
  float* op = a.out + (static_cast<long long>(b) * a.S * a.H + h) * a.dv + col0;
  auto fetch = [&](int c) {                                // rows past the end are zeros
    if (c < chunks) {
      const int st = c & 1, t0 = c * LC_C, kc = a.dk / 8, vc = cols / 8;
      for (int x = tid; x < LC_C * kc; x += 256) {
        const int r = x / kc, d = (x - r * kc) * 8, tok = min(t0 + r, n - 1);
        cp16_zfill(&sm.q[st][r * LC_LDK + d], qp + tok * a.q_ss + d, t0 + r < n);
        cp16_zfill(&sm.k[st][r * LC_LDK + d], kp + tok * a.k_ss + d, t0 + r < n);
      }
      for (int x = tid; x < LC_C * vc; x += 256) {
        const int r = x / vc, d = (x - r * vc) * 8, tok = min(t0 + r, n - 1);
        cp16_zfill(&sm.v[st][r * LC_LDV + d], vp + tok * a.v_ss + d, t0 + r < n);
      }
    }
    cp_commit();
  };
  fetch(0);
  float S[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
  // a lane's row and column for ldmatrix (csrc/mma_sync.cuh)
  const int lr = lane & 15, lc = (lane >> 4) * 8, br = (lane & 7) + ((lane >> 4) << 3), bc = ((lane >> 3) & 1) * 8;
  const int m0 = (warp >> 1) * 16, n0 = (warp & 1) * 32;
  for (int c = 0; c < chunks; ++c) {
    cp_wait<0>();
    __syncthreads();                                       // this chunk's rows and the state's mirror are there, the other stage is free
    fetch(c + 1);
    const int st = c & 1, m = min(LC_C, n - c * LC_C);
    const __nv_bfloat16 *q = sm.q[st], *k = sm.k[st], *v = sm.v[st];
    for (int x = tid; x < LC_C * LC_DV / 2; x += 256) {    // values times the decay up to the chunk's last token
      const int r = x / (LC_DV / 2), d = (x % (LC_DV / 2)) * 2;
      const float f = r < m ? sm.pw[m - 1 - r] : 0.f;
      const float2 u = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(v + r * LC_LDV + d));
      uint32_t w[3];
      lc_split(u.x * f, u.y * f, w);
#pragma unroll
      for (int i = 0; i < 3; ++i) *reinterpret_cast<uint32_t*>(&sm.dv[i][r * LC_LDV + d]) = w[i];
    }
    // ---- read-out of the state and products of the chunk's own tokens
    float o[4][4], p[8][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) p[i][0] = p[i][1] = p[i][2] = p[i][3] = 0.f;
#pragma unroll 2
    for (int x = 0; x < ks; ++x) {
      uint32_t qa[4];
      ldsm4(qa, q + (m0 + lr) * LC_LDK + x * 16 + lc);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (16 * j > m0) break;                            // later keys are not seen
        uint32_t kb[4];
        ldsm4(kb, k + (16 * j + br) * LC_LDK + x * 16 + bc);
        mma_bf16(p[2 * j], qa, kb[0], kb[1]);
        mma_bf16(p[2 * j + 1], qa, kb[2], kb[3]);
      }
      if (c > 0) {
#pragma unroll
        for (int i = 0; i < 3; ++i)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            uint32_t sb[4];
            ldsm4_t(sb, &sm.s[i][(x * 16 + lr) * LC_LDV + n0 + 16 * j + lc]);
            mma_bf16(o[2 * j], qa, sb[0], sb[1]);
            mma_bf16(o[2 * j + 1], qa, sb[2], sb[3]);
          }
      }
    }
    {
      const float f0 = sm.pw[m0 + g + 1], f1 = sm.pw[m0 + g + 9];
#pragma unroll
      for (int i = 0; i < 4; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (16 * j > m0) break;
      uint32_t pa[3][4];
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int d0 = m0 + g + 8 * r - (16 * j + 8 * e + 2 * t);
          uint32_t w[3];
          lc_split(d0 >= 0 ? p[2 * j + e][2 * r] * sm.pw[d0] : 0.f, d0 >= 1 ? p[2 * j + e][2 * r + 1] * sm.pw[d0 - 1] : 0.f, w);
#pragma unroll
          for (int i = 0; i < 3; ++i) pa[i][2 * e + r] = w[i];
        }
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        uint32_t vb[4];
        ldsm4_t(vb, v + (16 * j + lr) * LC_LDV + n0 + 16 * u + lc);
#pragma unroll
        for (int i = 0; i < 3; ++i) {
          mma_bf16(o[2 * u], pa[i], vb[0], vb[1]);
          mma_bf16(o[2 * u + 1], pa[i], vb[2], vb[3]);
        }
      }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int tok = c * LC_C + m0 + g + 8 * r;
      if (tok < a.S) {
        float* y = op + static_cast<long long>(tok) * a.H * a.dv;
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (n0 + 8 * i < cols) *reinterpret_cast<float2*>(y + n0 + 8 * i + 2 * t) = tok < n ? make_float2(o[i][2 * r], o[i][2 * r + 1]) : make_float2(0.f, 0.f);
      }
    }
    __syncthreads();                                       // decayed values complete, nobody reads the old mirror any more
    // ---- state of this warp's rows
    if (warp < ks) {
      const float f = sm.pw[m];
#pragma unroll
      for (int i = 0; i < 8; ++i) { S[i][0] *= f; S[i][1] *= f; S[i][2] *= f; S[i][3] *= f; }
#pragma unroll 1
      for (int x = 0; x < LC_C / 16; ++x) {
        uint32_t kt[4], ka[4];
        ldsm4_t(kt, k + (x * 16 + lr) * LC_LDK + warp * 16 + lc);      // 16 tokens x 16 channels, transposed: channels are the rows of A
        ka[0] = kt[0]; ka[1] = kt[2]; ka[2] = kt[1]; ka[3] = kt[3];
#pragma unroll
        for (int i = 0; i < 3; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint32_t vb[4];
            ldsm4_t(vb, &sm.dv[i][(x * 16 + lr) * LC_LDV + 16 * j + lc]);
            mma_bf16(S[2 * j], ka, vb[0], vb[1]);
            mma_bf16(S[2 * j + 1], ka, vb[2], vb[3]);
          }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t w[3];
          lc_split(S[i][2 * r], S[i][2 * r + 1], w);
#pragma unroll
          for (int e = 0; e < 3; ++e) *reinterpret_cast<uint32_t*>(&sm.s[e][(warp * 16 + g + 8 * r) * LC_LDV + 8 * i + 2 * t]) = w[e];
        }
    }
  }
  cp_wait<0>();
  const int done = min(a.S, chunks * LC_C);                // rows a chunk wrote; the padding after them is zero
  for (long long x = tid; x < static_cast<long long>(a.S - done) * cols; x += 256) op[(done + x / cols) * a.H * a.dv + x % cols] = 0.f;
  if (warp < ks) {
    float* sp = a.state + static_cast<long long>(blockIdx.y) * a.dk * a.dv + col0;
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int row = warp * 16 + g + 8 * r;
        if (row < a.dk && 8 * i < cols) *reinterpret_cast<float2*>(sp + static_cast<long long>(row) * a.dv + 8 * i + 2 * t) = make_float2(S[i][2 * r], S[i][2 * r + 1]);
      }
  }
}

// ---- one token per row ------------------------------------------------------------------------------------------------
constexpr int LS_COLS = 128, LS_UNROLL = 16;

// One CTA per (128 value columns, row and head): a warp reads every eighth state row as one 512-byte line, a lane owns four columns.
template <typename T>
__global__ void __launch_bounds__(256) lightning_step_kernel(LightningArgs a) {
  extern __shared__ __align__(16) float lt_smem[];
  float* const sk = lt_smem;                      // [dk]
  float* const sq = sk + a.dk;                    // [dk]
  __shared__ __align__(16) float part[8][LS_COLS];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.y / a.H, h = blockIdx.y % a.H, col = blockIdx.x * LS_COLS + lane * 4;
  float* const st = a.state + static_cast<long long>(blockIdx.y) * a.dk * a.dv;
  // the state was last written a step ago: bring it to the L2 while the kernel in front of this one still runs
  pdl_trigger();
  if (gridDim.x == 1 && tid < 8) {
    const long long bytes = static_cast<long long>(a.dk) * a.dv * 4 / 8 & ~15LL;
    if (bytes > 0) bulk_prefetch_l2(reinterpret_cast<const char*>(st) + tid * bytes, static_cast<uint32_t>(bytes));
  }
  pdl_wait();
  const double decay = a.decay[h];
  const float hi = static_cast<float>(decay), lo = static_cast<float>(decay - hi);
  const T* qp = static_cast<const T*>(a.q) + b * a.q_sb + h * a.q_sh;
  const T* kp = static_cast<const T*>(a.k) + b * a.k_sb + h * a.k_sh;
  const T* vp = static_cast<const T*>(a.v) + b * a.v_sb + h * a.v_sh + col;
  const bool live = col < a.dv;
  float4 x[LS_UNROLL];
  auto load = [&](int r0) {
#pragma unroll
    for (int i = 0; i < LS_UNROLL; ++i) {
      const int r = r0 + 8 * i;
      if (live && r < a.dk) x[i] = *reinterpret_cast<const float4*>(st + static_cast<long long>(r) * a.dv + col);
    }
  };
  load(warp);
  for (int d = tid; d < a.dk; d += 256) {
    sq[d] = lt_act(qp + d, a.silu);
    sk[d] = lt_act(kp + d, a.silu);
  }
  float v[4] = {0.f, 0.f, 0.f, 0.f}, o[4] = {0.f, 0.f, 0.f, 0.f};
  if (live)
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = lt_act(vp + e, a.silu);
  __syncthreads();
  for (int r0 = warp; r0 < a.dk; r0 += 8 * LS_UNROLL) {
    if (r0 != warp) load(r0);
    if (live)
#pragma unroll
      for (int i = 0; i < LS_UNROLL; ++i) {
        const int r = r0 + 8 * i;
        if (r >= a.dk) break;
        const float kr = sk[r], qr = sq[r];
        float y[4] = {x[i].x, x[i].y, x[i].z, x[i].w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          y[e] = fmaf(y[e], hi, fmaf(y[e], lo, kr * v[e]));
          o[e] += y[e] * qr;
        }
        *reinterpret_cast<float4*>(st + static_cast<long long>(r) * a.dv + col) = make_float4(y[0], y[1], y[2], y[3]);
      }
  }
  *reinterpret_cast<float4*>(&part[warp][lane * 4]) = make_float4(o[0], o[1], o[2], o[3]);
  __syncthreads();
  const int c = blockIdx.x * LS_COLS + tid;
  if (tid < LS_COLS && c < a.dv) {
    float sum = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) sum += part[w][tid];
    a.out[static_cast<long long>(blockIdx.y) * a.dv + c] = sum;
  }
}

}  // namespace tyr

using namespace tyr;

static LightningArgs lightning_args(const void* q, const void* k, const void* v, const double* decay, float* state, float* out, const int* lens,
                                    const long long* st, int S, int H, int dk, int dv, int silu) {
  return LightningArgs{q, k, v, decay, state, out, lens, st[0], st[1], st[2], st[3], st[4], st[5], st[6], st[7], st[8], S, H, dk, dv, silu};
}

// strides: (batch, token, head) element strides of q, k, v.  dtype: 0 = bf16, 1 = fp32 activations; silu: they come before SiLU.
extern "C" TYR_EXPORT int tyr_lightning_recurrent(const void* q, const void* k, const void* v, const double* decay, float* state, float* out,
                                                  const int* lens, const long long* strides, int B, int S, int H, int dk, int dv, int silu,
                                                  int dtype, void* stream) {
  if (B <= 0 || S <= 0 || H <= 0 || dk <= 0 || dv <= 0) return -1;
  const LightningArgs a = lightning_args(q, k, v, decay, state, out, lens, strides, S, H, dk, dv, silu);
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

// Fresh bf16 prompts, activated: the state starts at zero and is written.  dk (up to 128), dv and all strides multiples of 8, 16-byte
// aligned rows.
extern "C" TYR_EXPORT int tyr_lightning_chunk(const void* q, const void* k, const void* v, const double* decay, float* state, float* out,
                                              const int* lens, const long long* strides, int B, int S, int H, int dk, int dv, void* stream) {
  if (B <= 0 || S <= 0 || H <= 0 || dk <= 0 || dk > LC_DK || dv <= 0 || ((dk | dv) & 7) || static_cast<long long>(B) * H > 65535) return -1;
  for (int i = 0; i < 9; ++i)
    if (strides[i] & 7) return -3;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15) return -3;
  const LightningArgs a = lightning_args(q, k, v, decay, state, out, lens, strides, S, H, dk, dv, 0);
  static bool configured[64] = {};               // the attribute is per device
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
  if (!configured[dev]) {
    const cudaError_t e = cudaFuncSetAttribute(lightning_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(sizeof(ChunkSmem)));
    if (e != cudaSuccess) return 1000 + (int)e;
    configured[dev] = true;
  }
  return (int)launch_dependent(lightning_chunk_kernel, dim3((dv + LC_DV - 1) / LC_DV, B * H), dim3(256), sizeof(ChunkSmem), (cudaStream_t)stream, a);
}

// One token per row (S == 1), dv a multiple of 4; the rest as in tyr_lightning_recurrent.
extern "C" TYR_EXPORT int tyr_lightning_step(const void* q, const void* k, const void* v, const double* decay, float* state, float* out,
                                             const long long* strides, int B, int H, int dk, int dv, int silu, int dtype, void* stream) {
  if (B <= 0 || H <= 0 || dk <= 0 || dk > 4096 || dv <= 0 || (dv & 3) || static_cast<long long>(B) * H > 65535) return -1;
  if ((reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(out)) & 15) return -3;
  const LightningArgs a = lightning_args(q, k, v, decay, state, out, nullptr, strides, 1, H, dk, dv, silu);
  const dim3 grid((dv + LS_COLS - 1) / LS_COLS, B * H);
  const size_t smem = static_cast<size_t>(dk) * 2 * sizeof(float);
  return (int)(dtype == 1 ? launch_dependent(lightning_step_kernel<float>, grid, dim3(256), smem, (cudaStream_t)stream, a)
                          : launch_dependent(lightning_step_kernel<__nv_bfloat16>, grid, dim3(256), smem, (cudaStream_t)stream, a));
}
