// Decode-step attention with the KV append fused in and the sequence position read from device memory, so that a
// whole decode step can be replayed from a CUDA graph.
//
// One new query row per (batch, head); K/V stores [B, Hkv, cap, D] bf16 (plain or ring).  Grid (splits, Hkv, B): a CTA
// owns the G = Hq / Hkv <= 16 query heads of one K/V head over one slice of the retained keys (split-KV, 4 warps, 16 keys
// per warp step).  Both products run on mma.sync m16n8k16 with the operand fragments loaded straight from global
// memory, 16 bytes per lane (see the kernel's comment for the channel / key permutations that make this possible).
// The key at the new position is taken from k_new / v_new rather than from the store, so the append (done by split 0)
// cannot race with readers.  Split partials {m, l, acc} go to a workspace; the last CTA to arrive for a
// (batch, K/V head) combines them (atomic ticket, counter reset for the next launch).
//
// Each row of the batch has its own position.  Retained keys are walked by distance from the new token (a ring store by position
// modulo its capacity), so a window may be smaller than the ring and a penalty r1_h ln(1 + r2_h distance) can be taken off the
// scores (template parameter BIAS).  Key size DK and value size DV may differ.  The softmax denominator may also hold exp(sink_h),
// added once when a row's result is written, and the values may be the keys (one store: its rows are read from memory once).
// The first `keep` positions may stay visible past the window; a ring store then holds them in its first slots and the ring after them.
// Values that were rotated by their positions: the output's channel pairs (m, m + dv / 2) are turned back by the query's angles.
//
// The reference takes the library SDPA over a sliced cache for this step (cc/include/tyr_attention.h:58-130,
// Tyr/Inference/KVCache.lean:41-215).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "common.cuh"

namespace tyr {

constexpr int kDecWarps = 4;

struct DecodeAttnArgs {
  const __nv_bfloat16* q;        // [B, Hq, D], batch stride q_bs, head stride D
  const __nv_bfloat16* k_new;    // [B, Hkv, D], batch stride kn_bs, head stride D
  const __nv_bfloat16* v_new;    // same strides (vn_bs)
  __nv_bfloat16* k_cache;        // [B, Hkv, cap, DK] and [B, Hkv, cap, DV]
  __nv_bfloat16* v_cache;
  const int* pos;                // absolute position of the new token of row b: pos[b * pos_stride]
  int pos_stride;
  const float *r1, *r2;          // [Hq] distance penalty (BIAS forms)
  __nv_bfloat16* out;            // [B, Hq, dv], batch stride out_bs
  float* part_acc;               // [B, Hq, splits, DV]
  float* part_ml;                // [B, Hq, splits, 2]
  int* counters;                 // [B * Hkv], zero on entry, zero on exit
  long long q_bs, kn_bs, vn_bs;
  int B, Hq, Hkv, cap, ring, window, splits, append;
  float scale_log2;
  int* err;
  // optional output gate, applied when the result is written (mode 3: one value per (batch, head), out *= sigmoid(g)): mode 1 = one value per (batch, head), out *= softplus(g)
  // (Laguna); mode 2 = one value per element, out *= sigmoid(g) (Qwen3.5).  Element (b, h, d) is at gate + b * gate_bs +
  // h * gate_hs (+ d in mode 2).
  const __nv_bfloat16* gate;
  long long gate_bs, gate_hs;
  int gate_mode;
  const float* sink;             // [Hq] (nullable)
  long long out_bs;              // batch stride of out
  int dv;                        // channels of a head that are written (heads of out are packed)
  float out_scale;
  int keep;                      // positions 0 .. keep - 1 are visible past the window
  const float2* back;            // [positions, back_half] (cos, sin) of a position's turns (nullable)
  int back_half, back_rows;
};

__device__ __forceinline__ float decode_gate(const DecodeAttnArgs& a, int b, int h, int d) {
  if (a.gate_mode == 1) {
    const float g = __bfloat162float(a.gate[b * a.gate_bs + h * a.gate_hs]);
    return g > 20.f ? g : log1pf(__expf(g));
  }
  if (a.gate_mode >= 2) {
    const float g = __bfloat162float(a.gate[b * a.gate_bs + h * a.gate_hs + (a.gate_mode == 2 ? d : 0)]);
    return 1.f / (1.f + __expf(-g));
  }
  return 1.f;
}

// Channel d of a head: A / L over all keys relative to 2^M, with the sink, the gate and the factor.
__device__ __forceinline__ void decode_write(const DecodeAttnArgs& a, int b, int h, int d, float M, float L, float A) {
  if (d >= a.dv) return;
  if (a.sink != nullptr) {
    const float sk = a.sink[h] * 1.4426950408889634f, m = fmaxf(M, sk), f = exp2f(M - m);
    A *= f;
    L = L * f + exp2f(sk - m);
  }
  a.out[b * a.out_bs + static_cast<long long>(h) * a.dv + d] = __float2bfloat16((L > 0.f ? A / L : 0.f) * decode_gate(a, b, h, d) * a.out_scale);
}

// One m16n8k16 step.  `lo` accumulates the tile's rows 0..7 (query head g of the lane), `hi` rows 8..15 (head g + 8).
// With at most 8 query heads per K/V head the upper rows are padding: their A registers are zero and their accumulators
// scratch, which halves the live registers.
template <bool WIDE>
__device__ __forceinline__ void mma_bf16_16816(float (&lo)[2], float (&hi)[2], uint32_t a_lo0, uint32_t a_lo2, uint32_t a_hi0, uint32_t a_hi2,
                                               uint32_t b0, uint32_t b1) {
  if constexpr (WIDE) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(lo[0]), "+f"(lo[1]), "+f"(hi[0]), "+f"(hi[1])
                 : "r"(a_lo0), "r"(a_hi0), "r"(a_lo2), "r"(a_hi2), "r"(b0), "r"(b1));
  } else {
    float z0 = 0.f, z1 = 0.f;
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(lo[0]), "+f"(lo[1]), "+f"(z0), "+f"(z1)
                 : "r"(a_lo0), "r"(0u), "r"(a_lo2), "r"(0u), "r"(b0), "r"(b1));
  }
}

__device__ __forceinline__ uint32_t prmt(uint32_t a, uint32_t b, uint32_t sel) {
  uint32_t r;
  asm("prmt.b32 %0, %1, %2, %3;" : "=r"(r) : "r"(a), "r"(b), "r"(sel));
  return r;
}

// Channels d and d + back_half of a head, turned back by the angles of position `pos`.
__device__ __forceinline__ void decode_write_turned(const DecodeAttnArgs& a, int b, int h, int d, int pos, float M, float L, float u, float w) {
  const float2 cs = a.back[static_cast<long long>(pos) * a.back_half + d];
  decode_write(a, b, h, d, M, L, u * cs.x + w * cs.y);
  decode_write(a, b, h, d + a.back_half, M, L, w * cs.x - u * cs.y);
}

// The end of both kernels: combine the four warps' states {s_m, s_l, acc} (acc_warp: floats between two warps' accumulators), write the
// result of a single slice, or leave the partial and let the last CTA of this (batch, K/V head) merge all slices.
template <int DV, int GM>
__device__ __forceinline__ void decode_combine(const DecodeAttnArgs& a, int b, int hkv, int split, const float (*s_m)[GM], const float (*s_l)[GM],
                                               const float (*acc)[DV], int acc_warp, int* ticket) {
  const int tid = threadIdx.x, G = a.Hq / a.Hkv;
  // ---- combine the four warps -------------------------------------------------------------------------------
  __syncthreads();
  const int hq0 = hkv * G;
  for (int i = tid; i < G * DV; i += kDecWarps * 32) {
    const int g = i / DV, d = i - g * DV;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < kDecWarps; ++w) M = fmaxf(M, s_m[w][g]);
    float L = 0.f, A = 0.f, A2 = 0.f;
    const bool turned = a.splits == 1 && a.back != nullptr;
    if (turned && d >= a.back_half) continue;
    if (M > -INFINITY) {
#pragma unroll
      for (int w = 0; w < kDecWarps; ++w) {
        const float f = exp2f(s_m[w][g] - M);
        L += s_l[w][g] * f;
        A += acc[w * (acc_warp / DV) + g][d] * f;
        if (turned) A2 += acc[w * (acc_warp / DV) + g][d + a.back_half] * f;
      }
    }
    const long long row = static_cast<long long>(b) * a.Hq + hq0 + g;
    if (turned) {
      decode_write_turned(a, b, hq0 + g, d, a.pos[b * a.pos_stride], M, L, A, A2);
    } else if (a.splits == 1) {
      decode_write(a, b, hq0 + g, d, M, L, A);
    } else {
      a.part_acc[(row * a.splits + split) * DV + d] = A;
      if (d == 0) {
        a.part_ml[(row * a.splits + split) * 2] = M;
        a.part_ml[(row * a.splits + split) * 2 + 1] = L;
      }
    }
  }
  if (a.splits == 1) return;

  // ---- last CTA of this (batch, K/V head) merges the splits ---------------------------------------------------
  __threadfence();
  __syncthreads();
  if (tid == 0) *ticket = atomicAdd(&a.counters[b * a.Hkv + hkv], 1);
  __syncthreads();
  if (*ticket != a.splits - 1) return;
  __threadfence();
  for (int i = tid; i < G * DV; i += kDecWarps * 32) {
    const int g = i / DV, d = i - g * DV;
    const long long row = static_cast<long long>(b) * a.Hq + hq0 + g;
    float M = -INFINITY;
    if (a.back != nullptr && d >= a.back_half) continue;
    for (int sp = 0; sp < a.splits; ++sp) M = fmaxf(M, __ldcg(&a.part_ml[(row * a.splits + sp) * 2]));
    float L = 0.f, A = 0.f, A2 = 0.f;
    if (M > -INFINITY) {
      for (int sp = 0; sp < a.splits; ++sp) {
        const float f = exp2f(__ldcg(&a.part_ml[(row * a.splits + sp) * 2]) - M);
        L += __ldcg(&a.part_ml[(row * a.splits + sp) * 2 + 1]) * f;
        A += __ldcg(&a.part_acc[(row * a.splits + sp) * DV + d]) * f;
        if (a.back != nullptr) A2 += __ldcg(&a.part_acc[(row * a.splits + sp) * DV + d + a.back_half]) * f;
      }
    }
    if (a.back != nullptr) decode_write_turned(a, b, hq0 + g, d, a.pos[b * a.pos_stride], M, L, A, A2);
    else decode_write(a, b, hq0 + g, d, M, L, A);
  }
  if (tid == 0) a.counters[b * a.Hkv + hkv] = 0;
}

// Tensor-core formulation (mma.sync m16n8k16, bf16 in, fp32 accumulate); one warp consumes 16 keys per step.
//   S = Q K^T : M = query heads of the group (<= 8 real rows), N = 8 keys, K = 16 channels.  The reduction over channels
//   is order-free, so lane (g, t) feeds the B fragment straight from one 16-byte load of key row g (channels
//   32j + 8t .. +8) and Q is loaded once with the same addressing.
//   O += P V  : M = heads, N = 8 channels, K = 16 keys.  Lane (g, t) loads 16 bytes (8 channels) of the four key rows
//   {2t, 2t+1, 2t+8, 2t+9}; byte permutes pair the rows per channel.  The channel order of the accumulators is permuted
//   (undone when they are written out): accumulator (c, e, u) of lane (g, t) is channel 64c + 16t + 8u + e of head g.
template <int DK, int DV, bool WIDE, bool BIAS>
__global__ void __launch_bounds__(kDecWarps * 32) decode_attention_kernel(DecodeAttnArgs a) {
  pdl_entry();
  constexpr int NJ = DK / 32;                    // 16-byte chunks per lane of a K (or Q) row
  constexpr int NC = DV / 64;                    // 64-channel blocks of a V row
  constexpr int R = WIDE ? 2 : 1;                // query heads per lane: g, and g + 8 when more than 8 heads share a K/V head
  constexpr int GM = 8 * R;
  __shared__ float s_m[kDecWarps][GM], s_l[kDecWarps][GM];
  __shared__ float s_acc[kDecWarps][GM][DV];
  __shared__ int s_ticket;

  const int split = blockIdx.x, hkv = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int G = a.Hq / a.Hkv;
  const int pos = a.pos[b * a.pos_stride];
  if (pos < 0 || (!a.ring && pos >= a.cap) || (a.back != nullptr && pos >= a.back_rows)) {    // position outside the store or the turns: report, leave the output untouched
    if (tid == 0) report_error(a.err, ERR_BOUNDS, pos);
    return;
  }
  // Key index i of 0 .. n_keys - 1: the first k0 are the kept positions that the window has left behind, in slots of their own; the rest
  // is at distance n_keys - 1 - i from the new token and in slot slot0 + i - k0 (a ring: modulo its length).
  const int ring_len = a.cap - a.keep;
  int start = a.window > 0 && pos + 1 > a.window ? pos + 1 - a.window : 0;
  if (a.ring && pos + 1 - ring_len > start) start = pos + 1 - ring_len;
  const int k0 = min(a.keep, start);
  const int n_keys = k0 + pos + 1 - start;
  const int slot0 = (a.ring && start >= a.keep ? a.keep + (start - a.keep) % ring_len : start) - k0;
  const int slot_new = a.ring && pos >= a.keep ? a.keep + (pos - a.keep) % ring_len : pos;
  auto slot_of = [&](int i) {
    const int sl = slot0 + i;
    return i < k0 ? i : (sl >= a.cap ? sl - ring_len : sl);
  };
  int chunk = (n_keys + a.splits - 1) / a.splits;
  chunk = (chunk + 63) & ~63;
  const int lo = split * chunk;
  int hi = lo + chunk;
  if (hi > n_keys) hi = n_keys;

  const long long kv_row = (static_cast<long long>(b) * a.Hkv + hkv) * a.cap;
  __nv_bfloat16* kc = a.k_cache + kv_row * DK;
  __nv_bfloat16* vc = a.v_cache + kv_row * DV;
  const bool fresh = a.k_new != nullptr;         // otherwise the store already holds the new token
  const __nv_bfloat16* kn = fresh ? a.k_new + b * a.kn_bs + static_cast<long long>(hkv) * DK : nullptr;
  const __nv_bfloat16* vn = fresh ? a.v_new + b * a.vn_bs + static_cast<long long>(hkv) * DV : nullptr;

  if (a.append && split == 0) {                  // fused append; nobody reads this slot from the store in this launch
    for (int i = tid; i < DK / 8; i += kDecWarps * 32)
      reinterpret_cast<uint4*>(kc + static_cast<long long>(slot_new) * DK)[i] = reinterpret_cast<const uint4*>(kn)[i];
    for (int i = tid; i < DV / 8; i += kDecWarps * 32)
      reinterpret_cast<uint4*>(vc + static_cast<long long>(slot_new) * DV)[i] = reinterpret_cast<const uint4*>(vn)[i];
  }
  float r1[R], r2[R];                            // penalty of heads g and g + 8, in log2 units
  if constexpr (BIAS) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int head = g + 8 * r < G ? g + 8 * r : 0;
      r1[r] = a.r1[hkv * G + head];
      r2[r] = a.r2[hkv * G + head];
    }
  }

  uint4 qf[R][NJ];                               // A fragments of heads g (and g + 8); zero rows beyond G
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int head = g + 8 * r;
    const __nv_bfloat16* qrow = a.q + b * a.q_bs + static_cast<long long>(hkv * G + (head < G ? head : 0)) * DK;
#pragma unroll
    for (int j = 0; j < NJ; ++j) qf[r][j] = head < G ? *reinterpret_cast<const uint4*>(qrow + 32 * j + 8 * t) : make_uint4(0u, 0u, 0u, 0u);
  }
  float m[R], l[R];                              // running max (same in the four lanes of a head) and per-lane partial sum
  float o[R][NC][8][2];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    m[r] = -INFINITY;
    l[r] = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int e = 0; e < 8; ++e) o[r][c][e][0] = o[r][c][e][1] = 0.f;
  }

  for (int base = lo + warp * 16; base < hi; base += kDecWarps * 16) {
    // ---- S for 16 keys: key tiles base + [0, 8) and base + [8, 16) ----
    float s[R][2][2];
#pragma unroll
    for (int tile = 0; tile < 2; ++tile) {
      int row = base + 8 * tile + g;
      row = row < hi ? row : hi - 1;             // clamped rows are masked below
      const __nv_bfloat16* krow = (fresh && row == n_keys - 1) ? kn : kc + static_cast<long long>(slot_of(row)) * DK;
      uint4 kf[NJ];
#pragma unroll
      for (int j = 0; j < NJ; ++j) kf[j] = *reinterpret_cast<const uint4*>(krow + 32 * j + 8 * t);
      float c_lo[2] = {0.f, 0.f}, c_hi[2] = {0.f, 0.f};
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        mma_bf16_16816<WIDE>(c_lo, c_hi, qf[0][j].x, qf[0][j].y, qf[R - 1][j].x, qf[R - 1][j].y, kf[j].x, kf[j].y);
        mma_bf16_16816<WIDE>(c_lo, c_hi, qf[0][j].z, qf[0][j].w, qf[R - 1][j].z, qf[R - 1][j].w, kf[j].z, kf[j].w);
      }
      const int key0 = base + 8 * tile + 2 * t;
      s[0][tile][0] = key0 < hi ? c_lo[0] * a.scale_log2 : -INFINITY;
      s[0][tile][1] = key0 + 1 < hi ? c_lo[1] * a.scale_log2 : -INFINITY;
      if constexpr (WIDE) {
        s[1][tile][0] = key0 < hi ? c_hi[0] * a.scale_log2 : -INFINITY;
        s[1][tile][1] = key0 + 1 < hi ? c_hi[1] * a.scale_log2 : -INFINITY;
      }
      if constexpr (BIAS) {
        const float n0 = static_cast<float>(max(n_keys - 1 - key0, 0)), n1 = static_cast<float>(max(n_keys - 2 - key0, 0));
#pragma unroll
        for (int r = 0; r < R; ++r) {
          s[r][tile][0] -= r1[r] * __log2f(1.f + r2[r] * n0);
          s[r][tile][1] -= r1[r] * __log2f(1.f + r2[r] * n1);
        }
      }
    }
    // ---- V rows of this lane's four keys (issued before the softmax arithmetic so the loads overlap it) ----
    const __nv_bfloat16* vrow[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      int row = base + 2 * t + (i & 1) + 8 * (i >> 1);
      row = row < hi ? row : hi - 1;
      vrow[i] = (fresh && row == n_keys - 1) ? vn : vc + static_cast<long long>(slot_of(row)) * DV;
    }
    uint4 vf[NC][4];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int i = 0; i < 4; ++i) vf[c][i] = *reinterpret_cast<const uint4*>(vrow[i] + 64 * c + 8 * g);

    // ---- online softmax per head (its 16 scores live in the four lanes t = 0..3) ----
    uint32_t pa0[R], pa2[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      float mx = fmaxf(fmaxf(s[r][0][0], s[r][0][1]), fmaxf(s[r][1][0], s[r][1][1]));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      const float m_new = fmaxf(m[r], mx);       // finite: key `base` is always in range
      const float alpha = exp2f(m[r] - m_new);
      const float p00 = exp2f(s[r][0][0] - m_new), p01 = exp2f(s[r][0][1] - m_new);
      const float p10 = exp2f(s[r][1][0] - m_new), p11 = exp2f(s[r][1][1] - m_new);
      l[r] = l[r] * alpha + (p00 + p01) + (p10 + p11);
      if (__any_sync(0xffffffffu, m_new > m[r])) {
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
          for (int e = 0; e < 8; ++e) { o[r][c][e][0] *= alpha; o[r][c][e][1] *= alpha; }
      }
      m[r] = m_new;
      pa0[r] = pack_bf16x2(p00, p01);
      pa2[r] = pack_bf16x2(p10, p11);
    }

    // ---- O += P V ----
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const uint32_t v0[4] = {vf[c][0].x, vf[c][0].y, vf[c][0].z, vf[c][0].w};
      const uint32_t v1[4] = {vf[c][1].x, vf[c][1].y, vf[c][1].z, vf[c][1].w};
      const uint32_t v2[4] = {vf[c][2].x, vf[c][2].y, vf[c][2].z, vf[c][2].w};
      const uint32_t v3[4] = {vf[c][3].x, vf[c][3].y, vf[c][3].z, vf[c][3].w};
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const uint32_t sel = (e & 1) ? 0x7632u : 0x5410u;
        mma_bf16_16816<WIDE>(o[0][c][e], o[R - 1][c][e], pa0[0], pa2[0], pa0[R - 1], pa2[R - 1],
                             prmt(v0[e >> 1], v1[e >> 1], sel), prmt(v2[e >> 1], v3[e >> 1], sel));
      }
    }
  }

  // publish this warp's state: heads g (and g + 8), channels as laid out above
#pragma unroll
  for (int r = 0; r < R; ++r) {
    float lr = l[r];
    lr += __shfl_xor_sync(0xffffffffu, lr, 1);
    lr += __shfl_xor_sync(0xffffffffu, lr, 2);
    const int head = g + 8 * r;
    if (head < G) {
      if (t == 0) { s_m[warp][head] = m[r]; s_l[warp][head] = lr; }
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          s_acc[warp][head][64 * c + 16 * t + e] = o[r][c][e][0];
          s_acc[warp][head][64 * c + 16 * t + 8 + e] = o[r][c][e][1];
        }
    }
  }

  decode_combine<DV, GM>(a, b, hkv, split, s_m, s_l, s_acc[0], GM * DV, &s_ticket);
}

// The values are the keys (one store), at most 8 query heads per K/V head.  Every warp brings its 16-key tiles into a ring of its own in
// shared memory with cp.async, several tiles ahead, and takes the operands of both products from there: each row is read from memory
// once, and the bytes in flight do not depend on registers.  Rows of D channels are chunks of 16 bytes at position chunk ^ (row & 7).
constexpr int kRing = 4;

__device__ __forceinline__ void da_cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}

template <int D>
__global__ void __launch_bounds__(kDecWarps * 32, 3) decode_attention_shared_kernel(DecodeAttnArgs a) {
  constexpr int NJ = D / 32, NC = D / 64, GM = 8, CPR = D / 8;      // CPR: 16-byte chunks of a row
  constexpr int kTile = 16 * D * 2;
  extern __shared__ __align__(128) uint8_t da_ring[];
  __shared__ float s_m[kDecWarps][GM], s_l[kDecWarps][GM];
  __shared__ int s_ticket;
  const int split = blockIdx.x, hkv = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int G = a.Hq / a.Hkv;
  uint8_t* const ring = da_ring + warp * kRing * kTile;
  const uint32_t ring_u = smem_u32(ring);
  pdl_entry();
  const int pos = a.pos[b * a.pos_stride];
  if (pos < 0 || pos >= a.cap) {                 // position outside the store: report, leave the output untouched
    if (tid == 0) report_error(a.err, ERR_BOUNDS, pos);
    return;
  }
  const int n_keys = pos + 1;
  int chunk = (n_keys + a.splits - 1) / a.splits;
  chunk = (chunk + 63) & ~63;
  const int lo = split * chunk, hi = min(lo + chunk, n_keys);
  __nv_bfloat16* kc = a.k_cache + (static_cast<long long>(b) * a.Hkv + hkv) * a.cap * D;
  const __nv_bfloat16* kn = a.k_new + b * a.kn_bs + static_cast<long long>(hkv) * D;
  const int first = lo + warp * 16;
  auto fetch = [&](int base, int stage) {        // 16 rows, a row's chunks by adjacent lanes
    if (base < hi) {
#pragma unroll
      for (int i = 0; i < 16 * CPR / 32; ++i) {
        const int x = lane + 32 * i, r = x / CPR, c = x % CPR;
        const int row = min(base + r, hi - 1);   // clamped rows are masked below
        const __nv_bfloat16* src = row == n_keys - 1 ? kn : kc + static_cast<long long>(row) * D;
        da_cp_async16(ring_u + stage * kTile + (r * CPR + (c ^ (r & 7))) * 16, src + c * 8);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < kRing - 1; ++i) fetch(first + i * kDecWarps * 16, i);
  if (a.append && split == 0)                    // fused append; nobody reads this slot from the store in this launch
    for (int i = tid; i < CPR; i += kDecWarps * 32) reinterpret_cast<uint4*>(kc + static_cast<long long>(pos) * D)[i] = reinterpret_cast<const uint4*>(kn)[i];
  uint4 qf[NJ];                                  // A fragments of head g; zero rows beyond G
  {
    const __nv_bfloat16* qrow = a.q + b * a.q_bs + static_cast<long long>(hkv * G + (g < G ? g : 0)) * D;
#pragma unroll
    for (int j = 0; j < NJ; ++j) qf[j] = g < G ? *reinterpret_cast<const uint4*>(qrow + 32 * j + 8 * t) : make_uint4(0u, 0u, 0u, 0u);
  }
  float m = -INFINITY, l = 0.f, o[NC][8][2];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int e = 0; e < 8; ++e) o[c][e][0] = o[c][e][1] = 0.f;
  int stage = 0;
#pragma unroll 1
  for (int base = first; base < hi; base += kDecWarps * 16) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kRing - 2) : "memory");
    __syncwarp();                                // every lane's part of the tile has landed, and the stage fetched next is free
    fetch(base + (kRing - 1) * kDecWarps * 16, stage == 0 ? kRing - 1 : stage - 1);
    const uint8_t* kt = ring + stage * kTile;
    stage = stage + 1 == kRing ? 0 : stage + 1;
    auto chunk_at = [&](int r, int c) { return *reinterpret_cast<const uint4*>(kt + (r * CPR + (c ^ (r & 7))) * 16); };
    float s[2][2], none[2] = {0.f, 0.f};
#pragma unroll
    for (int tile = 0; tile < 2; ++tile) {
      float c_lo[2] = {0.f, 0.f};
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const uint4 kf = chunk_at(8 * tile + g, 4 * j + t);
        mma_bf16_16816<false>(c_lo, none, qf[j].x, qf[j].y, 0u, 0u, kf.x, kf.y);
        mma_bf16_16816<false>(c_lo, none, qf[j].z, qf[j].w, 0u, 0u, kf.z, kf.w);
      }
      const int key0 = base + 8 * tile + 2 * t;
      s[tile][0] = key0 < hi ? c_lo[0] * a.scale_log2 : -INFINITY;
      s[tile][1] = key0 + 1 < hi ? c_lo[1] * a.scale_log2 : -INFINITY;
    }
    float mx = fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1]));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    const float m_new = fmaxf(m, mx);            // finite: key `base` is always in range
    const float p00 = exp2f(s[0][0] - m_new), p01 = exp2f(s[0][1] - m_new), p10 = exp2f(s[1][0] - m_new), p11 = exp2f(s[1][1] - m_new);
    if (__any_sync(0xffffffffu, m_new > m)) {
      const float alpha = exp2f(m - m_new);
      l *= alpha;
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int e = 0; e < 8; ++e) { o[c][e][0] *= alpha; o[c][e][1] *= alpha; }
      m = m_new;
    }
    l += (p00 + p01) + (p10 + p11);
    const uint32_t pa0 = pack_bf16x2(p00, p01), pa2 = pack_bf16x2(p10, p11);
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const uint4 q0 = chunk_at(2 * t, 8 * c + g), q1 = chunk_at(2 * t + 1, 8 * c + g), q2 = chunk_at(2 * t + 8, 8 * c + g), q3 = chunk_at(2 * t + 9, 8 * c + g);
      const uint32_t v0[4] = {q0.x, q0.y, q0.z, q0.w}, v1[4] = {q1.x, q1.y, q1.z, q1.w}, v2[4] = {q2.x, q2.y, q2.z, q2.w}, v3[4] = {q3.x, q3.y, q3.z, q3.w};
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const uint32_t sel = (e & 1) ? 0x7632u : 0x5410u;
        mma_bf16_16816<false>(o[c][e], none, pa0, pa2, 0u, 0u, prmt(v0[e >> 1], v1[e >> 1], sel), prmt(v2[e >> 1], v3[e >> 1], sel));
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncwarp();
  // this warp's state: the accumulators go over its own ring
  float* acc = reinterpret_cast<float*>(ring);
  l += __shfl_xor_sync(0xffffffffu, l, 1);
  l += __shfl_xor_sync(0xffffffffu, l, 2);
  if (g < G) {
    if (t == 0) { s_m[warp][g] = m; s_l[warp][g] = l; }
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        acc[g * D + 64 * c + 16 * t + e] = o[c][e][0];
        acc[g * D + 64 * c + 16 * t + 8 + e] = o[c][e][1];
      }
  }
  decode_combine<D, GM>(a, b, hkv, split, s_m, s_l, reinterpret_cast<float(*)[D]>(da_ring), kRing * kTile / 4, &s_ticket);
}

}  // namespace tyr

// Workspace: floats for the split partials followed by the ticket counters.
extern "C" TYR_EXPORT long long tyr_decode_attention_workspace_bytes(int B, int Hq, int Hkv, int D, int splits) {
  return static_cast<long long>(B) * Hq * splits * (D + 2) * 4 + static_cast<long long>(B) * Hkv * 4;
}

static int decode_attention_launch(const void* q, const void* k_new, const void* v_new, void* k_cache, void* v_cache, const void* pos,
                                   int pos_stride, void* out, void* workspace, long long q_bs, long long kn_bs, long long vn_bs, int B,
                                   int Hq, int Hkv, int DK, int DV, int cap, int ring, int window, int splits, int append, float scale,
                                   const void* gate, long long gate_bs, long long gate_hs, int gate_mode, const float* r1,
                                   const float* r2, void* err, void* stream, const float* sink = nullptr, int dv_out = 0,
                                   long long out_bs = 0, float out_scale = 1.f, int keep = 0, const void* back = nullptr, int back_rows = 0) {
  using namespace tyr;
  if (gate_mode < 0 || gate_mode > 3 || (gate_mode != 0 && gate == nullptr)) return -5;
  if (B <= 0 || Hq <= 0 || Hkv <= 0 || Hq % Hkv != 0 || Hq / Hkv > 16 || cap <= 0 || splits < 1 || splits > 64) return -1;
  const bool wide = Hq / Hkv > 8;
  if ((q_bs | kn_bs | vn_bs) & 7) return -3;                       // 16-byte rows
  if ((r1 != nullptr) != (r2 != nullptr)) return -6;
  DecodeAttnArgs a;
  a.q = (const __nv_bfloat16*)q; a.k_new = (const __nv_bfloat16*)k_new; a.v_new = (const __nv_bfloat16*)v_new;
  a.k_cache = (__nv_bfloat16*)k_cache; a.v_cache = (__nv_bfloat16*)v_cache;
  a.pos = (const int*)pos; a.pos_stride = pos_stride; a.r1 = r1; a.r2 = r2; a.out = (__nv_bfloat16*)out;
  a.part_acc = (float*)workspace;
  a.part_ml = a.part_acc + static_cast<long long>(B) * Hq * splits * DV;
  a.counters = (int*)(a.part_ml + static_cast<long long>(B) * Hq * splits * 2);
  a.q_bs = q_bs; a.kn_bs = kn_bs; a.vn_bs = vn_bs;
  a.B = B; a.Hq = Hq; a.Hkv = Hkv; a.cap = cap; a.ring = ring; a.window = window; a.splits = splits; a.append = append;
  a.scale_log2 = scale * 1.4426950408889634f;
  a.err = (int*)err;
  a.gate = (const __nv_bfloat16*)gate; a.gate_bs = gate_bs; a.gate_hs = gate_hs; a.gate_mode = gate == nullptr ? 0 : gate_mode;
  a.sink = sink;
  a.dv = dv_out > 0 ? dv_out : DV;
  a.out_bs = out_bs > 0 ? out_bs : static_cast<long long>(Hq) * DV;
  a.out_scale = out_scale;
  if (keep < 0 || (ring && keep >= cap) || (keep > 0 && r1 != nullptr) || (append && k_new == nullptr) || (k_new == nullptr) != (v_new == nullptr)) return -7;
  a.keep = keep;
  a.back = (const float2*)back;
  a.back_half = a.dv / 2;
  a.back_rows = back_rows;
  if (back != nullptr && (a.dv & 1)) return -8;
  const dim3 grid(splits, Hkv, B);
  const cudaStream_t st = (cudaStream_t)stream;
  const dim3 block(kDecWarps * 32);
  if (k_cache == v_cache && k_new == v_new && DK == DV && (DK == 64 || DK == 128) && !wide && r1 == nullptr && !ring && window == 0 && k_new != nullptr) {
    const size_t smem = static_cast<size_t>(kDecWarps) * kRing * 16 * DK * 2;
    auto kernel = DK == 64 ? decode_attention_shared_kernel<64> : decode_attention_shared_kernel<128>;
    static bool configured[64][2] = {};          // the attribute is per device
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) dev = 0;
    bool& done = configured[dev][DK == 128 ? 1 : 0];
    if (!done) {
      const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return 1000 + (int)e;
      done = true;
    }
    return (int)launch_dependent(kernel, grid, block, smem, st, a);
  }
  const bool bias = r1 != nullptr;
#define TYR_DEC(DK_, DV_, WIDE_, BIAS_)                                  \
  if (DK == DK_ && DV == DV_ && wide == WIDE_ && bias == BIAS_)         \
    return (int)launch_dependent(decode_attention_kernel<DK_, DV_, WIDE_, BIAS_>, grid, block, 0, st, a);
  TYR_DEC(64, 64, false, false) TYR_DEC(64, 64, true, false)
  TYR_DEC(128, 128, false, false) TYR_DEC(128, 128, true, false)
  TYR_DEC(256, 256, false, false)                                  // 16 heads x 256 channels of accumulators do not fit a warp
  TYR_DEC(64, 128, false, false) TYR_DEC(64, 128, true, false)
  TYR_DEC(128, 64, false, false) TYR_DEC(128, 64, true, false)
  TYR_DEC(64, 64, false, true) TYR_DEC(64, 64, true, true)
  TYR_DEC(128, 128, false, true) TYR_DEC(128, 128, true, true)
  TYR_DEC(64, 128, false, true) TYR_DEC(64, 128, true, true)
  TYR_DEC(128, 64, false, true) TYR_DEC(128, 64, true, true)
#undef TYR_DEC
  return -2;
}

// `workspace` must be zero-filled once after allocation (the kernel leaves the counters at zero).  An output gate can be folded
// into the final write (see DecodeAttnArgs::gate).
extern "C" TYR_EXPORT int tyr_decode_attention_gated(const void* q, const void* k_new, const void* v_new, void* k_cache,
                                                     void* v_cache, const void* pos, void* out, void* workspace, long long q_bs,
                                                     long long kn_bs, long long vn_bs, int B, int Hq, int Hkv, int D, int cap,
                                                     int ring, int window, int splits, int append, float scale, const void* gate,
                                                     long long gate_bs, long long gate_hs, int gate_mode, void* err, void* stream) {
  return decode_attention_launch(q, k_new, v_new, k_cache, v_cache, pos, 0, out, workspace, q_bs, kn_bs, vn_bs, B, Hq, Hkv, D, D, cap,
                                 ring, window, splits, append, scale, gate, gate_bs, gate_hs, gate_mode, nullptr, nullptr, err, stream);
}

extern "C" TYR_EXPORT int tyr_decode_attention(const void* q, const void* k_new, const void* v_new, void* k_cache, void* v_cache,
                                               const void* pos, void* out, void* workspace, long long q_bs, long long kn_bs,
                                               long long vn_bs, int B, int Hq, int Hkv, int D, int cap, int ring, int window,
                                               int splits, int append, float scale, void* err, void* stream) {
  return tyr_decode_attention_gated(q, k_new, v_new, k_cache, v_cache, pos, out, workspace, q_bs, kn_bs, vn_bs, B, Hq, Hkv, D, cap,
                                    ring, window, splits, append, scale, nullptr, 0, 0, 0, err, stream);
}

// Distance penalty r1[h] ln(1 + r2[h] n) on the scores; own position per row (pos_stride 1) or one for all (0); DK, DV in {64, 128}.
extern "C" TYR_EXPORT int tyr_decode_attention_biased(const void* q, const void* k_new, const void* v_new, void* k_cache,
                                                      void* v_cache, const void* pos, int pos_stride, void* out, void* workspace,
                                                      long long q_bs, long long kn_bs, long long vn_bs, int B, int Hq, int Hkv, int DK,
                                                      int DV, int cap, int ring, int window, int splits, int append, float scale,
                                                      const float* r1, const float* r2, void* err, void* stream) {
  if (r1 == nullptr || r2 == nullptr) return -6;
  return decode_attention_launch(q, k_new, v_new, k_cache, v_cache, pos, pos_stride, out, workspace, q_bs, kn_bs, vn_bs, B, Hq, Hkv, DK,
                                 DV, cap, ring, window, splits, append, scale, nullptr, 0, 0, 0, r1, r2, err, stream);
}

// Sink per head (nullable), output gate out_scale * sigmoid(gate) (gate nullable: [B, Hq, dv] packed heads, batch stride gate_bs), own position
// per row (pos_stride 1) or one for all (0); stores of D in {64, 128} channels, of which dv are written to out [B, Hq, dv] (batch
// stride out_bs).  v_new / v_cache may be k_new / k_cache.
extern "C" TYR_EXPORT int tyr_decode_attention_sink(const void* q, const void* k_new, const void* v_new, void* k_cache, void* v_cache,
                                                    const void* pos, void* out, void* workspace, long long q_bs, long long kn_bs,
                                                    long long vn_bs, int B, int Hq, int Hkv, int D, int dv, int cap, int splits, int append,
                                                    int pos_stride, float scale, const float* sink, const void* gate, long long gate_bs,
                                                    long long out_bs, float out_scale, void* err, void* stream) {
  if (dv <= 0 || dv > D || (D != 64 && D != 128)) return -2;
  return decode_attention_launch(q, k_new, v_new, k_cache, v_cache, pos, pos_stride, out, workspace, q_bs, kn_bs, vn_bs, B, Hq, Hkv, D, D, cap, 0, 0,
                                 splits, append, scale, gate, gate_bs, dv, gate == nullptr ? 0 : 2, nullptr, nullptr, err, stream, sink, dv,
                                 out_bs, out_scale);
}

// Window (0: none) that leaves the first `keep` positions visible, in a plain store or one of `keep` slots followed by a ring; output gate
// sigmoid(head_gate[b * gate_bs + h]) (nullable); `back` (nullable): [back_rows, dv / 2] pairs (cos, sin) by which the output's channel pairs
// (m, m + dv / 2) are turned back.  k_new / v_new null: the store holds the new token already.  DK, DV in {64, 128}.
extern "C" TYR_EXPORT int tyr_decode_attention_kept(const void* q, const void* k_new, const void* v_new, void* k_cache, void* v_cache, const void* pos,
                                                    int pos_stride, void* out, void* workspace, long long q_bs, long long kn_bs, long long vn_bs,
                                                    int B, int Hq, int Hkv, int DK, int DV, int dv, int cap, int ring, int window, int keep, int splits,
                                                    int append, float scale, const void* head_gate, long long gate_bs, const void* back,
                                                    int back_rows, long long out_bs, void* err, void* stream) {
  if (dv <= 0 || dv > DV) return -2;
  return decode_attention_launch(q, k_new, v_new, k_cache, v_cache, pos, pos_stride, out, workspace, q_bs, kn_bs, vn_bs, B, Hq, Hkv, DK, DV, cap, ring,
                                 window, splits, append, scale, head_gate, gate_bs, 1, head_gate == nullptr ? 0 : 3, nullptr, nullptr, err, stream,
                                 nullptr, dv, out_bs, 1.f, keep, back, back_rows);
}
