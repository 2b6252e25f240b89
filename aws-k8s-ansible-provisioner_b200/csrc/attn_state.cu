// attn_state.cu -- mixers whose memory is a matrix state per head instead of a cache of keys and values: a head keeps
// S [dim][vdim] in fp32, every token updates it and reads it out, and the state of a sequence lives in a slot of the
// engine's sequence table.  The update rules share the kernels (StateGeom.rule):
//
//   STATE_RULE_DECAY   S <- diag(a_t) S + k_t v_t^T;                                  o_t = S^T q_t     (gated linear attention)
//   STATE_RULE_DELTA   S <- diag(a_t) S;  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t     (gated delta rule)
//
//   STATE_RULE_DELTA_HEAD   the same with ONE decay per head, S <- a_t S
//   STATE_RULE_DECAY_HEAD   S <- a_t S + d_t k_t v_t^T;  o_t = S^T q_t + D v_t                          (state-space recurrence, d_t the step size)
//   STATE_RULE_BONUS   o_t = (S + diag(u) k_t v_t^T)^T q_t;  S <- diag(a_t) S + k_t v_t^T               (time mixing with a bonus for the current token)
//
// a_t is a decay per head and key channel (or per head) in (0, 1); it scales the rows of S.  Query/key head of state head a is
// a / (heads / kv_heads).
//
// Everything here is fp32: the state, the decays (formed as exp(-rate * softplus(.)), never as a power of a rounded
// sigmoid), the step sizes, the unit norms, the read-out and its norm.  The inputs are the fp32 sums of the fused
// projection; only the gated read-out handed to the output projection is rounded to the operand type.
//
// A step must leave the same state when it is run twice from the same bookkeeping (the eager warm-up ahead of a graph
// capture): the state of a slot is kept twice, indexed by the parity of the last position it includes.  A portion that
// starts at position p reads copy (p - 1) & 1 (nothing when p == 0: a sequence starts from zero, so a slot that is
// used again needs no clearing) and writes copy (p + n - 1) & 1; a decode step therefore never overwrites what it
// reads.  The convolution keeps its last inputs in a ring of `taps` rows per slot indexed by position mod taps, for the
// same reason.
//
// The scan is sequential in time and parallel over (sequence, head, value column): a CTA owns up to 128 columns of one
// head's state for one portion, eight lanes share four neighbouring columns and split the key channels (channel i * 8 + j
// belongs to lane j), each lane keeps its channels of its columns in registers for the whole portion.  Tokens are staged through shared memory by asynchronous copies, a chunk ahead.  The arithmetic of a token does
// not depend on where the portion was cut, so prefill, chunked prefill and token-by-token decoding give the same bits.
//
// Kernels:
//   lowrank_act        y = act(W2 . lr + bias) for the low-rank second stages (decays, output gates), fp32; lowrank_act_tile: prompt-sized steps
//   conv_unit_finish   delta rule: causal convolution + silu on q | k | v (a thread per channel), then unit vectors and the query scale
//                      (a warp per head), beta
//   conv_unit_rows     the same for prompt-sized steps (a CTA walks down sixteen rows of one head)
//   conv_ring_store    the ring update, after every token of the step has read the ring (a decode step's tokens do it themselves)
//   conv_act           state-space mixer: causal convolution with bias + silu on x | B | C, step sizes and decays
//   state_scan         the recurrence; state_scan_head: the delta rule with one decay per head on packed fp32 pairs
//   state_scan_sum     the state-space and time-mixing rules on packed fp32 pairs
//   state_out_gate     per-head RMS norm of the read-out with a gain, times the gate (silu or given), operand type out
//   gate_part_norm     the read-out times silu(gate), RMS-normed in equal parts, operand type out
#include "kernels.h"

namespace b2 {

namespace {

__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }

typedef unsigned long long f32x2_t;
__device__ __forceinline__ f32x2_t x2_pack(float a, float b) {
  f32x2_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void x2_unpack(f32x2_t v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ f32x2_t x2_fma(f32x2_t a, f32x2_t b, f32x2_t c) {
  f32x2_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2_t x2_mul(f32x2_t a, f32x2_t b) {
  f32x2_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

__device__ __forceinline__ float lowrank_value(float z, int mode, float rate) {
  if (mode == LOWRANK_SIGMOID) return sigmoid_f(z);
  if (mode == LOWRANK_DECAY_SIGMOID_POW) return expf(-rate * softplus_f(-z));   // sigmoid(z)^rate
  if (mode == LOWRANK_DECAY_EXP) return expf(-expf(z));
  return expf(-rate * softplus_f(z));                                           // exp(-exp(A) softplus(z))
}

// A CTA takes LR_TOKENS tokens and NT output channels; a thread owns one channel, reads its row of w2 once (sixteen numbers at a
// time) and applies it to every token of the tile.  lr [T][ld] fp32 (rank numbers per token at column lr_off), staged in shared memory.
constexpr int LR_TOKENS = 8;
template <int NT>
__global__ void __launch_bounds__(NT) lowrank_act_kernel(const float* __restrict__ lr, int ld, int lr_off, int rank, const float* __restrict__ w2,
                                                          const float* __restrict__ bias, const float* __restrict__ rate_log, float rate,
                                                          int per_head, int mode, float* __restrict__ out, int C, int T) {
  extern __shared__ __align__(16) float lrs[];   // [LR_TOKENS][rank]
  pdl_wait();
  pdl_launch_dependents();
  const int t0 = blockIdx.x * LR_TOKENS, tn = min(LR_TOKENS, T - t0);
  for (int i = threadIdx.x; i < tn * rank; i += NT) {
    const float v = lr[(size_t)(t0 + i / rank) * ld + lr_off + i % rank];
    lrs[i] = mode == LOWRANK_DECAY_EXP ? tanhf(v) : v;
  }
  __syncthreads();
  const int c = blockIdx.y * NT + threadIdx.x;
  if (c >= C) return;
  const float* wr = w2 + (size_t)c * rank;
  const bool row16 = (rank & 3) == 0 && (reinterpret_cast<uintptr_t>(w2) & 15) == 0;
  float z[LR_TOKENS];
#pragma unroll
  for (int tt = 0; tt < LR_TOKENS; ++tt) z[tt] = 0.f;
  for (int r0 = 0; r0 < rank; r0 += 16) {
    float w[16];
#pragma unroll
    for (int x = 0; x < 16; x += 4) {
      if (row16) {
        const float4 v = r0 + x < rank ? *reinterpret_cast<const float4*>(wr + r0 + x) : make_float4(0.f, 0.f, 0.f, 0.f);
        w[x] = v.x; w[x + 1] = v.y; w[x + 2] = v.z; w[x + 3] = v.w;
      } else {
#pragma unroll
        for (int y = 0; y < 4; ++y) w[x + y] = r0 + x + y < rank ? wr[r0 + x + y] : 0.f;
      }
    }
#pragma unroll
    for (int tt = 0; tt < LR_TOKENS; ++tt) {
      if (tt < tn) {
        const float* l = lrs + tt * rank + r0;
        if ((rank & 3) == 0) {     // sixteen bytes of the token's low-rank values at a time
#pragma unroll
          for (int x = 0; x < 16; x += 4)
            if (r0 + x < rank) {
              const float4 lv = *reinterpret_cast<const float4*>(l + x);
              z[tt] = fmaf(w[x], lv.x, z[tt]);
              z[tt] = fmaf(w[x + 1], lv.y, z[tt]);
              z[tt] = fmaf(w[x + 2], lv.z, z[tt]);
              z[tt] = fmaf(w[x + 3], lv.w, z[tt]);
            }
        } else {
#pragma unroll
          for (int x = 0; x < 16; ++x)
            if (r0 + x < rank) z[tt] = fmaf(w[x], l[x], z[tt]);
        }
      }
    }
  }
  const float b = bias ? bias[c] : 0.f;
  const float rt = mode == LOWRANK_DECAY_SOFTPLUS ? expf(rate_log[c / per_head]) : rate;
#pragma unroll
  for (int tt = 0; tt < LR_TOKENS; ++tt) {
    if (tt >= tn) break;
    const float zz = z[tt] + b;
    out[(size_t)(t0 + tt) * C + c] = lowrank_value(zz, mode, rt);
  }
}

// Prompt-sized steps: a register-tiled product, 64 tokens x 128 channels at a time, a thread owns eight tokens (packed in pairs) of four channels.  The
// tokens' values are staged once (tanh applied there), then the CTA walks over its share of the channel tiles.  A channel's sum runs over the rank in
// order, as above.
constexpr int LT_T = 64, LT_C = 128, LT_K = 32, LT_MAX_RANK = 128;
__global__ void __launch_bounds__(256) lowrank_act_tile_kernel(const float* __restrict__ lr, int ld, int lr_off, int rank, const float* __restrict__ w2,
                                                               const float* __restrict__ bias, const float* __restrict__ rate_log, float rate, int per_head,
                                                               int mode, float* __restrict__ out, int C, int T, int tiles_per_cta) {
  extern __shared__ __align__(16) float lt_smem[];
  float(*As)[LT_T + 4] = reinterpret_cast<float(*)[LT_T + 4]>(lt_smem);                              // [rank][64 tokens]
  float(*Ws)[LT_C + 4] = reinterpret_cast<float(*)[LT_C + 4]>(lt_smem + (size_t)rank * (LT_T + 4));   // [LT_K][128 channels]
  pdl_wait();
  pdl_launch_dependents();
  const int t0 = blockIdx.x * LT_T, tid = threadIdx.x, tx = tid & 31, ty = tid >> 5;
  for (int i = tid; i < LT_T * rank; i += 256) {   // a warp takes 32 tokens of one column: the stores do not collide
    const int t = i % LT_T, r = i / LT_T;
    float v = t0 + t < T ? lr[(size_t)(t0 + t) * ld + lr_off + r] : 0.f;
    if (mode == LOWRANK_DECAY_EXP) v = tanhf(v);
    As[r][t] = v;
  }
  const bool row16 = (rank & 3) == 0 && (reinterpret_cast<uintptr_t>(w2) & 15) == 0;
  for (int ct = 0; ct < tiles_per_cta; ++ct) {
    const int c0 = (blockIdx.y * tiles_per_cta + ct) * LT_C;
    if (c0 >= C) return;
    f32x2_t acc[4][4];   // [token pair][channel]
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
      for (int b = 0; b < 4; ++b) acc[a][b] = 0ull;
    for (int k0 = 0; k0 < rank; k0 += LT_K) {
      const int kn = min(LT_K, rank - k0);
      __syncthreads();   // As is staged / the slab before this one is used up
      if (row16) {
        for (int i = tid; i < LT_C * (LT_K / 4); i += 256) {
          const int c = i % LT_C, r = (i / LT_C) * 4;
          const float4 v = r < kn && c0 + c < C ? *reinterpret_cast<const float4*>(w2 + (size_t)(c0 + c) * rank + k0 + r) : make_float4(0.f, 0.f, 0.f, 0.f);
          Ws[r][c] = v.x; Ws[r + 1][c] = v.y; Ws[r + 2][c] = v.z; Ws[r + 3][c] = v.w;
        }
      } else {
        for (int i = tid; i < LT_C * LT_K; i += 256) {
          const int c = i % LT_C, r = i / LT_C;
          Ws[r][c] = r < kn && c0 + c < C ? w2[(size_t)(c0 + c) * rank + k0 + r] : 0.f;
        }
      }
      __syncthreads();
#pragma unroll 4
      for (int r = 0; r < kn; ++r) {
        const ulonglong2 a0 = *reinterpret_cast<const ulonglong2*>(&As[k0 + r][ty * 8]), a1 = *reinterpret_cast<const ulonglong2*>(&As[k0 + r][ty * 8 + 4]);
        const float4 w = *reinterpret_cast<const float4*>(&Ws[r][tx * 4]);
        const f32x2_t av[4] = {a0.x, a0.y, a1.x, a1.y}, wv[4] = {x2_pack(w.x, w.x), x2_pack(w.y, w.y), x2_pack(w.z, w.z), x2_pack(w.w, w.w)};
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
          for (int b = 0; b < 4; ++b) acc[a][b] = x2_fma(av[a], wv[b], acc[a][b]);
      }
    }
    const int c = c0 + tx * 4;
    if (c >= C) continue;
    float bs[4], rt[4];
#pragma unroll
    for (int b = 0; b < 4; ++b) {
      const int cc = min(c + b, C - 1);
      bs[b] = bias ? bias[cc] : 0.f;
      rt[b] = mode == LOWRANK_DECAY_SOFTPLUS ? expf(rate_log[cc / per_head]) : rate;
    }
    const bool vec = c + 3 < C && C % 4 == 0;
#pragma unroll
    for (int a = 0; a < 4; ++a) {
      float lo[4], hi[4];
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        x2_unpack(acc[a][b], lo[b], hi[b]);
        lo[b] = lowrank_value(lo[b] + bs[b], mode, rt[b]);
        hi[b] = lowrank_value(hi[b] + bs[b], mode, rt[b]);
      }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = t0 + ty * 8 + 2 * a + h;
        if (t >= T) continue;
        const float* y = h ? hi : lo;
        float* dst = out + (size_t)t * C + c;
        if (vec) {
          *reinterpret_cast<float4*>(dst) = make_float4(y[0], y[1], y[2], y[3]);
        } else {
#pragma unroll
          for (int b = 0; b < 4; ++b)
            if (c + b < C) dst[b] = y[b];
        }
      }
    }
  }
}

// A CTA takes `upc` head units of one token (query heads, key heads, value heads, in the order of the projection's columns): first every
// thread convolves and activates channels of the CTA's range, then a warp per query / key head turns the head into a unit vector.
// proj [T][ld] fp32 = q (kv_heads*dim) | k (kv_heads*dim) | v (heads*vdim) | beta logits (heads) | ...; out [T][C] = the finished q | k | v,
// beta_out [T][heads]; with a_log one decay per head, exp(-exp(a_log) softplus(logit + dt_bias)), from the logits behind beta's.
template <int TAPS>   // 0: any number of taps
__global__ void __launch_bounds__(256) conv_unit_finish_kernel(const float* __restrict__ proj, int ld, StateGeom g, int taps_any,
                                                               const float* __restrict__ conv_w, const float* __restrict__ ring,
                                                               const int32_t* __restrict__ row_seq, const int32_t* __restrict__ row_first,
                                                               const int32_t* __restrict__ positions, const int32_t* __restrict__ slots,
                                                               float unit_eps, float* __restrict__ out, float* __restrict__ beta_out, int upc,
                                                               const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                                               float* __restrict__ decay_out, float* __restrict__ ring_store) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (slots[t] < 0) return;
  const int taps = TAPS > 0 ? TAPS : taps_any;
  const int pos = positions[t];
  const int nqk = g.kv_heads * g.dim, nv = g.heads * g.vdim, C = 2 * nqk + nv;
  const int units = 2 * g.kv_heads + g.heads, u_lo = blockIdx.y * upc, u_hi = min(units, u_lo + upc);
  auto unit_c0 = [&](int u) { return u < 2 * g.kv_heads ? u * g.dim : 2 * nqk + (u - 2 * g.kv_heads) * g.vdim; };
  const int c_lo = unit_c0(u_lo), c_hi = u_hi == units ? C : unit_c0(u_hi);
  const int back = t - row_first[t];
  const float* row = proj + (size_t)t * ld;
  const float* rg = ring + (size_t)row_seq[t] * taps * C;
  float* orow = out + (size_t)t * C;
  for (int c = c_lo + threadIdx.x; c < c_hi; c += 256) {
    float acc = 0.f;
    if constexpr (TAPS > 0) {                 // every load of the channel in flight at once
      float xx[TAPS], ww[TAPS];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int d = TAPS - 1 - j;
        ww[j] = conv_w[(size_t)c * TAPS + j];
        xx[j] = d <= back ? (row - (size_t)d * ld)[c] : (pos - d >= 0 ? rg[(size_t)((pos - d) % TAPS) * C + c] : 0.f);
      }
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(ww[j], xx[j], acc);
    } else {
      for (int j = 0; j < taps; ++j) {        // y_t = sum_j w[c][j] * x_(t - taps + 1 + j), the last column is the current token's
        const int d = taps - 1 - j;
        float xx = 0.f;
        if (d <= back) xx = (row - (size_t)d * ld)[c];
        else if (pos - d >= 0) xx = rg[(size_t)((pos - d) % taps) * C + c];
        acc = fmaf(conv_w[(size_t)c * taps + j], xx, acc);
      }
    }
    orow[c] = silu_f(acc);
    if (ring_store) ring_store[((size_t)row_seq[t] * taps + pos % taps) * C + c] = row[c];   // (a row of the ring that this launch does not read)
  }
  __syncthreads();   // (the CTA reads back only what it wrote itself)
  const float qscale = rsqrtf((float)g.dim);
  for (int u = u_lo + warp; u < min(u_hi, 2 * g.kv_heads); u += 8) {
    float* h = orow + u * g.dim;
    float ss = 0.f;
    for (int i = lane; i < g.dim; i += 32) ss = fmaf(h[i], h[i], ss);
    ss = warp_sum(ss);
    const float r = (1.0f / sqrtf(ss + unit_eps)) * (u < g.kv_heads ? qscale : 1.0f);
    for (int i = lane; i < g.dim; i += 32) h[i] *= r;
  }
  if (blockIdx.y == 0)
    for (int a = threadIdx.x; a < g.heads; a += 256) {
      beta_out[(size_t)t * g.heads + a] = sigmoid_f(row[C + a]);
      if (a_log) decay_out[(size_t)t * g.heads + a] = expf(-expf(a_log[a]) * softplus_f(row[C + g.heads + a] + dt_bias[a]));
    }
}

// Prompt-sized steps: a CTA takes CR_ROWS neighbouring token rows of one head unit (a query, key or value head).  A thread owns channels and walks
// down the rows with the last inputs in registers, so a projected row is read once; query and key heads then pass through shared memory for
// their unit vectors (a warp per row).
constexpr int CR_ROWS = 16;
template <int TAPS>
__global__ void __launch_bounds__(128) conv_unit_rows_kernel(const float* __restrict__ proj, int ld, StateGeom g, const float* __restrict__ conv_w,
                                                             const float* __restrict__ ring, const int32_t* __restrict__ row_seq,
                                                             const int32_t* __restrict__ row_first, const int32_t* __restrict__ positions,
                                                             const int32_t* __restrict__ slots, float unit_eps, float* __restrict__ out,
                                                             float* __restrict__ beta_out, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                                             float* __restrict__ decay_out, int T) {
  extern __shared__ float tile[];   // [CR_ROWS][dim] of a query or key head
  __shared__ int s_first[CR_ROWS], s_pos[CR_ROWS], s_seq[CR_ROWS];
  pdl_wait();
  pdl_launch_dependents();
  const int t0 = blockIdx.x * CR_ROWS, tn = min(CR_ROWS, T - t0), u = blockIdx.y;
  const int nqk = g.kv_heads * g.dim, C = 2 * nqk + g.heads * g.vdim;
  const bool unit = u < 2 * g.kv_heads;
  const int width = unit ? g.dim : g.vdim, ch0 = unit ? u * g.dim : 2 * nqk + (u - 2 * g.kv_heads) * g.vdim;
  if ((int)threadIdx.x < tn) {
    s_first[threadIdx.x] = slots[t0 + threadIdx.x] < 0 ? -1 : row_first[t0 + threadIdx.x];
    s_pos[threadIdx.x] = positions[t0 + threadIdx.x];
    s_seq[threadIdx.x] = row_seq[t0 + threadIdx.x];
  }
  __syncthreads();
  for (int cc = threadIdx.x; cc < width; cc += 128) {
    const int c = ch0 + cc;
    float w[TAPS], hist[TAPS];   // hist[d]: the input d rows back
#pragma unroll
    for (int d = 0; d < TAPS; ++d) w[d] = conv_w[(size_t)c * TAPS + TAPS - 1 - d];
    for (int i = 0; i < tn;) {   // runs of rows of one portion
      const int first = s_first[i], pos = s_pos[i], back = t0 + i - first;
      int e = i + 1;
      while (e < tn && s_first[e] == first) ++e;
#pragma unroll
      for (int d = 1; d < TAPS; ++d)
        hist[d] = first < 0 ? 0.f
                  : d <= back   ? proj[(size_t)(t0 + i - d) * ld + c]
                  : pos - d >= 0 ? ring[((size_t)s_seq[i] * TAPS + (pos - d) % TAPS) * C + c]
                                 : 0.f;
      while (i < e) {   // eight rows' loads in flight at a time
        const int m = min(8, e - i);
        float x[8];
#pragma unroll
        for (int r = 0; r < 8; ++r) x[r] = r < m ? proj[(size_t)(t0 + i + r) * ld + c] : 0.f;
#pragma unroll
        for (int r = 0; r < 8; ++r) {
          if (r < m) {
            float acc = 0.f;
#pragma unroll
            for (int d = TAPS - 1; d >= 1; --d) acc = fmaf(w[d], hist[d], acc);
            acc = fmaf(w[0], x[r], acc);
#pragma unroll
            for (int d = TAPS - 1; d >= 2; --d) hist[d] = hist[d - 1];
            hist[1] = x[r];
            const float y = silu_f(acc);
            if (unit) tile[(i + r) * width + cc] = y;
            else if (first >= 0) out[(size_t)(t0 + i + r) * C + c] = y;
          }
        }
        i += m;
      }
    }
  }
  if (unit) {
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float qscale = u < g.kv_heads ? rsqrtf((float)g.dim) : 1.0f;
    for (int i = warp; i < tn; i += 4) {
      const float* h = tile + i * width;
      float ss = 0.f;
      for (int d = lane; d < width; d += 32) ss = fmaf(h[d], h[d], ss);
      const float r = (1.0f / sqrtf(warp_sum(ss) + unit_eps)) * qscale;
      if (s_first[i] < 0) continue;
      for (int d = lane; d < width; d += 32) out[(size_t)(t0 + i) * C + ch0 + d] = h[d] * r;
    }
  }
  if (u == 0) {
    for (int i = threadIdx.x; i < tn * g.heads; i += 128) {
      const int t = t0 + i / g.heads, a = i % g.heads;
      const float* row = proj + (size_t)t * ld + C;
      beta_out[(size_t)t * g.heads + a] = sigmoid_f(row[a]);
      if (a_log) decay_out[(size_t)t * g.heads + a] = expf(-expf(a_log[a]) * softplus_f(row[g.heads + a] + dt_bias[a]));
    }
  }
}

// A thread owns a channel of x | B | C and walks down `rows` neighbouring token rows with the last inputs in registers (rows = 1 in short steps).  proj
// [T][ld] fp32 = x | B | C | step logits.  The first CTA column also forms the step sizes and decays.
template <int TAPS>   // 0: any number of taps
__global__ void __launch_bounds__(128) conv_act_kernel(const float* __restrict__ proj, int ld, int C, int heads, int taps_any, const float* __restrict__ conv_w,
                                                       const float* __restrict__ conv_b, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                                       const float* __restrict__ ring, float* __restrict__ ring_store, const int32_t* __restrict__ row_seq,
                                                       const int32_t* __restrict__ row_first, const int32_t* __restrict__ positions,
                                                       const int32_t* __restrict__ slots, float* __restrict__ out, float* __restrict__ step,
                                                       float* __restrict__ decay, int rows, int T) {
  const int t0 = blockIdx.x * rows, tn = min(rows, T - t0), c = blockIdx.y * 128 + threadIdx.x;
  const int taps = TAPS > 0 ? TAPS : taps_any;
  float w[TAPS > 0 ? TAPS : 1], bias = 0.f;   // constants of the model: readable before the kernel in front is done
  if (c < C) {
    bias = conv_b[c];
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int d = 0; d < TAPS; ++d) w[d] = conv_w[(size_t)c * TAPS + TAPS - 1 - d];
    }
  }
  pdl_wait();
  pdl_launch_dependents();
  if (c < C) {
    for (int i = 0; i < tn;) {   // runs of rows of one portion
      const int t = t0 + i, first = row_first[t], pos = positions[t], back = t - first;
      const bool live = slots[t] >= 0;
      const float* rg = ring + (size_t)row_seq[t] * taps * C + c;
      int e = i + 1;
      while (e < tn && row_first[t0 + e] == first) ++e;
      if constexpr (TAPS > 0) {
        float hist[TAPS];   // hist[d]: the input d rows back
#pragma unroll
        for (int d = 1; d < TAPS; ++d)
          hist[d] = !live       ? 0.f
                    : d <= back ? proj[(size_t)(t - d) * ld + c]
                    : pos >= d  ? rg[(size_t)((pos - d) % TAPS) * C]
                                : 0.f;
        while (i < e) {   // eight rows' loads in flight at a time
          const int m = min(8, e - i);
          float x[8];
#pragma unroll
          for (int r = 0; r < 8; ++r) x[r] = r < m ? proj[(size_t)(t0 + i + r) * ld + c] : 0.f;
#pragma unroll
          for (int r = 0; r < 8; ++r) {
            if (r < m) {
              float acc = bias;
#pragma unroll
              for (int d = TAPS - 1; d >= 1; --d) acc = fmaf(w[d], hist[d], acc);
              acc = fmaf(w[0], x[r], acc);
#pragma unroll
              for (int d = TAPS - 1; d >= 2; --d) hist[d] = hist[d - 1];
              if (TAPS > 1) hist[TAPS > 1 ? 1 : 0] = x[r];
              if (live) {
                out[(size_t)(t0 + i + r) * C + c] = silu_f(acc);
                if (ring_store) ring_store[((size_t)row_seq[t] * TAPS + pos % TAPS) * C + c] = x[r];   // (steps of single rows: an entry that no row reads)
              }
            }
          }
          i += m;
        }
      } else {
        for (; i < e; ++i) {
          const int tt = t0 + i, pp = positions[tt], bb = tt - first;
          if (!live) continue;
          float acc = bias;
          for (int d = taps - 1; d >= 0; --d) {
            const float xx = d <= bb ? proj[(size_t)(tt - d) * ld + c] : (pp >= d ? rg[(size_t)((pp - d) % taps) * C] : 0.f);
            acc = fmaf(conv_w[(size_t)c * taps + taps - 1 - d], xx, acc);
          }
          out[(size_t)tt * C + c] = silu_f(acc);
          if (ring_store) ring_store[((size_t)row_seq[tt] * taps + pp % taps) * C + c] = proj[(size_t)tt * ld + c];
        }
      }
    }
  }
  if (blockIdx.y == 0)
    for (int i = threadIdx.x; i < tn * heads; i += 128) {
      const int t = t0 + i / heads, a = i % heads;
      const float d = softplus_f(proj[(size_t)t * ld + C + a] + dt_bias[a]);
      step[(size_t)t * heads + a] = d;
      decay[(size_t)t * heads + a] = expf(-expf(a_log[a]) * d);
    }
}

// The same with four neighbouring channels per thread (prompt-sized steps; channels in multiples of four, rows on 16-byte boundaries).
template <int TAPS>
__global__ void __launch_bounds__(128) conv_act4_kernel(const float* __restrict__ proj, int ld, int C, int heads, const float* __restrict__ conv_w,
                                                        const float* __restrict__ conv_b, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                                        const float* __restrict__ ring, const int32_t* __restrict__ row_seq, const int32_t* __restrict__ row_first,
                                                        const int32_t* __restrict__ positions, const int32_t* __restrict__ slots, float* __restrict__ out,
                                                        float* __restrict__ step, float* __restrict__ decay, int rows, int T) {
  const int t0 = blockIdx.x * rows, tn = min(rows, T - t0), c = (blockIdx.y * 128 + threadIdx.x) * 4;
  float4 w[TAPS], bias = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < C) {
    bias = *reinterpret_cast<const float4*>(conv_b + c);
#pragma unroll
    for (int d = 0; d < TAPS; ++d) {
      const int k = TAPS - 1 - d;
      w[d] = make_float4(conv_w[(size_t)c * TAPS + k], conv_w[(size_t)(c + 1) * TAPS + k], conv_w[(size_t)(c + 2) * TAPS + k], conv_w[(size_t)(c + 3) * TAPS + k]);
    }
  }
  pdl_wait();
  pdl_launch_dependents();
  if (c < C) {
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int i = 0; i < tn;) {   // runs of rows of one portion
      const int t = t0 + i, first = row_first[t], pos = positions[t], back = t - first;
      const bool live = slots[t] >= 0;
      const float* rg = ring + (size_t)row_seq[t] * TAPS * C + c;
      int e = i + 1;
      while (e < tn && row_first[t0 + e] == first) ++e;
      float4 hist[TAPS];   // hist[d]: the inputs d rows back
#pragma unroll
      for (int d = 1; d < TAPS; ++d)
        hist[d] = !live       ? zero
                  : d <= back ? *reinterpret_cast<const float4*>(proj + (size_t)(t - d) * ld + c)
                  : pos >= d  ? *reinterpret_cast<const float4*>(rg + (size_t)((pos - d) % TAPS) * C)
                              : zero;
      while (i < e) {   // four rows' loads in flight at a time
        const int m = min(4, e - i);
        float4 x[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) x[r] = r < m ? *reinterpret_cast<const float4*>(proj + (size_t)(t0 + i + r) * ld + c) : zero;
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          if (r < m) {
            float4 acc = bias;
#pragma unroll
            for (int d = TAPS - 1; d >= 1; --d) {
              acc.x = fmaf(w[d].x, hist[d].x, acc.x); acc.y = fmaf(w[d].y, hist[d].y, acc.y);
              acc.z = fmaf(w[d].z, hist[d].z, acc.z); acc.w = fmaf(w[d].w, hist[d].w, acc.w);
            }
            acc.x = fmaf(w[0].x, x[r].x, acc.x); acc.y = fmaf(w[0].y, x[r].y, acc.y);
            acc.z = fmaf(w[0].z, x[r].z, acc.z); acc.w = fmaf(w[0].w, x[r].w, acc.w);
#pragma unroll
            for (int d = TAPS - 1; d >= 2; --d) hist[d] = hist[d - 1];
            if (TAPS > 1) hist[TAPS > 1 ? 1 : 0] = x[r];
            if (live) *reinterpret_cast<float4*>(out + (size_t)(t0 + i + r) * C + c) = make_float4(silu_f(acc.x), silu_f(acc.y), silu_f(acc.z), silu_f(acc.w));
          }
        }
        i += m;
      }
    }
  }
  if (blockIdx.y == 0)
    for (int i = threadIdx.x; i < tn * heads; i += 128) {
      const int t = t0 + i / heads, a = i % heads;
      const float d = softplus_f(proj[(size_t)t * ld + C + a] + dt_bias[a]);
      step[(size_t)t * heads + a] = d;
      decay[(size_t)t * heads + a] = expf(-expf(a_log[a]) * d);
    }
}

__global__ void __launch_bounds__(128) conv_ring_store_kernel(const float* __restrict__ proj, int ld, int C, int taps, float* __restrict__ ring,
                                                              const int32_t* __restrict__ row_seq, const int32_t* __restrict__ row_end,
                                                              const int32_t* __restrict__ positions, const int32_t* __restrict__ slots, int T) {
  pdl_wait();
  pdl_launch_dependents();
  const int mine = blockIdx.x * 32 + (threadIdx.x & 31), at = mine < T ? mine : 0;
  // every warp finds the block's rows to store: the last `taps` of a portion (a later token of the portion owns the others' entries)
  unsigned todo = __ballot_sync(0xffffffffu, mine < T && slots[at] >= 0 && row_end[at] - 1 - mine < taps);
  while (todo) {
    const int t = blockIdx.x * 32 + __ffs(todo) - 1;
    todo &= todo - 1;
    float* dst = ring + ((size_t)row_seq[t] * taps + positions[t] % taps) * C;
    const float* row = proj + (size_t)t * ld;
    for (int c = threadIdx.x; c < C; c += 128) dst[c] = row[c];
  }
}

constexpr int SC_LANES = 8;     // lanes that share a group of state columns and split the key channels
constexpr int SC_CHUNK = 8;     // tokens of one stage (two stages)

__device__ __forceinline__ void cp_async_f32(float* smem_dst, const float* gsrc) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(gsrc) : "memory");
}
__device__ __forceinline__ void cp_async_16(float* smem_dst, const float* gsrc) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(smem_dst)), "l"(gsrc) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// grid (portions, heads, column tiles); block (cols / NC) * 8.  Eight lanes share NC neighbouring columns of the state and split the key
// channels (channel i * 8 + j belongs to lane j; DPT channels per lane, dim <= 8 * DPT), so a value of q, k or the decay read from shared
// memory serves NC columns.  Shared-memory rows hold lane j's channels side by side (at j * (DPT + 4) + i; the pad of four words spreads the
// eight lanes over the banks) and are read sixteen bytes at a time.  Tokens arrive by asynchronous copies, the chunk after the one being
// worked on always in flight.  q is scaled at the read-out (S^T (c q) = c S^T q).
template <int DPT, int NC, int RULE>
__global__ void __launch_bounds__(256) state_scan_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ k, int ldk,
                                                         const float* __restrict__ v, int ldv, const float* __restrict__ decay,
                                                         const float* __restrict__ beta, StateGeom g, float qscale, float* __restrict__ state,
                                                         const int32_t* __restrict__ last_rows, const int32_t* __restrict__ row_seq,
                                                         const int32_t* __restrict__ row_first, const int32_t* __restrict__ row_end,
                                                         const int32_t* __restrict__ positions, const int32_t* __restrict__ slots,
                                                         float* __restrict__ out, int cols) {
  constexpr int LS = DPT + 4;               // words of one lane's channels in a staged row
  constexpr int RS = LS * SC_LANES;         // words of a staged row
  constexpr int CH = DPT >= 32 ? SC_CHUNK / 2 : SC_CHUNK;   // (static shared memory ends at 48 KB)
  constexpr int VW = DPT >= 4 ? 4 : DPT;    // channels per shared-memory load
  constexpr int DP = DPT * SC_LANES;
  constexpr int MAXC = 32 * NC;             // columns of a CTA at most
  constexpr bool HEAD = RULE == STATE_RULE_DELTA_HEAD || RULE == STATE_RULE_DECAY_HEAD;   // one decay per head and token: nothing staged per channel
  constexpr bool BETA = RULE != STATE_RULE_DECAY && RULE != STATE_RULE_BONUS;
  __shared__ __align__(16) float qs[2][CH][RS], ks[2][CH][RS], as[HEAD ? 1 : 2][HEAD ? 1 : CH][HEAD ? 4 : RS];
  __shared__ float ds[2][HEAD ? CH : 1];
  __shared__ __align__(16) float vs[2][CH][MAXC];
  __shared__ float bs[2][CH];
  pdl_wait();
  pdl_launch_dependents();
  const int r_last = last_rows ? last_rows[blockIdx.x] : (int)blockIdx.x;
  const int first = row_first[r_last], end = row_end[r_last];
  if (slots[first] < 0) return;   // padding row of a decode bucket
  const int a = blockIdx.y, kh = a / (g.heads / g.kv_heads);
  const int col0 = blockIdx.z * cols;
  const int grp = threadIdx.x / SC_LANES, j = threadIdx.x % SC_LANES;
  const int cl = grp * NC;                  // first of this thread's columns within the CTA's tile
  const int pos0 = positions[first], n = end - first;
  const int nthreads = blockDim.x;
  const size_t head_floats = (size_t)g.dim * g.vdim;
  float* sbase = state + ((size_t)row_seq[first] * 2 * g.heads) * head_floats;
  const float* s_in = sbase + ((size_t)((pos0 + 1) & 1) * g.heads + a) * head_floats;
  float* s_out = sbase + ((size_t)((pos0 + n - 1) & 1) * g.heads + a) * head_floats;
  // channels past dim and columns past vdim never change: zero keys, queries and values, a decay of one
  for (int i = threadIdx.x; i < 2 * CH * (DP - g.dim); i += nthreads) {
    const int st = i / (CH * (DP - g.dim)), rem = i % (CH * (DP - g.dim)), tt = rem / (DP - g.dim), d = g.dim + rem % (DP - g.dim);
    const int at = (d % SC_LANES) * LS + d / SC_LANES;
    qs[st][tt][at] = 0.f;
    ks[st][tt][at] = 0.f;
    if constexpr (!HEAD) {
      as[st][tt][at] = 1.f;
    }
  }
  const int vcols = min(cols, g.vdim - col0);
  if (vcols < cols)   // (only what no copy ever writes)
    for (int i = threadIdx.x; i < 2 * CH * (cols - vcols); i += nthreads) {
      const int row = i / (cols - vcols), c = vcols + i % (cols - vcols);
      vs[row / CH][row % CH][c] = 0.f;
    }
  __syncthreads();
  // (flat loops over a chunk's numbers keep every thread's copies in flight together; sizes that are powers of two -- the usual case --
  // index by shifts instead of divisions)
  const int dsh = (g.dim & (g.dim - 1)) == 0 ? 31 - __clz(g.dim) : -1, vsh = (vcols & (vcols - 1)) == 0 ? 31 - __clz(vcols) : -1;
  const float* qb = q + (size_t)first * ldq + kh * g.dim;
  const float* kb = k + (size_t)first * ldk + kh * g.dim;
  const float* ab = HEAD ? decay + (size_t)first * g.heads + a : decay + (size_t)first * ((size_t)g.heads * g.dim) + a * g.dim;
  const float* vb = v + (size_t)first * ldv + a * g.vdim + col0;
  const int lda = g.heads * g.dim;
  auto issue = [&](int c0, int st) {
    const int cn = min(CH, n - c0);
    for (int i = threadIdx.x; i < cn * g.dim; i += nthreads) {
      const int tt = dsh >= 0 ? i >> dsh : i / g.dim, d = dsh >= 0 ? i & (g.dim - 1) : i % g.dim, at = (d % SC_LANES) * LS + d / SC_LANES;
      const int row = c0 + tt;
      cp_async_f32(&qs[st][tt][at], qb + (size_t)row * ldq + d);
      cp_async_f32(&ks[st][tt][at], kb + (size_t)row * ldk + d);
      if constexpr (!HEAD) {
        cp_async_f32(&as[st][tt][at], ab + (size_t)row * lda + d);
      }
    }
    for (int i = threadIdx.x; i < cn * vcols; i += nthreads) {
      const int tt = vsh >= 0 ? i >> vsh : i / vcols, c = vsh >= 0 ? i & (vcols - 1) : i % vcols;
      cp_async_f32(&vs[st][tt][c], vb + (size_t)(c0 + tt) * ldv + c);
    }
    if (BETA) {   // (a plain `if`: a discarded loop without braces took the statement behind it along)
      for (int i = threadIdx.x; i < cn; i += nthreads) {
        cp_async_f32(&bs[st][i], beta + (size_t)(first + c0 + i) * g.heads + a);
        if (HEAD) {
          cp_async_f32(&ds[st][HEAD ? i : 0], ab + (size_t)(c0 + i) * g.heads);
        }
      }
    }
  };
  issue(0, 0);
  float s[DPT][NC];
#pragma unroll
  for (int i = 0; i < DPT; ++i) {
    const int d = i * SC_LANES + j;
#pragma unroll
    for (int c = 0; c < NC; ++c) s[i][c] = (pos0 > 0 && d < g.dim && col0 + cl + c < g.vdim) ? s_in[(size_t)d * g.vdim + col0 + cl + c] : 0.f;
  }
  float bonus[RULE == STATE_RULE_BONUS ? DPT : 1];   // this lane's channels
  if constexpr (RULE == STATE_RULE_BONUS) {
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
      const int d = i * SC_LANES + j;
      bonus[i] = d < g.dim ? g.bonus[a * g.dim + d] : 0.f;
    }
  }
  const float skip = RULE == STATE_RULE_DECAY_HEAD ? g.skip[a] : 0.f;
  auto load = [&](const float* p, int i, float* dst) {
    if constexpr (VW == 4) {
      const float4 x = *reinterpret_cast<const float4*>(p + i);
      dst[0] = x.x; dst[1] = x.y; dst[2] = x.z; dst[3] = x.w;
    } else if constexpr (VW == 2) {
      const float2 x = *reinterpret_cast<const float2*>(p + i);
      dst[0] = x.x; dst[1] = x.y;
    } else {
      dst[0] = p[i];
    }
  };
  int st = 0;
  for (int c0 = 0; c0 < n; c0 += CH, st ^= 1) {
    const int cn = min(CH, n - c0);
    cp_async_wait_all();                         // this chunk's copies (the only ones in flight)
    __syncthreads();                             // ... of every thread; and every thread has left the other stage
    if (c0 + CH < n) issue(c0 + CH, st ^ 1);     // the next chunk's copies run beside this chunk's arithmetic
    for (int tt = 0; tt < cn; ++tt) {
      float vc[NC];
      if constexpr (NC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(&vs[st][tt][cl]);
        vc[0] = x.x; vc[1] = x.y; vc[2] = x.z; vc[3] = x.w;
      } else {
#pragma unroll
        for (int c = 0; c < NC; ++c) vc[c] = vs[st][tt][cl + c];
      }
      const float* ap = HEAD ? nullptr : &as[st][tt][j * LS];
      const float* kp = &ks[st][tt][j * LS];
      const float* qp = &qs[st][tt][j * LS];
      float av[VW], kw[VW], qv[VW], acc[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) acc[c] = 0.f;
      if constexpr (RULE == STATE_RULE_DECAY) {
#pragma unroll
        for (int i = 0; i < DPT; i += VW) {
          load(ap, i, av);
          load(kp, i, kw);
          load(qp, i, qv);
#pragma unroll
          for (int x = 0; x < VW; ++x)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              s[i + x][c] = fmaf(av[x], s[i + x][c], kw[x] * vc[c]);
              acc[c] = fmaf(s[i + x][c], qv[x], acc[c]);
            }
        }
      } else if constexpr (RULE == STATE_RULE_DECAY_HEAD) {
        const float gd = ds[st][tt], bt = bs[st][tt];
        float wv[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) wv[c] = bt * vc[c];
#pragma unroll
        for (int i = 0; i < DPT; i += VW) {
          load(kp, i, kw);
          load(qp, i, qv);
#pragma unroll
          for (int x = 0; x < VW; ++x)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              s[i + x][c] = fmaf(kw[x], wv[c], gd * s[i + x][c]);
              acc[c] = fmaf(s[i + x][c], qv[x], acc[c]);
            }
        }
      } else if constexpr (RULE == STATE_RULE_BONUS) {
        float ruk = 0.f;   // sum of q u k over this lane's channels: every column's bonus is that times its v
#pragma unroll
        for (int i = 0; i < DPT; i += VW) {
          load(ap, i, av);
          load(kp, i, kw);
          load(qp, i, qv);
#pragma unroll
          for (int x = 0; x < VW; ++x) {
            ruk = fmaf(qv[x] * bonus[i + x], kw[x], ruk);
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              acc[c] = fmaf(s[i + x][c], qv[x], acc[c]);
              s[i + x][c] = fmaf(av[x], s[i + x][c], kw[x] * vc[c]);
            }
          }
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) acc[c] = fmaf(ruk, vc[c], acc[c]);
      } else if constexpr (HEAD) {
        // S' = g S + k u^T with u = beta (v - g S^T k): the decay is a number, so it leaves the sum over the key channels and joins the update
        const float gd = ds[st][tt], bt = bs[st][tt];
        float kv[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) kv[c] = 0.f;
#pragma unroll
        for (int i = 0; i < DPT; i += VW) {
          load(kp, i, kw);
#pragma unroll
          for (int x = 0; x < VW; ++x)
#pragma unroll
            for (int c = 0; c < NC; ++c) kv[c] = fmaf(s[i + x][c], kw[x], kv[c]);
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          kv[c] += __shfl_xor_sync(0xffffffffu, kv[c], 1);
          kv[c] += __shfl_xor_sync(0xffffffffu, kv[c], 2);
          kv[c] += __shfl_xor_sync(0xffffffffu, kv[c], 4);
          kv[c] = bt * fmaf(-gd, kv[c], vc[c]);     // u
        }
#pragma unroll
        for (int i = 0; i < DPT; i += VW) {
          load(kp, i, kw);
          load(qp, i, qv);
#pragma unroll
          for (int x = 0; x < VW; ++x)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              s[i + x][c] = fmaf(kw[x], kv[c], gd * s[i + x][c]);
              acc[c] = fmaf(s[i + x][c], qv[x], acc[c]);
            }
        }
      } else {
        float kv[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) kv[c] = 0.f;
#pragma unroll
        for (int i = 0; i < DPT; i += VW) {
          load(ap, i, av);
          load(kp, i, kw);
#pragma unroll
          for (int x = 0; x < VW; ++x)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              s[i + x][c] *= av[x];
              kv[c] = fmaf(s[i + x][c], kw[x], kv[c]);
            }
        }
        const float bt = bs[st][tt];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          kv[c] += __shfl_xor_sync(0xffffffffu, kv[c], 1);
          kv[c] += __shfl_xor_sync(0xffffffffu, kv[c], 2);
          kv[c] += __shfl_xor_sync(0xffffffffu, kv[c], 4);
          kv[c] = bt * (vc[c] - kv[c]);     // u
        }
#pragma unroll
        for (int i = 0; i < DPT; i += VW) {
          load(kp, i, kw);
          load(qp, i, qv);
#pragma unroll
          for (int x = 0; x < VW; ++x)
#pragma unroll
            for (int c = 0; c < NC; ++c) {
              s[i + x][c] = fmaf(kw[x], kv[c], s[i + x][c]);
              acc[c] = fmaf(s[i + x][c], qv[x], acc[c]);
            }
        }
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        acc[c] += __shfl_xor_sync(0xffffffffu, acc[c], 1);
        acc[c] += __shfl_xor_sync(0xffffffffu, acc[c], 2);
        acc[c] += __shfl_xor_sync(0xffffffffu, acc[c], 4);
      }
      if (j == 0) {
        float* orow = out + (size_t)(first + c0 + tt) * ((size_t)g.heads * g.vdim) + a * g.vdim + col0 + cl;
#pragma unroll
        for (int c = 0; c < NC; ++c)
          if (col0 + cl + c < g.vdim) orow[c] = RULE == STATE_RULE_DECAY_HEAD ? fmaf(skip, vc[c], acc[c] * qscale) : acc[c] * qscale;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < DPT; ++i) {
    const int d = i * SC_LANES + j;
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (d < g.dim && col0 + cl + c < g.vdim) s_out[(size_t)d * g.vdim + col0 + cl + c] = s[i][c];
  }
}

// ---- the delta rule with one decay per head, packed: the same grid, lanes and staging as state_scan_kernel with NC = 4, the state of a lane held
// as pairs of neighbouring channels so that every multiply-add works on two of them (fma.rn.f32x2, two independent fp32 operations).  The state is
// kept as a factor times a matrix: a decay multiplies the factor only, u enters divided by it, and the matrix takes the factor in (and the factor
// becomes one) before it could run out of range, so a decay of any size down to zero is exact to rounding.  The
// keys of a token stay in registers between the two sums that read them; the read-out's sum over the eight lanes leaves each column with
// one lane pair.
template <int DPT>   // channels per lane: 4, 8 or 16 (dim <= 8 DPT); lane j owns channels 32 m + 4 j + (0..3): rows are staged as they are, 16 bytes a copy
__global__ void __launch_bounds__(256) state_scan_head_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ k, int ldk,
                                                              const float* __restrict__ v, int ldv, const float* __restrict__ decay,
                                                              const float* __restrict__ beta, StateGeom g, float qscale, float* __restrict__ state,
                                                              const int32_t* __restrict__ last_rows, const int32_t* __restrict__ row_seq,
                                                              const int32_t* __restrict__ row_first, const int32_t* __restrict__ row_end,
                                                              const int32_t* __restrict__ positions, const int32_t* __restrict__ slots,
                                                              float* __restrict__ out, int cols) {
  constexpr int NC = 4, CH = SC_CHUNK, DP = DPT * SC_LANES, MAXC = 32 * NC, HP = DPT / 2;
  __shared__ __align__(16) float qs[2][CH][DP], ks[2][CH][DP];
  __shared__ __align__(16) float vs[2][CH][MAXC];
  __shared__ float bs[2][CH], ds[2][CH];
  pdl_wait();
  pdl_launch_dependents();
  const int r_last = last_rows ? last_rows[blockIdx.x] : (int)blockIdx.x;
  const int first = row_first[r_last], end = row_end[r_last];
  if (slots[first] < 0) return;   // padding row of a decode bucket
  const int a = blockIdx.y, kh = a / (g.heads / g.kv_heads);
  const int col0 = blockIdx.z * cols;
  const int grp = threadIdx.x / SC_LANES, j = threadIdx.x % SC_LANES, cl = grp * NC;
  const int pos0 = positions[first], n = end - first;
  const int nthreads = blockDim.x;
  const size_t head_floats = (size_t)g.dim * g.vdim;
  float* sbase = state + ((size_t)row_seq[first] * 2 * g.heads) * head_floats;
  const float* s_in = sbase + ((size_t)((pos0 + 1) & 1) * g.heads + a) * head_floats;
  float* s_out = sbase + ((size_t)((pos0 + n - 1) & 1) * g.heads + a) * head_floats;
  // channels past dim and columns past vdim never change: zero keys, queries and values
  for (int i = threadIdx.x; i < 2 * CH * (DP - g.dim); i += nthreads) {
    const int st = i / (CH * (DP - g.dim)), rem = i % (CH * (DP - g.dim)), tt = rem / (DP - g.dim), d = g.dim + rem % (DP - g.dim);
    qs[st][tt][d] = 0.f;
    ks[st][tt][d] = 0.f;
  }
  const int vcols = min(cols, g.vdim - col0);
  if (vcols < cols) {
    for (int i = threadIdx.x; i < 2 * CH * (cols - vcols); i += nthreads) {
      const int row = i / (cols - vcols), c = vcols + i % (cols - vcols);
      vs[row / CH][row % CH][c] = 0.f;
    }
  }
  __syncthreads();
  const int dq = g.dim >> 2, vq4 = vcols >> 2;   // 16-byte pieces of a row
  const int dsh = (dq & (dq - 1)) == 0 ? 31 - __clz(dq) : -1, vsh = (vq4 & (vq4 - 1)) == 0 ? 31 - __clz(vq4) : -1;
  const float* qb = q + (size_t)first * ldq + kh * g.dim;
  const float* kb = k + (size_t)first * ldk + kh * g.dim;
  const float* vb = v + (size_t)first * ldv + a * g.vdim + col0;
  auto issue = [&](int c0, int st) {
    const int cn = min(CH, n - c0);
    for (int i = threadIdx.x; i < cn * dq; i += nthreads) {
      const int tt = dsh >= 0 ? i >> dsh : i / dq, d = (i - tt * dq) * 4;
      cp_async_16(&qs[st][tt][d], qb + (size_t)(c0 + tt) * ldq + d);
      cp_async_16(&ks[st][tt][d], kb + (size_t)(c0 + tt) * ldk + d);
    }
    for (int i = threadIdx.x; i < cn * vq4; i += nthreads) {
      const int tt = vsh >= 0 ? i >> vsh : i / vq4, c = (i - tt * vq4) * 4;
      cp_async_16(&vs[st][tt][c], vb + (size_t)(c0 + tt) * ldv + c);
    }
    for (int i = threadIdx.x; i < cn; i += nthreads) {
      cp_async_f32(&bs[st][i], beta + (size_t)(first + c0 + i) * g.heads + a);
      cp_async_f32(&ds[st][i], decay + (size_t)(first + c0 + i) * g.heads + a);
    }
  };
  issue(0, 0);
  const bool live = col0 + cl + NC <= g.vdim;   // this group's four columns (vdim is a multiple of four)
  auto channel = [&](int i) { return (i >> 2) * 32 + 4 * j + (i & 3); };
  f32x2_t s[HP][NC];
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    float lo[NC], hi[NC];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = channel(2 * i + x);
      float* dst = x ? hi : lo;
      float4 w = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && pos0 > 0 && d < g.dim) w = *reinterpret_cast<const float4*>(s_in + (size_t)d * g.vdim + col0 + cl);
      dst[0] = w.x; dst[1] = w.y; dst[2] = w.z; dst[3] = w.w;
    }
#pragma unroll
    for (int c = 0; c < NC; ++c) s[i][c] = x2_pack(lo[c], hi[c]);
  }
  float fac = 1.0f;   // the state is fac * s: a decay multiplies one number
  int st = 0;
  for (int c0 = 0; c0 < n; c0 += CH, st ^= 1) {
    const int cn = min(CH, n - c0);
    cp_async_wait_all();                         // this chunk's copies (the only ones in flight)
    __syncthreads();                             // ... of every thread; and every thread has left the other stage
    if (c0 + CH < n) issue(c0 + CH, st ^ 1);     // the next chunk's copies run beside this chunk's arithmetic
    for (int tt = 0; tt < cn; ++tt) {
      const float4 vq = *reinterpret_cast<const float4*>(&vs[st][tt][cl]);
      const float vc[NC] = {vq.x, vq.y, vq.z, vq.w};
      const float bt = bs[st][tt];
      fac *= ds[st][tt];
      if (fac < 1e-12f) {   // (the same in every thread of the CTA)
        const f32x2_t f2 = x2_pack(fac, fac);
#pragma unroll
        for (int i = 0; i < HP; ++i)
#pragma unroll
          for (int c = 0; c < NC; ++c) s[i][c] = x2_mul(f2, s[i][c]);
        fac = 1.0f;
      }
      const float inv = __fdividef(1.0f, fac);   // (1e-12 <= fac <= 1)
      const ulonglong2* kp = reinterpret_cast<const ulonglong2*>(&ks[st][tt][4 * j]);   // (32 channels on: eight pieces of 16 bytes)
      const ulonglong2* qp = reinterpret_cast<const ulonglong2*>(&qs[st][tt][4 * j]);
      f32x2_t kk[HP], sum[NC];
#pragma unroll
      for (int i = 0; i < HP; i += 2) {
        const ulonglong2 w = kp[(i >> 1) * 8];
        kk[i] = w.x;
        kk[i + 1] = w.y;
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) sum[c] = x2_mul(s[0][c], kk[0]);
#pragma unroll
      for (int i = 1; i < HP; ++i)
#pragma unroll
        for (int c = 0; c < NC; ++c) sum[c] = x2_fma(s[i][c], kk[i], sum[c]);
      f32x2_t u2[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        float lo, hi;
        x2_unpack(sum[c], lo, hi);
        float kv = lo + hi;
        kv += __shfl_xor_sync(0xffffffffu, kv, 1);
        kv += __shfl_xor_sync(0xffffffffu, kv, 2);
        kv += __shfl_xor_sync(0xffffffffu, kv, 4);
        const float u = bt * fmaf(vc[c], inv, -kv);   // beta (v - fac S^T k) / fac
        u2[c] = x2_pack(u, u);
      }
#pragma unroll
      for (int i = 0; i < HP; i += 2) {
        const ulonglong2 w = qp[(i >> 1) * 8];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          s[i][c] = x2_fma(kk[i], u2[c], s[i][c]);
          s[i + 1][c] = x2_fma(kk[i + 1], u2[c], s[i + 1][c]);
          sum[c] = i == 0 ? x2_mul(s[0][c], w.x) : x2_fma(s[i][c], w.x, sum[c]);
          sum[c] = x2_fma(s[i + 1][c], w.y, sum[c]);
        }
      }
      // sum over the eight lanes: each exchange halves the columns a lane still holds, then the last two lanes of a column add
      float o[NC];
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        float lo, hi;
        x2_unpack(sum[c], lo, hi);
        o[c] = lo + hi;
      }
      const bool up1 = (j & 1) != 0, up2 = (j & 2) != 0;
      const float a0 = (up1 ? o[2] : o[0]) + __shfl_xor_sync(0xffffffffu, up1 ? o[0] : o[2], 1);
      const float a1 = (up1 ? o[3] : o[1]) + __shfl_xor_sync(0xffffffffu, up1 ? o[1] : o[3], 1);
      float r = (up2 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, up2 ? a0 : a1, 2);
      r += __shfl_xor_sync(0xffffffffu, r, 4);
      const int c = (up1 ? 2 : 0) + (up2 ? 1 : 0);   // the column this lane ended with
      if (j < 4 && live)
        out[(size_t)(first + c0 + tt) * ((size_t)g.heads * g.vdim) + a * g.vdim + col0 + cl + c] = r * (qscale * fac);
    }
  }
  const f32x2_t f2 = x2_pack(fac, fac);
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    float lo[NC], hi[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c) x2_unpack(x2_mul(f2, s[i][c]), lo[c], hi[c]);
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = channel(2 * i + x);
      const float* src = x ? hi : lo;
      if (live && d < g.dim) *reinterpret_cast<float4*>(s_out + (size_t)d * g.vdim + col0 + cl) = make_float4(src[0], src[1], src[2], src[3]);
    }
  }
}

// ---- the rules whose write does not read the state (DECAY_HEAD, BONUS), packed the same way.  DECAY_HEAD: the state is a factor times a matrix, as above.
// BONUS: decays per channel are staged beside the keys; the read-out sees the state before the write, and the bonus of a token is the number
// sum_d q_d u_d k_d times its value.
template <int DPT, int RULE>
__global__ void __launch_bounds__(256) state_scan_sum_kernel(const float* __restrict__ q, int ldq, const float* __restrict__ k, int ldk,
                                                             const float* __restrict__ v, int ldv, const float* __restrict__ decay,
                                                             const float* __restrict__ beta, StateGeom g, float qscale, float* __restrict__ state,
                                                             const int32_t* __restrict__ last_rows, const int32_t* __restrict__ row_seq,
                                                             const int32_t* __restrict__ row_first, const int32_t* __restrict__ row_end,
                                                             const int32_t* __restrict__ positions, const int32_t* __restrict__ slots,
                                                             float* __restrict__ out, int cols) {
  constexpr int NC = 4, CH = SC_CHUNK, DP = DPT * SC_LANES, MAXC = 32 * NC, HP = DPT / 2;
  constexpr bool HEAD = RULE == STATE_RULE_DECAY_HEAD;
  __shared__ __align__(16) float qs[2][CH][DP], ks[2][CH][DP], as[HEAD ? 1 : 2][HEAD ? 1 : CH][HEAD ? 4 : DP];
  __shared__ __align__(16) float vs[2][CH][MAXC];
  __shared__ float bs[2][CH], ds[2][CH];
  pdl_wait();
  pdl_launch_dependents();
  const int r_last = last_rows ? last_rows[blockIdx.x] : (int)blockIdx.x;
  const int first = row_first[r_last], end = row_end[r_last];
  if (slots[first] < 0) return;   // padding row of a decode bucket
  const int a = blockIdx.y, kh = a / (g.heads / g.kv_heads);
  const int col0 = blockIdx.z * cols;
  const int grp = threadIdx.x / SC_LANES, j = threadIdx.x % SC_LANES, cl = grp * NC;
  const int pos0 = positions[first], n = end - first;
  const int nthreads = blockDim.x;
  const size_t head_floats = (size_t)g.dim * g.vdim;
  float* sbase = state + ((size_t)row_seq[first] * 2 * g.heads) * head_floats;
  const float* s_in = sbase + ((size_t)((pos0 + 1) & 1) * g.heads + a) * head_floats;
  float* s_out = sbase + ((size_t)((pos0 + n - 1) & 1) * g.heads + a) * head_floats;
  // channels past dim and columns past vdim never change: zero keys, queries, decays and values
  for (int i = threadIdx.x; i < 2 * CH * (DP - g.dim); i += nthreads) {
    const int st = i / (CH * (DP - g.dim)), rem = i % (CH * (DP - g.dim)), tt = rem / (DP - g.dim), d = g.dim + rem % (DP - g.dim);
    qs[st][tt][d] = 0.f;
    ks[st][tt][d] = 0.f;
    if (!HEAD) {
      as[HEAD ? 0 : st][HEAD ? 0 : tt][HEAD ? 0 : d] = 0.f;
    }
  }
  const int vcols = min(cols, g.vdim - col0);
  if (vcols < cols) {
    for (int i = threadIdx.x; i < 2 * CH * (cols - vcols); i += nthreads) {
      const int row = i / (cols - vcols), c = vcols + i % (cols - vcols);
      vs[row / CH][row % CH][c] = 0.f;
    }
  }
  __syncthreads();
  const int dq = g.dim >> 2, vq4 = vcols >> 2;   // 16-byte pieces of a row
  const int dsh = (dq & (dq - 1)) == 0 ? 31 - __clz(dq) : -1, vsh = (vq4 & (vq4 - 1)) == 0 ? 31 - __clz(vq4) : -1;
  const int lda = g.heads * g.dim;
  const float* qb = q + (size_t)first * ldq + kh * g.dim;
  const float* kb = k + (size_t)first * ldk + kh * g.dim;
  const float* ab = HEAD ? decay : decay + (size_t)first * lda + a * g.dim;
  const float* vb = v + (size_t)first * ldv + a * g.vdim + col0;
  auto issue = [&](int c0, int st) {
    const int cn = min(CH, n - c0);
    for (int i = threadIdx.x; i < cn * dq; i += nthreads) {
      const int tt = dsh >= 0 ? i >> dsh : i / dq, d = (i - tt * dq) * 4;
      cp_async_16(&qs[st][tt][d], qb + (size_t)(c0 + tt) * ldq + d);
      cp_async_16(&ks[st][tt][d], kb + (size_t)(c0 + tt) * ldk + d);
      if (!HEAD) {
        cp_async_16(&as[HEAD ? 0 : st][HEAD ? 0 : tt][HEAD ? 0 : d], ab + (size_t)(c0 + tt) * lda + d);
      }
    }
    for (int i = threadIdx.x; i < cn * vq4; i += nthreads) {
      const int tt = vsh >= 0 ? i >> vsh : i / vq4, c = (i - tt * vq4) * 4;
      cp_async_16(&vs[st][tt][c], vb + (size_t)(c0 + tt) * ldv + c);
    }
    if (HEAD) {
      for (int i = threadIdx.x; i < cn; i += nthreads) {
        cp_async_f32(&bs[st][i], beta + (size_t)(first + c0 + i) * g.heads + a);
        cp_async_f32(&ds[st][i], decay + (size_t)(first + c0 + i) * g.heads + a);
      }
    }
  };
  issue(0, 0);
  const bool live = col0 + cl + NC <= g.vdim;   // this group's four columns (vdim is a multiple of four)
  auto channel = [&](int i) { return (i >> 2) * 32 + 4 * j + (i & 3); };
  f32x2_t s[HP][NC], bonus[HEAD ? 1 : HP];
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    float lo[NC], hi[NC];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = channel(2 * i + x);
      float* dst = x ? hi : lo;
      float4 w = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && pos0 > 0 && d < g.dim) w = *reinterpret_cast<const float4*>(s_in + (size_t)d * g.vdim + col0 + cl);
      dst[0] = w.x; dst[1] = w.y; dst[2] = w.z; dst[3] = w.w;
    }
#pragma unroll
    for (int c = 0; c < NC; ++c) s[i][c] = x2_pack(lo[c], hi[c]);
    if (!HEAD) {
      const int d0 = channel(2 * i), d1 = channel(2 * i + 1);
      bonus[HEAD ? 0 : i] = x2_pack(d0 < g.dim ? g.bonus[a * g.dim + d0] : 0.f, d1 < g.dim ? g.bonus[a * g.dim + d1] : 0.f);
    }
  }
  const float skip = HEAD ? g.skip[a] : 0.f;
  const bool up1 = (j & 1) != 0, up2 = (j & 2) != 0;
  const int ccol = (up1 ? 2 : 0) + (up2 ? 1 : 0);   // the column this lane ends a token with
  const size_t ostep = (size_t)g.heads * g.vdim;
  float* optr = out + (size_t)first * ostep + a * g.vdim + col0 + cl + ccol;
  float fac = 1.0f;
  int st = 0;
  for (int c0 = 0; c0 < n; c0 += CH, st ^= 1) {
    const int cn = min(CH, n - c0);
    cp_async_wait_all();                         // this chunk's copies (the only ones in flight)
    __syncthreads();                             // ... of every thread; and every thread has left the other stage
    if (c0 + CH < n) issue(c0 + CH, st ^ 1);     // the next chunk's copies run beside this chunk's arithmetic
    // one token: wr is the write's factor (DECAY_HEAD), ofac the read-out's
    auto token = [&](int tt, float wr, float ofac) {
      const float4 vq = *reinterpret_cast<const float4*>(&vs[st][tt][cl]);
      const float vc[NC] = {vq.x, vq.y, vq.z, vq.w};
      const ulonglong2* kp = reinterpret_cast<const ulonglong2*>(&ks[st][tt][4 * j]);   // (32 channels on: eight pieces of 16 bytes)
      const ulonglong2* qp = reinterpret_cast<const ulonglong2*>(&qs[st][tt][4 * j]);
      f32x2_t sum[NC], w2[NC];
      float o[NC];
      if constexpr (HEAD) {
#pragma unroll
        for (int c = 0; c < NC; ++c) w2[c] = x2_pack(vc[c] * wr, vc[c] * wr);
#pragma unroll
        for (int i = 0; i < HP; i += 2) {
          const ulonglong2 kw = kp[(i >> 1) * 8], qw = qp[(i >> 1) * 8];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            s[i][c] = x2_fma(kw.x, w2[c], s[i][c]);
            s[i + 1][c] = x2_fma(kw.y, w2[c], s[i + 1][c]);
            sum[c] = i == 0 ? x2_mul(s[0][c], qw.x) : x2_fma(s[i][c], qw.x, sum[c]);
            sum[c] = x2_fma(s[i + 1][c], qw.y, sum[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float lo, hi;
          x2_unpack(sum[c], lo, hi);
          o[c] = lo + hi;
        }
      } else {
        const ulonglong2* ap = reinterpret_cast<const ulonglong2*>(&as[HEAD ? 0 : st][HEAD ? 0 : tt][HEAD ? 0 : 4 * j]);
        f32x2_t ruk = 0ull;
#pragma unroll
        for (int c = 0; c < NC; ++c) w2[c] = x2_pack(vc[c], vc[c]);
#pragma unroll
        for (int i = 0; i < HP; i += 2) {
          const ulonglong2 kw = kp[(i >> 1) * 8], qw = qp[(i >> 1) * 8], aw = ap[(i >> 1) * 8];
          ruk = x2_fma(x2_mul(qw.x, bonus[HEAD ? 0 : i]), kw.x, ruk);
          ruk = x2_fma(x2_mul(qw.y, bonus[HEAD ? 0 : i + 1]), kw.y, ruk);
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            sum[c] = i == 0 ? x2_mul(s[0][c], qw.x) : x2_fma(s[i][c], qw.x, sum[c]);
            sum[c] = x2_fma(s[i + 1][c], qw.y, sum[c]);
            s[i][c] = x2_fma(aw.x, s[i][c], x2_mul(kw.x, w2[c]));
            s[i + 1][c] = x2_fma(aw.y, s[i + 1][c], x2_mul(kw.y, w2[c]));
          }
        }
        float rl, rh;
        x2_unpack(ruk, rl, rh);
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float lo, hi;
          x2_unpack(sum[c], lo, hi);
          o[c] = fmaf(rl + rh, vc[c], lo + hi);
        }
      }
      // sum over the eight lanes: each exchange halves the columns a lane still holds, then the last two lanes of a column add
      const float a0 = (up1 ? o[2] : o[0]) + __shfl_xor_sync(0xffffffffu, up1 ? o[0] : o[2], 1);
      const float a1 = (up1 ? o[3] : o[1]) + __shfl_xor_sync(0xffffffffu, up1 ? o[1] : o[3], 1);
      float r = (up2 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, up2 ? a0 : a1, 2);
      r += __shfl_xor_sync(0xffffffffu, r, 4);
      r *= ofac;
      if (HEAD) r = fmaf(skip, up1 ? (up2 ? vc[3] : vc[2]) : (up2 ? vc[1] : vc[0]), r);
      if (j < 4 && live) *optr = r;
      optr += ostep;
    };
    if constexpr (HEAD) {
#pragma unroll 1
      for (int tt = 0; tt < cn; ++tt) {
        fac *= ds[st][tt];
        if (fac < 1e-12f) {   // (the same in every thread of the CTA)
          const f32x2_t f2 = x2_pack(fac, fac);
#pragma unroll
          for (int i = 0; i < HP; ++i)
#pragma unroll
            for (int c = 0; c < NC; ++c) s[i][c] = x2_mul(f2, s[i][c]);
          fac = 1.0f;
        }
        token(tt, bs[st][tt] * __fdividef(1.0f, fac), qscale * fac);   // (1e-12 <= fac <= 1)
      }
    } else if (cn == CH) {
#pragma unroll 2
      for (int tt = 0; tt < CH; ++tt) token(tt, 0.f, qscale);
    } else {
#pragma unroll 1
      for (int tt = 0; tt < cn; ++tt) token(tt, 0.f, qscale);
    }
  }
  const f32x2_t f2 = x2_pack(fac, fac);
#pragma unroll
  for (int i = 0; i < HP; ++i) {
    float lo[NC], hi[NC];
#pragma unroll
    for (int c = 0; c < NC; ++c) x2_unpack(x2_mul(f2, s[i][c]), lo[c], hi[c]);
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int d = channel(2 * i + x);
      const float* src = x ? hi : lo;
      if (live && d < g.dim) *reinterpret_cast<float4*>(s_out + (size_t)d * g.vdim + col0 + cl) = make_float4(src[0], src[1], src[2], src[3]);
    }
  }
}

// One warp per (token, head): y = o / sqrt(mean(o^2) + eps) * gain * gate, gate = silu(gate_in) or gate_in as it is.
template <typename TX>
__global__ void __launch_bounds__(128) state_out_gate_kernel(const float* __restrict__ o, const float* __restrict__ gain,
                                                             const float* __restrict__ gate, int gate_ld, int gate_silu, TX* __restrict__ out,
                                                             int heads, int vdim, float eps, int T, int gain_per_head, float scale, int out_ld) {
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long unit = (long)blockIdx.x * 4 + warp;
  if (unit >= (long)T * heads) return;
  const int t = (int)(unit / heads), a = (int)(unit % heads);
  const float* orow = o + ((size_t)t * heads + a) * vdim;
  const float* grow = gate + (size_t)t * gate_ld + (size_t)a * vdim;
  float ss = 0.f;
  for (int i = lane; i < vdim; i += 32) ss = fmaf(orow[i], orow[i], ss);
  ss = warp_sum(ss);
  const float r = scale / sqrtf(ss / (float)vdim + eps);
  TX* dst = out + (size_t)t * out_ld + (size_t)a * vdim;
  if (gain_per_head) gain += (size_t)a * vdim;
  if (vdim % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0 && (reinterpret_cast<uintptr_t>(gate) & 15) == 0) {   // sixteen bytes at a time
    for (int i = lane * 4; i < vdim; i += 128) {
      const float4 ov = *reinterpret_cast<const float4*>(orow + i), gv = *reinterpret_cast<const float4*>(grow + i);
      const float4 nv = *reinterpret_cast<const float4*>(gain + i);
      const float oo[4] = {ov.x, ov.y, ov.z, ov.w}, gg[4] = {gv.x, gv.y, gv.z, gv.w}, nn[4] = {nv.x, nv.y, nv.z, nv.w};
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) y[k] = oo[k] * r * nn[k] * (gate_silu ? silu_f(gg[k]) : gg[k]);
      if constexpr (sizeof(TX) == 4) {
        *reinterpret_cast<float4*>(dst + i) = make_float4(y[0], y[1], y[2], y[3]);
      } else {
        uint2 pk;
        pk.x = pack_bf16x2(y[0], y[1]);
        pk.y = pack_bf16x2(y[2], y[3]);
        *reinterpret_cast<uint2*>(dst + i) = pk;
      }
    }
    return;
  }
  for (int i = lane; i < vdim; i += 32) {
    const float gt = gate_silu ? silu_f(grow[i]) : grow[i];
    dst[i] = (TX)(orow[i] * r * gain[i] * gt);
  }
}

// One CTA of NT threads per (token, part): v = o * silu(gate) is formed once and kept in registers (R groups of four numbers a thread) or, for other
// sizes (R = 0), in shared memory.
template <typename TX, int NT, int R>
__global__ void __launch_bounds__(NT) gate_part_norm_kernel(const float* __restrict__ o, const float* __restrict__ gate, int gate_ld,
                                                            const float* __restrict__ gain, float scale, TX* __restrict__ out, int out_ld, int N, int part,
                                                            float eps) {
  extern __shared__ float vrow[];
  __shared__ float red[NT / 32];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, c0 = blockIdx.y * part;
  const float* orow = o + (size_t)t * N + c0;
  const float* grow = gate + (size_t)t * gate_ld + c0;
  TX* dst = out + (size_t)t * out_ld + c0;
  float ss = 0.f;
  float4 v[R > 0 ? R : 1];
  if constexpr (R > 0) {
    float4 gv[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x + r * NT;
      const bool in = 4 * i < part;
      v[r] = in ? reinterpret_cast<const float4*>(orow)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
      gv[r] = in ? reinterpret_cast<const float4*>(grow)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      v[r].x *= silu_f(gv[r].x); v[r].y *= silu_f(gv[r].y); v[r].z *= silu_f(gv[r].z); v[r].w *= silu_f(gv[r].w);
      ss += (v[r].x * v[r].x + v[r].y * v[r].y) + (v[r].z * v[r].z + v[r].w * v[r].w);
    }
  } else {
    for (int i = threadIdx.x; i < part; i += NT) {
      const float x = orow[i] * silu_f(grow[i]);
      vrow[i] = x;
      ss = fmaf(x, x, ss);
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; ++w) tot += red[w];
  const float rn = scale / sqrtf(tot / (float)part + eps);
  if constexpr (R > 0) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int i = threadIdx.x + r * NT;
      if (4 * i >= part) continue;
      const float4 gn = reinterpret_cast<const float4*>(gain + c0)[i];
      const float y[4] = {v[r].x * rn * gn.x, v[r].y * rn * gn.y, v[r].z * rn * gn.z, v[r].w * rn * gn.w};
      if constexpr (sizeof(TX) == 4) {
        *reinterpret_cast<float4*>(dst + 4 * i) = make_float4(y[0], y[1], y[2], y[3]);
      } else {
        uint2 pk;
        pk.x = pack_bf16x2(y[0], y[1]);
        pk.y = pack_bf16x2(y[2], y[3]);
        *reinterpret_cast<uint2*>(dst + 4 * i) = pk;
      }
    }
  } else {
    for (int i = threadIdx.x; i < part; i += NT) dst[i] = (TX)(vrow[i] * rn * gain[c0 + i]);   // (a thread's own columns)
  }
}

template <typename TX>
int gate_part_norm_typed(const float* o, const float* gate, int gate_ld, const float* gain, int parts, float scale, TX* out, int out_ld, int N, float eps,
                         int T, cudaStream_t s) {
  const int part = N / parts;
  const dim3 grid(T, parts);
#define B2_GPN(NT, R)                                                                                                                              \
  do {                                                                                                                                             \
    B2_CUDA_OK(b2_launch(gate_part_norm_kernel<TX, NT, R>, grid, dim3(NT), 0, s, o, gate, gate_ld, gain, scale, out, out_ld, N, part, eps));        \
    return 0;                                                                                                                                      \
  } while (0)
  const bool vec = part % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  if (vec && part <= 512) B2_GPN(128, 1);
  if (vec && part <= 1024) B2_GPN(128, 2);
  if (vec && part <= 2048) B2_GPN(256, 2);
  if (vec && part <= 4096) B2_GPN(512, 2);
  if (vec && part <= 8192) B2_GPN(512, 4);
#undef B2_GPN
  B2_REQUIRE((size_t)part * 4 <= 160 * 1024, "gate_part_norm: a part of %d numbers does not fit in shared memory", part);
  static B2PerDeviceOnce once;
  if ((size_t)part * 4 > 48 * 1024) b2_prefer_max_smem(gate_part_norm_kernel<TX, 256, 0>, once);
  B2_CUDA_OK(b2_launch(gate_part_norm_kernel<TX, 256, 0>, grid, dim3(256), (size_t)part * 4, s, o, gate, gate_ld, gain, scale, out, out_ld, N, part, eps));
  return 0;
}

// The same for heads of 4 L numbers (L = 4 .. 32 lanes per head): a lane keeps its four numbers in registers.
template <typename TX, int L>
__global__ void __launch_bounds__(256) state_out_gate_lanes_kernel(const float* __restrict__ o, const float* __restrict__ gain,
                                                                   const float* __restrict__ gate, int gate_ld, int gate_silu, TX* __restrict__ out,
                                                                   int heads, float eps, int T, int gain_per_head, float scale, int out_ld) {
  constexpr int V = 4 * L;
  pdl_wait();
  pdl_launch_dependents();
  const long unit = ((long)blockIdx.x * 256 + threadIdx.x) / L;
  const bool in = unit < (long)T * heads;
  const int t = in ? (int)(unit / heads) : 0, a = in ? (int)(unit - (long)t * heads) : 0, i = (threadIdx.x % L) * 4;
  const float4 ov = *reinterpret_cast<const float4*>(o + ((size_t)t * heads + a) * V + i);
  const float4 gv = *reinterpret_cast<const float4*>(gate + (size_t)t * gate_ld + (size_t)a * V + i);
  const float4 nv = *reinterpret_cast<const float4*>(gain + (gain_per_head ? (size_t)a * V : 0) + i);
  float ss = (ov.x * ov.x + ov.y * ov.y) + (ov.z * ov.z + ov.w * ov.w);
#pragma unroll
  for (int m = L / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  if (!in) return;
  const float r = scale / sqrtf(ss / (float)V + eps);
  const float oo[4] = {ov.x, ov.y, ov.z, ov.w}, gg[4] = {gv.x, gv.y, gv.z, gv.w}, nn[4] = {nv.x, nv.y, nv.z, nv.w};
  float y[4];
#pragma unroll
  for (int k = 0; k < 4; ++k) y[k] = oo[k] * r * nn[k] * (gate_silu ? silu_f(gg[k]) : gg[k]);
  TX* dst = out + (size_t)t * out_ld + (size_t)a * V + i;
  if constexpr (sizeof(TX) == 4) {
    *reinterpret_cast<float4*>(dst) = make_float4(y[0], y[1], y[2], y[3]);
  } else {
    uint2 pk;
    pk.x = pack_bf16x2(y[0], y[1]);
    pk.y = pack_bf16x2(y[2], y[3]);
    *reinterpret_cast<uint2*>(dst) = pk;
  }
}

template <typename TX>
int state_out_gate_typed(const float* o, const float* gain, const float* gate, int gate_ld, int gate_silu, TX* out, int heads, int vdim, float eps, int T,
                         int gain_per_head, float scale, int out_ld, cudaStream_t s) {
  const long units = (long)T * heads;
  const bool vec = gate_ld % 4 == 0 && out_ld % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(gain) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
#define B2_OUT_GATE(L)                                                                                                                                     \
  if (vec && vdim == 4 * (L)) {                                                                                                                            \
    B2_CUDA_OK(b2_launch(state_out_gate_lanes_kernel<TX, L>, dim3((unsigned)((units * (L) + 255) / 256)), dim3(256), 0, s, o, gain, gate, gate_ld, gate_silu, out, \
                         heads, eps, T, gain_per_head, scale, out_ld));                                                                                    \
    return 0;                                                                                                                                              \
  }
  B2_OUT_GATE(4) B2_OUT_GATE(8) B2_OUT_GATE(16) B2_OUT_GATE(32)
#undef B2_OUT_GATE
  B2_CUDA_OK(b2_launch(state_out_gate_kernel<TX>, dim3((unsigned)((units + 3) / 4)), dim3(128), 0, s, o, gain, gate, gate_ld, gate_silu, out, heads, vdim, eps, T,
                       gain_per_head, scale, out_ld));
  return 0;
}

template <int RULE>
int launch_scan_rule(int dpt, dim3 grid, dim3 block, cudaStream_t s, const float* q, int ldq, const float* k, int ldk, const float* v, int ldv,
                     const float* decay, const float* beta, const StateGeom& g, float qscale, float* state, const int32_t* last_rows,
                     const int32_t* row_seq, const int32_t* row_first, const int32_t* row_end, const int32_t* positions, const int32_t* slots,
                     float* out, int cols) {
#define B2_SCAN_CASE(D, N)                                                                                                                    \
  case D:                                                                                                                                     \
    B2_CUDA_OK(b2_launch(state_scan_kernel<D, N, RULE>, grid, block, 0, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows,  \
                         row_seq, row_first, row_end, positions, slots, out, cols));                                                          \
    return 0;
  switch (dpt) {
    B2_SCAN_CASE(1, 4)
    B2_SCAN_CASE(2, 4)
    B2_SCAN_CASE(4, 4)
    B2_SCAN_CASE(8, 4)
    B2_SCAN_CASE(16, 4)
    B2_SCAN_CASE(32, 2)
  }
#undef B2_SCAN_CASE
  b2_set_error("state_scan: key width %d not built (at most 256)", g.dim);
  return -22;
}

}  // namespace

int launch_lowrank_act(const float* lr, int ld, int lr_off, int rank, const float* w2, const float* bias, int mode, float rate,
                       const float* rate_log, int per_head, float* out, int T, int C, cudaStream_t s) {
  if (T <= 0 || C <= 0) return 0;
  B2_REQUIRE(rank >= 1 && rank <= 1024, "lowrank_act: rank %d (at most 1024)", rank);
  B2_REQUIRE(mode != LOWRANK_DECAY_SOFTPLUS || (rate_log != nullptr && per_head >= 1), "lowrank_act: the softplus decay needs a rate per head");
  if (T >= 256 && rank <= LT_MAX_RANK) {
    const int tb = (T + LT_T - 1) / LT_T, tiles = (C + LT_C - 1) / LT_C;
    int ys = 1;   // as few shares of the channel tiles as still give every SM several CTAs
    while (ys < tiles && tb * ys < 4 * device_num_sms()) ys *= 2;
    const int per = (tiles + ys - 1) / ys;
    const size_t smem = ((size_t)rank * (LT_T + 4) + (size_t)LT_K * (LT_C + 4)) * 4;
    static B2PerDeviceOnce attr_once;
    if (attr_once.need())
      B2_CUDA_OK(cudaFuncSetAttribute(lowrank_act_tile_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                      (int)(((size_t)LT_MAX_RANK * (LT_T + 4) + (size_t)LT_K * (LT_C + 4)) * 4)));
    B2_CUDA_OK(b2_launch(lowrank_act_tile_kernel, dim3(tb, (tiles + per - 1) / per), dim3(256), smem, s, lr, ld, lr_off, rank, w2, bias, rate_log, rate,
                         per_head > 0 ? per_head : 1, mode, out, C, T, per));
    return 0;
  }
  const dim3 grid((T + LR_TOKENS - 1) / LR_TOKENS, (C + 63) / 64);
  B2_CUDA_OK(b2_launch(lowrank_act_kernel<64>, grid, dim3(64), (size_t)LR_TOKENS * rank * 4, s, lr, ld, lr_off, rank, w2, bias, rate_log, rate,
                       per_head > 0 ? per_head : 1, mode, out, C, T));
  return 0;
}

int launch_conv_unit_finish(const float* proj, int ld, const StateGeom& g, int taps, const float* conv_w, float* ring, const int32_t* row_seq,
                            const int32_t* row_first, const int32_t* row_end, const int32_t* positions, const int32_t* slots, float unit_eps,
                            float* out, float* beta_out, int T, cudaStream_t s, const float* a_log, const float* dt_bias, float* decay_out, int single_rows) {
  if (T <= 0) return 0;
  B2_REQUIRE(a_log == nullptr || (dt_bias != nullptr && decay_out != nullptr), "conv_unit_finish: a decay per head needs its bias and its output");
  B2_REQUIRE(taps >= 1 && conv_w && (ring || taps == 1) && row_seq && row_first && row_end, "conv_unit_finish: the convolution needs its weights and state");
  const int C = 2 * g.kv_heads * g.dim + g.heads * g.vdim;
  const int units = 2 * g.kv_heads + g.heads, upc = T >= 256 ? units : std::max(1, (units + 15) / 16);   // few tokens: up to sixteen CTAs each
  const dim3 grid(T, (units + upc - 1) / upc);
#define B2_CONV_FINISH(TAPS)                                                                                                                      \
  B2_CUDA_OK(b2_launch(conv_unit_finish_kernel<TAPS>, grid, dim3(256), 0, s, proj, ld, g, taps, conv_w, (const float*)ring, row_seq, row_first, positions, \
                       slots, unit_eps, out, beta_out, upc, a_log, dt_bias, decay_out, single_rows && taps > 1 ? ring : (float*)nullptr))
#define B2_CONV_ROWS(TAPS)                                                                                                                        \
  B2_CUDA_OK(b2_launch(conv_unit_rows_kernel<TAPS>, dim3((T + CR_ROWS - 1) / CR_ROWS, units), dim3(128), (size_t)CR_ROWS * g.dim * 4, s, proj, ld, g, conv_w, \
                       (const float*)ring, row_seq, row_first, positions, slots, unit_eps, out, beta_out, a_log, dt_bias, decay_out, T))
  const bool rows = !single_rows && T >= 512 && taps >= 2 && taps <= 4 && g.dim <= 512;
  if (rows && taps == 4) B2_CONV_ROWS(4);
  else if (rows && taps == 3) B2_CONV_ROWS(3);
  else if (rows) B2_CONV_ROWS(2);
  else if (taps == 4) B2_CONV_FINISH(4);
  else if (taps == 3) B2_CONV_FINISH(3);
  else if (taps == 2) B2_CONV_FINISH(2);
  else B2_CONV_FINISH(0);
#undef B2_CONV_FINISH
#undef B2_CONV_ROWS
  if (taps > 1 && !single_rows)
    B2_CUDA_OK(b2_launch(conv_ring_store_kernel, dim3((T + 31) / 32), dim3(128), 0, s, proj, ld, C, taps, ring, row_seq, row_end, positions, slots, T));
  return 0;
}

int launch_state_scan(const float* q, int ldq, const float* k, int ldk, const float* v, int ldv, const float* decay, const float* beta,
                      const StateGeom& g, float qscale, float* state, int portions, const int32_t* last_rows, const int32_t* row_seq,
                      const int32_t* row_first, const int32_t* row_end, const int32_t* positions, const int32_t* slots, float* out,
                      cudaStream_t s) {
  if (portions <= 0) return 0;
  B2_REQUIRE(g.heads >= 1 && g.kv_heads >= 1 && g.heads % g.kv_heads == 0 && g.dim >= 1 && g.vdim >= 1, "state_scan: bad sizes");
  B2_REQUIRE(g.rule == STATE_RULE_DECAY || (g.rule == STATE_RULE_BONUS && g.bonus != nullptr) ||
                 (g.rule == STATE_RULE_DECAY_HEAD && g.skip != nullptr && beta != nullptr) || ((g.rule == STATE_RULE_DELTA || g.rule == STATE_RULE_DELTA_HEAD) && beta != nullptr), "state_scan: rule %d", g.rule);
  int dpt = 1;
  while (dpt * SC_LANES < g.dim) dpt *= 2;
  B2_REQUIRE(dpt <= 32, "state_scan: key width %d not built (at most 256)", g.dim);
  // a warp is four groups of eight lanes, a group owns nc neighbouring columns; as many columns per CTA (at most eight warps) as still
  // leave two CTAs for every SM (a column's arithmetic does not depend on the tile it falls into)
  const int nc = dpt >= 32 ? 2 : 4, step = 4 * nc;
  int cols = std::min(32 * nc, (g.vdim + step - 1) / step * step);
  while (cols > step && (long)portions * g.heads * ((g.vdim + cols - 1) / cols) < 2L * device_num_sms()) cols = (cols / 2 + step - 1) / step * step;
  const dim3 grid(portions, g.heads, (g.vdim + cols - 1) / cols), block(cols / nc * SC_LANES);
  if (g.rule == STATE_RULE_DECAY)
    return launch_scan_rule<STATE_RULE_DECAY>(dpt, grid, block, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows, row_seq,
                                              row_first, row_end, positions, slots, out, cols);
  static const bool packed = [] { const char* e = getenv("B2_SCAN_PACKED"); return !(e && *e == '0'); }();   // 0: the generic form (cross-check)
  const bool rows16 = g.dim % 4 == 0 && g.vdim % 4 == 0 && ldq % 4 == 0 && ldk % 4 == 0 && ldv % 4 == 0 &&
                      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15) == 0;
  if ((g.rule == STATE_RULE_DECAY_HEAD || g.rule == STATE_RULE_BONUS) && packed && rows16 && dpt <= 16 && (reinterpret_cast<uintptr_t>(decay) & 15) == 0) {
#define B2_SCAN_SUM(D, R)                                                                                                                          \
  B2_CUDA_OK(b2_launch(state_scan_sum_kernel<D, R>, grid, block, 0, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows, row_seq,   \
                       row_first, row_end, positions, slots, out, cols))
    if (g.rule == STATE_RULE_DECAY_HEAD) {
      if (dpt <= 4) B2_SCAN_SUM(4, STATE_RULE_DECAY_HEAD);
      else if (dpt == 8) B2_SCAN_SUM(8, STATE_RULE_DECAY_HEAD);
      else B2_SCAN_SUM(16, STATE_RULE_DECAY_HEAD);
    } else {
      if (dpt <= 4) B2_SCAN_SUM(4, STATE_RULE_BONUS);
      else if (dpt == 8) B2_SCAN_SUM(8, STATE_RULE_BONUS);
      else B2_SCAN_SUM(16, STATE_RULE_BONUS);
    }
#undef B2_SCAN_SUM
    return 0;
  }
  if (g.rule == STATE_RULE_DECAY_HEAD)
    return launch_scan_rule<STATE_RULE_DECAY_HEAD>(dpt, grid, block, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows, row_seq,
                                                   row_first, row_end, positions, slots, out, cols);
  if (g.rule == STATE_RULE_BONUS)
    return launch_scan_rule<STATE_RULE_BONUS>(dpt, grid, block, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows, row_seq,
                                              row_first, row_end, positions, slots, out, cols);
  if (g.rule == STATE_RULE_DELTA_HEAD && packed && rows16 && dpt <= 16) {
#define B2_SCAN_HEAD(D)                                                                                                                          \
  B2_CUDA_OK(b2_launch(state_scan_head_kernel<D>, grid, block, 0, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows, row_seq,   \
                       row_first, row_end, positions, slots, out, cols))
    if (dpt <= 4) B2_SCAN_HEAD(4);
    else if (dpt == 8) B2_SCAN_HEAD(8);
    else B2_SCAN_HEAD(16);
#undef B2_SCAN_HEAD
    return 0;
  }
  if (g.rule == STATE_RULE_DELTA_HEAD)
    return launch_scan_rule<STATE_RULE_DELTA_HEAD>(dpt, grid, block, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows, row_seq,
                                                   row_first, row_end, positions, slots, out, cols);
  return launch_scan_rule<STATE_RULE_DELTA>(dpt, grid, block, s, q, ldq, k, ldk, v, ldv, decay, beta, g, qscale, state, last_rows, row_seq,
                                            row_first, row_end, positions, slots, out, cols);
}

size_t state_floats_per_slot(const StateGeom& g) { return (size_t)2 * g.heads * g.dim * g.vdim; }

int launch_state_out_gate(const float* o, const float* gain, const float* gate, int gate_ld, int gate_silu, void* out, int out_f32,
                          int heads, int vdim, float eps, int T, cudaStream_t s, int gain_per_head, float scale, int out_ld) {
  if (T <= 0) return 0;
  if (out_ld <= 0) out_ld = heads * vdim;
  return out_f32 ? state_out_gate_typed<float>(o, gain, gate, gate_ld, gate_silu, (float*)out, heads, vdim, eps, T, gain_per_head, scale, out_ld, s)
                 : state_out_gate_typed<bf16>(o, gain, gate, gate_ld, gate_silu, (bf16*)out, heads, vdim, eps, T, gain_per_head, scale, out_ld, s);
}

int launch_conv_act_finish(const float* proj, int ld, int channels, int heads, int taps, const float* conv_w, const float* conv_b, const float* a_log,
                           const float* dt_bias, float* ring, const int32_t* row_seq, const int32_t* row_first, const int32_t* row_end,
                           const int32_t* positions, const int32_t* slots, float* out, float* step, float* decay, int T, int single_rows, cudaStream_t s) {
  if (T <= 0) return 0;
  B2_REQUIRE(taps >= 1 && (ring != nullptr || taps == 1), "conv_act_finish: a convolution of %d taps needs its ring", taps);
  const int rows = single_rows || T < 512 ? 1 : CR_ROWS;
  const dim3 grid((T + rows - 1) / rows, (channels + 127) / 128);
  float* store = single_rows && taps > 1 ? ring : nullptr;
#define B2_CONV_ACT(TAPS)                                                                                                                        \
  B2_CUDA_OK(b2_launch(conv_act_kernel<TAPS>, grid, dim3(128), 0, s, proj, ld, channels, heads, taps, conv_w, conv_b, a_log, dt_bias, (const float*)ring, store, \
                       row_seq, row_first, positions, slots, out, step, decay, rows, T))
#define B2_CONV_ACT4(TAPS)                                                                                                                       \
  B2_CUDA_OK(b2_launch(conv_act4_kernel<TAPS>, dim3((T + rows - 1) / rows, (channels / 4 + 127) / 128), dim3(128), 0, s, proj, ld, channels, heads, conv_w, conv_b, \
                       a_log, dt_bias, (const float*)ring, row_seq, row_first, positions, slots, out, step, decay, rows, T))
  const bool four = rows > 1 && taps >= 2 && taps <= 4 && channels % 4 == 0 && ld % 4 == 0 && ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(conv_b)) & 15) == 0;
  if (four && taps == 4) B2_CONV_ACT4(4);
  else if (four && taps == 3) B2_CONV_ACT4(3);
  else if (four) B2_CONV_ACT4(2);
  else if (taps == 4) B2_CONV_ACT(4);
  else if (taps == 3) B2_CONV_ACT(3);
  else if (taps == 2) B2_CONV_ACT(2);
  else B2_CONV_ACT(0);
#undef B2_CONV_ACT
#undef B2_CONV_ACT4
  if (taps > 1 && !single_rows)
    B2_CUDA_OK(b2_launch(conv_ring_store_kernel, dim3((T + 31) / 32), dim3(128), 0, s, proj, ld, channels, taps, ring, row_seq, row_end, positions, slots, T));
  return 0;
}

int launch_gate_part_norm(const float* o, const float* gate, int gate_ld, const float* gain, int parts, float scale, void* out, int out_f32, int out_ld,
                          int N, float eps, int T, cudaStream_t s) {
  if (T <= 0) return 0;
  B2_REQUIRE(parts >= 1 && N % parts == 0, "gate_part_norm: %d numbers in %d parts", N, parts);
  return out_f32 ? gate_part_norm_typed<float>(o, gate, gate_ld, gain, parts, scale, (float*)out, out_ld, N, eps, T, s)
                 : gate_part_norm_typed<bf16>(o, gate, gate_ld, gain, parts, scale, (bf16*)out, out_ld, N, eps, T, s);
}

}  // namespace b2
