// moe_route.cu -- the router of a routed-experts feed-forward, and the bookkeeping that turns its choices into ragged
// groups for gemm_any.cu.
//
// Router (all fp32): z = R x (+ a bias), s = sigmoid(z) or a softmax of z over all experts (RouteGeom.softmax).  The CHOICE uses s + correction (an
// optional per-expert offset that steers load and may make a choice score negative); the mixing WEIGHTS use s alone.  Experts are
// `groups` equal runs of neighbours; a group's score is the sum of its two best choice scores (or its best one, group_best) and only the
// `keep` best groups may supply experts (the others are out, not zero).  Of the allowed experts the `top` with the best choice scores
// are taken; their s, divided by their sum (+ 1e-20) or as they are times a constant (raw_weights, scale), are the weights.  Ties go to
// the lower index.  A router matrix may carry one more row, whose sigmoid gates a shared expert.
//
// route_permute is a counting sort of the (token, choice) pairs by expert: slots of expert e are [offsets[e], offsets[e+1]).
// Which slot of its expert a pair gets depends on the order of atomic arrivals, and that is harmless: gemm_any.cu sums every
// output row on its own, so a row's result does not depend on its slot or on its tile mates -- nor, therefore, on the other
// requests of the batch.  route_combine adds the weighted expert outputs (and the mixer branch) onto the fp32 residual
// stream in choice order.
#include "kernels.h"

namespace b2 {

namespace {

// One warp: a token's router products s [E] (and, with a softmax, still logits) become scores, the choices and their weights.  ch [E] and
// gs [groups] are the warp's scratch in shared memory.
__device__ void route_pick(float* s, float* ch, float* gs, const RouteGeom& g, const float* __restrict__ correction, int t, int32_t* __restrict__ idx,
                           float* __restrict__ weight) {
  const int lane = threadIdx.x & 31, E = g.experts;
  if (g.softmax) {
    float m = -INFINITY, sum = 0.f;
    for (int e = lane; e < E; e += 32) m = fmaxf(m, s[e]);
    m = warp_max(m);
    for (int e = lane; e < E; e += 32) {
      const float p = expf(s[e] - m);
      s[e] = p;
      sum += p;
    }
    const float inv = 1.0f / warp_sum(sum);
    for (int e = lane; e < E; e += 32) s[e] *= inv;   // (a lane's own entries)
  }
  for (int e = lane; e < E; e += 32) ch[e] = s[e] + (correction ? correction[e] : 0.f);
  __syncwarp();
  // groups: all but the `keep` best are out (choice = -inf).  Ranks are formed from the untouched scores first, then applied.
  const int per = E / g.groups;
  if (g.keep < g.groups) {
    for (int gi = lane; gi < g.groups; gi += 32) {
      float b1 = -INFINITY, b2 = -INFINITY;
      for (int e = gi * per; e < (gi + 1) * per; ++e) {
        const float v = ch[e];
        if (v > b1) { b2 = b1; b1 = v; } else if (v > b2) { b2 = v; }
      }
      gs[gi] = (per >= 2 && !g.group_best) ? b1 + b2 : b1;
    }
    __syncwarp();
    for (int gi = lane; gi < g.groups; gi += 32) {
      int beat = 0;  // groups ranked ahead of gi (lower index wins a tie)
      for (int gj = 0; gj < g.groups; ++gj) {
        if (gj == gi) continue;
        if (gs[gj] > gs[gi] || (gs[gj] == gs[gi] && gj < gi)) ++beat;
      }
      if (beat >= g.keep)
        for (int e = gi * per; e < (gi + 1) * per; ++e) ch[e] = -INFINITY;
    }
    __syncwarp();
  }
  float sum = 0.f;
  const float scale = g.scale != 0.f ? g.scale : 1.0f;
  for (int k = 0; k < g.top; ++k) {
    float bv = -INFINITY;   // -inf = out or already taken
    int best = 0x7fffffff;
    for (int e = lane; e < E; e += 32)
      if (ch[e] > bv) { best = e; bv = ch[e]; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {   // the first index wins a tie
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, best, o);
      if (ov > bv || (ov == bv && oi < best)) { bv = ov; best = oi; }
    }
    if (best >= E) best = k < E ? k : 0;  // only for rows that hold no numbers (padding rows of a graph bucket): keep the index valid
    const float w = s[best];
    if (lane == 0) {
      idx[(size_t)t * g.top + k] = best;
      weight[(size_t)t * g.top + k] = g.raw_weights ? w * scale : w;
      ch[best] = -INFINITY;
    }
    sum += w;
    __syncwarp();
  }
  if (g.raw_weights) return;   // the scores as they are (times the scale)
  const float inv = 1.0f / (sum + 1e-20f);
  if (lane == 0)
    for (int k = 0; k < g.top; ++k) weight[(size_t)t * g.top + k] *= inv;
}

// A CTA takes NTOK tokens: their rows are staged once as fp32, warp w takes router rows w, w + 16, ... (a row is read once for all tokens of
// the CTA), then one warp per token forms the scores and selects.  A token's arithmetic does not depend on NTOK.
template <typename TX, int NTOK, int RT_WARPS>
__global__ void __launch_bounds__(RT_WARPS * 32) route_kernel(const TX* __restrict__ x, const float* __restrict__ router,
                                                              const float* __restrict__ correction, RouteGeom g, int32_t* __restrict__ idx,
                                                              float* __restrict__ weight, int T, int W, float* __restrict__ gate_out) {
  extern __shared__ __align__(16) float sm[];  // x rows [NTOK][W rounded up to 4] (read as float4), then per token: s [E + 1], choice [E], group scores [groups]
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * NTOK, tn = min(NTOK, T - t0);
  const int E = g.experts, ER = E + (gate_out != nullptr ? 1 : 0), Wp = (W + 3) & ~3, per_tok = 2 * E + 1 + g.groups;
  float* xs = sm;
  float* sc = xs + NTOK * Wp;
  for (int i = threadIdx.x; i < NTOK * W; i += RT_WARPS * 32) {
    const int tt = i / W, c = i - tt * W;
    xs[tt * Wp + c] = tt < tn ? (float)x[(size_t)(t0 + tt) * W + c] : 0.f;
  }
  __syncthreads();
  const bool vec = (W % 4 == 0);
  for (int e = warp; e < ER; e += RT_WARPS) {
    const float* rr = router + (size_t)e * W;
    float acc[NTOK];
#pragma unroll
    for (int tt = 0; tt < NTOK; ++tt) acc[tt] = 0.f;
    if (vec) {
#pragma unroll 8
      for (int i = lane * 4; i < W; i += 128) {
        const float4 r4 = *reinterpret_cast<const float4*>(rr + i);
#pragma unroll
        for (int tt = 0; tt < NTOK; ++tt) {
          const float4 x4 = *reinterpret_cast<const float4*>(xs + tt * Wp + i);
          acc[tt] = fmaf(x4.x, r4.x, acc[tt]); acc[tt] = fmaf(x4.y, r4.y, acc[tt]); acc[tt] = fmaf(x4.z, r4.z, acc[tt]); acc[tt] = fmaf(x4.w, r4.w, acc[tt]);
        }
      }
    } else {
      for (int i = lane; i < W; i += 32) {
        const float r = rr[i];
#pragma unroll
        for (int tt = 0; tt < NTOK; ++tt) acc[tt] = fmaf(xs[tt * Wp + i], r, acc[tt]);
      }
    }
#pragma unroll
    for (int tt = 0; tt < NTOK; ++tt) {
      const float z = warp_sum(acc[tt]);
      if (lane == 0) {
        const float zb = z + (g.logit_bias && e < E ? g.logit_bias[e] : 0.f);
        sc[tt * per_tok + e] = (g.softmax && e < E) ? zb : 1.0f / (1.0f + expf(-zb));   // (the extra row is a gate: always a sigmoid)
      }
    }
  }
  __syncthreads();
  if (warp >= tn) return;
  const int t = t0 + warp;
  float* s = sc + warp * per_tok;
  float* ch = s + E + 1;
  float* gs = ch + E;
  if (gate_out != nullptr && lane == 0) gate_out[t] = s[E];
  route_pick(s, ch, gs, g, correction, t, idx, weight);
}

// The same behind a product that has formed the logits z [T][ld] already (experts, then the gate's): one warp per token.
__global__ void __launch_bounds__(256) route_select_kernel(const float* __restrict__ z, int ld, const float* __restrict__ correction, RouteGeom g,
                                                           int32_t* __restrict__ idx, float* __restrict__ weight, int T, float* __restrict__ gate_out) {
  extern __shared__ __align__(16) float sm[];
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 8 + warp, E = g.experts;
  if (t >= T) return;
  float* s = sm + warp * (2 * E + g.groups);
  const float* zr = z + (size_t)t * ld;
  for (int e = lane; e < E; e += 32) {
    const float zb = zr[e] + (g.logit_bias ? g.logit_bias[e] : 0.f);
    s[e] = g.softmax ? zb : 1.0f / (1.0f + expf(-zb));
  }
  if (gate_out != nullptr && lane == 0) gate_out[t] = 1.0f / (1.0f + expf(-zr[E]));
  __syncwarp();
  route_pick(s, s + E, s + 2 * E, g, correction, t, idx, weight);
}

// the permutation in three steps: histogram (any number of CTAs), scan (one thread; experts are few), placement
__global__ void __launch_bounds__(256) route_count_kernel(const int32_t* __restrict__ idx, int npairs, int E, int* __restrict__ counts) {
  extern __shared__ int hist[];
  pdl_wait();
  pdl_launch_dependents();
  for (int e = threadIdx.x; e < E; e += 256) hist[e] = 0;
  __syncthreads();
  const int p = blockIdx.x * 256 + threadIdx.x;
  if (p < npairs) atomicAdd(&hist[idx[p]], 1);
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += 256)
    if (hist[e]) atomicAdd(&counts[e], hist[e]);
}
__global__ void route_scan_kernel(int* __restrict__ counts, int E, int32_t* __restrict__ offsets, int* __restrict__ cursor) {
  pdl_wait();
  pdl_launch_dependents();
  if (threadIdx.x != 0) return;
  int run = 0;
  for (int e = 0; e < E; ++e) {
    offsets[e] = run;
    cursor[e] = run;
    run += counts[e];
    counts[e] = 0;  // ready for the next call
  }
  offsets[E] = run;
}
__global__ void __launch_bounds__(256) route_place_kernel(const int32_t* __restrict__ idx, int npairs, int top, int* __restrict__ cursor,
                                                          int32_t* __restrict__ slot_token, int32_t* __restrict__ pair_slot) {
  pdl_wait();
  pdl_launch_dependents();
  const int p = blockIdx.x * 256 + threadIdx.x;
  if (p >= npairs) return;
  const int slot = atomicAdd(&cursor[idx[p]], 1);
  slot_token[slot] = p / top;
  pair_slot[p] = slot;
}

// few pairs (a decode step): the three steps in one CTA, histogram and cursors in shared memory
__global__ void __launch_bounds__(1024) route_permute_small_kernel(const int32_t* __restrict__ idx, int npairs, int top, int E,
                                                                   int32_t* __restrict__ offsets, int32_t* __restrict__ slot_token,
                                                                   int32_t* __restrict__ pair_slot) {
  extern __shared__ int cur[];  // [E]
  pdl_wait();
  pdl_launch_dependents();
  for (int e = threadIdx.x; e < E; e += 1024) cur[e] = 0;
  __syncthreads();
  const int p = threadIdx.x;
  const int mine = p < npairs ? idx[p] : -1;
  if (mine >= 0) atomicAdd(&cur[mine], 1);
  __syncthreads();
  if (threadIdx.x == 0) {
    int run = 0;
    for (int e = 0; e < E; ++e) {
      const int c = cur[e];
      offsets[e] = run;
      cur[e] = run;
      run += c;
    }
    offsets[E] = run;
  }
  __syncthreads();
  if (mine >= 0) {
    const int slot = atomicAdd(&cur[mine], 1);
    slot_token[slot] = p / top;
    pair_slot[p] = slot;
  }
}

constexpr int COMBINE_MAX_TOP = 16;   // choices staged in shared memory; wider routers read them from global memory
__global__ void __launch_bounds__(256) route_combine_kernel(float* __restrict__ h, const float* __restrict__ mix, const float* __restrict__ y,
                                                            const float* __restrict__ weight, const int32_t* __restrict__ pair_slot, int W,
                                                            int top) {
  __shared__ float w_s[COMBINE_MAX_TOP];
  __shared__ int slot_s[COMBINE_MAX_TOP];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const bool staged = top <= COMBINE_MAX_TOP;
  if (staged && (int)threadIdx.x < top) {
    w_s[threadIdx.x] = weight[(size_t)t * top + threadIdx.x];
    slot_s[threadIdx.x] = pair_slot[(size_t)t * top + threadIdx.x];
  }
  __syncthreads();
  if (staged && W % 4 == 0) {   // (rows of h, mix and y start on 16-byte boundaries: W * 4 bytes apart from aligned bases)
    float4* hr = reinterpret_cast<float4*>(h + (size_t)t * W);
    const float4* mr = mix != nullptr ? reinterpret_cast<const float4*>(mix + (size_t)t * W) : nullptr;
    for (int i = threadIdx.x; i < W / 4; i += 256) {
      float4 acc = mr != nullptr ? mr[i] : make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < top; ++k) {   // choice order
        const float4 v = reinterpret_cast<const float4*>(y + (size_t)slot_s[k] * W)[i];
        const float w = w_s[k];
        acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y); acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
      }
      float4 o = hr[i];
      o.x += acc.x; o.y += acc.y; o.z += acc.z; o.w += acc.w;
      hr[i] = o;
    }
    return;
  }
  for (int i = threadIdx.x; i < W; i += 256) {
    float acc = mix != nullptr ? mix[(size_t)t * W + i] : 0.f;
    for (int k = 0; k < top; ++k) acc = fmaf(weight[(size_t)t * top + k], y[(size_t)pair_slot[(size_t)t * top + k] * W + i], acc);
    h[(size_t)t * W + i] += acc;
  }
}

// slot_weight[pair_slot[p]] = weight[p]: the pairs' weights in expert (slot) order, for experts whose INPUT the weight multiplies
__global__ void __launch_bounds__(256) route_slot_weights_kernel(const float* __restrict__ weight, const int32_t* __restrict__ pair_slot,
                                                                 float* __restrict__ slot_weight, int npairs) {
  pdl_wait();
  pdl_launch_dependents();
  const int p = blockIdx.x * 256 + threadIdx.x;
  if (p < npairs) slot_weight[pair_slot[p]] = weight[p];
}

// No router: a table row per token id names the token's experts, each weighted 1 / top.  idx [T][top], weight [T][top].
__global__ void __launch_bounds__(256) route_table_kernel(const int32_t* __restrict__ ids, const int32_t* __restrict__ table, int vocab, int experts,
                                                          int top, int32_t* __restrict__ idx, float* __restrict__ weight, int npairs) {
  pdl_wait();
  pdl_launch_dependents();
  const int p = blockIdx.x * 256 + threadIdx.x;
  if (p >= npairs) return;
  const int t = p / top, k = p - t * top;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  int x = table[(size_t)id * top + k];
  x = x < 0 ? 0 : (x >= experts ? experts - 1 : x);
  idx[p] = x;
  weight[p] = 1.0f / (float)top;
}

// act = bf16(max(up, 0)^2): the experts' activation between the two dense products of a prompt-sized step
__global__ void __launch_bounds__(256) relu2_round_kernel(const float4* __restrict__ up, uint2* __restrict__ act, size_t n4) {
  pdl_wait();
  pdl_launch_dependents();
  for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n4; i += (size_t)gridDim.x * 256) {
    const float4 v = up[i];
    const float a = fmaxf(v.x, 0.f), b = fmaxf(v.y, 0.f), c = fmaxf(v.z, 0.f), d = fmaxf(v.w, 0.f);
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a * a, b * b), hi = __floats2bfloat162_rn(c * c, d * d);
    uint2 o;
    o.x = *reinterpret_cast<const uint32_t*>(&lo);
    o.y = *reinterpret_cast<const uint32_t*>(&hi);
    act[i] = o;
  }
}

}  // namespace

int launch_relu2_round(const float* up, bf16* act, size_t n, cudaStream_t s) {
  if (n == 0) return 0;
  if (n % 4 != 0) return -22;   // (rows are multiples of 64 wide on this path)
  const size_t n4 = n / 4;
  const int grid = (int)std::min<size_t>((n4 + 255) / 256, 148 * 16);
  B2_CUDA_OK(b2_launch(relu2_round_kernel, dim3(grid), dim3(256), 0, s, (const float4*)up, (uint2*)act, n4));
  return 0;
}

int launch_route(const void* x, int x_f32, const float* router, const float* correction, const RouteGeom& g, int32_t* idx, float* weight,
                 int T, int W, cudaStream_t s, float* gate_out) {
  if (T <= 0) return 0;
  B2_REQUIRE(g.experts >= 1 && g.groups >= 1 && g.groups <= 64 && g.experts % g.groups == 0, "route: %d experts do not form %d equal groups", g.experts, g.groups);
  B2_REQUIRE(g.keep >= 1 && g.keep <= g.groups, "route: keep %d outside [1, %d]", g.keep, g.groups);
  B2_REQUIRE(g.top >= 1 && g.top <= g.keep * (g.experts / g.groups), "route: top %d exceeds the %d experts of the kept groups", g.top,
             g.keep * (g.experts / g.groups));
  auto bytes = [&](int ntok) { return (size_t)ntok * (2 * g.experts + 1 + g.groups + ((W + 3) & ~3)) * sizeof(float); };
  B2_REQUIRE(bytes(1) <= 48 * 1024, "route: %d experts and width %d need %zu bytes of shared memory", g.experts, W, bytes(1));
  // prompt-sized steps: several tokens per CTA share one pass over the router's rows
  const int ntok = T >= 1024 && bytes(4) <= 48 * 1024 ? 4 : T >= 512 && bytes(2) <= 48 * 1024 ? 2 : 1;
  const dim3 grid((T + ntok - 1) / ntok);
#define B2_ROUTE(TX, N) B2_CUDA_OK(b2_launch(route_kernel<TX, N, (N == 1 ? 32 : 16)>, grid, dim3(N == 1 ? 1024 : 512), bytes(N), s, (const TX*)x, router, correction, g, idx, weight, T, W, gate_out))
  if (x_f32) {
    if (ntok == 4) B2_ROUTE(float, 4);
    else if (ntok == 2) B2_ROUTE(float, 2);
    else B2_ROUTE(float, 1);
  } else {
    if (ntok == 4) B2_ROUTE(bf16, 4);
    else if (ntok == 2) B2_ROUTE(bf16, 2);
    else B2_ROUTE(bf16, 1);
  }
#undef B2_ROUTE
  return 0;
}

int launch_route_select(const float* z, int ld, const float* correction, const RouteGeom& g, int32_t* idx, float* weight, int T, cudaStream_t s, float* gate_out) {
  if (T <= 0) return 0;
  B2_REQUIRE(g.experts >= 1 && g.groups >= 1 && g.groups <= 64 && g.experts % g.groups == 0 && g.keep >= 1 && g.keep <= g.groups && g.top >= 1 &&
                 g.top <= g.keep * (g.experts / g.groups),
             "route_select: bad sizes (experts %d, groups %d, keep %d, top %d)", g.experts, g.groups, g.keep, g.top);
  const size_t smem = (size_t)8 * (2 * g.experts + g.groups) * sizeof(float);
  B2_REQUIRE(smem <= 48 * 1024, "route_select: %d experts", g.experts);
  B2_CUDA_OK(b2_launch(route_select_kernel, dim3((T + 7) / 8), dim3(256), smem, s, z, ld, correction, g, idx, weight, T, gate_out));
  return 0;
}

int launch_route_permute(const int32_t* idx, int T, int top, int experts, int32_t* offsets, int stride, int32_t* slot_token,
                         int32_t* pair_slot, cudaStream_t s) {
  if (T <= 0) return 0;
  B2_REQUIRE(stride >= experts + 1, "route_permute: stride %d < experts + 1", stride);
  int* counts = offsets + stride;   // zero between calls (the scan step clears what the histogram added)
  int* cursor = counts + stride;
  const int npairs = T * top;
  B2_REQUIRE((size_t)experts * sizeof(int) <= 48 * 1024, "route_permute: %d experts", experts);
  if (npairs <= 1024) {
    B2_CUDA_OK(b2_launch(route_permute_small_kernel, dim3(1), dim3(1024), (size_t)experts * sizeof(int), s, idx, npairs, top, experts, offsets,
                         slot_token, pair_slot));
    return 0;
  }
  B2_CUDA_OK(b2_launch(route_count_kernel, dim3((npairs + 255) / 256), dim3(256), (size_t)experts * sizeof(int), s, idx, npairs, experts, counts));
  B2_CUDA_OK(b2_launch(route_scan_kernel, dim3(1), dim3(32), 0, s, counts, experts, offsets, cursor));
  B2_CUDA_OK(b2_launch(route_place_kernel, dim3((npairs + 255) / 256), dim3(256), 0, s, idx, npairs, top, cursor, slot_token, pair_slot));
  return 0;
}

int launch_route_table(const int32_t* ids, const int32_t* table, int vocab, int experts, int top, int32_t* idx, float* weight, int T, cudaStream_t s) {
  if (T <= 0) return 0;
  const int npairs = T * top;
  B2_CUDA_OK(b2_launch(route_table_kernel, dim3((npairs + 255) / 256), dim3(256), 0, s, ids, table, vocab, experts, top, idx, weight, npairs));
  return 0;
}

int launch_route_slot_weights(const float* weight, const int32_t* pair_slot, float* slot_weight, int npairs, cudaStream_t s) {
  if (npairs <= 0) return 0;
  B2_CUDA_OK(b2_launch(route_slot_weights_kernel, dim3((npairs + 255) / 256), dim3(256), 0, s, weight, pair_slot, slot_weight, npairs));
  return 0;
}

int launch_route_combine(float* h, const float* mix, const float* y, const float* weight, const int32_t* pair_slot, int T, int W, int top,
                         cudaStream_t s) {
  if (T <= 0) return 0;
  B2_CUDA_OK(b2_launch(route_combine_kernel, dim3(T), dim3(256), 0, s, h, mix, y, weight, pair_slot, W, top));
  return 0;
}

}  // namespace b2
