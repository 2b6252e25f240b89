// attn_latent_decode.cu -- the decode step of attention over a shared per-token latent (bf16 cache, absorbed form; see attn_latent.cu for the
// mathematics): every sequence brings one token, i.e. `heads` query rows that all read the same cached rows.
//
// A cluster of eight CTAs takes one sequence and sixteen heads; each CTA takes an eighth of the visible keys.  A sequence of a thousand tokens is
// then about 128 keys per CTA -- four tiles of 32, two of them in flight; two CTAs fit on an SM.  Per tile:
//   S [16 x 32]   = Q . K^T      warp w: keys 8w .. 8w + 7, mma.m16n8k16 (bf16 operands, fp32 sums)
//   P             = exp(S - m)   eight threads per head, running maximum and sum in registers; bf16 P (the summed weights are the rounded ones)
//   O [16 x rank] += P . C       warp w: a quarter of the latent, accumulators in registers; rescaled when a row's maximum moved
// The eight partial results (maximum, sum, unnormalised latents) meet through distributed shared memory: CTA z folds its eighth of the latent for all
// sixteen heads, with the sink as one more term of the denominator, and writes it.  No partials go through global memory and no merge launch follows.
#include "kernels.h"

namespace b2 {

namespace {

constexpr int LD_SPLITS = 8;       // CTAs of a cluster: shares of the keys
constexpr int LD_HEADS = 16, LD_KEYS = 32, LD_THREADS = 128, LD_WARPS = LD_THREADS / 32;
constexpr int LD_SS = LD_KEYS + 8; // row stride of S and P

__device__ __forceinline__ void ld_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ld_matrix4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_matrix4_trans(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ float ld_peer_f32(uint32_t local_addr, int rank) {   // the same shared-memory word of another CTA of the cluster
  uint32_t a;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
  return v;
}
__device__ __forceinline__ void ld_cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

struct LatentDecodeArgs {
  const float* q_abs;
  const float* q_rot;
  const bf16* cache;
  LatentGeom g;
  const int32_t* block_table;
  int bt_stride;
  const int32_t* positions;
  const int32_t* seq_lens;
  const float* sink;
  bf16* out_lat;
  int pages_cap;   // pages of a CTA's share at most
};

__host__ __device__ inline int ld_row_elems(const LatentGeom& g) { return ((g.kv_rank + g.rot_dim + 31) & ~31) + 8; }   // padded row of Q and K
inline size_t ld_smem(const LatentGeom& g, int pages_cap) {
  const int dp = ld_row_elems(g);
  return (size_t)(LD_HEADS + 2 * LD_KEYS) * dp * 2 + (size_t)LD_HEADS * LD_SS * (4 + 2) + (size_t)(5 * LD_HEADS + LD_HEADS * LD_SPLITS) * 4 + (size_t)pages_cap * 4;
}

// NF: 16-wide pieces of the latent per warp (kv_rank <= 64 NF)
template <int NF>
__global__ void __launch_bounds__(LD_THREADS, 2) latent_decode_kernel(LatentDecodeArgs a) {
  extern __shared__ __align__(128) unsigned char smraw[];
  const LatentGeom& g = a.g;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x, h0 = blockIdx.y * LD_HEADS, b = blockIdx.z;
  const int R = g.kv_rank, D = R + g.rot_dim, DP = ld_row_elems(g), D32 = DP - 8, R16 = (R + 15) & ~15, nh = min(LD_HEADS, g.heads - h0);
  bf16* Qs = reinterpret_cast<bf16*>(smraw);                  // [16][DP]
  bf16* Ks = Qs + LD_HEADS * DP;                              // [2][64][DP]
  float* Ss = reinterpret_cast<float*>(Ks + 2 * LD_KEYS * DP);   // [16][72]
  bf16* Ps = reinterpret_cast<bf16*>(Ss + LD_HEADS * LD_SS);  // [16][72]
  float* row_m = reinterpret_cast<float*>(Ps + LD_HEADS * LD_SS);   // [16] maximum and sum of this CTA's share
  float* row_l = row_m + LD_HEADS;
  float* row_f = row_l + LD_HEADS;                            // [16] rescale factor of the tile; afterwards 1 / denominator
  float* wgt = row_f + 3 * LD_HEADS;                          // [16][8] weights of the shares
  int* pages = reinterpret_cast<int*>(wgt + LD_HEADS * LD_SPLITS);
  float* Os = reinterpret_cast<float*>(Ks);                   // after the sweep: [16][R16 + 4]
  // Lengths, positions, the block table and the cached rows (the newest one too) are older than the kernel right before this one, which made the
  // absorbed queries: the keys are on their way before the wait.
  if (a.seq_lens[b] <= 0) {   // (all CTAs of the cluster)
    pdl_wait();
    pdl_launch_dependents();
    return;
  }
  const int pos = a.positions[b];
  // this CTA's keys: 16-key units [u0, u1) of the visible range
  const int lo = g.window > 0 ? max(0, pos - g.window + 1) : 0;
  const int ub = lo >> 4, ue = (pos >> 4) + 1, per = (ue - ub + LD_SPLITS - 1) / LD_SPLITS;
  const int u0 = min(ub + split * per, ue), u1 = min(u0 + per, ue);
  const int k_begin = u0 << 4, k_end = min(u1 << 4, pos + 1);
  const int n_tiles = k_end > k_begin ? (k_end - k_begin + LD_KEYS - 1) / LD_KEYS : 0;
  for (int i = tid; i < u1 - u0; i += LD_THREADS) pages[i] = a.block_table[(size_t)b * a.bt_stride + u0 + i];
  __syncthreads();
  const int cpr = D >> 3;                                     // 16-byte pieces per cached row
  const int csh = (cpr & (cpr - 1)) == 0 ? 31 - __clz(cpr) : -1;
  auto issue = [&](int t) {
    const int k0 = k_begin + t * LD_KEYS;
    const uint32_t base = smem_u32(Ks + (t & 1) * LD_KEYS * DP);
    for (int i = tid; i < LD_KEYS * cpr; i += LD_THREADS) {
      const int j = csh >= 0 ? i >> csh : i / cpr, c = i - j * cpr, kp = k0 + j;
      const bool in = kp < k_end;
      const bf16* src = a.cache + ((size_t)pages[((in ? kp : k_begin) - k_begin) >> 4] * 16 + (kp & 15)) * D + c * 8;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(base + (uint32_t)(j * DP + c * 8) * 2u), "l"(src), "r"(in ? 16 : 0) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (n_tiles > 0) issue(0);
  if (n_tiles > 1) issue(1);
  pdl_wait();
  pdl_launch_dependents();
  // queries, rounded to the operand type; columns past D and heads past the last one are zeros
  if (D == D32 && R % 4 == 0) {   // eight threads per head row, four numbers at a time: independent loads, many in flight together
    const int r = tid >> 3;
    const size_t row = (size_t)b * g.heads + h0 + (r < nh ? r : 0);
    const float4* qa = reinterpret_cast<const float4*>(a.q_abs + row * R);
    const float4* qr = reinterpret_cast<const float4*>(a.q_rot + row * g.rot_dim);
    const int r4 = R >> 2;
#pragma unroll 9
    for (int c = tid & 7; c < (D >> 2); c += 8) {
      const float4 v = c < r4 ? __ldg(qa + c) : __ldg(qr + (c - r4));
      uint2 pk;
      pk.x = r < nh ? pack_bf16x2(v.x, v.y) : 0u;
      pk.y = r < nh ? pack_bf16x2(v.z, v.w) : 0u;
      *reinterpret_cast<uint2*>(Qs + r * DP + c * 4) = pk;
    }
  } else
  for (int i = tid; i < LD_HEADS * (D32 >> 1); i += LD_THREADS) {
    const int r = i / (D32 >> 1), d = (i - r * (D32 >> 1)) * 2;
    float v[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const size_t row = (size_t)b * g.heads + h0 + r;
      v[x] = r >= nh || d + x >= D ? 0.f : (d + x < R ? a.q_abs[row * R + d + x] : a.q_rot[row * g.rot_dim + d + x - R]);
    }
    *reinterpret_cast<uint32_t*>(Qs + r * DP + d) = pack_bf16x2(v[0], v[1]);
  }
  if (D < D32)
    for (int i = tid; i < 2 * LD_KEYS * (D32 - D); i += LD_THREADS) Ks[(i / (D32 - D)) * DP + D + i % (D32 - D)] = __float2bfloat16_rn(0.f);
  float oacc[NF][2][4];
#pragma unroll
  for (int f = 0; f < NF; ++f)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) oacc[f][n][x] = 0.f;
  const int sr = tid >> 3, sq = tid & 7;                      // softmax: head row, and which four keys
  float m_run = -INFINITY, l_run = 0.f;
  const uint32_t q_addr = smem_u32(Qs) + (uint32_t)((lane & 15) * DP + (lane >> 4) * 8) * 2u;
  const uint32_t p_addr = smem_u32(Ps) + (uint32_t)((lane & 15) * LD_SS + (lane >> 4) * 8) * 2u;
  for (int t = 0; t < n_tiles; ++t) {
    if (t + 1 < n_tiles) {
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const uint32_t ks = smem_u32(Ks + (t & 1) * LD_KEYS * DP);
    {   // ---- scores ----
      float acc[2][4];
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[0][x] = acc[1][x] = 0.f;
      const uint32_t k_addr = ks + (uint32_t)((warp * 8 + (lane & 7)) * DP + (lane >> 3) * 8) * 2u;
#pragma unroll 4
      for (int d = 0; d < D32; d += 32) {
        uint32_t qa[4], qb[4], kf[4];
        ld_matrix4(qa, q_addr + d * 2);
        ld_matrix4(qb, q_addr + d * 2 + 32);
        ld_matrix4(kf, k_addr + d * 2);
        ld_mma(acc[0], qa, kf[0], kf[1]);
        ld_mma(acc[1], qb, kf[2], kf[3]);
      }
      const int r = lane >> 2, c = warp * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(Ss + r * LD_SS + c) = make_float2((acc[0][0] + acc[1][0]) * g.scale, (acc[0][1] + acc[1][1]) * g.scale);
      *reinterpret_cast<float2*>(Ss + (r + 8) * LD_SS + c) = make_float2((acc[0][2] + acc[1][2]) * g.scale, (acc[0][3] + acc[1][3]) * g.scale);
    }
    __syncthreads();
    {   // ---- weights ----
      const float4 s4 = *reinterpret_cast<const float4*>(Ss + sr * LD_SS + sq * 4);
      float s[4] = {s4.x, s4.y, s4.z, s4.w};
      const int kp = k_begin + t * LD_KEYS + sq * 4;
      float mx = -INFINITY;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        if (kp + x < lo || kp + x >= k_end) s[x] = -INFINITY;
        mx = fmaxf(mx, s[x]);
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_new = fmaxf(m_run, mx), f = m_run == -INFINITY ? 0.f : expf(m_run - m_new);
      float p[4], sum = 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        p[x] = s[x] == -INFINITY ? 0.f : __bfloat162float(__float2bfloat16_rn(expf(s[x] - m_new)));   // the weights that are summed are the weights
        sum += p[x];                                                                                  // that multiply the latents
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      l_run = l_run * f + sum;
      m_run = m_new;
      uint2 pk;
      pk.x = pack_bf16x2(p[0], p[1]);
      pk.y = pack_bf16x2(p[2], p[3]);
      *reinterpret_cast<uint2*>(Ps + sr * LD_SS + sq * 4) = pk;
      if (sq == 0) row_f[sr] = f;
    }
    __syncthreads();
    {   // ---- weighted latents ----
      const float f0 = row_f[lane >> 2], f1 = row_f[(lane >> 2) + 8];
#pragma unroll
      for (int f = 0; f < NF; ++f)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          oacc[f][n][0] *= f0; oacc[f][n][1] *= f0; oacc[f][n][2] *= f1; oacc[f][n][3] *= f1;
        }
      const uint32_t v_addr = ks + (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * DP + (lane >> 4) * 8) * 2u;
#pragma unroll
      for (int kk = 0; kk < LD_KEYS; kk += 16) {
        uint32_t pa[4];
        ld_matrix4(pa, p_addr + kk * 2);
#pragma unroll
        for (int f = 0; f < NF; ++f) {
          const int d0 = (warp * NF + f) * 16;
          if (d0 >= R16) continue;   // warp-uniform
          uint32_t vb[4];
          ld_matrix4_trans(vb, v_addr + (uint32_t)(kk * DP + d0) * 2u);
          ld_mma(oacc[f][0], pa, vb[0], vb[1]);
          ld_mma(oacc[f][1], pa, vb[2], vb[3]);
        }
      }
    }
    __syncthreads();   // the tile has been read: its stage may be filled again (and after the last one, become the output)
    if (t + 2 < n_tiles) issue(t + 2);
  }
  __syncthreads();
  const int OLD = R16 + 4;
#pragma unroll
  for (int f = 0; f < NF; ++f) {
    const int d0 = (warp * NF + f) * 16;
    if (d0 >= R16) continue;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int r = lane >> 2, d = d0 + n * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(Os + r * OLD + d) = make_float2(oacc[f][n][0], oacc[f][n][1]);
      *reinterpret_cast<float2*>(Os + (r + 8) * OLD + d) = make_float2(oacc[f][n][2], oacc[f][n][3]);
    }
  }
  if (sq == 0) {
    row_m[sr] = m_run;
    row_l[sr] = l_run;
  }
  __syncwarp();
  ld_cluster_sync();
  // ---- the shares of the keys meet: this CTA folds dims [split * dw, ...) of every head ----
  if (tid < LD_HEADS) {
    float mz[LD_SPLITS], lz[LD_SPLITS];
#pragma unroll
    for (int z = 0; z < LD_SPLITS; ++z) {
      mz[z] = ld_peer_f32(smem_u32(row_m + tid), z);
      lz[z] = ld_peer_f32(smem_u32(row_l + tid), z);
    }
    const float sk = a.sink != nullptr && tid < nh ? a.sink[h0 + tid] : -INFINITY;
    float mf = sk;
#pragma unroll
    for (int z = 0; z < LD_SPLITS; ++z) mf = fmaxf(mf, mz[z]);
    float den = sk == -INFINITY ? 0.f : expf(sk - mf);
#pragma unroll
    for (int z = 0; z < LD_SPLITS; ++z) {
      const float w = mz[z] == -INFINITY ? 0.f : expf(mz[z] - mf);
      wgt[tid * LD_SPLITS + z] = w;
      den = fmaf(lz[z], w, den);
    }
    row_f[tid] = 1.0f / den;
  }
  __syncthreads();
  const int dw = (R + LD_SPLITS - 1) / LD_SPLITS, d_lo = split * dw, dn = max(0, min(dw, R - d_lo));
  for (int i = tid; i < nh * dn; i += LD_THREADS) {
    const int r = i / dn, d = d_lo + i - r * dn;
    float v[LD_SPLITS], acc = 0.f;
#pragma unroll
    for (int z = 0; z < LD_SPLITS; ++z) v[z] = ld_peer_f32(smem_u32(Os + r * OLD + d), z);
#pragma unroll
    for (int z = 0; z < LD_SPLITS; ++z) acc = fmaf(v[z], wgt[r * LD_SPLITS + z], acc);
    a.out_lat[((size_t)b * g.heads + h0 + r) * R + d] = __float2bfloat16_rn(acc * row_f[r]);
  }
  __syncwarp();
  ld_cluster_sync();   // nobody leaves while a peer may still read its shared memory
}

template <int NF>
int launch_ld(const LatentDecodeArgs& a, int B, size_t smem, cudaStream_t s) {
  static B2PerDeviceOnce once;
  if (once.need()) B2_CUDA_OK(cudaFuncSetAttribute(latent_decode_kernel<NF>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(LD_SPLITS, (a.g.heads + LD_HEADS - 1) / LD_HEADS, B);
  cfg.blockDim = dim3(LD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = LD_SPLITS;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = b2_pdl_enabled() ? 2 : 1;
  B2_CUDA_OK(cudaLaunchKernelEx(&cfg, latent_decode_kernel<NF>, a));
  return 0;
}

}  // namespace

bool latent_decode_ok(const LatentGeom& g, int block_size, int B, int max_context) {
  static const bool on = [] { const char* e = getenv("B2_LATENT_DECODE"); return !(e && *e == '0'); }();   // 0: the key-split kernel of attn_latent.cu (cross-check)
  const int pages_cap = ((max_context + 15) / 16 + LD_SPLITS - 1) / LD_SPLITS + 1;
  if (!on || block_size != 16 || max_context <= 0 || g.kv_rank > 512 || (g.kv_rank + g.rot_dim) % 8 != 0 || ld_smem(g, pages_cap) > 220 * 1024) return false;
  // few sequences over a very long cache leave most SMs idle with eight shares each: the other kernel cuts finer
  const int clusters = B * ((g.heads + LD_HEADS - 1) / LD_HEADS);
  return clusters >= 8 || max_context <= 4096;
}

int launch_latent_decode(const float* q_abs, const float* q_rot, const bf16* cache, const LatentGeom& g, const int32_t* block_table, int bt_stride,
                         const int32_t* positions, const int32_t* seq_lens, const float* sink, bf16* out_lat, int B, int max_context, cudaStream_t s) {
  if (B <= 0) return 0;
  const int pages_cap = ((max_context + 15) / 16 + LD_SPLITS - 1) / LD_SPLITS + 1;
  const LatentDecodeArgs a{q_abs, q_rot, cache, g, block_table, bt_stride, positions, seq_lens, sink, out_lat, pages_cap};
  const size_t smem = ld_smem(g, pages_cap);
  const int nf = (g.kv_rank + 16 * LD_WARPS - 1) / (16 * LD_WARPS);
  if (nf <= 1) return launch_ld<1>(a, B, smem, s);
  if (nf == 2) return launch_ld<2>(a, B, smem, s);
  if (nf <= 4) return launch_ld<4>(a, B, smem, s);
  return launch_ld<8>(a, B, smem, s);
}

}  // namespace b2
