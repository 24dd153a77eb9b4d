// Attention over a latent that all heads share (SpanAttention without a V pool).
//
//   prepare  from projection rows to the cached latent and key part and the rotated parts of the queries
//   tokens   decoded tokens of wide latents: one CTA reads every latent once for up to 32 heads
//   gather   latents of whole contexts side by side, for prompts: a matrix product then makes keys and
//            values of all heads, and attention_span_mma.cu runs over those
#include <algorithm>

#include "layered_ops.h"
#include "prep_core.cuh"
#include "span_core.cuh"

namespace hb {

// One CTA per row.  V > 1: all widths and offsets are multiples of V, and so is the number of pairs.
template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) latent_prepare_kernel(const LatentPrep a) {
  pdl_trigger();
  extern __shared__ float s_cs[];  // [pairs] cosines, [pairs] sines
  __shared__ float red[33];
  pdl_grid_wait();
  const int64_t row = blockIdx.x, slot = a.slots[row];
  const int tid = threadIdx.x, P = a.pairs, R = a.rot_dim, C = a.rank, QD = a.dim + R, KD = C + R;
  const bool keep = slot >= 0 && slot < a.num_blocks * HB_BLOCK_SIZE;
  T* pr = (T*)a.p + row * a.ld;
  const T* latent = pr + a.off_c;
  float f[V], g[V];
  if (tid * V < C) Run<T, V>::load(f, latent + tid * V);  // on its way while the angles are formed
  angles_of(s_cs, a.rotation, P, a.pos[row], a.rotation_gain);
  float ss = 0.f;
  for (int i = tid * V; i < C; i += kPrepThreads * V) {
    if (i >= kPrepThreads * V) Run<T, V>::load(f, latent + i);
#pragma unroll
    for (int j = 0; j < V; ++j) ss = fmaf(f[j], f[j], ss);
  }
  ss = block_sum(ss, red);  // (its barriers also publish the angles)
  T* entry = keep ? (T*)a.kc + pool_at(slot, 1, 0, KD, 0) : nullptr;
  if (keep) {
    const float r = 1.f / sqrtf(ss / (float)C + a.eps);
    for (int i = tid * V; i < C; i += kPrepThreads * V) {
      if (C > kPrepThreads * V) Run<T, V>::load(f, latent + i);
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] *= r * a.norm[i + j];
      Run<T, V>::store(entry + i, f);
    }
  }
  // rotated parts: one per head of the queries, then the key's
  const int turned = P / V, per = turned + (R - 2 * P) / V;
  for (int i = tid; i < (a.heads + (keep ? 1 : 0)) * per; i += kPrepThreads) {
    const int h = i / per, u = i % per, d = u < turned ? u * V : P + u * V;
    T* src = pr + (h < a.heads ? a.off_q + h * QD + a.dim : a.off_c + C) + d;
    T* dst = (h < a.heads ? (T*)a.q + row * a.ld_q + (int64_t)h * KD : entry) + C + d;
    Run<T, V>::load(f, src);
    if (u < turned) {
      Run<T, V>::load(g, src + P);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        float x, y;
        rope_rotate(f[j], g[j], s_cs[d + j], s_cs[P + d + j], &x, &y);
        f[j] = x;
        g[j] = y;
      }
      Run<T, V>::store(dst + P, g);
      if (h < a.heads) {
        Run<T, V>::store(src, f);
        Run<T, V>::store(src + P, g);
      }
    }
    Run<T, V>::store(dst, f);
  }
}

int latent_prepare(cudaStream_t st, const LatentPrep& a, int64_t rows, hb_dtype dtype) {
  if (rows == 0) return HB_OK;
  if (2 * a.pairs > a.rot_dim || a.pairs > 5000 || a.rank < 1)
    return fail(HB_ERR_INVALID_ARG, "latent_prepare: %d pairs of %d channels", a.pairs, a.rot_dim);
  const int n = (int)(16 / dtype_size(dtype));
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = a.dim % n == 0 && a.rot_dim % n == 0 && a.rank % n == 0 && a.pairs % n == 0 && a.off_q % n == 0 &&
                   a.off_c % n == 0 && a.ld % n == 0 && a.ld_q % n == 0 && al(a.p) && al(a.q) && al(a.kc);
  auto launch = [&](auto* k) -> int {
    HB_CUDA_CHECK(launch_pdl(k, dim3((unsigned)rows), dim3(kPrepThreads), (size_t)a.pairs * 2 * sizeof(float), st, a));
    return HB_OK;
  };
  if (dtype == HB_F32) return vec ? launch(latent_prepare_kernel<float, 4>) : launch(latent_prepare_kernel<float, 1>);
  if (dtype == HB_BF16)
    return vec ? launch(latent_prepare_kernel<__nv_bfloat16, 8>) : launch(latent_prepare_kernel<__nv_bfloat16, 1>);
  return fail(HB_ERR_UNSUPPORTED_DTYPE, "latent_prepare runs in bf16 or f32");
}

__global__ void latent_gather_kernel(uint4* __restrict__ dst, const uint4* __restrict__ pool, const int32_t* __restrict__ list, int per,
                                     int64_t num_blocks) {
  pdl_trigger();
  pdl_grid_wait();
  int64_t b = list[blockIdx.x];
  if (b < 0 || b >= num_blocks) b = 0;  // never outside the pool
  for (int i = threadIdx.x; i < per; i += blockDim.x) dst[(int64_t)blockIdx.x * per + i] = pool[b * per + i];
}

int latent_gather(cudaStream_t st, void* dst, const void* pool, const int32_t* list, int n_blocks, int width, int64_t num_blocks,
                  hb_dtype dtype) {
  if (n_blocks == 0) return HB_OK;
  const int per = (int)(width * dtype_size(dtype) * HB_BLOCK_SIZE / 16);
  HB_CUDA_CHECK(launch_pdl(latent_gather_kernel, dim3((unsigned)n_blocks), dim3(256), 0, st, (uint4*)dst, (const uint4*)pool, list, per,
                           num_blocks));
  return HB_OK;
}

// Decoded tokens.  CTA = (row, kv head and slice of up to 8 NT query heads, split).  Its warps work on the
// 64-key tiles of the row side by side:
//   1 warp    brings the tiles in, one bulk copy per key, `stages` tiles ahead
//   4 warps   scores S^T[16 keys, 8 heads] = K Q^T of one block each, softmax, weights to shared memory
//   8 warps   O^T[16 values, 8 heads] += V^T P^T for MT of the value tiles each, one tile behind
// The weights are pairs of bf16 numbers, in two buffers.  Tiles and buffers change hands through mbarriers;
// every wait is bounded: when one runs out the CTA goes on without waiting, and *err is set.
// n_splits > 1: partials (O, m, l) that span_attention_merge sums up.
constexpr int kLatThreads = 13 * 32;
constexpr int kLatKeys = 64;
constexpr int kLatP = kLatKeys + 8;  // padded row of weights
// most query heads of a CTA (the accumulators of wider values leave registers for fewer)
static int latent_most_heads(const SpanAttention& a) { return a.vdim > 512 ? 16 : 32; }
constexpr int kLatStages = 3;        // most tiles in shared memory

template <int MT, int NT>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_tokens_kernel(const SpanAttention a, const int32_t* __restrict__ rows, int n_splits, int stages, float* __restrict__ part) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int HP = NT * 8;
  const HeadSlice hs(a, blockIdx.y);
  const int R = hs.n, D = a.dim, DP = pad16(D), KS = DP + 8, VD = a.vdim, VT = pad16(VD) / 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gi = lane >> 2, t = lane & 3, split = blockIdx.z;
  __nv_bfloat16* s_q = (__nv_bfloat16*)smem;                  // [HP][KS]
  __nv_bfloat16* s_k = s_q + HP * KS;                         // [stages][64][KS]
  __nv_bfloat16* s_p = s_k + (size_t)stages * kLatKeys * KS;  // [2] hi [HP][kLatP], lo [HP][kLatP]
  __shared__ float s_max[2][4][HP], s_alpha[2][HP], s_m[HP], s_sum[4][HP];
  __shared__ __align__(8) uint64_t b_full[kLatStages], b_empty[kLatStages], b_weights[2], b_used[2];
  __shared__ int s_abort;
  if (tid == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(smem_u32(&b_full[s]), 1);
      mbar_init(smem_u32(&b_empty[s]), 12);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(smem_u32(&b_weights[b]), 4);
      mbar_init(smem_u32(&b_used[b]), 8);
    }
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (D % 16)  // padding columns stay zero
    for (int i = tid; i < HP + stages * kLatKeys; i += kLatThreads)
      *reinterpret_cast<uint4*>(s_q + i * KS + D) = make_uint4(0, 0, 0, 0);
  __syncthreads();
  pdl_grid_wait();
  const int64_t row = rows[blockIdx.x];
  const int pos = a.pos[row], lo = a.first_seen(pos);
  const BlockRuns runs = block_runs(pos, pos, a);
  const int n_all = (runs.n + 3) / 4, per = (n_all + n_splits - 1) / n_splits;
  const int first = split * per, n_tiles = max(0, min(n_all, first + per) - first);
  float o[MT][NT][4];  // of the eight warps

  if (warp == 0) {
    const int32_t* table = a.tables + (int64_t)a.row_seg[row] * a.max_blocks;
    const uint32_t bytes = (uint32_t)D * 2;
    int issued = 0;
    for (int i = 0; i < n_tiles; ++i, ++issued) {
      const int s = i % stages;
      if (i >= stages && !__all_sync(0xffffffffu, mbar_wait(smem_u32(&b_empty[s]), (uint32_t)(i / stages - 1) & 1u, &s_abort))) break;
      const uint32_t bar = smem_u32(&b_full[s]);
      if (lane == 0) mbar_expect_tx(bar, kLatKeys * bytes);
      __syncwarp();
#pragma unroll
      for (int r = lane; r < kLatKeys; r += 32) {
        // past the last block: any block will do, its keys are masked
        const int lb = runs.block(min((first + i) * 4 + r / kBS, runs.n - 1));
        int64_t phys = lb < a.max_blocks ? table[lb] : 0;
        if (phys < 0 || phys >= a.num_blocks) phys = 0;  // never outside the pool
        bulk_load(smem_u32(s_k + ((size_t)s * kLatKeys + r) * KS), (const __nv_bfloat16*)a.kc + ((phys * a.kv_heads + hs.kvh) * kBS + r % kBS) * D,
                  bytes, bar);
      }
    }
    if (*(volatile int*)&s_abort)  // let every issued copy land before this CTA's shared memory can be reused
      for (int i = max(0, issued - stages); i < issued; ++i)
        for (uint32_t it = 0; it < kSpinLimit && !mbar_try(smem_u32(&b_full[i % stages]), (uint32_t)(i / stages) & 1u); ++it) {
        }
    __syncwarp();
  } else {
    const __nv_bfloat16* q = (const __nv_bfloat16*)a.q + row * a.ld_q + (int64_t)hs.first * D;
    for (int i = tid - 32; i < HP * (D / 8); i += kLatThreads - 32) {
      const int m = i / (D / 8), c = i % (D / 8) * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (m < R) v = *reinterpret_cast<const uint4*>(q + m * D + c);
      *reinterpret_cast<uint4*>(s_q + m * KS + c) = v;
    }
    asm volatile("bar.sync 1, %0;" ::"n"(kLatThreads - 32) : "memory");
  }
  if (warp >= 1 && warp <= 4) {
    const int blk = warp - 1;
    const float sc = a.scale * kLog2e, cap = a.softcap * kLog2e, cap_k = cap > 0.f ? 2.f / a.softcap : 0.f;
    const uint32_t q_addr = smem_u32(s_q + (lane & 7) * KS + (lane >> 3) * 8);  // B fragments of two 16-channel steps
    const uint32_t k_off = (uint32_t)((blk * 16 + (lane & 15)) * KS + (lane >> 4) * 8) * 2;
    float m_run[NT][2], l_run[NT][2];
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      m_run[n][0] = m_run[n][1] = -INFINITY;
      l_run[n][0] = l_run[n][1] = 0.f;
    }
    for (int i = 0; i < n_tiles; ++i) {
      const int st = i % stages, b = i & 1;
      mbar_wait(smem_u32(&b_full[st]), (uint32_t)(i / stages) & 1u, &s_abort);
      __syncwarp();
      const uint32_t base = smem_u32(s_k + (size_t)st * kLatKeys * KS);
      float s[NT][2][4];  // two partial sums, so that neighbouring steps do not wait for each other
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][0][e] = s[n][1][e] = 0.f;
#pragma unroll 3
      for (int ks = 0; ks < DP / 16; ks += 2) {
        uint32_t k0[4], k1[4];
        ldsm_x4(base + k_off + ks * 32, k0[0], k0[1], k0[2], k0[3]);
        const bool two = ks + 1 < DP / 16;
        if (two) ldsm_x4(base + k_off + ks * 32 + 32, k1[0], k1[1], k1[2], k1[3]);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          uint32_t b0, b1, b2, b3;
          // (a lone last step also reads the 16 elements behind it: unused)
          ldsm_x4(q_addr + (n * 8 * KS + ks * 16) * 2, b0, b1, b2, b3);
          mma_bf16_16816(s[n][0], k0, b0, b1);
          if (two) mma_bf16_16816(s[n][1], k1, b2, b3);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&b_empty[st]));
      const int vb = (first + i) * 4 + blk, key0 = vb < runs.n ? runs.block(vb) * kBS : -1;
      const bool full = key0 >= 0 && all_visible(key0, pos, lo, a.keep_first);
      const bool see0 = full || (key0 >= 0 && visible(key0 + gi, pos, lo, a.keep_first));
      const bool see1 = full || (key0 >= 0 && visible(key0 + gi + 8, pos, lo, a.keep_first));
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        float (&p)[4] = s[n][0];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float x = (s[n][0][e] + s[n][1][e]) * sc;
          if (cap > 0.f) x = capped(x, cap, cap_k);
          p[e] = (e < 2 ? see0 : see1) ? x : -INFINITY;
        }
        float x0 = fmaxf(p[0], p[2]), x1 = fmaxf(p[1], p[3]);
#pragma unroll
        for (int w = 4; w < 32; w <<= 1) {
          x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, w));
          x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, w));
        }
        if (gi == 0) { s_max[b][blk][n * 8 + 2 * t] = x0; s_max[b][blk][n * 8 + 2 * t + 1] = x1; }
      }
      asm volatile("bar.sync 2, 128;" ::: "memory");  // the four blocks' maxima
      if (i >= 2) mbar_wait(smem_u32(&b_used[b]), (uint32_t)(i / 2 - 1) & 1u, &s_abort);
      __nv_bfloat16* weights = s_p + b * 2 * HP * kLatP;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int h = n * 8 + 2 * t;
        float (&p)[4] = s[n][0];
        float top[2];
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const float x = fmaxf(fmaxf(s_max[b][0][h + c], s_max[b][1][h + c]), fmaxf(s_max[b][2][h + c], s_max[b][3][h + c]));
          const float m_new = fmaxf(m_run[n][c], x);
          top[c] = m_new == -INFINITY ? 0.f : m_new;  // nothing visible yet
          const float al = ex2(m_run[n][c] - top[c]);
          m_run[n][c] = m_new;
          l_run[n][c] *= al;
          if (blk == 0 && gi == 0) s_alpha[b][h + c] = al;
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          p[e] = ex2(p[e] - top[e & 1]);
          l_run[n][e & 1] += p[e];
          const __nv_bfloat16 hi = __float2bfloat16_rn(p[e]);
          __nv_bfloat16* dst = weights + (h + (e & 1)) * kLatP + blk * 16 + gi + (e < 2 ? 0 : 8);
          dst[0] = hi;
          dst[HP * kLatP] = __float2bfloat16_rn(p[e] - __bfloat162float(hi));
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&b_weights[b]));
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float ll = l_run[n][c];
#pragma unroll
        for (int w = 4; w < 32; w <<= 1) ll += __shfl_xor_sync(0xffffffffu, ll, w);
        if (gi == 0) {
          s_sum[blk][n * 8 + 2 * t + c] = ll;
          if (blk == 0) s_m[n * 8 + 2 * t + c] = m_run[n][c];
        }
      }
  } else if (warp >= 5) {
    const uint32_t v_off = (uint32_t)(((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int k = 0; k < MT; ++k)
#pragma unroll
      for (int n = 0; n < NT; ++n) o[k][n][0] = o[k][n][1] = o[k][n][2] = o[k][n][3] = 0.f;
    for (int i = 0; i < n_tiles; ++i) {
      const int st = i % stages, b = i & 1;
      mbar_wait(smem_u32(&b_full[st]), (uint32_t)(i / stages) & 1u, &s_abort);
      mbar_wait(smem_u32(&b_weights[b]), (uint32_t)(i / 2) & 1u, &s_abort);
      __syncwarp();
      const uint32_t base = smem_u32(s_k + (size_t)st * kLatKeys * KS);
      const __nv_bfloat16* weights = s_p + b * 2 * HP * kLatP;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const float a0 = s_alpha[b][n * 8 + 2 * t], a1 = s_alpha[b][n * 8 + 2 * t + 1];
        if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f))
#pragma unroll
          for (int k = 0; k < MT; ++k) { o[k][n][0] *= a0; o[k][n][1] *= a1; o[k][n][2] *= a0; o[k][n][3] *= a1; }
      }
#pragma unroll
      for (int kb = 0; kb < 4; ++kb) {
        uint32_t hi[NT][2], low[NT][2];
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const uint32_t* p = reinterpret_cast<const uint32_t*>(weights + (n * 8 + gi) * kLatP + kb * 16 + 2 * t);
          hi[n][0] = p[0]; hi[n][1] = p[4];
          low[n][0] = p[HP * kLatP / 2]; low[n][1] = p[HP * kLatP / 2 + 4];
        }
#pragma unroll
        for (int k = 0; k < MT; ++k) {
          const int vt = warp - 5 + 8 * k;
          if (vt < VT) {
            uint32_t va[4];
            ldsm_x4_trans(base + v_off + (kb * 16 * KS + vt * 16) * 2, va[0], va[1], va[2], va[3]);
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_bf16_16816(o[k][n], va, hi[n][0], hi[n][1]);
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_bf16_16816(o[k][n], va, low[n][0], low[n][1]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) {
        mbar_arrive(smem_u32(&b_empty[st]));
        mbar_arrive(smem_u32(&b_used[b]));
      }
    }
  }
  pdl_trigger();
  __syncthreads();
  if (tid == 0 && s_abort && a.err) atomicExch(a.err, HB_ERR_TIMEOUT);
  if (warp < 5) return;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int h = n * 8 + 2 * t + c;
      if (h < R) {
        const int64_t head = hs.first + h;
        const float l = (s_sum[0][h] + s_sum[1][h]) + (s_sum[2][h] + s_sum[3][h]), m = s_m[h];
        float* p = part + (((int64_t)blockIdx.x * a.heads + head) * n_splits + split) * (VD + 2);
        float inv = 1.f / l;
        if (a.sink) {
          const float k = a.sink[head] * kLog2e, top = fmaxf(m, k), f = ex2(m - top);
          inv = f / fmaf(l, f, ex2(k - top));
        }
#pragma unroll
        for (int k = 0; k < MT; ++k)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int col = (warp - 5 + 8 * k) * 16 + gi + e * 8;
            if (col >= VD) continue;
            float x = o[k][n][2 * e + c];
            if (n_splits > 1) {
              p[col] = x;
            } else {
              x *= inv;
              if (a.gate) x *= sigmoid_of(((const uint16_t*)a.gate)[row * a.ld_gate + head * VD + col]);
              ((__nv_bfloat16*)a.out)[row * a.ld_out + head * VD + col] = __float2bfloat16_rn(x);
            }
          }
        if (n_splits > 1 && warp == 5 && gi == 0) {
          p[VD] = m;
          p[VD + 1] = l;
        }
      }
    }
}

static size_t latent_tokens_smem(const SpanAttention& a, int heads, int stages) {
  const size_t KS = pad16(a.dim) + 8;
  return (heads * KS + (size_t)stages * kLatKeys * KS + (size_t)4 * heads * kLatP) * 2;
}
static int latent_heads(const SpanAttention& a) {  // of a slice, padded
  SpanAttention s = a;
  s.cut(latent_most_heads(s));
  return s.slice <= 8 ? 8 : s.slice <= 16 ? 16 : 32;
}

// Narrow latents are left to the kernel of attention_span_mma.cu, whose warps need no barriers.
bool latent_tokens_supported(const SpanAttention& a, hb_dtype dtype) {
  return span_attention_mma_ok(a, dtype) && !a.vc && !a.key_scale && !a.dist_bias && a.vdim > 128 && a.vdim <= 1024 &&
         latent_tokens_smem(a, latent_heads(a), 2) <= kSmemCap;
}

int latent_tokens_units(const SpanAttention& args) {
  SpanAttention a = args;
  a.cut(latent_most_heads(a));
  return a.kv_heads * a.slices();
}

int latent_tokens(cudaStream_t st, const SpanAttention& args, const int32_t* rows, int n_rows, int n_splits, float* part) {
  if (n_rows == 0) return HB_OK;
  SpanAttention a = args;
  a.cut(latent_most_heads(a));
  const int heads = latent_heads(a), stages = latent_tokens_smem(a, heads, kLatStages) <= kSmemCap ? kLatStages : 2;
  const size_t smem = latent_tokens_smem(a, heads, stages);
  auto launch = [&](auto* k) -> int {
    HB_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemCap));
    HB_CUDA_CHECK(launch_pdl(k, dim3((unsigned)n_rows, (unsigned)(a.kv_heads * a.slices()), (unsigned)n_splits), dim3(kLatThreads),
                             smem, st, a, rows, n_splits, stages, part));
    return HB_OK;
  };
  int rc;
#define HB_LATENT(MT)                                            \
  rc = heads == 8 ? launch(latent_tokens_kernel<MT, 1>)          \
       : heads == 16 || MT > 4 ? launch(latent_tokens_kernel<MT, 2>) : launch(latent_tokens_kernel<MT, (MT > 4 ? 2 : 4)>)
  if (a.vdim <= 256) HB_LATENT(2);
  else if (a.vdim <= 512) HB_LATENT(4);
  else HB_LATENT(8);
#undef HB_LATENT
  return rc || n_splits == 1 ? rc : span_attention_merge(st, a, rows, n_rows, n_splits, part);
}

template <typename E>
__global__ void transpose_kernel(E* __restrict__ dst, const E* __restrict__ src, int64_t rows, int64_t cols) {
  __shared__ E tile[32][33];
  const int64_t at = (int64_t)blockIdx.z * rows * cols;
  const int64_t r0 = (int64_t)blockIdx.y * 32, c0 = (int64_t)blockIdx.x * 32;
  for (int i = threadIdx.y; i < 32; i += 8)
    if (r0 + i < rows && c0 + threadIdx.x < cols) tile[i][threadIdx.x] = src[at + (r0 + i) * cols + c0 + threadIdx.x];
  __syncthreads();
  for (int i = threadIdx.y; i < 32; i += 8)
    if (c0 + i < cols && r0 + threadIdx.x < rows) dst[at + (c0 + i) * rows + r0 + threadIdx.x] = tile[threadIdx.x][i];
}

int transpose_matrices(cudaStream_t st, void* dst, const void* src, int64_t n, int64_t rows, int64_t cols, size_t es) {
  const dim3 grid((unsigned)((cols + 31) / 32), (unsigned)((rows + 31) / 32), (unsigned)n), block(32, 8);
  if (n < 1 || n > 65535 || grid.y > 65535) return fail(HB_ERR_INVALID_ARG, "transpose: %lld matrices", (long long)n);
  if (es == 2) transpose_kernel<uint16_t><<<grid, block, 0, st>>>((uint16_t*)dst, (const uint16_t*)src, rows, cols);
  else transpose_kernel<uint32_t><<<grid, block, 0, st>>>((uint32_t*)dst, (const uint32_t*)src, rows, cols);
  HB_LAUNCH_CHECK();
  return HB_OK;
}

}  // namespace hb
