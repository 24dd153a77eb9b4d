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
  T* qr = a.qs ? (T*)a.qs + row * a.ld_qs : pr + a.off_q;
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
  if (!a.halves) {  // neighbours
    const int per = (V == 1 ? P : 0) + (V == 1 ? R - 2 * P : R / V);
    for (int i = tid; i < (a.heads + (keep ? 1 : 0)) * per; i += kPrepThreads) {
      const int h = i / per, u = i % per;
      T* src = h < a.heads ? qr + h * QD + a.dim : pr + a.off_c + C;
      T* dst = (h < a.heads ? (T*)a.q + row * a.ld_q + (int64_t)h * KD : entry) + C;
      if constexpr (V == 1) {  // a pair, or a channel behind them
        if (u < P) {
          float x, y;
          rope_rotate(to_f32<T>(src[2 * u]), to_f32<T>(src[2 * u + 1]), s_cs[u], s_cs[P + u], &x, &y);
          dst[2 * u] = from_f32<T>(x);
          dst[2 * u + 1] = from_f32<T>(y);
          if (h < a.heads) {
            src[2 * u] = from_f32<T>(x);
            src[2 * u + 1] = from_f32<T>(y);
          }
        } else {
          dst[P + u] = src[P + u];
        }
      } else {
        const int d = u * V;
        Run<T, V>::load(f, src + d);
        if (d < 2 * P) {
#pragma unroll
          for (int j = 0; j < V; j += 2) {
            float x, y;
            rope_rotate(f[j], f[j + 1], s_cs[(d + j) / 2], s_cs[P + (d + j) / 2], &x, &y);
            f[j] = x;
            f[j + 1] = y;
          }
          if (h < a.heads) Run<T, V>::store(src + d, f);
        }
        Run<T, V>::store(dst + d, f);
      }
    }
    return;
  }
  const int turned = P / V, per = turned + (R - 2 * P) / V;
  for (int i = tid; i < (a.heads + (keep ? 1 : 0)) * per; i += kPrepThreads) {
    const int h = i / per, u = i % per, d = u < turned ? u * V : P + u * V;
    T* src = (h < a.heads ? qr + h * QD + a.dim : pr + a.off_c + C) + d;
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
  const bool vec = a.dim % n == 0 && a.rot_dim % n == 0 && a.rank % n == 0 && (a.halves ? a.pairs % n == 0 : 2 * a.pairs % n == 0) &&
                   (a.qs ? a.ld_qs % n == 0 && al(a.qs) : a.off_q % n == 0) &&
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
// 16-key blocks of the row side by side:
//   4 warps   bring the blocks in, every fourth each, into a ring of `ring` blocks (bulk copies, one per key,
//             were slower: their issue took longer than the block's arithmetic)
//   4 warps   scores S^T[16 keys, 8 heads] = K Q^T of every fourth block each, weights to shared memory
//   8 warps   O^T[16 values, 8 heads] += V^T P^T for MT of the value tiles each, block after block
// The weights 2^(score - ref) are pairs of bf16 numbers and come with their references: the largest score
// of the first four blocks, until a warp meets one that lies kLatSlack above its own.  So the warps need no
// barrier after their first blocks, and the accumulating warps bring blocks of different references
// together where there are any.  Blocks and weights change hands through mbarriers; every wait
// is bounded: when one runs out the CTA goes on without waiting, and *err is set.
// n_splits > 1: partials (O, ref, l) that span_attention_merge sums up.
constexpr int kLatLoaders = 4, kLatThreads = (kLatLoaders + 4 + 8) * 32;
constexpr int kLatP = kBS + 8;       // padded row of weights
constexpr int kLatWeights = 8;       // blocks of weights
constexpr float kLatSlack = 8.f;
constexpr int kLatRing = 16;         // most blocks in shared memory
// Where block j lies in the ring, and the parity of the ring's round, without divisions.
struct RingPlace {
  int at;
  uint32_t parity = 0;
  __device__ __forceinline__ void step(int by, int ring) {
    at += by;
    if (at >= ring) {
      at -= ring;
      parity ^= 1u;
    }
  }
};
// most query heads of a CTA (the accumulators of wider values leave registers for fewer)
static int latent_most_heads(const SpanAttention& a) { return a.vdim > 512 ? 16 : 32; }

template <int MT, int NT>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_tokens_kernel(const SpanAttention a, const int32_t* __restrict__ rows, int n_splits, int ring, float* __restrict__ part) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int HP = NT * 8;
  const HeadSlice hs(a, blockIdx.y);
  const int R = hs.n, D = a.dim, DP = pad16(D), KS = DP + 8, VD = a.vdim, VT = pad16(VD) / 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gi = lane >> 2, t = lane & 3, split = blockIdx.z;
  __nv_bfloat16* s_q = (__nv_bfloat16*)smem;                  // [HP][KS]
  __nv_bfloat16* s_k = s_q + HP * KS;                         // [ring][16][KS]
  __nv_bfloat16* s_p = s_k + (size_t)ring * kBS * KS;         // [kLatWeights] hi [HP][kLatP], lo [HP][kLatP]
  __shared__ float s_ref[kLatWeights][HP], s_first[4][HP], s_last[4][HP], s_sum[4][HP];
  __shared__ __align__(8) uint64_t b_full[kLatRing], b_empty[kLatRing], b_weights[kLatWeights], b_used[kLatWeights];
  __shared__ int s_abort;
  if (tid == 0) {
    for (int s = 0; s < ring; ++s) {
      mbar_init(smem_u32(&b_full[s]), 32);
      mbar_init(smem_u32(&b_empty[s]), 1 + 8);
    }
    for (int b = 0; b < kLatWeights; ++b) {
      mbar_init(smem_u32(&b_weights[b]), 1);
      mbar_init(smem_u32(&b_used[b]), 8);
    }
    s_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (D % 16)  // padding columns stay zero
    for (int i = tid; i < HP + ring * kBS; i += kLatThreads)
      *reinterpret_cast<uint4*>(s_q + i * KS + D) = make_uint4(0, 0, 0, 0);
  __syncthreads();
  pdl_grid_wait();
  const int64_t row = rows[blockIdx.x];
  const int pos = a.pos[row], lo = a.first_seen(pos);
  const BlockRuns runs = block_runs(pos, pos, a);
  const int per = (runs.n + n_splits - 1) / n_splits;
  const int first = split * per, n_blocks = max(0, min(runs.n, first + per) - first);
  float o[MT][NT][4], ref[NT][2], col[NT];  // of the eight warps: sums, references of heads 8n + 2t (+ 1) and 8n + gi

  if (warp < kLatLoaders) {
    const int32_t* table = a.tables + (int64_t)a.row_seg[row] * a.max_blocks;
    const BlockCopy copy(D, lane);
    int tab = 0;
    RingPlace place{warp};
    for (int j = warp, i = 0; j < n_blocks; j += 4, ++i, place.step(4, ring)) {
      const int s = place.at;
      if (i % 32 == 0) {  // block table entries of this warp, 32 at a time, one per lane
        const int lb = runs.block(min(first + j + 4 * lane, runs.n - 1));
        tab = lb < a.max_blocks ? table[lb] : 0;
        if (tab < 0 || tab >= a.num_blocks) tab = 0;  // never outside the pool
      }
      if (j >= ring && !__all_sync(0xffffffffu, mbar_wait(smem_u32(&b_empty[s]), place.parity ^ 1u, &s_abort))) break;
      const int64_t phys = __shfl_sync(0xffffffffu, tab, i % 32);
      copy(smem_u32(s_k + (size_t)s * kBS * KS), KS * 2,
           (const __nv_bfloat16*)a.kc + (phys * a.kv_heads + hs.kvh) * kBS * D, D);
      mbar_arrive_copies(smem_u32(&b_full[s]));
    }
    cp_async_wait<0>();
  } else {
    const __nv_bfloat16* q = (const __nv_bfloat16*)a.q + row * a.ld_q + (int64_t)hs.first * D;
    for (int i = tid - kLatLoaders * 32; i < HP * (D / 8); i += kLatThreads - kLatLoaders * 32) {
      const int m = i / (D / 8), c = i % (D / 8) * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (m < R) v = *reinterpret_cast<const uint4*>(q + m * D + c);
      *reinterpret_cast<uint4*>(s_q + m * KS + c) = v;
    }
    asm volatile("bar.sync 1, %0;" ::"n"(kLatThreads - kLatLoaders * 32) : "memory");
  }
  if (warp >= kLatLoaders && warp < kLatLoaders + 4) {
    const int blk = warp - kLatLoaders;
    const float sc = a.scale * kLog2e, cap = a.softcap * kLog2e, cap_k = cap > 0.f ? 2.f / a.softcap : 0.f;
    const uint32_t q_addr = smem_u32(s_q + (lane & 7) * KS + (lane >> 3) * 8);  // B fragments of two 16-channel steps
    const uint32_t k_off = (uint32_t)((lane & 15) * KS + (lane >> 4) * 8) * 2;
    float ref[NT][2], l[NT][2];  // of heads 8n + 2t, 8n + 2t + 1
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      ref[n][0] = ref[n][1] = -INFINITY;
      l[n][0] = l[n][1] = 0.f;
    }
    auto raise = [&](int n, int c, float to) {
      l[n][c] *= ref[n][c] == -INFINITY ? 0.f : ex2(ref[n][c] - to);
      ref[n][c] = to;
    };
    auto meet = [&] {  // one reference for the first blocks of all four warps
#pragma unroll
      for (int n = 0; n < NT; ++n)
        if (gi == 0) { s_first[blk][n * 8 + 2 * t] = ref[n][0]; s_first[blk][n * 8 + 2 * t + 1] = ref[n][1]; }
      asm volatile("bar.sync 2, 128;" ::: "memory");
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int h = n * 8 + 2 * t + c;
          ref[n][c] = fmaxf(fmaxf(s_first[0][h], s_first[1][h]), fmaxf(s_first[2][h], s_first[3][h]));
        }
    };
    if (blk >= n_blocks) meet();
    RingPlace place{blk};
    for (int j = blk; j < n_blocks; j += 4, place.step(4, ring)) {
      const int st = place.at, b = j % kLatWeights;
      mbar_wait(smem_u32(&b_full[st]), place.parity, &s_abort);
      __syncwarp();
      const uint32_t base = smem_u32(s_k + (size_t)st * kBS * KS);
      float s[NT][2][4];  // two partial sums, so that neighbouring steps do not wait for each other
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[n][0][e] = s[n][1][e] = 0.f;
      // fragments of two 16-channel steps; the next ones are fetched before the current ones are used
      uint32_t k[2][2][4], qf[2][NT][4];
      const int n_ks = (DP / 16 + 1) / 2;
      auto fetch = [&](uint32_t (&kk)[2][4], uint32_t (&qq)[NT][4], int ks) {
        // (behind the last step: the padding of the row and the first channels of the next one, unused)
        ldsm_x4(base + k_off + ks * 64, kk[0][0], kk[0][1], kk[0][2], kk[0][3]);
        if (2 * ks + 1 < DP / 16) ldsm_x4(base + k_off + ks * 64 + 32, kk[1][0], kk[1][1], kk[1][2], kk[1][3]);
#pragma unroll
        for (int n = 0; n < NT; ++n) ldsm_x4(q_addr + (n * 8 * KS + ks * 32) * 2, qq[n][0], qq[n][1], qq[n][2], qq[n][3]);
      };
      auto use = [&](const uint32_t (&kk)[2][4], const uint32_t (&qq)[NT][4], int ks) {
#pragma unroll
        for (int n = 0; n < NT; ++n) mma_bf16_16816(s[n][0], kk[0], qq[n][0], qq[n][1]);
        if (2 * ks + 1 < DP / 16)
#pragma unroll
          for (int n = 0; n < NT; ++n) mma_bf16_16816(s[n][1], kk[1], qq[n][2], qq[n][3]);
      };
      fetch(k[0], qf[0], 0);
      for (int ks = 0; ks < n_ks; ks += 2) {
        if (ks + 1 < n_ks) fetch(k[1], qf[1], ks + 1);
        use(k[0], qf[0], ks);
        if (ks + 1 < n_ks) {
          if (ks + 2 < n_ks) fetch(k[0], qf[0], ks + 2);
          use(k[1], qf[1], ks + 1);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&b_empty[st]));
      const int key0 = runs.block(first + j) * kBS;
      const bool full = all_visible(key0, pos, lo, a.keep_first);
      const bool see0 = full || visible(key0 + gi, pos, lo, a.keep_first);
      const bool see1 = full || visible(key0 + gi + 8, pos, lo, a.keep_first);
      bool above = false;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        float (&p)[4] = s[n][0];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float x = (s[n][0][e] + s[n][1][e]) * sc;
          if (cap > 0.f) x = capped(x, cap, cap_k);
          p[e] = (e < 2 ? see0 : see1) ? x : -INFINITY;
          above = above || p[e] > ref[n][e & 1] + kLatSlack;
        }
      }
      if (__any_sync(0xffffffffu, above)) {
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            float x = fmaxf(s[n][0][c], s[n][0][2 + c]);
#pragma unroll
            for (int w = 4; w < 32; w <<= 1) x = fmaxf(x, __shfl_xor_sync(0xffffffffu, x, w));
            const float r = fmaxf(ref[n][c], x);
            if (r > ref[n][c]) raise(n, c, r);
          }
      }
      if (j == blk) meet();
      if (j >= kLatWeights) mbar_wait(smem_u32(&b_used[b]), (uint32_t)(j / kLatWeights - 1) & 1u, &s_abort);
      __nv_bfloat16* weights = s_p + b * 2 * HP * kLatP;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const int h = n * 8 + 2 * t;
        float (&p)[4] = s[n][0];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          p[e] = p[e] == -INFINITY ? 0.f : ex2(p[e] - ref[n][e & 1]);
          l[n][e & 1] += p[e];
          const __nv_bfloat16 hi = __float2bfloat16_rn(p[e]);
          __nv_bfloat16* dst = weights + (h + (e & 1)) * kLatP + gi + (e < 2 ? 0 : 8);
          dst[0] = hi;
          dst[HP * kLatP] = __float2bfloat16_rn(p[e] - __bfloat162float(hi));
        }
        if (gi == 0) { s_ref[b][h] = ref[n][0]; s_ref[b][h + 1] = ref[n][1]; }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&b_weights[b]));
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float ll = l[n][c];
#pragma unroll
        for (int w = 4; w < 32; w <<= 1) ll += __shfl_xor_sync(0xffffffffu, ll, w);
        if (gi == 0) {
          s_sum[blk][n * 8 + 2 * t + c] = ll;
          s_last[blk][n * 8 + 2 * t + c] = ref[n][c];
        }
      }
  } else if (warp >= kLatLoaders + 4) {
    const uint32_t v_off = (uint32_t)(((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int k = 0; k < MT; ++k)
#pragma unroll
      for (int n = 0; n < NT; ++n) o[k][n][0] = o[k][n][1] = o[k][n][2] = o[k][n][3] = 0.f;
#pragma unroll
    for (int n = 0; n < NT; ++n) col[n] = ref[n][0] = ref[n][1] = -INFINITY;
    RingPlace place{0};
    for (int j = 0; j < n_blocks; ++j, place.step(1, ring)) {
      const int st = place.at, b = j % kLatWeights;
      mbar_wait(smem_u32(&b_full[st]), place.parity, &s_abort);
      mbar_wait(smem_u32(&b_weights[b]), (uint32_t)(j / kLatWeights) & 1u, &s_abort);
      __syncwarp();
      const uint32_t base = smem_u32(s_k + (size_t)st * kBS * KS);
      const __nv_bfloat16* weights = s_p + b * 2 * HP * kLatP;
      uint32_t hi[NT][2], low[NT][2];
      bool moved = false;
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        const uint32_t* p = reinterpret_cast<const uint32_t*>(weights + (n * 8 + gi) * kLatP + 2 * t);
        hi[n][0] = p[0]; hi[n][1] = p[4];
        low[n][0] = p[HP * kLatP / 2]; low[n][1] = p[HP * kLatP / 2 + 4];
        const float g = s_ref[b][n * 8 + gi];
        moved = moved || g != col[n];
      }
      if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
        for (int n = 0; n < NT; ++n) {
#pragma unroll
          for (int c = 0; c < 2; ++c) {  // the sums so far
            const float to = fmaxf(ref[n][c], s_ref[b][n * 8 + 2 * t + c]);
            const float f = ref[n][c] == to ? 1.f : ex2(ref[n][c] - to);
            ref[n][c] = to;
#pragma unroll
            for (int k = 0; k < MT; ++k) { o[k][n][c] *= f; o[k][n][2 + c] *= f; }
          }
          const float g = s_ref[b][n * 8 + gi], to = fmaxf(col[n], g);
          const float f = g == to ? 1.f : ex2(g - to);  // the block's weights
          col[n] = to;
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const float2 h2 = unpack_bf16(hi[n][x]), l2 = unpack_bf16(low[n][x]);
            split_bf16((h2.x + l2.x) * f, (h2.y + l2.y) * f, hi[n][x], low[n][x]);
          }
        }
      }
      {
        // two value tiles at a time, the next two fetched before the current ones are used; the low halves of
        // the weights follow the high ones of both
        uint32_t va[2][2][4];
        auto fetch = [&](uint32_t (&v)[2][4], int k) {
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            const int vt = min(warp - kLatLoaders - 4 + 8 * (k + x), VT - 1);  // past the last: unused
            ldsm_x4_trans(base + v_off + vt * 32, v[x][0], v[x][1], v[x][2], v[x][3]);
          }
        };
        fetch(va[0], 0);
#pragma unroll
        for (int k = 0; k < MT; k += 2) {
          if (k + 2 < MT) fetch(va[(k / 2 + 1) & 1], k + 2);
          const uint32_t (&v)[2][4] = va[(k / 2) & 1];
#pragma unroll
          for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_bf16_16816(o[k + x][n], v[x], hi[n][0], hi[n][1]);
#pragma unroll
          for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_bf16_16816(o[k + x][n], v[x], low[n][0], low[n][1]);
        }
        __syncwarp();
        if (lane == 0) {
          mbar_arrive(smem_u32(&b_empty[st]));
          mbar_arrive(smem_u32(&b_used[b]));
        }
      }
    }
  }
  pdl_trigger();
  __syncthreads();
  if (tid == 0 && s_abort && a.err) atomicExch(a.err, HB_ERR_TIMEOUT);
  if (warp < kLatLoaders + 4) return;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int h = n * 8 + 2 * t + c;
      if (h < R) {
        const int64_t head = hs.first + h;
        const float m = ref[n][c];
        float l = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w)
          if (s_last[w][h] != -INFINITY) l = fmaf(s_sum[w][h], ex2(s_last[w][h] - m), l);
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
            const int col = (warp - kLatLoaders - 4 + 8 * k) * 16 + gi + e * 8;
            if (col >= VD) continue;
            float x = o[k][n][2 * e + c];
            if (n_splits > 1) {
              p[col] = x;
            } else {
              x *= inv;
              if (a.gate) x *= sigmoid_of(((const uint16_t*)a.gate)[a.gate_at(row, head, col)]);
              ((__nv_bfloat16*)a.out)[row * a.ld_out + head * VD + col] = __float2bfloat16_rn(x);
            }
          }
        if (n_splits > 1 && warp == kLatLoaders + 4 && gi == 0) {
          p[VD] = m;
          p[VD + 1] = l;
        }
      }
    }
}

// Blocks the ring may have beside everything else.
static int latent_ring(const SpanAttention& a, int heads) {
  const size_t row = (size_t)(pad16(a.dim) + 8) * 2, fixed = heads * row + (size_t)kLatWeights * 2 * heads * kLatP * 2;
  return fixed < kSmemCap ? (int)std::min<size_t>(kLatRing, (kSmemCap - fixed) / (kBS * row)) : 0;
}
static size_t latent_tokens_smem(const SpanAttention& a, int heads) {
  const size_t row = (size_t)(pad16(a.dim) + 8) * 2;
  return heads * row + (size_t)kLatWeights * 2 * heads * kLatP * 2 + latent_ring(a, heads) * kBS * row;
}
static int latent_heads(const SpanAttention& a) {  // of a slice, padded
  SpanAttention s = a;
  s.cut(latent_most_heads(s));
  return s.slice <= 8 ? 8 : s.slice <= 16 ? 16 : 32;
}

// Narrow latents are left to the kernel of attention_span_mma.cu, whose warps need no barriers.
bool latent_tokens_supported(const SpanAttention& a, hb_dtype dtype) {
  return span_attention_mma_ok(a, dtype) && !a.vc && !a.key_scale && !a.dist_bias && a.vdim > 128 && a.vdim <= 1024 &&
         latent_ring(a, latent_heads(a)) >= 6;
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
  const int heads = latent_heads(a);
  const size_t smem = latent_tokens_smem(a, heads);
  auto launch = [&](auto* k) -> int {
    HB_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemCap));
    HB_CUDA_CHECK(launch_pdl(k, dim3((unsigned)n_rows, (unsigned)(a.kv_heads * a.slices()), (unsigned)n_splits), dim3(kLatThreads),
                             smem, st, a, rows, n_splits, latent_ring(a, heads), part));
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
