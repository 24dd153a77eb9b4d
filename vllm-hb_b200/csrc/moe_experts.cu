// Mixture of experts with top-k routing (softmax over the chosen logits; sigmoid scores with the choice
// limited to the best groups of experts; or softmax over all with a corrected choice, where some outputs
// may hand the row itself on), each expert run on its own rows only.
//
//   route   logits, the top experts of every row and their weights; every (row, expert) draws a rank
//           among the expert's rows; the last CTA turns the counts into batch tiles
//   gather  rows to the places of their experts (tiles of m_pad places that belong to one expert)
//   (two grouped GEMMs, gemm_tc.cu / gemm_simt.cu; the weighted sum is part of streams_mix)
//
// The order of the rows inside an expert depends on timing; no result does, because rows do not
// meet before the weighted sum, which runs in the order of the router.
#include <algorithm>

#include "gemm.h"
#include "layered_ops.h"

namespace hb {

constexpr int kRouteThreads = 256;
constexpr int kRouteWarps = kRouteThreads / 32;

// RB rows per CTA share every router row they read.
template <typename T, int RB>
__global__ void __launch_bounds__(kRouteThreads)
moe_route_top_kernel(const MoeRouting m, const T* __restrict__ h, int64_t ld_h, const T* __restrict__ router,
                     const float* __restrict__ bias, int64_t rows, int64_t width) {
  pdl_trigger();
  extern __shared__ float s_logit[];  // [RB][outputs], then [RB][groups] and (softmax_all) [RB][outputs] scores
  __shared__ int s_last;
  pdl_grid_wait();
  constexpr int N = Vec16<T>::N;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, E = m.experts, O = m.outputs();
  const int64_t row0 = (int64_t)blockIdx.x * RB;
  const int nr = (int)min((int64_t)RB, rows - row0);
  const bool vec = width % N == 0 && ld_h % N == 0;
  for (int e = warp; e < O; e += kRouteWarps) {
    const T* w = router + (int64_t)e * width;
    float acc[RB];
#pragma unroll
    for (int r = 0; r < RB; ++r) acc[r] = 0.f;
    if (vec) {
#pragma unroll 4
      for (int64_t v = lane; v < width / N; v += 32) {
        Vec16<T> a, b;
        b.load(w + v * N);
        float fa[N], fb[N];
        b.unpack(fb);
#pragma unroll
        for (int r = 0; r < RB; ++r) {
          if (r < nr) {
            a.load(h + (row0 + r) * ld_h + v * N);
            a.unpack(fa);
#pragma unroll
            for (int j = 0; j < N; ++j) acc[r] = fmaf(fa[j], fb[j], acc[r]);
          }
        }
      }
    } else {
      for (int64_t i = lane; i < width; i += 32) {
        const float b = to_f32<T>(w[i]);
#pragma unroll
        for (int r = 0; r < RB; ++r)
          if (r < nr) acc[r] = fmaf(to_f32<T>(h[(row0 + r) * ld_h + i]), b, acc[r]);
      }
    }
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      const float s = warp_sum(acc[r]);
      if (lane == 0) {
        const float z = bias ? s + bias[e] : s;
        s_logit[r * O + e] = m.sigmoid ? 1.f / (1.f + expf(-z)) : z;
      }
    }
  }
  __syncthreads();
  // one warp per row: the largest logit `top` times, the lower expert among equals
  for (int r = warp; r < nr; r += kRouteWarps) {
    float *z = s_logit + r * O, *score = s_logit + RB * (O + m.groups) + r * O;
    const int64_t at = (row0 + r) * m.picks();
    if (m.keep < m.groups) {
      // groups by the sum of their two largest scores; experts of the others cannot be chosen
      float* gs = s_logit + RB * O + r * m.groups;
      const int size = E / m.groups;
      for (int g = lane; g < m.groups; g += 32) {
        float a = -INFINITY, b = -INFINITY;
        for (int e = g * size; e < (g + 1) * size; ++e) {
          const float v = z[e];
          if (v > a) { b = a; a = v; }
          else if (v > b) b = v;
        }
        gs[g] = size > 1 ? a + b : a;
      }
      __syncwarp();
      for (int g = lane; g < m.groups; g += 32) {
        int better = 0;  // groups that go first: larger, or equal and lower
        for (int o = 0; o < m.groups; ++o) better += gs[o] > gs[g] || (gs[o] == gs[g] && o < g);
        if (better >= m.keep)
          for (int e = g * size; e < (g + 1) * size; ++e) z[e] = __int_as_float(0x7fc00000);
      }
      __syncwarp();
    }
    if (m.softmax_all) {
      float mx = -INFINITY, total = 0.f;
      for (int e = lane; e < O; e += 32) mx = fmaxf(mx, z[e]);
      mx = warp_max(mx);
      for (int e = lane; e < O; e += 32) {
        score[e] = expf(z[e] - mx);
        total += score[e];
      }
      total = warp_sum(total);
      for (int e = lane; e < O; e += 32) {
        score[e] /= total;
        z[e] = m.correction ? score[e] + m.correction[e] : score[e];
      }
      __syncwarp();
    }
    float first = 0.f, sum = 0.f;
    int mine = 0;        // lane k keeps choice k (of every 32) and its unscaled weight
    float mine_p = 0.f;
    for (int k = 0; k < m.top; ++k) {
      float best = -INFINITY;
      int who = O;
      for (int e = lane; e < O; e += 32)
        if (z[e] > best || who == O) {
          if (!isnan(z[e])) { best = z[e]; who = e; }
        }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float b = __shfl_xor_sync(0xffffffffu, best, o);
        const int w = __shfl_xor_sync(0xffffffffu, who, o);
        if (w < O && (who == O || b > best || (b == best && w < who))) { best = b; who = w; }
      }
      const int e = min(who, O - 1);  // a row of NaNs still names an expert
      if (k == 0) first = best;
      const float p = m.softmax_all ? score[e] : m.sigmoid ? best : expf(best - first);
      sum += p;
      if (lane == 0) z[e] = __int_as_float(0x7fc00000);  // taken
      if (lane == (k & 31)) {
        mine = e;
        mine_p = p;
      }
      __syncwarp();
      if ((k & 31) == 31 || k == m.top - 1) {
        const int at_k = (k & ~31) + lane;
        if (at_k <= k) {
          m.ids[at + at_k] = mine;
          m.weight[at + at_k] = mine_p;
          m.rank[at + at_k] = mine < E ? atomicAdd(m.count + mine, 1) : 0;
        }
      }
    }
    __syncwarp();
    if (!m.softmax_all)
      for (int k = lane; k < m.top; k += 32) m.weight[at + k] /= m.sigmoid ? sum + 1e-20f : sum;  // written by this lane
    if (m.shared && lane == 0) {
      m.ids[at + m.top] = E;
      m.weight[at + m.top] = 1.f;
      m.rank[at + m.top] = (int)(row0 + r);
    }
  }
  // the last CTA: every expert's tiles
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(m.count + E, 1) == (int)gridDim.x - 1;
  __syncthreads();
  if (!s_last || warp != 0) return;
  __threadfence();
  int tile = 0;  // tiles of the experts before this group of 32
  for (int e0 = 0; e0 < E; e0 += 32) {
    const int e = e0 + lane;
    const int n = e < E ? (__ldcg(m.count + e) + m.m_pad - 1) / m.m_pad : 0;
    int incl = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += v;
    }
    const int at = tile + incl - n;
    if (e < E) {
      m.first[e] = at * m.m_pad;
      m.count[e] = 0;
      for (int i = 0; i < n && at + i < m.max_tiles; ++i) m.tile_group[at + i] = e;
    }
    tile += __shfl_sync(0xffffffffu, incl, 31);
  }
  if (m.shared) {
    const int n = (int)((rows + m.m_pad - 1) / m.m_pad);
    if (lane == 0) m.first[E] = tile * m.m_pad;
    for (int i = lane; i < n && tile + i < m.max_tiles; i += 32) m.tile_group[tile + i] = E;
    tile += n;
  }
  for (int i = tile + lane; i < m.max_tiles; i += 32) m.tile_group[i] = -1;
  if (lane == 0) m.count[E] = 0;
}

template <typename T>
__global__ void __launch_bounds__(kRouteThreads)
moe_gather_kernel(const MoeRouting m, T* __restrict__ x, const T* __restrict__ h, int64_t ld) {
  pdl_trigger();
  extern __shared__ int32_t s_place[];  // [picks]
  pdl_grid_wait();
  constexpr int N = Vec16<T>::N;
  const int64_t row = blockIdx.x, places = (int64_t)m.max_tiles * m.m_pad;
  const int picks = m.picks();
  Vec16<T> a;
  int64_t v = threadIdx.x;
  if (v < ld / N) a.load(h + row * ld + v * N);  // on its way while the places are looked up
  for (int k = threadIdx.x; k < picks; k += kRouteThreads) {
    const int64_t at = row * picks + k;
    const int id = m.ids[at];
    const bool expert = id < m.experts || (m.shared && k == m.top);
    const int p = expert ? m.first[id] + m.rank[at] : -1;
    s_place[k] = p < places ? p : 0;  // never outside the buffer
    m.place[at] = s_place[k];
  }
  __syncthreads();
  for (; v < ld / N; v += kRouteThreads) {
    if (v >= kRouteThreads) a.load(h + row * ld + v * N);
    for (int k = 0; k < picks; ++k)
      if (s_place[k] >= 0) a.store(x + (int64_t)s_place[k] * ld + v * N);
  }
}

int moe_route_top(cudaStream_t st, const MoeRouting& m, const void* h, int64_t ld_h, const void* router, const float* bias,
                  int64_t rows, int64_t width, hb_dtype dtype) {
  if (rows == 0) return HB_OK;
  if (m.experts < 1 || m.identity < 0 || m.outputs() > kMoeMaxExperts || m.top < 1 || m.top > m.outputs() || m.m_pad < 1)
    return fail(HB_ERR_INVALID_ARG, "moe_route_top: %d of %d experts (at most %d)", m.top, m.outputs(), kMoeMaxExperts);
  if (((m.identity || m.softmax_all) && m.groups > 1) || (m.identity && m.shared) || (m.correction && !m.softmax_all) ||
      (m.sigmoid && m.softmax_all))
    return fail(HB_ERR_INVALID_ARG, "moe_route_top: scores, groups, identity and shared experts do not go together");
  if (m.groups < 1 || m.experts % m.groups || m.keep < 1 || m.keep > m.groups ||
      (m.groups > 1 && m.top > m.experts / m.groups * m.keep))
    return fail(HB_ERR_INVALID_ARG, "moe_route_top: %d of %d groups of %d experts, top %d", m.keep, m.groups, m.experts, m.top);
  auto launch = [&](auto* k, int rb, auto* t) -> int {
    using T = std::remove_pointer_t<decltype(t)>;
    HB_CUDA_CHECK(launch_pdl(k, dim3((unsigned)((rows + rb - 1) / rb)), dim3(kRouteThreads),
                             (size_t)rb * (m.outputs() * (m.softmax_all ? 2 : 1) + m.groups) * sizeof(float), st, m, (const T*)h, ld_h, (const T*)router, bias, rows, width));
    return HB_OK;
  };
  const bool few = rows <= 296;
  if (dtype == HB_F32)
    return few ? launch(moe_route_top_kernel<float, 1>, 1, (float*)nullptr) : launch(moe_route_top_kernel<float, 4>, 4, (float*)nullptr);
  if (dtype == HB_BF16)
    return few ? launch(moe_route_top_kernel<__nv_bfloat16, 1>, 1, (__nv_bfloat16*)nullptr)
               : launch(moe_route_top_kernel<__nv_bfloat16, 4>, 4, (__nv_bfloat16*)nullptr);
  return fail(HB_ERR_UNSUPPORTED_DTYPE, "moe_route_top runs in bf16 or f32");
}

int moe_gather(cudaStream_t st, const MoeRouting& m, void* x, const void* h, int64_t ld, int64_t rows, hb_dtype dtype) {
  if (rows == 0) return HB_OK;
  const int n = (int)(16 / dtype_size(dtype));
  if (ld % n || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(h) & 15))
    return fail(HB_ERR_INVALID_ARG, "moe_gather: rows must be multiples of 16 bytes");
  const size_t smem = (size_t)m.picks() * sizeof(int32_t);
  if (dtype == HB_F32)
    HB_CUDA_CHECK(launch_pdl(moe_gather_kernel<float>, dim3((unsigned)rows), dim3(kRouteThreads), smem, st, m, (float*)x,
                             (const float*)h, ld));
  else if (dtype == HB_BF16)
    HB_CUDA_CHECK(launch_pdl(moe_gather_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(kRouteThreads), smem, st, m,
                             (__nv_bfloat16*)x, (const __nv_bfloat16*)h, ld));
  else
    return fail(HB_ERR_UNSUPPORTED_DTYPE, "moe_gather runs in bf16 or f32");
  return HB_OK;
}

// ------------------------------------------------------------------- gated activation
// tile_group (may be null): rows of negative groups are skipped, those of group `further` have inter2
// and act2.
template <typename T>
__global__ void gated_act_kernel(T* __restrict__ out, int64_t ld_out, const T* __restrict__ gu, int64_t ld_gu, int64_t inter,
                                 GatedAct act, const int32_t* __restrict__ tile_group, int m_pad, int further, int64_t inter2,
                                 GatedAct act2, const float* __restrict__ gate_bias, const float* __restrict__ up_bias) {
  pdl_trigger();
  pdl_grid_wait();
  const int64_t row = blockIdx.x;
  if (tile_group) {
    const int group = tile_group[row / m_pad];
    if (group < 0) return;
    if (group == further) {
      inter = inter2;
      act = act2;
    }
  }
  if (act.single) {
    for (int64_t i = threadIdx.x; i < inter; i += blockDim.x) {
      const float z = to_f32<T>(gu[row * ld_gu + i]), g = fminf(z, act.limit);
      const float f = act.form == GatedAct::kTanh ? act.limit * tanhf(z / act.limit)
                      : act.form == GatedAct::kErf ? g * normcdff(g)
                                                   : g / (1.f + expf(-act.slope * (g + act.cubic * g * g * g)));
      out[row * ld_out + i] = from_f32<T>(f);
    }
    return;
  }
  for (int64_t i = threadIdx.x; i < inter; i += blockDim.x) {
    const float gb = gate_bias ? gate_bias[i] : 0.f, ub = up_bias ? up_bias[i] : 0.f;
    const float g = fminf(to_f32<T>(gu[row * ld_gu + i]) + gb, act.limit);
    const float u = fminf(fmaxf(to_f32<T>(gu[row * ld_gu + inter + i]) + ub, -act.limit), act.limit);
    const float f = act.form == GatedAct::kErf ? g * normcdff(g) : g / (1.f + expf(-act.slope * (g + act.cubic * g * g * g)));
    out[row * ld_out + i] = from_f32<T>(f * (u + act.shift));
  }
}

int gated_act(cudaStream_t st, void* out, const void* gate_up, int64_t M, int64_t inter, const GatedAct& act, hb_dtype dtype,
              const float* gate_bias, const float* up_bias) {
  if (M == 0) return HB_OK;
  HB_DISPATCH_DTYPE(dtype, T, {
    HB_CUDA_CHECK(launch_pdl(gated_act_kernel<T>, dim3((unsigned)M), dim3(256), 0, st, (T*)out, inter, (const T*)gate_up,
                             act.single ? inter : 2 * inter, inter, act, nullptr, 1, -1, 0, act, gate_bias, up_bias));
  });
  return HB_OK;
}

int gated_act_grouped(cudaStream_t st, void* out, int64_t ld_out, const void* gate_up, int64_t ld_gu, int64_t inter,
                      const GatedAct& act, hb_dtype dtype, const TcGroups& g, const int32_t* tile_group) {
  const int64_t rows = (int64_t)g.max_tiles * g.m_pad;
  if (rows == 0) return HB_OK;
  HB_DISPATCH_DTYPE(dtype, T, {
    HB_CUDA_CHECK(launch_pdl(gated_act_kernel<T>, dim3((unsigned)rows), dim3(256), 0, st, (T*)out, ld_out, (const T*)gate_up,
                             ld_gu, inter, act, tile_group, g.m_pad, g.shared_w ? g.groups : -1, act.single ? g.shared_n : g.shared_n / 2, g.shared_act,
                             nullptr, nullptr));
  });
  return HB_OK;
}

}  // namespace hb
