// From a layer's projection rows to queries in place and keys and values in their slots: biases,
// norms over whole projections, rotation of channel pairs, all in fp32, one CTA per row.
#include "layered_ops.h"
#include "prep_core.cuh"

namespace hb {

template <typename T, int V>
__device__ __forceinline__ void copy_values(const AttentionPrep& a, const T* pr, int64_t slot) {
  const int vper = a.vdim / V;
  for (int i = threadIdx.x; i < a.kv_heads * vper; i += kPrepThreads) {
    const int g = i / vper, d = i % vper * V;
    float f[V];
    Run<T, V>::load(f, pr + a.off_v + g * a.vdim + d);
    Run<T, V>::store((T*)a.vc + pool_at(slot, a.kv_heads, g, a.vdim, d), f);
  }
}

// Rotation of neighbouring channels.  V > 1: runs of V channels (widths and the number of rotated channels
// are multiples of V); V == 1: pair by pair.
template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) attention_rotate_kernel(const AttentionPrep a) {
  pdl_trigger();
  extern __shared__ float s_cs[];  // [pairs] cosines, [pairs] sines
  pdl_grid_wait();
  const int64_t row = blockIdx.x, slot = a.slots[row];
  const int tid = threadIdx.x, P = a.pairs, D = a.dim;
  const bool keep = a.kc && slot >= 0 && slot < a.num_blocks * HB_BLOCK_SIZE;
  T* pr = (T*)a.p + row * a.ld;
  constexpr int W = V == 1 ? 2 : V;           // channels a thread turns at a time
  const int per = (D + W - 1) / W, total = (a.heads + (a.kc ? a.kv_heads : 0)) * per;
  // channels i of head i / per: queries first, then keys
  auto source = [&](int i) { return pr + (i < a.heads * per ? a.off_q : a.off_k - a.heads * D) + i / per * D + i % per * W; };
  Vec16<T> ahead;  // the first run of every thread is on its way while the angles are formed
  if constexpr (V > 1)
    if (tid < total) ahead.load(source(tid));
  angles_of(s_cs, a.rotation, P, a.pos[row], a.rotation_gain);
  __syncthreads();
  for (int i = tid; i < total; i += kPrepThreads) {
    const int head = i / per, d = i % per * W;
    const bool query = head < a.heads;
    const int g = query ? head : head - a.heads;
    const float* bias = query ? a.q_bias : a.k_bias;
    T* src = source(i);
    float f[W];
    if constexpr (V == 1) {
      f[0] = to_f32<T>(src[0]);
      f[1] = d + 1 < D ? to_f32<T>(src[1]) : 0.f;
    } else {
      if (i >= kPrepThreads) ahead.load(src);
      ahead.unpack(f);
    }
    if (bias)
#pragma unroll
      for (int j = 0; j < W; ++j)
        if (d + j < D) f[j] += bias[g * D + d + j];
    if (d / 2 < P) {
#pragma unroll
      for (int j = 0; j < W; j += 2) {
        const float c = s_cs[d / 2 + j / 2], s = s_cs[P + d / 2 + j / 2], u = f[j], v = f[j + 1];
        f[j] = u * c - v * s;
        f[j + 1] = v * c + u * s;
      }
    }
    if (!query && !keep) continue;
    T* dst = query ? src : (T*)a.kc + pool_at(slot, a.kv_heads, g, D, d);
    if constexpr (V == 1) {
      dst[0] = from_f32<T>(f[0]);
      if (d + 1 < D) dst[1] = from_f32<T>(f[1]);
    } else {
      Run<T, V>::store(dst, f);
    }
  }
  if (keep) copy_values<T, V>(a, pr, slot);
}

// Channel i turned with channel i + pairs.  A thread takes V pairs, or V channels behind the pairs, at
// a time (V > 1: widths and the number of pairs are multiples of V).
template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) attention_rotate_halves_kernel(const AttentionPrep a) {
  pdl_trigger();
  extern __shared__ float s_cs[];  // [pairs] cosines, [pairs] sines
  pdl_grid_wait();
  const int64_t row = blockIdx.x, slot = a.slots[row];
  const int tid = threadIdx.x, P = a.pairs, D = a.dim;
  const bool keep = a.kc && slot >= 0 && slot < a.num_blocks * HB_BLOCK_SIZE;
  T* pr = (T*)a.p + row * a.ld;
  const int turned = P / V, per = turned + (D - 2 * P) / V, total = (a.heads + (keep ? a.kv_heads : 0)) * per;
  auto channel = [&](int u) { return u < turned ? u * V : P + u * V; };  // first channel of unit u of a head
  auto source = [&](int i) { return pr + (i < a.heads * per ? a.off_q : a.off_k - a.heads * D) + i / per * D + channel(i % per); };
  float f[V], g[V];
  auto load = [&](int i) {
    const T* src = source(i);
    Run<T, V>::load(f, src);
    if (i % per < turned) Run<T, V>::load(g, src + P);
  };
  if (tid < total) load(tid);  // on its way while the angles are formed
  angles_of(s_cs, a.rotation, P, a.pos[row], a.rotation_gain);
  __syncthreads();
  for (int i = tid; i < total; i += kPrepThreads) {
    if (i >= kPrepThreads) load(i);
    const int head = i / per, u = i % per, d = channel(u);
    const bool query = head < a.heads, pair = u < turned;
    const int h = query ? head : head - a.heads;
    const float* bias = query ? a.q_bias : a.k_bias;
    if (bias)
#pragma unroll
      for (int j = 0; j < V; ++j) {
        f[j] += bias[h * D + d + j];
        if (pair) g[j] += bias[h * D + d + P + j];
      }
    if (pair) {
#pragma unroll
      for (int j = 0; j < V; ++j) {
        float x, y;
        rope_rotate(f[j], g[j], s_cs[d + j], s_cs[P + d + j], &x, &y);
        f[j] = x;
        g[j] = y;
      }
    }
    T* dst = query ? source(i) : (T*)a.kc + pool_at(slot, a.kv_heads, h, D, d);
    Run<T, V>::store(dst, f);
    if (pair) Run<T, V>::store(dst + P, g);
  }
  if (keep) copy_values<T, V>(a, pr, slot);
}

// RMS norms over all query rows and all key rows of a position.  A thread keeps its first kHeld runs
// of queries and its first run of keys in registers between the sums and the results.
constexpr int kHeld = 2;
template <typename T, int V>
__global__ void __launch_bounds__(kPrepThreads) attention_norm_kernel(const AttentionPrep a) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float red[2][33];
  const int64_t row = blockIdx.x, slot = a.slots[row];
  const int tid = threadIdx.x, D = a.dim, nq = a.heads * D, nk = a.kv_heads * D, rep = a.heads / a.kv_heads;
  const bool keep = slot >= 0 && slot < a.num_blocks * HB_BLOCK_SIZE, tied = a.key_scale != nullptr;
  T* q = (T*)a.p + row * a.ld + a.off_q;
  const T* k = (const T*)a.p + row * a.ld + a.off_k;
  constexpr int step = kPrepThreads * V;
  auto load = [&](float (&f)[V], const T* src, const float* bias, int i) {
    Run<T, V>::load(f, src + i);
    if (bias)
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] += bias[i + j];
  };
  auto squares = [&](const float (&f)[V], float s) {
#pragma unroll
    for (int j = 0; j < V; ++j) s = fmaf(f[j], f[j], s);
    return s;
  };
  float sq = 0.f, sk = 0.f, f[V], held[kHeld][V], key[V];
#pragma unroll
  for (int n = 0; n < kHeld; ++n)
    if (tid * V + n * step < nq) load(held[n], q, a.q_bias, tid * V + n * step);
  if (tid * V < nk) load(key, k, a.k_bias, tid * V);
#pragma unroll
  for (int n = 0; n < kHeld; ++n)
    if (tid * V + n * step < nq) sq = squares(held[n], sq);
  if (tid * V < nk) sk = squares(key, sk);
  for (int i = tid * V + kHeld * step; i < nq; i += step) {
    load(f, q, a.q_bias, i);
    sq = squares(f, sq);
  }
  for (int i = tid * V + step; i < nk; i += step) {
    load(f, k, a.k_bias, i);
    sk = squares(f, sk);
  }
  // both sums behind one barrier
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = sq;
    red[1][tid >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < kPrepThreads / 32; ++w) {
    sq += red[0][w];
    sk += red[1][w];
  }
  const float rq = 1.f / sqrtf(sq / (float)nq + a.eps), rk = 1.f / sqrtf(sk / (float)nk + a.eps);
  auto query = [&](float (&v)[V], int i) {
    const int at = tied ? i / (rep * D) * D + i % D : 0;  // the key channel this query channel meets
#pragma unroll
    for (int j = 0; j < V; ++j) {
      v[j] *= rq * a.q_norm[i + j];
      if (tied) v[j] *= a.k_norm[at + j];
    }
    Run<T, V>::store(q + i, v);
  };
  auto keyed = [&](float (&v)[V], int i) {
    if (!tied)
#pragma unroll
      for (int j = 0; j < V; ++j) v[j] *= rk * a.k_norm[i + j];
    Run<T, V>::store((T*)a.kc + pool_at(slot, a.kv_heads, i / D, D, i % D), v);
  };
#pragma unroll
  for (int n = 0; n < kHeld; ++n)
    if (tid * V + n * step < nq) query(held[n], tid * V + n * step);
  for (int i = tid * V + kHeld * step; i < nq; i += step) {
    load(f, q, a.q_bias, i);
    query(f, i);
  }
  if (!keep) return;
  if (tid * V < nk) keyed(key, tid * V);
  for (int i = tid * V + step; i < nk; i += step) {
    load(f, k, a.k_bias, i);
    keyed(f, i);
  }
  if (tied) {
    if (tid == 0) a.key_scale[slot] = rk;
    return;
  }
  const int nv = a.kv_heads * a.vdim;
  for (int i = tid * V; i < nv; i += step) {
    Run<T, V>::load(f, (const T*)a.p + row * a.ld + a.off_v + i);
    Run<T, V>::store((T*)a.vc + pool_at(slot, a.kv_heads, i / a.vdim, a.vdim, i % a.vdim), f);
  }
}

int attention_prepare(cudaStream_t st, const AttentionPrep& a, int64_t rows, hb_dtype dtype) {
  if (rows == 0) return HB_OK;
  const bool norm = a.q_norm || a.k_norm;
  if (norm && (!a.q_norm || !a.k_norm || a.pairs))
    return fail(HB_ERR_INVALID_ARG, "attention_prepare: norms come for queries and keys, and without a rotation");
  if (a.key_scale && (!norm || a.vdim != a.dim))
    return fail(HB_ERR_INVALID_ARG, "attention_prepare: keys that are the values have a norm and their width");
  if (!a.kc && norm)
    return fail(HB_ERR_INVALID_ARG, "attention_prepare: queries without keys are only rotated");
  if (2 * a.pairs > a.dim || a.pairs > 5000) return fail(HB_ERR_INVALID_ARG, "attention_prepare: %d pairs of %d channels", a.pairs, a.dim);
  const int es = (int)dtype_size(dtype), n = 16 / es;
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = a.dim % n == 0 && a.vdim % n == 0 && (a.halves ? a.pairs : 2 * a.pairs) % n == 0 && a.off_q % n == 0 && a.off_k % n == 0 &&
                   a.off_v % n == 0 && a.ld % n == 0 && al(a.p) && al(a.kc) && al(a.vc);
  const dim3 grid((unsigned)rows), block(kPrepThreads);
  const size_t smem = (size_t)a.pairs * 2 * sizeof(float);
  auto launch = [&](auto* rotate, auto* halves, auto* normed) -> int {
    if (a.halves) rotate = halves;
    if (norm) HB_CUDA_CHECK(launch_pdl(normed, grid, block, 0, st, a));
    else HB_CUDA_CHECK(launch_pdl(rotate, grid, block, smem, st, a));
    return HB_OK;
  };
  if (dtype == HB_F32)
    return vec ? launch(attention_rotate_kernel<float, 4>, attention_rotate_halves_kernel<float, 4>, attention_norm_kernel<float, 4>)
               : launch(attention_rotate_kernel<float, 1>, attention_rotate_halves_kernel<float, 1>, attention_norm_kernel<float, 1>);
  if (dtype == HB_BF16)
    return vec ? launch(attention_rotate_kernel<__nv_bfloat16, 8>, attention_rotate_halves_kernel<__nv_bfloat16, 8>,
                         attention_norm_kernel<__nv_bfloat16, 8>)
               : launch(attention_rotate_kernel<__nv_bfloat16, 1>, attention_rotate_halves_kernel<__nv_bfloat16, 1>,
                         attention_norm_kernel<__nv_bfloat16, 1>);
  return fail(HB_ERR_UNSUPPORTED_DTYPE, "attention_prepare runs in bf16 or f32");
}

__global__ void expand_distance_bias_kernel(float* __restrict__ out, const float* __restrict__ rel,
                                            const int32_t* __restrict__ bucket, int heads, int dist_len) {
  const int d = blockIdx.x * blockDim.x + threadIdx.x;
  if (d < dist_len) out[(int64_t)blockIdx.y * dist_len + d] = rel[(int64_t)bucket[d] * heads + blockIdx.y];
}

int expand_distance_bias(cudaStream_t st, float* out, const float* rel, const int32_t* bucket, int heads, int dist_len) {
  expand_distance_bias_kernel<<<dim3((unsigned)((dist_len + 255) / 256), (unsigned)heads), 256, 0, st>>>(out, rel, bucket, heads,
                                                                                                    dist_len);
  HB_LAUNCH_CHECK();
  return HB_OK;
}

}  // namespace hb
