// Paged attention over a span of positions: the last `window` of them (or all), or those of the
// position's own chunk, and the first `keep_first`; keys and values of any (different) widths, a
// bias by distance, a sink, a gate on the outputs.
//
// The visible keys of a query at position p are two runs, [0, keep) and [lo, p] with
// lo = SpanAttention::first_seen(p) and keep = min(keep_first, lo); only their blocks are read.
#include <algorithm>
#include <climits>

#include "layered_ops.h"

namespace hb {

constexpr int kSpanThreads = 128;
constexpr int kSpanWarps = kSpanThreads / 32;
constexpr int kSpanTile = 64;  // keys per softmax tile

// K and V of a step's rows into the paged pools; V16: 16-byte vectors.
template <typename E>
__global__ void span_kv_write_kernel(E* __restrict__ kc, E* __restrict__ vc, const E* __restrict__ k, const E* __restrict__ v,
                                     int64_t ld, const int64_t* __restrict__ slots, int G, int kw, int vw, int64_t num_blocks) {
  pdl_trigger();
  pdl_grid_wait();
  const int64_t row = blockIdx.x, slot = slots[row];
  if (slot < 0 || slot >= num_blocks * HB_BLOCK_SIZE) return;
  const int64_t blk = slot / HB_BLOCK_SIZE, off = slot % HB_BLOCK_SIZE;
  for (int i = threadIdx.x; i < G * kw; i += blockDim.x)
    kc[((blk * G + i / kw) * HB_BLOCK_SIZE + off) * kw + i % kw] = k[row * ld + i];
  for (int i = threadIdx.x; i < G * vw; i += blockDim.x)
    vc[((blk * G + i / vw) * HB_BLOCK_SIZE + off) * vw + i % vw] = v[row * ld + i];
}

int span_kv_write(cudaStream_t st, const SpanAttention& a, const void* k, const void* v, int64_t ld_kv, const int64_t* slots,
                  int64_t rows, hb_dtype dtype) {
  const size_t es = dtype_size(dtype);
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = (a.dim * es) % 16 == 0 && (a.vdim * es) % 16 == 0 && (ld_kv * es) % 16 == 0 && al(k) && al(v);
  const dim3 grid((unsigned)rows), block(kSpanThreads);
  if (vec) {
    const int n = (int)(16 / es);
    HB_CUDA_CHECK(launch_pdl(span_kv_write_kernel<uint4>, grid, block, 0, st, (uint4*)a.kc, (uint4*)a.vc, (const uint4*)k,
                             (const uint4*)v, ld_kv / n, slots, a.kv_heads, a.dim / n, a.vdim / n, a.num_blocks));
  } else if (es == 2) {
    HB_CUDA_CHECK(launch_pdl(span_kv_write_kernel<uint16_t>, grid, block, 0, st, (uint16_t*)a.kc, (uint16_t*)a.vc,
                             (const uint16_t*)k, (const uint16_t*)v, ld_kv, slots, a.kv_heads, a.dim, a.vdim, a.num_blocks));
  } else {
    HB_CUDA_CHECK(launch_pdl(span_kv_write_kernel<uint32_t>, grid, block, 0, st, (uint32_t*)a.kc, (uint32_t*)a.vc,
                             (const uint32_t*)k, (const uint32_t*)v, ld_kv, slots, a.kv_heads, a.dim, a.vdim, a.num_blocks));
  }
  return HB_OK;
}

// One CTA per (row, kv head, slice of its query heads): scores and running softmax of all query heads of the group in
// fp32 on CUDA cores.  The kernel for fp32 models and for sizes the tensor-core kernels do not take.
template <typename T>
__global__ void __launch_bounds__(kSpanThreads)
span_attention_rows_kernel(const SpanAttention a, const int32_t* __restrict__ row_list) {
  pdl_grid_wait();
  extern __shared__ float sm[];
  const HeadSlice hs(a, blockIdx.y);
  const int R = hs.n, D = a.dim, VD = a.vdim;
  float* s_q = sm;                    // [R][D]
  float* s_p = s_q + R * D;           // [R][kSpanTile]
  float* s_acc = s_p + R * kSpanTile; // [R][VD]
  float* s_m = s_acc + R * VD;        // [R] running maximum
  float* s_l = s_m + R;               // [R] running sum
  float* s_a = s_l + R;               // [R] rescale of this tile
  __shared__ int64_t s_key[kSpanTile];  // (block * kv_heads + head) * 16 + offset of the tile's keys
  __shared__ float s_ks[kSpanTile];     // scale of the keys
  __shared__ int s_dist[kSpanTile];     // their distance, up to the last of the bias table
  const T* values = (const T*)(a.vc ? a.vc : a.kc);
  const int ld_v = a.vc ? VD : D;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = hs.kvh;
  const int64_t row = row_list[blockIdx.x];
  const int pos = a.pos[row];
  const int lo = a.first_seen(pos);
  const int keep = min(a.keep_first, lo);
  const int n_keys = keep + (pos - lo + 1);
  const int32_t* table = a.tables + (int64_t)a.row_seg[row] * a.max_blocks;
  const T* q = (const T*)a.q + row * a.ld_q + (int64_t)hs.first * D;
  for (int i = tid; i < R * D; i += kSpanThreads) s_q[i] = to_f32<T>(q[i]) * a.scale;
  for (int i = tid; i < R * VD; i += kSpanThreads) s_acc[i] = 0.f;
  for (int i = tid; i < R; i += kSpanThreads) { s_m[i] = -INFINITY; s_l[i] = 0.f; }
  for (int t0 = 0; t0 < n_keys; t0 += kSpanTile) {
    const int nt = min(kSpanTile, n_keys - t0);
    __syncthreads();
    for (int i = tid; i < nt; i += kSpanThreads) {
      const int j = t0 + i < keep ? t0 + i : lo + (t0 + i - keep);
      int64_t blk = j / HB_BLOCK_SIZE < a.max_blocks ? table[j / HB_BLOCK_SIZE] : 0;
      if (blk < 0 || blk >= a.num_blocks) blk = 0;  // never outside the pool
      s_key[i] = (blk * a.kv_heads + g) * HB_BLOCK_SIZE + j % HB_BLOCK_SIZE;
      s_ks[i] = a.key_scale ? a.key_scale[blk * HB_BLOCK_SIZE + j % HB_BLOCK_SIZE] : 1.f;
      s_dist[i] = min(pos - j, a.dist_len - 1);
    }
    __syncthreads();
    for (int i = warp; i < nt; i += kSpanWarps) {
      const T* kr = (const T*)a.kc + s_key[i] * D;
      for (int h = 0; h < R; ++h) {
        float s = 0.f;
        for (int d = lane; d < D; d += 32) s = fmaf(s_q[h * D + d], to_f32<T>(kr[d]), s);
        s = warp_sum(s);
        if (lane == 0) {
          s *= s_ks[i];
          if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
          s_p[h * kSpanTile + i] = s + (a.dist_bias ? a.dist_bias[(int64_t)(hs.first + h) * a.dist_len + s_dist[i]] : 0.f);
        }
      }
    }
    __syncthreads();
    for (int h = warp; h < R; h += kSpanWarps) {
      float mx = -INFINITY;
      for (int i = lane; i < nt; i += 32) mx = fmaxf(mx, s_p[h * kSpanTile + i]);
      mx = warp_max(mx);
      const float m_old = s_m[h], m_new = fmaxf(m_old, mx);
      float l = 0.f;
      for (int i = lane; i < nt; i += 32) {
        const float p = expf(s_p[h * kSpanTile + i] - m_new);
        s_p[h * kSpanTile + i] = p;
        l += p;
      }
      l = warp_sum(l);
      __syncwarp();
      if (lane == 0) {
        const float al = m_old == -INFINITY ? 0.f : expf(m_old - m_new);
        s_a[h] = al;
        s_m[h] = m_new;
        s_l[h] = s_l[h] * al + l;
      }
    }
    __syncthreads();
    for (int d = tid; d < VD; d += kSpanThreads) {
      for (int h = 0; h < R; ++h) s_acc[h * VD + d] *= s_a[h];
      for (int i = 0; i < nt; ++i) {
        const float v = to_f32<T>(values[s_key[i] * ld_v + d]);
        for (int h = 0; h < R; ++h) s_acc[h * VD + d] = fmaf(s_p[h * kSpanTile + i], v, s_acc[h * VD + d]);
      }
    }
  }
  __syncthreads();
  if (a.sink)  // one more member of the softmax, without a value
    for (int h = tid; h < R; h += kSpanThreads) {
      const float k = a.sink[hs.first + h], top = fmaxf(s_m[h], k), f = expf(s_m[h] - top);
      s_a[h] = f;
      s_l[h] = fmaf(s_l[h], f, expf(k - top));
    }
  __syncthreads();
  T* out = (T*)a.out + row * a.ld_out + (int64_t)hs.first * VD;
  const T* gate = a.gate ? (const T*)a.gate + a.gate_at(row, hs.first, 0) : nullptr;
  for (int i = tid; i < R * VD; i += kSpanThreads) {
    float o = s_acc[i] / s_l[i / VD];
    if (a.sink) o *= s_a[i / VD];
    if (gate) o /= 1.f + expf(-to_f32<T>(gate[a.gate_per_head ? i / VD : i]));
    out[i] = from_f32<T>(o);
  }
}

int span_attention_rows(cudaStream_t st, const SpanAttention& args, const int32_t* row_list, int n_rows, hb_dtype dtype) {
  if (n_rows == 0) return HB_OK;
  SpanAttention a = args;
  const size_t per_head = (size_t)(a.dim + kSpanTile + a.vdim + 3) * sizeof(float);
  a.cut(std::max(1, (int)(100 * 1024 / per_head)));
  const size_t smem = a.slice * per_head;
  if (smem > 200 * 1024)
    return fail(HB_ERR_INVALID_ARG, "attention: a head of %d + %d channels does not fit shared memory", a.dim, a.vdim);
  auto launch = [&](auto* kernel) -> int {
    if (smem > 48 * 1024)
      HB_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    HB_CUDA_CHECK(launch_pdl(kernel, dim3((unsigned)n_rows, (unsigned)(a.kv_heads * a.slices())), dim3(kSpanThreads), smem,
                             st, a, row_list));
    return HB_OK;
  };
  if (dtype == HB_F32) return launch(span_attention_rows_kernel<float>);
  if (dtype == HB_BF16) return launch(span_attention_rows_kernel<__nv_bfloat16>);
  return fail(HB_ERR_UNSUPPORTED_DTYPE, "span attention runs in bf16 or f32");
}

}  // namespace hb
