// Attention over a latent that all heads share: from projection rows to the cached latent and key part
// and the rotated parts of the queries (the attention itself: attention_span*.cu, without a V pool).
#include "layered_ops.h"
#include "prep_core.cuh"

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
  const T* pr = (const T*)a.p + row * a.ld;
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
    const T* src = (h < a.heads ? pr + a.off_q + h * QD + a.dim : latent + C) + d;
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
