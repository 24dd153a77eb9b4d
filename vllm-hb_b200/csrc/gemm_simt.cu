// Y[M,N] = X[M,K] . W[N,K]^T on CUDA cores, any dtype and any shape.
//
// This is the coverage kernel: F32/F16 models (the reference's CPU and default CUDA
// dtypes, src/engine/dtype.rs:22-28), and bf16 shapes the tensor-core kernel does not
// take (K not a multiple of 64).  One warp per output column n streams W[n,:] once
// with 128-bit loads and keeps kMB rows of the batch in fp32 accumulators.
#include "common.h"
#include "gemm.h"

namespace hb {

constexpr int kSimtWarps = 8;
constexpr int kMB = 8;

// g.tile_group (may be null): rows m belong to group tile_group[m / m_pad], whose weights are the
// group-th [N, K] matrix of W (the further group's: w2 [n2, k2]); rows of a negative group are
// skipped (m_pad is a multiple of kMB).
struct SimtGroups {
  const int32_t* tile_group = nullptr;
  int m_pad = 1, further = -1;
  const void* w2 = nullptr;
  int64_t n2 = 0, k2 = 0;
  int heads = 0;  // TcHeads: blockIdx.z is the head
  int64_t x_step = 0, y_step = 0;
};
template <typename T, typename OutT, bool VEC>
__global__ void __launch_bounds__(kSimtWarps * 32)
gemm_simt_kernel(OutT* __restrict__ Y, const T* __restrict__ X, const T* __restrict__ W, int64_t M,
                 int64_t N, int64_t K, int64_t ldx, int64_t ldy, const SimtGroups g) {
  constexpr int NV = Vec16<T>::N;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int64_t n = (int64_t)blockIdx.x * kSimtWarps + warp;
  const int64_t m0 = (int64_t)blockIdx.y * kMB;
  const T* wr = W + n * K;
  if (g.heads) {
    wr += (int64_t)blockIdx.z * N * K;
    X += (int64_t)blockIdx.z * g.x_step;
    Y += (int64_t)blockIdx.z * g.y_step;
  }
  if (g.tile_group) {
    const int group = g.tile_group[m0 / g.m_pad];
    if (group < 0) return;
    wr += (int64_t)group * N * K;
    if (group == g.further) {
      N = g.n2;
      K = g.k2;
      wr = (const T*)g.w2 + n * K;
    }
  }
  if (n >= N) return;
  float acc[kMB];
#pragma unroll
  for (int i = 0; i < kMB; ++i) acc[i] = 0.f;
  if (VEC) {
    for (int64_t k = (int64_t)lane * NV; k < K; k += 32 * NV) {
      Vec16<T> wv;
      wv.load(wr + k);
      float wf[NV];
      wv.unpack(wf);
#pragma unroll
      for (int i = 0; i < kMB; ++i) {
        if (m0 + i < M) {
          Vec16<T> xv;
          xv.load(X + (m0 + i) * ldx + k);
          float xf[NV];
          xv.unpack(xf);
#pragma unroll
          for (int j = 0; j < NV; ++j) acc[i] = fmaf(xf[j], wf[j], acc[i]);
        }
      }
    }
  } else {
    for (int64_t k = lane; k < K; k += 32) {
      const float wf = to_f32<T>(wr[k]);
#pragma unroll
      for (int i = 0; i < kMB; ++i)
        if (m0 + i < M) acc[i] = fmaf(to_f32<T>(X[(m0 + i) * ldx + k]), wf, acc[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < kMB; ++i) {
    const float s = warp_sum(acc[i]);
    if (lane == 0 && m0 + i < M) Y[(m0 + i) * ldy + n] = from_f32<OutT>(s);
  }
}

template <typename T, typename OutT>
static int launch_simt(cudaStream_t st, OutT* Y, const T* X, const T* W, int64_t M, int64_t N,
                       int64_t K, int64_t ldx, int64_t ldy, const SimtGroups& g = SimtGroups()) {
  constexpr int NV = Vec16<T>::N;
  const bool vec = K % NV == 0 && ldx % NV == 0 && g.k2 % NV == 0 && g.x_step % NV == 0 && (reinterpret_cast<uintptr_t>(g.w2) & 15) == 0 && (reinterpret_cast<uintptr_t>(X) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(W) & 15) == 0;
  const int64_t widest = N > g.n2 ? N : g.n2;
  dim3 grid((unsigned)((widest + kSimtWarps - 1) / kSimtWarps), (unsigned)((M + kMB - 1) / kMB),
            (unsigned)(g.heads ? g.heads : 1));
  if (vec)
    gemm_simt_kernel<T, OutT, true><<<grid, kSimtWarps * 32, 0, st>>>(Y, X, W, M, N, K, ldx, ldy, g);
  else
    gemm_simt_kernel<T, OutT, false><<<grid, kSimtWarps * 32, 0, st>>>(Y, X, W, M, N, K, ldx, ldy, g);
  HB_LAUNCH_CHECK();
  return HB_OK;
}

int gemm_simt(cudaStream_t st, void* Y, const void* X, const void* W, int64_t M, int64_t N,
              int64_t K, hb_dtype dtype, bool out_f32) {
  if (M == 0 || N == 0) return HB_OK;
  HB_DISPATCH_DTYPE(dtype, T, {
    if (out_f32)
      return (launch_simt<T, float>(st, (float*)Y, (const T*)X, (const T*)W, M, N, K, K, N));
    return (launch_simt<T, T>(st, (T*)Y, (const T*)X, (const T*)W, M, N, K, K, N));
  });
  return HB_OK;
}

int gemm_simt_heads(cudaStream_t st, void* Y, const void* X, const void* W, int64_t M, int64_t N, int64_t K, hb_dtype dtype,
                    bool out_f32, const TcHeads& heads) {
  if (heads.heads < 1 || heads.heads > 65535) return fail(HB_ERR_INVALID_ARG, "gemm_simt_heads: %d heads", heads.heads);
  if (M == 0 || N == 0) return HB_OK;
  SimtGroups g;
  g.heads = heads.heads; g.x_step = heads.x_step; g.y_step = heads.y_step;
  HB_DISPATCH_DTYPE(dtype, T, {
    if (out_f32)
      return (launch_simt<T, float>(st, (float*)Y, (const T*)X, (const T*)W, M, N, K, heads.ldx, heads.ldy, g));
    return (launch_simt<T, T>(st, (T*)Y, (const T*)X, (const T*)W, M, N, K, heads.ldx, heads.ldy, g));
  });
  return HB_OK;
}

int gemm_simt_grouped(cudaStream_t st, void* Y, const void* X, const void* W, int64_t N, int64_t K, hb_dtype dtype, bool out_f32,
                      const TcGroups& groups, const int32_t* tile_group) {
  if (groups.m_pad % kMB || groups.m_pad < 1)
    return fail(HB_ERR_INVALID_ARG, "gemm_simt_grouped: tiles of %d rows", groups.m_pad);
  const int64_t M = (int64_t)groups.max_tiles * groups.m_pad;
  if (M == 0 || N == 0) return HB_OK;
  SimtGroups g;
  g.tile_group = tile_group; g.m_pad = groups.m_pad;
  if (groups.shared_w) { g.further = groups.groups; g.w2 = groups.shared_w; g.n2 = groups.shared_n; g.k2 = groups.shared_k; }
  const int64_t ldx = groups.ldx ? groups.ldx : K, ldy = groups.ldy ? groups.ldy : N;
  HB_DISPATCH_DTYPE(dtype, T, {
    if (out_f32)
      return (launch_simt<T, float>(st, (float*)Y, (const T*)X, (const T*)W, M, N, K, ldx, ldy, g));
    return (launch_simt<T, T>(st, (T*)Y, (const T*)X, (const T*)W, M, N, K, ldx, ldy, g));
  });
  return HB_OK;
}

}  // namespace hb
