// Residual streams in fp32 and the norms around them.
//
// A sublayer boundary is one kernel: the output of the sublayer goes back into all streams (or
// first the mean of two normed branch outputs), the next sublayer's input is read from the new
// streams and normalised — one read and one write of the streams per sublayer.
#include "layered_ops.h"

namespace hb {

constexpr int kStreamThreads = 256;
constexpr int kWideThreads = 512;   // few rows (decoding): more loads in flight per row
constexpr int kFewRows = 592;

template <typename T, int VEC>
__device__ __forceinline__ void load_vec(float (&f)[VEC], const T* p);
template <> __device__ __forceinline__ void load_vec<float, 4>(float (&f)[4], const float* p) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
template <> __device__ __forceinline__ void load_vec<__nv_bfloat16, 4>(float (&f)[4], const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&v.x), b = *reinterpret_cast<const __nv_bfloat162*>(&v.y);
  f[0] = __low2float(a); f[1] = __high2float(a); f[2] = __low2float(b); f[3] = __high2float(b);
}
template <> __device__ __forceinline__ void load_vec<float, 1>(float (&f)[1], const float* p) { f[0] = *p; }
template <> __device__ __forceinline__ void load_vec<__nv_bfloat16, 1>(float (&f)[1], const __nv_bfloat16* p) {
  f[0] = __bfloat162float(*p);
}
template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[VEC]);
template <> __device__ __forceinline__ void store_vec<float, 4>(float* p, const float (&f)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
template <> __device__ __forceinline__ void store_vec<__nv_bfloat16, 4>(__nv_bfloat16* p, const float (&f)[4]) {
  uint2 v;
  *reinterpret_cast<__nv_bfloat162*>(&v.x) = __floats2bfloat162_rn(f[0], f[1]);
  *reinterpret_cast<__nv_bfloat162*>(&v.y) = __floats2bfloat162_rn(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = v;
}
template <> __device__ __forceinline__ void store_vec<float, 1>(float* p, const float (&f)[1]) { *p = f[0]; }
template <> __device__ __forceinline__ void store_vec<__nv_bfloat16, 1>(__nv_bfloat16* p, const float (&f)[1]) {
  *p = __float2bfloat16_rn(f[0]);
}

__device__ __forceinline__ float inv_rms(float sum_sq, int64_t n, float eps) { return 1.0f / sqrtf(sum_sq / (float)n + eps); }

template <typename T, int VEC>
__global__ void __launch_bounds__(kStreamThreads)
streams_embed_kernel(float* __restrict__ x, T* __restrict__ h, const T* __restrict__ embed, const T* __restrict__ pos_table,
                     const uint32_t* __restrict__ ids, const int32_t* __restrict__ pos, const float* __restrict__ in,
                     const float* __restrict__ norm, float norm_offset, int S, int64_t W, int64_t ld_h, int64_t vocab,
                     int64_t max_positions, float eps, float embed_scale) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float red[33];
  const int64_t row = blockIdx.x;
  const int64_t id = min((int64_t)ids[row], vocab - 1);                       // never outside the tables
  const int64_t p = max((int64_t)0, min((int64_t)pos[row], max_positions - 1));
  const T* er = embed + id * W;
  const T* pr = pos_table ? pos_table + p * W : nullptr;
  float* xr = x + row * S * W;
  float in_sum = 0.f;
  for (int s = 0; s < S; ++s) in_sum += in[s];
  float ss = 0.f;
  for (int64_t i = (int64_t)threadIdx.x * VEC; i < W; i += kStreamThreads * VEC) {
    float a[VEC], b[VEC];
    load_vec<T, VEC>(a, er + i);
    if (pr) load_vec<T, VEC>(b, pr + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      a[j] *= embed_scale;
      if (pr) a[j] += b[j];
      const float u = in_sum * a[j];
      ss = fmaf(u, u, ss);
    }
    for (int s = 0; s < S; ++s) store_vec<float, VEC>(xr + s * W + i, a);
  }
  const float r = inv_rms(block_sum(ss, red), W, eps);
  for (int64_t i = (int64_t)threadIdx.x * VEC; i < W; i += kStreamThreads * VEC) {
    float a[VEC], w[VEC];
    load_vec<float, VEC>(a, xr + i);  // written by this thread
    load_vec<float, VEC>(w, norm + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) a[j] = in_sum * a[j] * r * (norm_offset + w[j]);
    store_vec<T, VEC>(h + row * ld_h + i, a);
  }
}

template <typename T, int VEC, int NS, bool TWO>
__global__ void __launch_bounds__(NS <= 4 ? kWideThreads : kStreamThreads)
streams_mix_kernel(float* __restrict__ x, T* __restrict__ h, const float* __restrict__ y, const float* __restrict__ y2,
                   int64_t ld_y, StreamMix m, int S, int64_t W, int64_t ld_h, float eps) {
  pdl_trigger();
  extern __shared__ float s_u[];  // [W] the next sublayer's input before its norm
  __shared__ float red[33];
  __shared__ float s_mix[NS][NS], s_out[NS], s_in[NS];
  const int tid = threadIdx.x, threads = blockDim.x;
  // mixing weights are parameters: they may be read before the producing kernel has finished
  for (int i = tid; i < NS * NS; i += threads) {
    const int a = i / NS, b = i % NS;
    s_mix[a][b] = (a < S && b < S) ? m.mix[a * S + b] : 0.f;
  }
  for (int i = tid; i < NS; i += threads) {
    s_out[i] = i < S ? m.out[i] : 0.f;
    s_in[i] = (i < S && m.next_norm) ? m.next_in[i] : 0.f;
  }
  pdl_grid_wait();
  const int64_t row = blockIdx.x;
  const float* yr = y ? y + row * ld_y : nullptr;
  const float* y2r = TWO ? y2 + row * ld_y : nullptr;
  float r1 = 0.f, r2 = 0.f;
  if (TWO) {
    float a1 = 0.f, a2 = 0.f;
    for (int64_t i = (int64_t)tid * VEC; i < W; i += threads * VEC) {
      float f[VEC], g[VEC];
      load_vec<float, VEC>(f, yr + i);
      load_vec<float, VEC>(g, y2r + i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        a1 = fmaf(f[j], f[j], a1);
        a2 = fmaf(g[j], g[j], a2);
      }
    }
    r1 = inv_rms(block_sum(a1, red), W, eps);
    r2 = inv_rms(block_sum(a2, red), W, eps);
  } else {
    __syncthreads();
  }
  float* xr = x + row * S * W;
  float ss = 0.f;
  for (int64_t i = (int64_t)tid * VEC; i < W; i += threads * VEC) {
    float xs[NS][VEC], f[VEC];
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      if (s < S) load_vec<float, VEC>(xs[s], xr + s * W + i);
      else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) xs[s][j] = 0.f;
      }
    }
    if (TWO || yr) {
      load_vec<float, VEC>(f, yr + i);
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) f[j] = 0.f;
    }
    if (!TWO && m.bias) {
      float b[VEC];
      load_vec<float, VEC>(b, m.bias + i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) f[j] += b[j];
    }
    if (!TWO && m.top) {
      const int32_t* place = m.expert_place + row * m.top;
      const float* weight = m.expert_weight + row * m.top;
#pragma unroll 4
      for (int k = 0; k < m.top; ++k) {
        float e[VEC];
        load_vec<T, VEC>(e, (const T*)m.expert_y + (int64_t)place[k] * ld_y + i);
        const float w = weight[k];
#pragma unroll
        for (int j = 0; j < VEC; ++j) f[j] = fmaf(w, e[j], f[j]);
      }
    }
    if (TWO) {
      float g[VEC], w1[VEC], w2[VEC];
      load_vec<float, VEC>(g, y2r + i);
      load_vec<float, VEC>(w1, m.w1 + i);
      load_vec<float, VEC>(w2, m.w2 + i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) f[j] = 0.5f * (f[j] * r1 * w1[j] + g[j] * r2 * w2[j]);
    }
    float u[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = 0.f;
#pragma unroll
    for (int t = 0; t < NS; ++t) {
      if (t < S) {
        float n[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          float a = s_out[t] * f[j];
#pragma unroll
          for (int s = 0; s < NS; ++s) a = fmaf(s_mix[s][t], xs[s][j], a);
          n[j] = a;
          u[j] = fmaf(s_in[t], a, u[j]);
        }
        store_vec<float, VEC>(xr + t * W + i, n);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(u[j], u[j], ss);
    store_vec<float, VEC>(s_u + i, u);
  }
  if (!m.next_norm) return;
  const float r = inv_rms(block_sum(ss, red), W, eps);
  for (int64_t i = (int64_t)tid * VEC; i < W; i += threads * VEC) {
    float u[VEC], w[VEC];
    load_vec<float, VEC>(u, s_u + i);  // written by this thread
    load_vec<float, VEC>(w, m.next_norm + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = u[j] * r * (m.norm_offset + w[j]);
    store_vec<T, VEC>(h + row * ld_h + i, u);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kStreamThreads)
streams_final_kernel(T* __restrict__ h, const float* __restrict__ x, const int32_t* __restrict__ want,
                     const float* __restrict__ norm, float norm_offset, int S, int64_t W, int64_t ld_h, float eps, float scale) {
  pdl_trigger();
  pdl_grid_wait();
  extern __shared__ float s_u[];
  __shared__ float red[33];
  const float* xr = x + (int64_t)want[blockIdx.x] * S * W;
  float ss = 0.f;
  for (int64_t i = (int64_t)threadIdx.x * VEC; i < W; i += kStreamThreads * VEC) {
    float u[VEC];
    load_vec<float, VEC>(u, xr + i);
    for (int s = 1; s < S; ++s) {
      float a[VEC];
      load_vec<float, VEC>(a, xr + s * W + i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) u[j] += a[j];
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(u[j], u[j], ss);
    store_vec<float, VEC>(s_u + i, u);
  }
  const float r = scale * inv_rms(block_sum(ss, red), W, eps);
  for (int64_t i = (int64_t)threadIdx.x * VEC; i < W; i += kStreamThreads * VEC) {
    float u[VEC], w[VEC];
    load_vec<float, VEC>(u, s_u + i);
    load_vec<float, VEC>(w, norm + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) u[j] = u[j] * r * (norm_offset + w[j]);
    store_vec<T, VEC>(h + (int64_t)blockIdx.x * ld_h + i, u);
  }
}

// Groups of up to a warp's worth of work are normed by one warp each; a single wide group by the
// whole CTA.
template <typename T, bool WARP, int VEC>
__global__ void __launch_bounds__(kStreamThreads)
gated_group_norm_kernel(T* __restrict__ out, int64_t ld_out, const float* __restrict__ o, int64_t ld_o,
                        const T* __restrict__ gate, int64_t ld_gate, const float* __restrict__ weight, const GroupNorm n) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float red[33];
  const int64_t row = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, groups = n.groups, size = n.size;
  const int group = WARP ? blockIdx.y * (kStreamThreads / 32) + warp : blockIdx.y;
  const int first = (WARP ? lane : (int)threadIdx.x) * VEC, step = (WARP ? 32 : kStreamThreads) * VEC;
  if (WARP && group >= groups) return;
  const int64_t at = (int64_t)group * size;
  const float* og = o + row * ld_o + at;
  const T* gg = gate + row * ld_gate + at;
  T* dst = out + row * ld_out + at;
  if (n.own_weights) weight += at;
  auto act = [&](float g) {
    const float sg = 1.f / (1.f + expf(-g));
    return n.gate_silu ? g * sg : sg;
  };
  float ss = 0.f;
#pragma unroll 4
  for (int i = first; i < size; i += step) {
    float f[VEC];
    load_vec<float, VEC>(f, og + i);
    if (n.gate_first) {
      float g[VEC];
      load_vec<T, VEC>(g, gg + i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) f[j] *= act(g[j]);
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss = fmaf(f[j], f[j], ss);
  }
  ss = WARP ? warp_sum(ss) : block_sum(ss, red);
  const float r = inv_rms(ss, size, n.eps);
#pragma unroll 2
  for (int i = first; i < size; i += step) {
    float f[VEC], g[VEC], w[VEC];
    load_vec<float, VEC>(f, og + i);
    load_vec<T, VEC>(g, gg + i);
    load_vec<float, VEC>(w, weight + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) f[j] = f[j] * act(g[j]) * r * w[j];
    store_vec<T, VEC>(dst + i, f);
  }
}

// bf16 serves, fp32 checks; F16 models do not come in these designs
#define HB_DISPATCH_LAYERED(dtype, T, ...)                                                               \
  switch (dtype) {                                                                                       \
    case HB_F32: { using T = float; __VA_ARGS__; break; }                                                \
    case HB_BF16: { using T = __nv_bfloat16; __VA_ARGS__; break; }                                       \
    default: return ::hb::fail(HB_ERR_UNSUPPORTED_DTYPE, "layered models run in bf16 or f32, not dtype %d", (int)(dtype)); \
  }

int streams_embed(cudaStream_t st, float* x, void* h, const void* embed, const void* pos_table, const uint32_t* ids,
                  const int32_t* pos, const float* in, const float* norm, float norm_offset, int64_t rows, int streams,
                  int64_t width, int64_t ld_h, int64_t vocab, int64_t max_positions, float eps, hb_dtype dtype, float embed_scale) {
  HB_DISPATCH_LAYERED(dtype, T, {
    auto* k = width % 4 == 0 ? streams_embed_kernel<T, 4> : streams_embed_kernel<T, 1>;
    HB_CUDA_CHECK(launch_pdl(k, dim3((unsigned)rows), dim3(kStreamThreads), 0, st, x, (T*)h, (const T*)embed,
                             (const T*)pos_table, ids, pos, in, norm, norm_offset, streams, width, ld_h, vocab, max_positions, eps,
                             embed_scale));
  });
  return HB_OK;
}

// The row's sublayer input waits for its norm in shared memory; rows above 48 KB need the opt-in.
template <typename K>
static int row_smem(K kernel, int64_t width) {
  if (width * 4 > 200 * 1024) return fail(HB_ERR_INVALID_ARG, "a width of %lld is not supported", (long long)width);
  if (width * 4 > 47 * 1024) HB_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  return HB_OK;
}

template <typename T, int VEC, int NS, bool TWO>
static int launch_mix(cudaStream_t st, float* x, void* h, const float* y, const float* y2, int64_t ld_y, const StreamMix& m,
                      int64_t rows, int streams, int64_t width, int64_t ld_h, float eps) {
  const int threads = NS <= 4 && rows <= kFewRows && width >= kWideThreads * VEC ? kWideThreads : kStreamThreads;
  const int rc = row_smem(streams_mix_kernel<T, VEC, NS, TWO>, width);
  if (rc) return rc;
  HB_CUDA_CHECK(launch_pdl(streams_mix_kernel<T, VEC, NS, TWO>, dim3((unsigned)rows), dim3((unsigned)threads),
                           (size_t)width * 4, st, x, (T*)h, y, y2, ld_y, m, streams, width, ld_h, eps));
  return HB_OK;
}

int streams_mix(cudaStream_t st, float* x, void* h, const float* y, const float* y2, int64_t ld_y, const StreamMix& m,
                int64_t rows, int streams, int64_t width, int64_t ld_h, float eps, hb_dtype dtype) {
#define HB_MIX_NS(T, VEC, NS)                                                                                      \
  return y2 ? (launch_mix<T, VEC, NS, true>(st, x, h, y, y2, ld_y, m, rows, streams, width, ld_h, eps))            \
            : (launch_mix<T, VEC, NS, false>(st, x, h, y, y2, ld_y, m, rows, streams, width, ld_h, eps))
#define HB_MIX(T, VEC)                          \
  do {                                          \
    if (streams == 1) HB_MIX_NS(T, VEC, 1);     \
    if (streams == 2) HB_MIX_NS(T, VEC, 2);     \
    if (streams == 3) HB_MIX_NS(T, VEC, 3);     \
    if (streams == 4) HB_MIX_NS(T, VEC, 4);     \
    if (streams <= 8) HB_MIX_NS(T, VEC, 8);     \
    HB_MIX_NS(T, VEC, 16);                      \
  } while (0)
  if (streams < 1 || streams > kMaxStreams) return fail(HB_ERR_INVALID_ARG, "%d residual streams (1 to %d)", streams, kMaxStreams);
  HB_DISPATCH_LAYERED(dtype, T, {
    if (width % 4 == 0) HB_MIX(T, 4);
    HB_MIX(T, 1);
  });
  return HB_OK;
}

int streams_final(cudaStream_t st, void* h, const float* x, const int32_t* want, const float* norm, float norm_offset,
                  int64_t n_want, int streams, int64_t width, int64_t ld_h, float eps, hb_dtype dtype, float scale) {
  if (n_want == 0) return HB_OK;
  HB_DISPATCH_LAYERED(dtype, T, {
    auto* k = width % 4 == 0 ? streams_final_kernel<T, 4> : streams_final_kernel<T, 1>;
    const int rc = row_smem(k, width);
    if (rc) return rc;
    HB_CUDA_CHECK(launch_pdl(k, dim3((unsigned)n_want), dim3(kStreamThreads), (size_t)width * 4, st, (T*)h, x, want, norm,
                             norm_offset, streams, width, ld_h, eps, scale));
  });
  return HB_OK;
}

int gated_group_norm(cudaStream_t st, void* out, int64_t ld_out, const float* o, int64_t ld_o, const void* gate,
                     int64_t ld_gate, const float* weight, int64_t rows, const GroupNorm& n, hb_dtype dtype) {
  const int groups = n.groups, size = n.size;
  const bool warp = groups > 1 && size <= 1024;
  const unsigned gy = warp ? (unsigned)((groups + kStreamThreads / 32 - 1) / (kStreamThreads / 32)) : (unsigned)groups;
  HB_DISPATCH_LAYERED(dtype, T, {
    const uintptr_t bits = (uintptr_t)o | (uintptr_t)weight | ((uintptr_t)gate * (16 / (4 * sizeof(T)))) |
                           ((uintptr_t)out * (16 / (4 * sizeof(T))));
    const bool vec = (bits & 15) == 0 && size % 4 == 0 && ld_o % 4 == 0 && ld_gate % 4 == 0 && ld_out % 4 == 0;
    auto* k = vec ? (warp ? gated_group_norm_kernel<T, true, 4> : gated_group_norm_kernel<T, false, 4>)
                  : (warp ? gated_group_norm_kernel<T, true, 1> : gated_group_norm_kernel<T, false, 1>);
    HB_CUDA_CHECK(launch_pdl(k, dim3((unsigned)rows, gy), dim3(kStreamThreads), 0, st, (T*)out, ld_out, o, ld_o,
                             (const T*)gate, ld_gate, weight, n));
  });
  return HB_OK;
}

}  // namespace hb
