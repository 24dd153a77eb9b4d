// Causal convolution per channel with a few taps, bias and SiLU; what it needs of earlier steps is
// part of the sequence's state.
#include "layered_ops.h"
#include "prep_core.cuh"

namespace hb {

constexpr int kConvThreads = 256;
constexpr int kConvHeld = 4;                         // taps whose inputs stay in registers

// CTA = (segment or chunk of one, LANES * V channels); the other threads share its tokens.  The CTA of a segment's first tokens is the
// only one that reads the old state, and writes the new one at its end.  HELD: at most kConvHeld taps.
template <typename T, int V, bool HELD, int LANES>
__global__ void __launch_bounds__(kConvThreads)
short_conv_kernel(const ShortConv a, const int32_t* __restrict__ list, int n_list, const RowRange* __restrict__ chunks) {
  pdl_trigger();
  constexpr int kConvRun = kRecChunk / (kConvThreads / LANES);  // consecutive tokens of a thread
  const int c = (blockIdx.y * LANES + threadIdx.x % LANES) * V, run = threadIdx.x / LANES;
  const bool live = c < a.channels;
  const int back = a.taps - 1;
  float w[HELD ? kConvHeld : 1][V], bias[V];
  if (live) {  // parameters: they may be read before the producing kernel has finished
#pragma unroll
    for (int j = 0; j < V; ++j) bias[j] = a.bias[c + j];
    if (HELD)
#pragma unroll
      for (int k = 0; k < kConvHeld; ++k)
#pragma unroll
        for (int j = 0; j < V; ++j) w[k][j] = k < kConvHeld - a.taps ? 0.f : a.w[(int64_t)(k - kConvHeld + a.taps) * a.channels + c + j];
  }
  pdl_grid_wait();
  const bool whole = (int)blockIdx.x < n_list;
  RowRange t;
  if (!whole) t = chunks[blockIdx.x - n_list];
  const SegInfo seg = a.segs[whole ? list[blockIdx.x] : t.seg];
  if (whole) { t.row0 = seg.row0; t.n = seg.n; t.index = 0; }
  const int first = t.row0 - seg.row0;             // token of the segment
  T* state = (T*)a.state + (int64_t)seg.slot * back * a.channels + c;
  // input of token i of the segment (negative: of earlier steps)
  auto input = [&](float (&f)[V], int i) {
    if (i >= 0) {
      Run<T, V>::load(f, (const T*)a.p + (int64_t)(seg.row0 + i) * a.ld + a.off + c);
    } else if (seg.pos0 > 0) {
      Run<T, V>::load(f, state + (int64_t)(back + i) * a.channels);
    } else {  // a new sequence starts from zero
#pragma unroll
      for (int j = 0; j < V; ++j) f[j] = 0.f;
    }
  };
  const int i0 = run * kConvRun, i1 = min(t.n, i0 + kConvRun);
  if (live && i0 < i1) {
    float x[kConvHeld][V];  // inputs of the last tokens, oldest first
    if (HELD) {
#pragma unroll
      for (int k = 0; k + 1 < kConvHeld; ++k) {
        if (kConvHeld - 1 - k <= back) input(x[k + 1], first + i0 - (kConvHeld - 1 - k));
        else
#pragma unroll
          for (int j = 0; j < V; ++j) x[k + 1][j] = 0.f;
      }
    }
    for (int i = i0; i < i1; ++i) {
      float acc[V];
#pragma unroll
      for (int j = 0; j < V; ++j) acc[j] = bias[j];
      if (HELD) {
#pragma unroll
        for (int k = 0; k + 1 < kConvHeld; ++k)
#pragma unroll
          for (int j = 0; j < V; ++j) x[k][j] = x[k + 1][j];
        input(x[kConvHeld - 1], first + i);
#pragma unroll
        for (int k = 0; k < kConvHeld; ++k)
#pragma unroll
          for (int j = 0; j < V; ++j) acc[j] = fmaf(w[k][j], x[k][j], acc[j]);
      } else {
        for (int k = 0; k <= back; ++k) {
          float f[V];
          input(f, first + i - back + k);
#pragma unroll
          for (int j = 0; j < V; ++j) acc[j] = fmaf(a.w[(int64_t)k * a.channels + c + j], f[j], acc[j]);
        }
      }
#pragma unroll
      for (int j = 0; j < V; ++j) acc[j] = acc[j] / (1.f + expf(-acc[j]));
      Run<T, V>::store((T*)a.out + (int64_t)(t.row0 + i) * a.ld_out + c, acc);
    }
  }
  if (t.index != 0) return;
  __syncthreads();  // the old state has been read
  if (live && run == 0)
    for (int k = 0; k < back; ++k) {  // ascending: an entry moves to an earlier place
      float f[V];
      input(f, seg.n - back + k);
      Run<T, V>::store(state + (int64_t)k * a.channels, f);
    }
}

int short_conv(cudaStream_t st, const ShortConv& a, const int32_t* list, int n_list, const RowRange* chunks, int n_chunks,
               hb_dtype dtype) {
  if (n_list + n_chunks == 0) return HB_OK;
  if (a.taps < 1 || a.taps > kConvMaxTaps || a.channels < 1)
    return fail(HB_ERR_INVALID_ARG, "short_conv: %d taps of %d channels (at most %d taps)", a.taps, a.channels, kConvMaxTaps);
  const int n = (int)(16 / dtype_size(dtype));
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = a.channels % n == 0 && a.off % n == 0 && a.ld % n == 0 && a.ld_out % n == 0 && al(a.p) && al(a.out) && al(a.state);
  // whole segments are a few tokens: their CTAs spread over the channels
  auto launch = [&](auto* wide, auto* narrow, int v) -> int {
    auto grid = [&](int cta, int lanes) { return dim3((unsigned)cta, (unsigned)((a.channels + lanes * v - 1) / (lanes * v))); };
    if (n_list) HB_CUDA_CHECK(launch_pdl(wide, grid(n_list, 256), dim3(kConvThreads), 0, st, a, list, n_list, chunks));
    if (n_chunks) HB_CUDA_CHECK(launch_pdl(narrow, grid(n_chunks, 32), dim3(kConvThreads), 0, st, a, list, 0, chunks));
    return HB_OK;
  };
  const bool held = a.taps <= kConvHeld;
#define HB_CONV(T, V)                                                                                          \
  return held ? launch(short_conv_kernel<T, V, true, 256>, short_conv_kernel<T, V, true, 32>, V)               \
              : launch(short_conv_kernel<T, V, false, 256>, short_conv_kernel<T, V, false, 32>, V)
  if (dtype == HB_F32) {
    if (vec) HB_CONV(float, 4);
    HB_CONV(float, 1);
  }
  if (dtype == HB_BF16) {
    if (vec) HB_CONV(__nv_bfloat16, 8);
    HB_CONV(__nv_bfloat16, 1);
  }
#undef HB_CONV
  return fail(HB_ERR_UNSUPPORTED_DTYPE, "short_conv runs in bf16 or f32");
}

}  // namespace hb
