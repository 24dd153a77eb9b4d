// Pieces of the tensor-core attention kernels over a span of positions.
#pragma once

#include "layered_ops.h"
#include "mma_sync.cuh"
#include "tc_core.cuh"

namespace hb {
namespace {

constexpr int kBS = HB_BLOCK_SIZE;
constexpr size_t kSmemCap = 224 * 1024;
__host__ __device__ constexpr int pad16(int n) { return (n + 15) / 16 * 16; }

// The blocks a CTA reads: [0, na) of the kept tokens, then [b0, b1].
struct BlockRuns {
  int na, b0, n;
  __device__ __forceinline__ int block(int i) const { return i < na ? i : b0 + (i - na); }
};
__device__ __forceinline__ BlockRuns block_runs(int first_pos, int last_pos, const SpanAttention& a) {
  BlockRuns r;
  const int lo = a.first_seen(first_pos);
  r.b0 = lo / kBS;
  r.na = min((min(a.keep_first, lo) + kBS - 1) / kBS, r.b0);
  r.n = r.na + last_pos / kBS - r.b0 + 1;
  return r;
}
// lo: first_seen() of the position
__device__ __forceinline__ bool visible(int key, int pos, int lo, int keep_first) {
  return key <= pos && (key >= lo || key < keep_first);
}
// Every key of the block that starts at `key` is visible from all positions of a range: `first` is
// the earliest, `lo` what the latest of them sees first (it grows with the position).
__device__ __forceinline__ bool all_visible(int key, int first, int lo, int keep_first) {
  return key + kBS - 1 <= first && (key >= lo || key + kBS <= keep_first);
}
constexpr float kLog2e = 1.4426950408889634f;
// cap * tanh(s / cap) for a score and a cap in units of log2, tanh(y) = 1 - 2 / (1 + e^(2y)); k = 2 / softcap
__device__ __forceinline__ float capped(float s, float cap, float k) { return cap - __fdividef(2.f * cap, 1.f + ex2(s * k)); }
__device__ __forceinline__ float sigmoid_of(uint32_t bits16) {
  const float z = __uint_as_float(bits16 << 16);  // a bf16 number
  return __fdividef(1.f, 1.f + __expf(-z));
}
// A warp copies a block of 16 (or `rows`) rows of `w` 16-byte vectors a row into rows of `stride` bytes; (j, c) is the
// lane's first (row, vector), stepped without divisions.
struct BlockCopy {
  int w, j, c, dj, dc;
  __device__ __forceinline__ BlockCopy(int width, int lane) : w(width / 8), j(lane / w), c(lane % w), dj(32 / w), dc(32 % w) {}
  __device__ __forceinline__ void operator()(uint32_t dst, int stride, const __nv_bfloat16* src, int64_t src_row, int rows = kBS) const {
    if (dc == 0 && dj > 0) {  // whole rows at a time: a lane stays in its column
      dst += j * stride + c * 16;
      src += j * src_row + c * 8;
      for (int jj = j; jj < rows; jj += dj, dst += dj * stride, src += dj * src_row) cp_async_16(dst, src);
      return;
    }
    int jj = j, cc = c;
#pragma unroll 4
    while (jj < rows) {
      cp_async_16(dst + jj * stride + cc * 16, src + jj * src_row + cc * 8);
      jj += dj;
      cc += dc;
      if (cc >= w) { cc -= w; ++jj; }
    }
  }
};

}  // namespace
}  // namespace hb
