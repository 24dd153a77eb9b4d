// Residual of designs that norm what a sublayer puts out and hand the residual itself to the next one.
//
// One kernel per sublayer boundary: the output (a product's rows, the weighted outputs of experts, or
// embedding rows) is normed in equal parts of the width and added to the residual; at the end of a layer
// the residual becomes a weighted sum over the results of all layers so far; and the next sublayer's
// input is formed, with a causal convolution over the tokens of the sequence.
//
// Norm parts are independent of each other throughout, so a CTA takes a run of tokens and one or several
// parts; a thread owns its channels and keeps the last inputs of the convolution in registers.  The first
// taps - 1 tokens ahead of a run are worked out again (they read what their own CTA reads, so both get the
// same bits).  What earlier steps leave for the convolution is a ring per sequence, an entry per position
// modulo taps - 1; it is written one boundary later, when nobody reads it any more: the residual that a
// convolution read is the residual the next boundary adds to.
#include <algorithm>

#include "layered_ops.h"

namespace hb {

constexpr int kResidualThreads = 512;  // most threads of a part
constexpr int kHeldTaps = 4;           // taps whose inputs stay in registers

template <typename T, int VEC>
__device__ __forceinline__ void load_row(float (&f)[VEC], const T* p) {
  if constexpr (VEC == 1) {
    f[0] = to_f32<T>(*p);
  } else if constexpr (VEC == 2 && sizeof(T) == 4) {
    const float2 v = *reinterpret_cast<const float2*>(p);
    f[0] = v.x; f[1] = v.y;
  } else if constexpr (VEC == 2) {
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    f[0] = v.x; f[1] = v.y;
  } else if constexpr (sizeof(T) == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  } else {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_row(T* p, const float (&f)[VEC]) {
  if constexpr (VEC == 1) {
    *p = from_f32<T>(f[0]);
  } else if constexpr (VEC == 2 && sizeof(T) == 4) {
    *reinterpret_cast<float2*>(p) = make_float2(f[0], f[1]);
  } else if constexpr (VEC == 2) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(f[0], f[1]);
  } else if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    uint2 v;
    *reinterpret_cast<__nv_bfloat162*>(&v.x) = __floats2bfloat162_rn(f[0], f[1]);
    *reinterpret_cast<__nv_bfloat162*>(&v.y) = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = v;
  }
}

// Threads of a part: team of consecutive ones, sums by warps and, where a team has several, through
// shared memory (`red`, two sets that take turns so that one barrier per sum is enough).
struct Team {
  int size, rank, first_warp;
  __device__ __forceinline__ Team(int size_) : size(size_), rank(threadIdx.x % size_), first_warp((threadIdx.x - threadIdx.x % size_) >> 5) {}
  __device__ __forceinline__ float sum(float v, float* red) const {
    v = warp_sum(v);
    if (size == 32) return v;
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < size >> 5; ++w) t += red[first_warp + w];
    return t;
  }
};

// The sublayer's output of a row, VEC channels from c on.
template <typename T, int VEC>
__device__ __forceinline__ void sublayer_output(float (&f)[VEC], const ResidualStep& a, int64_t W, int64_t row, int64_t c) {
  if (a.embed) {
    const int64_t id = min((int64_t)a.ids[row], a.vocab - 1);  // never outside the table
    load_row<T, VEC>(f, (const T*)a.embed + id * W + c);
    return;
  }
  if (a.y) {
    load_row<float, VEC>(f, a.y + row * a.ld_y + c);
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) f[j] = 0.f;
  }
  const int32_t* place = a.expert_place + row * a.top;
  const float* weight = a.expert_weight + row * a.top;
#pragma unroll 4
  for (int k = 0; k < a.top; ++k) {
    const int p = place[k];
    const T* src = p < 0 ? (const T*)a.input + row * a.ld_input : (const T*)a.expert_y + (int64_t)p * a.ld_y;
    float e[VEC];
    load_row<T, VEC>(e, src + c);
    const float w = weight[k];
#pragma unroll
    for (int j = 0; j < VEC; ++j) f[j] = fmaf(w, e[j], f[j]);
  }
}

// NC: runs of VEC channels a thread owns.  HELD: at most kHeldTaps taps; else `win` [taps - 1][NC * VEC]
// per thread lies in shared memory.
template <typename T, int VEC, int NC, bool HELD>
__global__ void __launch_bounds__(kResidualThreads)
residual_kernel(const ResidualStep a, const RowRange* __restrict__ tiles, const SegInfo* __restrict__ segs, int64_t W, int team_size) {
  extern __shared__ float s_win[];
  __shared__ float red[2][kResidualThreads / 32];
  pdl_trigger();
  pdl_grid_wait();
  const Team team(team_size);
  const int teams = blockDim.x / team_size, size = (int)(W / a.groups);
  const int group = blockIdx.y * teams + threadIdx.x / team_size;
  const bool member = group < a.groups;
  const RowRange tile = tiles[blockIdx.x];
  const SegInfo seg = segs[tile.seg];
  const int back = a.conv ? a.taps - 1 : 0, ring = a.taps - 1, first = tile.row0 - seg.row0;
  const int64_t c0 = (int64_t)group * size;
  auto chan = [&](int k) { return (team.rank + k * team.size) * VEC; };  // of the part
  auto live = [&](int k) { return member && chan(k) < size; };

  auto output = [&](float (&f)[VEC], int64_t row, int64_t c) { sublayer_output<T, VEC>(f, a, W, row, c); };

  const int i0 = max(-first, -back);
  float win[HELD ? kHeldTaps - 1 : 1][NC][VEC];  // inputs of the tokens ahead of i0, oldest first
  auto held = [&](int b, int k, int j) -> float& {  // b tokens back (from 1), not HELD
    return s_win[((b - 1) * NC * VEC + k * VEC + j) * blockDim.x + threadIdx.x];
  };
  if (a.conv) {
#pragma unroll
    for (int b = 1; b < (HELD ? kHeldTaps : a.taps); ++b) {
      const int64_t p = (int64_t)seg.pos0 - b;
#pragma unroll
      for (int k = 0; k < NC; ++k) {
        float f[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) f[j] = 0.f;
        // where the run's past reaches back beyond this step (else it is all worked out below)
        if (b <= back && first + i0 == 0 && p >= 0 && live(k))
          load_row<float, VEC>(f, a.state + ((int64_t)seg.slot * ring + p % ring) * W + c0 + chan(k));
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          if constexpr (HELD) win[kHeldTaps - 1 - b][k][j] = f[j];
          else held(b, k, j) = f[j];
        }
      }
    }
  }

  float next[NC][VEC];
#pragma unroll
  for (int k = 0; k < NC; ++k)
    if (live(k)) output(next[k], tile.row0 + i0, c0 + chan(k));
  for (int i = i0; i < tile.n; ++i) {
    const int64_t row = tile.row0 + i;
    float v[NC][VEC], ss = 0.f;
#pragma unroll
    for (int k = 0; k < NC; ++k) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        v[k][j] = live(k) ? next[k][j] : 0.f;
        ss = fmaf(v[k][j], v[k][j], ss);
      }
    }
    float x[NC][VEC];
#pragma unroll
    for (int k = 0; k < NC; ++k) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) x[k][j] = 0.f;
      if (live(k)) {
        if (a.x) load_row<float, VEC>(x[k], a.x + row * W + c0 + chan(k));
        if (i + 1 < tile.n) output(next[k], row + 1, c0 + chan(k));  // on its way during the sum
      }
    }
    const float r = 1.f / sqrtf(team.sum(ss, red[i & 1]) / (float)size + a.eps);
    // the residual that the last convolution read: part of the sequence's state
    const bool keep = a.past && ring > 0 && i >= 0 && first + i >= seg.n - ring;
#pragma unroll
    for (int k = 0; k < NC; ++k) {
      if (!live(k)) continue;
      const int64_t c = c0 + chan(k);
      if (keep) store_row<float, VEC>(a.past + ((int64_t)seg.slot * ring + ((int64_t)seg.pos0 + first + i) % ring) * W + c, x[k]);
      float w[VEC];
      load_row<float, VEC>(w, a.norm + c);
#pragma unroll
      for (int j = 0; j < VEC; ++j) x[k][j] = fmaf(v[k][j] * r, w[j], x[k][j]);
      if (a.result && i >= 0) store_row<float, VEC>(a.result + row * W + c, x[k]);
      if (a.depth) {
        const float own = a.depth[a.n_earlier];
#pragma unroll
        for (int j = 0; j < VEC; ++j) x[k][j] *= own;
        const float* e = a.earlier + row * W + c;
#pragma unroll 4
        for (int l = 0; l < a.n_earlier; ++l, e += a.step) {
          float f[VEC];
          load_row<float, VEC>(f, e);
          const float d = a.depth[l];
#pragma unroll
          for (int j = 0; j < VEC; ++j) x[k][j] = fmaf(d, f[j], x[k][j]);
        }
      }
      if (a.x_out && i >= 0) store_row<float, VEC>(a.x_out + row * W + c, x[k]);
      if (!a.h) continue;
      float h[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) h[j] = x[k][j];
      if (a.conv) {
        const float* cw = a.conv + (int64_t)back * W + c;  // the token's own tap; older ones before it
        float f[VEC];
        if (i >= 0) {
          load_row<float, VEC>(f, cw);
          float acc[VEC];
#pragma unroll
          for (int j = 0; j < VEC; ++j) acc[j] = f[j] * x[k][j];
#pragma unroll
          for (int b = 1; b < (HELD ? kHeldTaps : a.taps); ++b) {
            if (b <= back) {
              load_row<float, VEC>(f, cw - (int64_t)b * W);
#pragma unroll
              for (int j = 0; j < VEC; ++j) {
                float old;
                if constexpr (HELD) old = win[kHeldTaps - 1 - b][k][j];
                else old = held(b, k, j);
                acc[j] = fmaf(f[j], old, acc[j]);
              }
            }
          }
#pragma unroll
          for (int j = 0; j < VEC; ++j) h[j] += acc[j];
        }
        if constexpr (HELD) {
#pragma unroll
          for (int b = 0; b + 2 < kHeldTaps; ++b)
#pragma unroll
            for (int j = 0; j < VEC; ++j) win[b][k][j] = win[b + 1][k][j];
#pragma unroll
          for (int j = 0; j < VEC; ++j) win[kHeldTaps - 2][k][j] = x[k][j];
        } else if (back) {
          for (int b = back; b > 1; --b)
#pragma unroll
            for (int j = 0; j < VEC; ++j) held(b, k, j) = held(b - 1, k, j);
#pragma unroll
          for (int j = 0; j < VEC; ++j) held(1, k, j) = x[k][j];
        }
      }
      if (i >= 0) store_row<T, VEC>((T*)a.h + row * a.ld_h + c, h);
    }
  }
}

// The same in two kernels, for many rows: the factors of all parts of all rows first (and the experts' outputs
// summed up); then a thread takes
// two channels of a run and all of the run's rows at once, with nothing to wait for but its loads.
template <typename T>
__global__ void __launch_bounds__(kResidualThreads)
residual_scale_kernel(const ResidualStep a, int64_t W, int team_size) {
  __shared__ float red[kResidualThreads / 32];
  pdl_trigger();
  pdl_grid_wait();
  const Team team(team_size);
  const int size = (int)(W / a.groups), group = blockIdx.y * (blockDim.x / team_size) + threadIdx.x / team_size;
  const int64_t row = blockIdx.x;
  float ss = 0.f;
  if (group < a.groups)
    for (int i = team.rank * 4; i < size; i += team.size * 4) {
      float f[4];
      sublayer_output<T, 4>(f, a, W, row, (int64_t)group * size + i);
      if (a.top) store_row<float, 4>(a.mixed + row * a.ld_y + (int64_t)group * size + i, f);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss = fmaf(f[j], f[j], ss);
    }
  const float r = 1.f / sqrtf(team.sum(ss, red) / (float)size + a.eps);
  if (group < a.groups && team.rank == 0) a.scale[row * a.groups + group] = r;
}

constexpr int kRunThreads = 128;
template <typename T>
__global__ void __launch_bounds__(kRunThreads)
residual_run_kernel(const ResidualStep a, const RowRange* __restrict__ tiles, const SegInfo* __restrict__ segs, int64_t W) {
  constexpr int H = kHeldTaps - 1, N = H + kResidualRun, V = 2;  // rows ahead of the run, all rows, channels
  pdl_trigger();
  pdl_grid_wait();
  const int64_t c = ((int64_t)blockIdx.y * kRunThreads + threadIdx.x) * V;
  if (c >= W) return;
  const RowRange tile = tiles[blockIdx.x];
  const SegInfo seg = segs[tile.seg];
  const int back = a.conv ? a.taps - 1 : 0, ring = a.taps - 1, first = tile.row0 - seg.row0, group = (int)(c / (W / a.groups));
  // row i is token first + i - H of the segment; rows that are not there are read as the run's first one, so
  // that no load waits for a branch, and come to nothing
  auto row = [&](int i) { return (int64_t)tile.row0 + (i < H ? (first + i < H ? 0 : i - H) : i - H < tile.n ? i - H : 0); };
  float x[N][V];
  const float* y = a.top ? a.mixed : a.y;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    if (a.embed) load_row<T, V>(x[i], (const T*)a.embed + min((int64_t)a.ids[row(i)], a.vocab - 1) * W + c);
    else load_row<float, V>(x[i], y + row(i) * a.ld_y + c);
  }
  float w[V], f[N][V];
  load_row<float, V>(w, a.norm + c);
#pragma unroll
  for (int i = 0; i < N; ++i) {
#pragma unroll
    for (int j = 0; j < V; ++j) f[i][j] = 0.f;
    if (a.x) load_row<float, V>(f[i], a.x + row(i) * W + c);
  }
  if (a.past && ring > 0 && first + tile.n > seg.n - ring) {  // (the end of the segment)
#pragma unroll
    for (int i = H; i < N; ++i) {
      const int token = first + i - H;
      if (i - H < tile.n && token >= seg.n - ring)
        store_row<float, V>(a.past + ((int64_t)seg.slot * ring + ((int64_t)seg.pos0 + token) % ring) * W + c, f[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const float r = a.scale[row(i) * a.groups + group];
#pragma unroll
    for (int j = 0; j < V; ++j) x[i][j] = fmaf(x[i][j] * r, w[j], f[i][j]);
  }
  if (a.result) {
#pragma unroll
    for (int i = H; i < N; ++i)
      if (i - H < tile.n) store_row<float, V>(a.result + row(i) * W + c, x[i]);
  }
  if (a.depth) {
    const float d = a.depth[a.n_earlier];
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int j = 0; j < V; ++j) x[i][j] *= d;
    const float* e = a.earlier + c;
    for (int l = 0; l < a.n_earlier; ++l, e += a.step) {
#pragma unroll
      for (int i = 0; i < N; ++i) load_row<float, V>(f[i], e + row(i) * W);
      const float d = a.depth[l];
#pragma unroll
      for (int i = 0; i < N; ++i)
#pragma unroll
        for (int j = 0; j < V; ++j) x[i][j] = fmaf(d, f[i][j], x[i][j]);
    }
  }
  if (a.x_out) {
#pragma unroll
    for (int i = H; i < N; ++i)
      if (i - H < tile.n) store_row<float, V>(a.x_out + row(i) * W + c, x[i]);
  }
  if (!a.h) return;
  if (a.conv) {
    float tap[kHeldTaps][V];  // by distance
#pragma unroll
    for (int b = 0; b < kHeldTaps; ++b) {
#pragma unroll
      for (int j = 0; j < V; ++j) tap[b][j] = 0.f;
      if (b <= back) load_row<float, V>(tap[b], a.conv + (int64_t)(back - b) * W + c);
    }
    if (first < H) {  // the run's past reaches back beyond this step
#pragma unroll
      for (int i = 0; i < H; ++i) {
        const int token = first + i - H;
        if (token >= 0) continue;
#pragma unroll
        for (int j = 0; j < V; ++j) x[i][j] = 0.f;
        if (H - i <= back && seg.pos0 + token >= 0)
          load_row<float, V>(x[i], a.state + ((int64_t)seg.slot * ring + ((int64_t)seg.pos0 + token) % ring) * W + c);
      }
    }
#pragma unroll
    for (int i = N - 1; i >= H; --i) {  // the last row first: it is the one no other row needs any more
      float acc[V];
#pragma unroll
      for (int j = 0; j < V; ++j) acc[j] = tap[0][j] * x[i][j];
#pragma unroll
      for (int b = 1; b < kHeldTaps; ++b)
#pragma unroll
        for (int j = 0; j < V; ++j) acc[j] = fmaf(tap[b][j], x[i - b][j], acc[j]);
#pragma unroll
      for (int j = 0; j < V; ++j) x[i][j] += acc[j];
    }
  }
#pragma unroll
  for (int i = H; i < N; ++i)
    if (i - H < tile.n) store_row<T, V>((T*)a.h + row(i) * a.ld_h + c, x[i]);
}

// Rows normed in parts, wherever they lie: CTA = (row, one or several parts).
template <typename T, typename IN, int VEC>
__global__ void __launch_bounds__(kResidualThreads)
parts_norm_kernel(T* __restrict__ out, int64_t ld_out, const IN* __restrict__ in, int64_t ld_in, const int32_t* __restrict__ list,
                  const float* __restrict__ weight, int groups, int size, float eps, int team_size) {
  __shared__ float red[kResidualThreads / 32];
  pdl_trigger();
  pdl_grid_wait();
  const Team team(team_size);
  const int group = blockIdx.y * (blockDim.x / team_size) + threadIdx.x / team_size;
  const int64_t at = (int64_t)group * size;
  const IN* src = in + (list ? list[blockIdx.x] : (int64_t)blockIdx.x) * ld_in + at;
  float ss = 0.f;
  if (group < groups)
    for (int i = team.rank * VEC; i < size; i += team.size * VEC) {
      float f[VEC];
      load_row<IN, VEC>(f, src + i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss = fmaf(f[j], f[j], ss);
    }
  const float r = 1.f / sqrtf(team.sum(ss, red) / (float)size + eps);
  if (group >= groups) return;
  for (int i = team.rank * VEC; i < size; i += team.size * VEC) {
    float f[VEC], w[VEC];
    load_row<IN, VEC>(f, src + i);
    load_row<float, VEC>(w, weight + at + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) f[j] = f[j] * r * w[j];
    store_row<T, VEC>(out + (int64_t)blockIdx.x * ld_out + at + i, f);
  }
}

// Threads of a part with about `runs` runs of vec channels each, and of a CTA.
static int team_threads(int64_t size, int vec, int runs) {
  int t = 32;
  while (t < kResidualThreads && (int64_t)t * vec * runs < size) t *= 2;
  return t;
}

int residual_step(cudaStream_t st, const ResidualStep& a, const RowRange* tiles, int n_tiles, const SegInfo* segs, int64_t width,
                  hb_dtype dtype) {
  if (n_tiles == 0) return HB_OK;
  if (a.groups < 1 || width < 1 || width % a.groups || a.taps < 1 || a.taps > kResidualMaxTaps || (a.conv && !a.h))
    return fail(HB_ERR_INVALID_ARG, "residual_step: a width of %lld in %d parts, %d taps", (long long)width, a.groups, a.taps);
  const int64_t size = width / a.groups;
  auto al = [](const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const size_t es = 4 * dtype_size(dtype);
  const bool vec = size % 4 == 0 && a.ld_y % 4 == 0 && a.ld_input % 4 == 0 && a.ld_h % 4 == 0 && a.step % 4 == 0 && al(a.y, 16) &&
                   al(a.norm, 16) && al(a.x, 16) && al(a.x_out, 16) && al(a.result, 16) && al(a.earlier, 16) && al(a.conv, 16) &&
                   al(a.state, 16) && al(a.past, 16) && al(a.mixed, 16) && al(a.expert_y, es) && al(a.input, es) && al(a.embed, es) && al(a.h, es);
  const int v = vec ? 4 : 1, team = team_threads(size, v, 2);
  const int runs = (int)((size + (int64_t)team * v - 1) / ((int64_t)team * v));
  if (runs > 8) return fail(HB_ERR_INVALID_ARG, "residual_step: parts of %lld channels are not supported", (long long)size);
  const int threads = std::max(team, 128), teams = threads / team;
  const bool held = a.taps <= kHeldTaps;
  const dim3 grid((unsigned)n_tiles, (unsigned)((a.groups + teams - 1) / teams));
  if (residual_in_two(a) && vec) {
    auto two = [&](auto* scale, auto* run) -> int {
      HB_CUDA_CHECK(launch_pdl(scale, dim3((unsigned)a.rows, grid.y), dim3((unsigned)threads), 0, st, a, width, team));
      HB_CUDA_CHECK(launch_pdl(run, dim3((unsigned)n_tiles, (unsigned)((width / 2 + kRunThreads - 1) / kRunThreads)), dim3(kRunThreads), 0, st,
                               a, tiles, segs, width));
      return HB_OK;
    };
    if (dtype == HB_F32) return two(residual_scale_kernel<float>, residual_run_kernel<float>);
    if (dtype == HB_BF16) return two(residual_scale_kernel<__nv_bfloat16>, residual_run_kernel<__nv_bfloat16>);
  }
  auto launch = [&](auto* k, int nc) -> int {
    const size_t smem = held || !a.conv ? 0 : (size_t)(a.taps - 1) * nc * v * threads * sizeof(float);
    if (smem > 200 * 1024) return fail(HB_ERR_INVALID_ARG, "residual_step: %d taps of parts of %lld channels are not supported", a.taps, (long long)size);
    if (smem > 40 * 1024) HB_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    HB_CUDA_CHECK(launch_pdl(k, grid, dim3((unsigned)threads), smem, st, a, tiles, segs, width, team));
    return HB_OK;
  };
#define HB_RESIDUAL_NC(T, VEC, NC) \
  return held ? launch(residual_kernel<T, VEC, NC, true>, NC) : launch(residual_kernel<T, VEC, NC, false>, NC)
#define HB_RESIDUAL(T, VEC)                       \
  do {                                            \
    if (runs <= 1) HB_RESIDUAL_NC(T, VEC, 1);     \
    if (runs <= 2) HB_RESIDUAL_NC(T, VEC, 2);     \
    if (runs <= 4) HB_RESIDUAL_NC(T, VEC, 4);     \
    HB_RESIDUAL_NC(T, VEC, 8);                    \
  } while (0)
  if (dtype == HB_F32) {
    if (vec) HB_RESIDUAL(float, 4);
    HB_RESIDUAL(float, 1);
  }
  if (dtype == HB_BF16) {
    if (vec) HB_RESIDUAL(__nv_bfloat16, 4);
    HB_RESIDUAL(__nv_bfloat16, 1);
  }
#undef HB_RESIDUAL
#undef HB_RESIDUAL_NC
  return fail(HB_ERR_UNSUPPORTED_DTYPE, "residual_step runs in bf16 or f32");
}

int parts_norm(cudaStream_t st, void* out, int64_t ld_out, const void* in, int64_t ld_in, bool in_f32, const int32_t* list,
               const float* weight, int64_t rows, int groups, int64_t size, float eps, hb_dtype dtype) {
  if (rows == 0) return HB_OK;
  if (groups < 1 || size < 1) return fail(HB_ERR_INVALID_ARG, "parts_norm: %d parts of %lld channels", groups, (long long)size);
  const size_t es = dtype_size(dtype), ins = in_f32 ? 4 : es;
  auto al = [](const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  const bool vec = size % 4 == 0 && ld_in % 4 == 0 && ld_out % 4 == 0 && al(in, 4 * ins) && al(out, 4 * es) && al(weight, 16);
  const int team = team_threads(size, vec ? 4 : 1, 2), threads = std::max(team, 128), teams = threads / team;
  const dim3 grid((unsigned)rows, (unsigned)((groups + teams - 1) / teams));
  auto launch = [&](auto* k, auto* o, auto* i) -> int {
    using O = std::remove_pointer_t<decltype(o)>;
    using I = std::remove_pointer_t<decltype(i)>;
    HB_CUDA_CHECK(launch_pdl(k, grid, dim3((unsigned)threads), 0, st, (O*)out, ld_out, (const I*)in, ld_in, list, weight, groups,
                             (int)size, eps, team));
    return HB_OK;
  };
  using B = __nv_bfloat16;
  if (dtype == HB_F32)
    return vec ? launch(parts_norm_kernel<float, float, 4>, (float*)nullptr, (float*)nullptr)
               : launch(parts_norm_kernel<float, float, 1>, (float*)nullptr, (float*)nullptr);
  if (dtype != HB_BF16) return fail(HB_ERR_UNSUPPORTED_DTYPE, "parts_norm runs in bf16 or f32");
  if (in_f32)
    return vec ? launch(parts_norm_kernel<B, float, 4>, (B*)nullptr, (float*)nullptr)
               : launch(parts_norm_kernel<B, float, 1>, (B*)nullptr, (float*)nullptr);
  return vec ? launch(parts_norm_kernel<B, B, 4>, (B*)nullptr, (B*)nullptr)
             : launch(parts_norm_kernel<B, B, 1>, (B*)nullptr, (B*)nullptr);
}

}  // namespace hb
