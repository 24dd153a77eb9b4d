// Chunked form of the linear recurrence (see recurrence.cu) for prompt portions.
//
// With b_i the running sum of log2 decays inside a chunk of C = 64 tokens (per key channel, fp32),
//   o_i   = (q_i 2^b_i)^T S_0 + sum_{j <= i} [sum_d q_i[d] k_j[d] 2^(b_i[d] - b_j[d])] v_j
//   S_end = diag(2^b_end) S_0 + sum_j (k_j 2^(b_end - b_j)) v_j^T
// where S_0 is the state before the chunk.  All exponents that are formed are <= 0: keys are
// scaled to the end of their own 16-token block, queries from there on, and inside a block the
// difference b_i - b_j is formed per pair, so that any decay (0 and 1 included) is safe.
//
// Products run on tensor cores with both operands as pairs of bf16 numbers (hi + lo), which keeps
// fp32-like precision; sums, decays and states are fp32.
//
// With a decay per token and head (selective state space) b_i is one number per token, so scores are
// q_i . k_j * 2^(b_i - b_j) * step_j; q, k and v are exact bf16 numbers and need no second half.
//
//   decay   running log2 decays of a chunk (low-rank decay), also steps (decay per token)
//   state   per (chunk, head, 64 state columns): the chunk's own contribution to the state
//   scan    per element of the state: over the chunks of a segment, contribution -> state before
//   output  per (chunk, head): scores, outputs
#include <algorithm>

#include "layered_ops.h"
#include "mma_sync.cuh"
#include "tc_core.cuh"

namespace hb {

namespace {
constexpr int kC = kRecChunk;
constexpr int kT = 128;        // threads: four warps of 16 tokens
constexpr int kVT = 64;        // state columns of a tile
constexpr int kVS = kVT + 8;   // padded row of a bf16 tile
constexpr float kLog2e = 1.4426950408889634f;
using bf16 = __nv_bfloat16;
enum Decay { kConstant, kLowRank, kPerToken };

__device__ __forceinline__ float rec_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float log2_sigmoid(float z) { return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * kLog2e; }
__device__ __forceinline__ float ld_proj(const Recurrence& a, int64_t row, int col) {
  return __bfloat162float(((const bf16*)a.p)[row * a.ld + col]);
}
// log2 of a constant decay to the power n (n = 0: exactly 0, also for decay 0)
__device__ __forceinline__ float log2_pow(float log2_decay, int n) { return n == 0 ? 0.f : log2_decay * (float)n; }
__device__ __forceinline__ int pad16d(int n) { return (n + 15) / 16 * 16; }
// Eight neighbouring columns of a projection row (16 bytes where they are aligned); columns from
// `valid` on are zero.
__device__ __forceinline__ void ld_proj8(float (&f)[8], const Recurrence& a, int64_t row, int col, int valid) {
  const bf16* p = (const bf16*)a.p + row * a.ld + col;
  if (valid >= 8 && (reinterpret_cast<uintptr_t>(p) & 15) == 0) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&w[i]);
      f[2 * i] = __low2float(b);
      f[2 * i + 1] = __high2float(b);
    }
  } else {
#pragma unroll
    for (int i = 0; i < 8; ++i) f[i] = i < valid ? __bfloat162float(p[i]) : 0.f;
  }
}
// hi/lo pairs of eight values to 16-byte aligned shared memory
__device__ __forceinline__ void put_split8(bf16* hi, bf16* lo, const float (&f)[8]) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) split_bf16(f[2 * i], f[2 * i + 1], h[i], l[i]);
  *reinterpret_cast<uint4*>(hi) = make_uint4(h[0], h[1], h[2], h[3]);
  *reinterpret_cast<uint4*>(lo) = make_uint4(l[0], l[1], l[2], l[3]);
}
__device__ __forceinline__ void put8(bf16* dst, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}
// Calls f(token, first channel) for every group of eight channels of a [64][DP] tile, spread over the
// CTA's threads without divisions in the loop.
template <typename F>
__device__ __forceinline__ void for_groups(int DP, F f) {
  const int w = DP / 8, dj = kT / w, dc = kT % w;
  int j = threadIdx.x / w, c = threadIdx.x % w;
  while (j < kC) {
    f(j, c * 8);
    j += dj;
    c += dc;
    if (c >= w) { c -= w; ++j; }
  }
}
// Two neighbouring outputs of an accumulator row
__device__ __forceinline__ void put_pair(float* p, float x, float y, int valid) {
  if (valid >= 2 && (reinterpret_cast<uintptr_t>(p) & 7) == 0) *reinterpret_cast<float2*>(p) = make_float2(x, y);
  else {
    if (valid >= 1) p[0] = x;
    if (valid >= 2) p[1] = y;
  }
}
}  // namespace

__global__ void __launch_bounds__(256)
recurrence_decay_kernel(const Recurrence a, const RowRange* __restrict__ chunks, float* __restrict__ cum) {
  extern __shared__ float s_t[];  // [64][rank]
  pdl_trigger();
  pdl_grid_wait();
  const RowRange ch = chunks[blockIdx.x];
  for (int i = threadIdx.x; i < ch.n * a.rank; i += blockDim.x)
    s_t[i] = ld_proj(a, ch.row0 + i / a.rank, a.off_a1 + i % a.rank);
  __syncthreads();
  const int hd = a.heads * a.dim, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= hd) return;
  const float* w = a.a2 + (int64_t)c * a.rank;
  const float bias = a.a2_bias[c];
  float b = 0.f;
  if (a.rank == 16) {
    float wr[16];
#pragma unroll
    for (int r = 0; r < 16; ++r) wr[r] = w[r];
    for (int i = 0; i < ch.n; ++i) {
      float z = bias;
#pragma unroll
      for (int r = 0; r < 16; ++r) z = fmaf(wr[r], s_t[i * 16 + r], z);
      b = fmaf(log2_sigmoid(z), a.inv_tau, b);
      cum[(int64_t)(ch.row0 + i) * hd + c] = b;
    }
  } else {
    for (int i = 0; i < ch.n; ++i) {
      float z = bias;
      for (int r = 0; r < a.rank; ++r) z = fmaf(w[r], s_t[i * a.rank + r], z);
      b = fmaf(log2_sigmoid(z), a.inv_tau, b);
      cum[(int64_t)(ch.row0 + i) * hd + c] = b;
    }
  }
}

// Decay per token: CTA = (chunk, 32 heads).
constexpr int kStepHeads = 32;
__global__ void __launch_bounds__(256)
recurrence_step_kernel(const Recurrence a, const RowRange* __restrict__ chunks, float* __restrict__ cum) {
  __shared__ float s_t[kC][kStepHeads + 1];
  pdl_trigger();
  pdl_grid_wait();
  const RowRange ch = chunks[blockIdx.x];
  const int h0 = blockIdx.y * kStepHeads, n = min(kStepHeads, a.heads - h0), x = threadIdx.x % kStepHeads;
  const float bias = x < n ? a.dt_bias[h0 + x] : 0.f;
#pragma unroll 4
  for (int i = threadIdx.x / kStepHeads; i < ch.n; i += 256 / kStepHeads) {
    if (x >= n) continue;
    const float z = __bfloat162float(((const bf16*)a.dt)[(int64_t)(ch.row0 + i) * a.ld_dt + h0 + x]) + bias;
    const float t = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
    s_t[i][x] = t;
    cum[((int64_t)(ch.row0 + i) * 2 + 1) * a.heads + h0 + x] = t;
  }
  __syncthreads();
  if ((int)threadIdx.x >= n) return;
  const float rate = -expf(a.a_log[h0 + threadIdx.x]) * kLog2e;
  float b = 0.f;
  for (int i = 0; i < ch.n; ++i) {
    b = fmaf(rate, s_t[i][threadIdx.x], b);
    cum[(int64_t)(ch.row0 + i) * 2 * a.heads + h0 + threadIdx.x] = b;
  }
}

// Value tile [64 tokens][64 columns] as hi/lo pairs (EXACT: as they are); rows and columns outside are
// zero.
template <bool EXACT>
__device__ __forceinline__ void load_values(const Recurrence& a, const RowRange& ch, int h, int v0, bf16* hi, bf16* lo) {
#pragma unroll 4
  for (int i = threadIdx.x; i < kC * kVT / 8; i += kT) {
    const int j = i / (kVT / 8), c = i % (kVT / 8) * 8;
    float v[8];
    ld_proj8(v, a, ch.row0 + min(j, ch.n - 1), a.off_v + h * a.vdim + v0 + c, j < ch.n ? a.vdim - v0 - c : 0);
    if (a.silu_qkv) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = rec_silu(v[e]);
    }
    if (EXACT) put8(hi + j * kVS + c, v);
    else put_split8(hi + j * kVS + c, lo + j * kVS + c, v);
  }
}

template <int MODE>
__global__ void __launch_bounds__(kT)
recurrence_state_kernel(const Recurrence a, const RowRange* __restrict__ chunks, const float* __restrict__ cum,
                        float* __restrict__ out) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int D = a.dim, DP = pad16d(D), KS = DP + 8, h = blockIdx.y, v0 = blockIdx.z * kVT;
  bf16* k_hi = (bf16*)smem;
  bf16* k_lo = k_hi + kC * KS;
  bf16* v_hi = k_lo + kC * KS;
  bf16* v_lo = v_hi + kC * kVS;                   // not with a decay per token
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  pdl_grid_wait();
  const RowRange ch = chunks[blockIdx.x];
  const int hd = a.heads * D, hk = a.qk(h);
  const float ld2 = MODE == kConstant ? log2f(a.decay[h]) : 0.f;
  __shared__ float s_f[kC];                       // decay per token: factors of the keys
  if (MODE == kPerToken) {
    if (tid < ch.n) {
      const float* own = cum + (int64_t)(ch.row0 + tid) * 2 * a.heads + h;
      s_f[tid] = own[a.heads] * ex2(cum[(int64_t)(ch.row0 + ch.n - 1) * 2 * a.heads + h] - own[0]);
    }
    __syncthreads();
  }
  for_groups(DP, [&](int j, int d) {
    float k[8];
    const bool live = j < ch.n;
    ld_proj8(k, a, ch.row0 + min(j, ch.n - 1), a.off_k + hk * D + d, live ? D - d : 0);
    if (live) {
      const float f = MODE == kConstant ? ex2(log2_pow(ld2, ch.n - 1 - j)) : MODE == kPerToken ? s_f[j] : 1.f;
      const float* end = cum + (int64_t)(ch.row0 + ch.n - 1) * hd + h * D + d;
      const float* own = cum + (int64_t)(ch.row0 + j) * hd + h * D + d;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        if (a.silu_qkv) k[e] = rec_silu(k[e]);
        k[e] *= MODE != kLowRank ? f : (d + e < D ? ex2(end[e] - own[e]) : 0.f);
      }
    }
    put_split8(k_hi + j * KS + d, k_lo + j * KS + d, k);
  });
  load_values<MODE == kPerToken>(a, ch, h, v0, v_hi, v_lo);
  __syncthreads();
  float* o = out + ((int64_t)blockIdx.x * a.heads + h) * D * a.vdim + v0;
  // A = (scaled keys)^T: stored [token][channel], read transposed.  Matrices of the x4 load: channels
  // 0-7 / 8-15 of tokens 0-7, then of tokens 8-15.
  const uint32_t ah = smem_u32(k_hi + ((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8);
  const uint32_t al = smem_u32(k_lo + ((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8);
  const uint32_t bh = smem_u32(v_hi + (lane & 15) * kVS + (lane >> 4) * 8);
  const uint32_t bl = smem_u32(v_lo + (lane & 15) * kVS + (lane >> 4) * 8);
  for (int mt = warp; mt < DP / 16; mt += kT / 32) {
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < kC / 16; ++ks) {
      uint32_t hi[4], lo[4];
      ldsm_x4_trans(ah + (ks * 16 * KS + mt * 16) * 2, hi[0], hi[1], hi[2], hi[3]);
      ldsm_x4_trans(al + (ks * 16 * KS + mt * 16) * 2, lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
      for (int nv = 0; nv < 4; ++nv) {
        uint32_t b[4], c[4];
        ldsm_x4_trans(bh + (ks * 16 * kVS + nv * 16) * 2, b[0], b[1], b[2], b[3]);
        if (MODE == kPerToken) {
          mma_pair(acc[2 * nv], hi, lo, b[0], b[1]);
          mma_pair(acc[2 * nv + 1], hi, lo, b[2], b[3]);
          continue;
        }
        ldsm_x4_trans(bl + (ks * 16 * kVS + nv * 16) * 2, c[0], c[1], c[2], c[3]);
        mma_split(acc[2 * nv], hi, lo, b[0], b[1], c[0], c[1]);
        mma_split(acc[2 * nv + 1], hi, lo, b[2], b[3], c[2], c[3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int d = mt * 16 + g + r * 8, c = i * 8 + 2 * t;
        if (d < D) put_pair(o + (int64_t)d * a.vdim + c, acc[i][2 * r], acc[i][2 * r + 1], a.vdim - v0 - c);
      }
  }
}

// One thread per VEC neighbouring state elements.
template <int VEC, int MODE>
__global__ void __launch_bounds__(256)
recurrence_scan_kernel(const Recurrence a, const RowRange* __restrict__ segs, const RowRange* __restrict__ chunks,
                       const float* __restrict__ cum, float* __restrict__ chunk_state) {
  pdl_grid_wait();
  const int64_t per_head = (int64_t)a.dim * a.vdim;
  const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (i >= per_head) return;
  const int h = blockIdx.y, d = (int)(i / a.vdim), hd = a.heads * a.dim;
  const RowRange sg = segs[blockIdx.z];
  const SegInfo info = a.segs[sg.seg];
  float* state = a.state + ((int64_t)info.slot * a.heads + h) * per_head + i;
  const float ld2 = MODE == kConstant ? log2f(a.decay[h]) : 0.f;
  float s[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) s[j] = info.pos0 > 0 ? state[j] : 0.f;  // a new sequence starts from zero
  constexpr int AHEAD = 4;  // chunks fetched together
  const int64_t stride = (int64_t)a.heads * per_head;
  float* u = chunk_state + ((int64_t)sg.row0 * a.heads + h) * per_head + i;
  for (int c0 = 0; c0 < sg.n; c0 += AHEAD) {
    float v[AHEAD][VEC], f[AHEAD];
#pragma unroll
    for (int c = 0; c < AHEAD; ++c) {
      f[c] = 0.f;
      if (c0 + c < sg.n) {
        const RowRange ch = chunks[sg.row0 + c0 + c];
        const int64_t end = ch.row0 + ch.n - 1;
        f[c] = MODE == kConstant ? log2_pow(ld2, ch.n) : MODE == kPerToken ? cum[end * 2 * a.heads + h] : cum[end * hd + h * a.dim + d];
        if (VEC == 4) {
          const float4 x = *reinterpret_cast<const float4*>(u + c * stride);
          v[c][0] = x.x; v[c][1 % VEC] = x.y; v[c][2 % VEC] = x.z; v[c][3 % VEC] = x.w;
        } else {
          v[c][0] = u[c * stride];
        }
      }
    }
#pragma unroll
    for (int c = 0; c < AHEAD; ++c) {
      if (c0 + c < sg.n) {
        if (VEC == 4) *reinterpret_cast<float4*>(u + c * stride) = make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]);
        else u[c * stride] = s[0];
        const float k = ex2(f[c]);
#pragma unroll
        for (int j = 0; j < VEC; ++j) s[j] = fmaf(k, s[j], v[c][j]);
      }
    }
    u += AHEAD * stride;
  }
  pdl_trigger();
#pragma unroll
  for (int j = 0; j < VEC; ++j) state[j] = s[j];
}

template <int MODE>
__global__ void __launch_bounds__(kT)
recurrence_output_kernel(const Recurrence a, const RowRange* __restrict__ chunks, const float* __restrict__ cum,
                         const float* __restrict__ chunk_state) {
  extern __shared__ __align__(16) uint8_t smem[];
  // LR: q and k are exact bf16, decays per channel
  constexpr bool LR = MODE == kLowRank, TOKEN = MODE == kPerToken;
  const int D = a.dim, DP = pad16d(D), KS = DP + 8, BS = DP + 4, h = blockIdx.y, hk = a.qk(h);
  // low rank: q | b | k | scaled k (hi, lo);  constant: q (hi, lo) | k (hi, lo);  per token: q | k.  The
  // keys' part is reused by the value and state tiles of the second phase.
  bf16* q_hi = (bf16*)smem;                       // [64][KS]
  bf16* q_lo = q_hi + kC * KS;                    // constant decay only
  float* s_b = (float*)(q_hi + kC * KS);          // LR only: [64][BS]
  uint8_t* keys = LR ? (uint8_t*)(s_b + kC * BS) : TOKEN ? (uint8_t*)(q_hi + kC * KS) : (uint8_t*)(q_lo + kC * KS);
  __shared__ float s_cum[kC], s_step[kC];         // decay per token
  bf16* k_raw = (bf16*)keys;                      // LR only
  bf16* k_hi = LR ? k_raw + kC * KS : (bf16*)keys;
  bf16* k_lo = k_hi + kC * KS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  pdl_grid_wait();
  const RowRange ch = chunks[blockIdx.x];
  const int hd = a.heads * D;
  const float ld2 = MODE == kConstant ? log2f(a.decay[h]) : 0.f;
  if (TOKEN && tid < kC) {  // tokens past the end keep the last decay
    const float* own = cum + (int64_t)(ch.row0 + min(tid, ch.n - 1)) * 2 * a.heads + h;
    s_cum[tid] = own[0];
    s_step[tid] = own[a.heads];
  }
  if (LR) {
    for_groups(DP, [&](int j, int d) {
      // tokens past the end keep the last decay: every exponent stays <= 0
      const float* c = cum + (int64_t)(ch.row0 + min(j, ch.n - 1)) * hd + h * D + d;
#pragma unroll
      for (int e = 0; e < 8; ++e) s_b[j * BS + d + e] = d + e < D ? c[e] : 0.f;
    });
    __syncthreads();
  }
  for_groups(DP, [&](int j, int d) {
    float q[8], k[8];
    const int valid = j < ch.n ? D - d : 0;
    const int64_t row = ch.row0 + min(j, ch.n - 1);
    ld_proj8(q, a, row, a.off_q + hk * D + d, valid);
    ld_proj8(k, a, row, a.off_k + hk * D + d, valid);
    if (a.silu_qkv) {
#pragma unroll
      for (int e = 0; e < 8; ++e) { q[e] = rec_silu(q[e]); k[e] = rec_silu(k[e]); }
    }
    if (LR) {
      put8(q_hi + j * KS + d, q);   // exact; the scale is applied to the results
      put8(k_raw + j * KS + d, k);
      const float *end = s_b + (j | 15) * BS + d, *own = s_b + j * BS + d;
#pragma unroll
      for (int e = 0; e < 8; ++e) k[e] *= ex2(end[e] - own[e]);
      put_split8(k_hi + j * KS + d, k_lo + j * KS + d, k);
    } else if (TOKEN) {
      put8(q_hi + j * KS + d, q);
      put8(k_hi + j * KS + d, k);
    } else {
      put_split8(q_hi + j * KS + d, q_lo + j * KS + d, q);
      put_split8(k_hi + j * KS + d, k_lo + j * KS + d, k);
    }
  });
  __syncthreads();

  // ---- scores of this warp's 16 tokens with all tokens up to them: s[n] = keys 8n .. 8n+7
  float s[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
  const int i0 = warp * 16 + g, i1 = i0 + 8;
  const uint32_t kh = smem_u32(k_hi + ((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8);
  const uint32_t kl = smem_u32(k_lo + ((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8);
  const uint32_t qh = smem_u32(q_hi + (warp * 16 + (lane & 15)) * KS + (lane >> 4) * 8);
  const uint32_t ql = smem_u32(q_lo + (warp * 16 + (lane & 15)) * KS + (lane >> 4) * 8);
  // query fragment of one 16-channel step, scaled by 2^(b_i - e) with e the reference of the key
  // block (ref < 0: the start of the chunk, e = 0)
  auto q_frag = [&](int ks, int ref, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int d = ks * 16 + half * 8 + 2 * t;
      const float e0 = ref < 0 ? 0.f : s_b[ref * BS + d], e1 = ref < 0 ? 0.f : s_b[ref * BS + d + 1];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int i = r ? i1 : i0;
        const __nv_bfloat162 q2 = *reinterpret_cast<const __nv_bfloat162*>(q_hi + i * KS + d);
        split_bf16(__low2float(q2) * ex2(s_b[i * BS + d] - e0), __high2float(q2) * ex2(s_b[i * BS + d + 1] - e1),
                   hi[half * 2 + r], lo[half * 2 + r]);
      }
    }
  };
#pragma unroll
  for (int nb = 0; nb < 4; ++nb) {   // blocks of 16 keys
    if (LR ? nb < warp : nb <= warp) {
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t hi[4], lo[4], b[4], c[4];
        if (LR) {
          q_frag(ks, nb * 16 + 15, hi, lo);
        } else {
          ldsm_x4(qh + ks * 32, hi[0], hi[1], hi[2], hi[3]);
          if (!TOKEN) ldsm_x4(ql + ks * 32, lo[0], lo[1], lo[2], lo[3]);
        }
        if (TOKEN) {
          ldsm_x4(kh + (nb * 16 * KS + ks * 16) * 2, b[0], b[1], b[2], b[3]);
          mma_bf16_16816(s[2 * nb], hi, b[0], b[1]);
          mma_bf16_16816(s[2 * nb + 1], hi, b[2], b[3]);
          continue;
        }
        ldsm_x4(kh + (nb * 16 * KS + ks * 16) * 2, b[0], b[1], b[2], b[3]);
        ldsm_x4(kl + (nb * 16 * KS + ks * 16) * 2, c[0], c[1], c[2], c[3]);
        mma_split(s[2 * nb], hi, lo, b[0], b[1], c[0], c[1]);
        mma_split(s[2 * nb + 1], hi, lo, b[2], b[3], c[2], c[3]);
      }
    }
    if (LR && nb == warp) {
      // inside the block the decay differs per pair: fp32 on CUDA cores (pairs with j > i are dropped
      // below, whatever their exponential is).  Keys 8-15 of the block never
      // meet queries 0-7.
      float p[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) p[e] = 0.f;
      const int j0 = warp * 16 + 2 * t;
      auto bf2 = [](const bf16* p2) {
        const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(p2);
        return make_float2(__low2float(v), __high2float(v));
      };
      auto fl2 = [](const float* p2) { return *reinterpret_cast<const float2*>(p2); };
      auto pair = [](float& acc, float2 q, float2 k, float2 bi, float2 bj) {
        acc = fmaf(q.x * k.x, ex2(bi.x - bj.x), acc);
        acc = fmaf(q.y * k.y, ex2(bi.y - bj.y), acc);
      };
      for (int d = 0; d < D; d += 2) {  // channels past D are zero
        const float2 b0 = fl2(s_b + i0 * BS + d), b1 = fl2(s_b + i1 * BS + d);
        const float2 q0 = bf2(q_hi + i0 * KS + d), q1 = bf2(q_hi + i1 * KS + d);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float2 kj = bf2(k_raw + (j0 + e) * KS + d), bj = fl2(s_b + (j0 + e) * BS + d);
          const float2 kj8 = bf2(k_raw + (j0 + 8 + e) * KS + d), bj8 = fl2(s_b + (j0 + 8 + e) * BS + d);
          pair(p[e], q0, kj, b0, bj);
          pair(p[2 + e], q1, kj, b1, bj);
          pair(p[6 + e], q1, kj8, b1, bj8);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) { s[2 * nb][e] = p[e]; s[2 * nb + 1][e] = p[4 + e]; }
    }
  }
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = e < 2 ? i0 : i1, j = n * 8 + 2 * t + (e & 1);
      if (j > i) s[n][e] = 0.f;
      else if (TOKEN) s[n][e] *= ex2(s_cum[i] - s_cum[j]) * s_step[j];
      else if (!LR) s[n][e] *= ex2(log2_pow(ld2, i - j));
    }
  __syncthreads();  // keys are done with: their memory holds the tiles of phase two

  bf16* v_hi = (bf16*)keys;            // [64][kVS] values
  bf16* v_lo = v_hi + kC * kVS;
  bf16* t_hi = TOKEN ? v_lo : v_lo + kC * kVS;  // [64][kVS] 64 channels of the state before the chunk
  bf16* t_lo = t_hi + kC * kVS;
  const uint32_t vh = smem_u32(v_hi + (lane & 15) * kVS + (lane >> 4) * 8), vl = smem_u32(v_lo + (lane & 15) * kVS + (lane >> 4) * 8);
  const uint32_t th = smem_u32(t_hi + (lane & 15) * kVS + (lane >> 4) * 8), tl = smem_u32(t_lo + (lane & 15) * kVS + (lane >> 4) * 8);
  const float f0 = LR ? 1.f : ex2(TOKEN ? s_cum[i0] : log2_pow(ld2, i0 + 1)), f1 = LR ? 1.f : ex2(TOKEN ? s_cum[i1] : log2_pow(ld2, i1 + 1));
  const float skip = a.skip ? a.skip[h] : 0.f;
  const float* st = chunk_state + ((int64_t)blockIdx.x * a.heads + h) * D * a.vdim;
  const bool live = warp * 16 < ch.n;
  for (int v0 = 0; v0 < a.vdim; v0 += kVT) {
    float o[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    for (int d0 = 0; d0 < DP; d0 += 64) {
      const bool aligned = a.vdim % 4 == 0;
#pragma unroll 4
      for (int i = tid; i < 64 * kVT / 8; i += kT) {
        const int r = i / (kVT / 8), d = d0 + r, c = i % (kVT / 8) * 8;
        const float* src = st + (int64_t)d * a.vdim + v0 + c;
        float f[8];
        if (aligned && d < D && v0 + c + 8 <= a.vdim) {
          const float4 x = *reinterpret_cast<const float4*>(src), y = *reinterpret_cast<const float4*>(src + 4);
          f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w;
          f[4] = y.x; f[5] = y.y; f[6] = y.z; f[7] = y.w;
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = d < D && v0 + c + e < a.vdim ? src[e] : 0.f;
        }
        put_split8(t_hi + r * kVS + c, t_lo + r * kVS + c, f);
      }
      if (d0 == 0) load_values<TOKEN>(a, ch, h, v0, v_hi, v_lo);
      __syncthreads();
      if (live) {
        const int n_ks = min(4, (DP - d0) / 16);
        for (int ks = 0; ks < n_ks; ++ks) {
          uint32_t hi[4], lo[4];
          if (LR) {
            q_frag(d0 / 16 + ks, -1, hi, lo);
          } else {
            ldsm_x4(qh + (d0 / 16 + ks) * 32, hi[0], hi[1], hi[2], hi[3]);
            if (!TOKEN) ldsm_x4(ql + (d0 / 16 + ks) * 32, lo[0], lo[1], lo[2], lo[3]);
          }
#pragma unroll
          for (int nv = 0; nv < 4; ++nv) {
            uint32_t b[4], c[4];
            ldsm_x4_trans(th + (ks * 16 * kVS + nv * 16) * 2, b[0], b[1], b[2], b[3]);
            ldsm_x4_trans(tl + (ks * 16 * kVS + nv * 16) * 2, c[0], c[1], c[2], c[3]);
            if (TOKEN) {
              mma_bf16_16816(o[2 * nv], hi, b[0], b[1]);
              mma_bf16_16816(o[2 * nv + 1], hi, b[2], b[3]);
              mma_bf16_16816(o[2 * nv], hi, c[0], c[1]);
              mma_bf16_16816(o[2 * nv + 1], hi, c[2], c[3]);
              continue;
            }
            mma_split(o[2 * nv], hi, lo, b[0], b[1], c[0], c[1]);
            mma_split(o[2 * nv + 1], hi, lo, b[2], b[3], c[2], c[3]);
          }
        }
      }
      if (d0 + 64 < DP) __syncthreads();  // the state tile is refilled
    }
    if (live) {
      if (!LR) {
#pragma unroll
        for (int i = 0; i < 8; ++i) { o[i][0] *= f0; o[i][1] *= f0; o[i][2] *= f1; o[i][3] *= f1; }
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        if (kk <= warp) {
          uint32_t hi[4], lo[4];
          split_bf16(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
          split_bf16(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
          split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
          split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
          for (int nv = 0; nv < 4; ++nv) {
            uint32_t b[4], c[4];
            ldsm_x4_trans(vh + (kk * 16 * kVS + nv * 16) * 2, b[0], b[1], b[2], b[3]);
            if (TOKEN) {
              mma_pair(o[2 * nv], hi, lo, b[0], b[1]);
              mma_pair(o[2 * nv + 1], hi, lo, b[2], b[3]);
              continue;
            }
            ldsm_x4_trans(vl + (kk * 16 * kVS + nv * 16) * 2, c[0], c[1], c[2], c[3]);
            mma_split(o[2 * nv], hi, lo, b[0], b[1], c[0], c[1]);
            mma_split(o[2 * nv + 1], hi, lo, b[2], b[3], c[2], c[3]);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = e ? i1 : i0, c = i * 8 + 2 * t;
          if (r < ch.n) {
            float x = o[i][2 * e] * a.q_scale, y = o[i][2 * e + 1] * a.q_scale;
            if (TOKEN) {  // the values' own way around the state
              const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(v_hi + r * kVS + c);
              x = fmaf(skip, __low2float(v), x);
              y = fmaf(skip, __high2float(v), y);
            }
            put_pair(a.o + (int64_t)(ch.row0 + r) * a.ld_o + (int64_t)h * a.vdim + v0 + c, x, y, a.vdim - v0 - c);
          }
        }
    }
    __syncthreads();
  }
  pdl_trigger();
}

static int pad16h(int n) { return (n + 15) / 16 * 16; }
static size_t state_smem(const Recurrence& a) { return (size_t)2 * kC * (pad16h(a.dim) + 8 + kVS) * 2; }
static size_t output_smem(const Recurrence& a) {
  const size_t ks = (size_t)kC * (pad16h(a.dim) + 8) * 2, tiles = (size_t)(a.dt ? 3 : 4) * kC * kVS * 2;
  if (a.dt) return ks + std::max(ks, tiles);
  return a.decay ? 2 * ks + std::max(2 * ks, tiles)
                 : ks + (size_t)kC * (pad16h(a.dim) + 4) * 4 + std::max(3 * ks, tiles);
}

bool recurrence_chunks_supported(const Recurrence& a, hb_dtype dtype) {
  static const bool off = [] { const char* e = getenv("HB_RECURRENCE"); return e && e[0] == 't'; }();
  return !off && dtype == HB_BF16 && !(a.dt && (a.silu_qkv || a.q_scale != 1.f)) && !(a.skip && !a.dt) && output_smem(a) <= 224 * 1024 && state_smem(a) <= 224 * 1024 &&
         (size_t)kC * a.rank * 4 <= 48 * 1024;
}

int recurrence_chunks(cudaStream_t st, const Recurrence& a, const RecurrenceChunks& c, int64_t* launches) {
  if (c.n_chunks == 0) return HB_OK;
  const unsigned nc = (unsigned)c.n_chunks, H = (unsigned)a.heads;
  auto opt_in = [](auto* k, size_t smem) -> int {
    if (smem > 48 * 1024) HB_CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
    return HB_OK;
  };
  int rc;
  if (a.dt) {
    HB_CUDA_CHECK(launch_pdl(recurrence_step_kernel, dim3(nc, (unsigned)((a.heads + kStepHeads - 1) / kStepHeads)), dim3(256), 0, st,
                             a, c.chunks, c.cum));
    ++*launches;
  } else if (!a.decay) {
    HB_CUDA_CHECK(launch_pdl(recurrence_decay_kernel, dim3(nc, (unsigned)((a.heads * a.dim + 255) / 256)), dim3(256),
                             (size_t)kC * a.rank * 4, st, a, c.chunks, c.cum));
    ++*launches;
  }
  const size_t ss = state_smem(a), os = output_smem(a);
  const int64_t per_head = (int64_t)a.dim * a.vdim;
  const int vec = a.vdim % 4 == 0 ? 4 : 1;
  auto run = [&](auto* own, auto* scan, auto* out) -> int {
    if ((rc = opt_in(own, ss)) || (rc = opt_in(out, os))) return rc;
    HB_CUDA_CHECK(launch_pdl(own, dim3(nc, H, (unsigned)((a.vdim + kVT - 1) / kVT)), dim3(kT), ss, st, a, c.chunks,
                             (const float*)c.cum, c.state));
    HB_CUDA_CHECK(launch_pdl(scan, dim3((unsigned)((per_head / vec + 255) / 256), H, (unsigned)c.n_segs), dim3(256), 0, st, a,
                             c.segs, c.chunks, (const float*)c.cum, c.state));
    HB_CUDA_CHECK(launch_pdl(out, dim3(nc, H), dim3(kT), os, st, a, c.chunks, (const float*)c.cum, (const float*)c.state));
    *launches += 3;
    return HB_OK;
  };
#define HB_RECURRENCE(MODE)                                                                                   \
  return run(recurrence_state_kernel<MODE>, vec == 4 ? recurrence_scan_kernel<4, MODE> : recurrence_scan_kernel<1, MODE>, \
             recurrence_output_kernel<MODE>)
  if (a.dt) HB_RECURRENCE(kPerToken);
  if (a.decay) HB_RECURRENCE(kConstant);
  HB_RECURRENCE(kLowRank);
#undef HB_RECURRENCE
}

}  // namespace hb
