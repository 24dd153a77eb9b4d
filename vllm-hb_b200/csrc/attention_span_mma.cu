// Span attention (see attention_span.cu) on tensor cores: bf16, key and value widths that are
// multiples of 8.  S = Q K^T with bf16 operands and fp32 accumulation, softmax in fp32, and
// O += P V with P as a pair of bf16 numbers (P = hi + lo), so that the weights keep fp32-like
// precision.  Kernels instantiated with EXT also take a bias by distance, a cap on the scores, and keys
// that are or contain their values: K and V are then one tile of shared memory, read once.
//
//   tiles  (prompt portions): CTA = 64 rows = up to 64 / R consecutive positions of one segment x
//          the R query heads of a kv head; four warps of 16 rows share every 64-key tile.
//   tokens (decoded tokens): CTA = one row and kv head with its R <= 16 query heads; each of four
//          warps streams every fourth 16-key block through a ring of its own and the warps'
//          (m, l, O) meet in shared memory.
//
// Both read only the 16-key blocks that some row of the CTA sees: those of the first kept tokens
// and those from the earliest window on.  Rows of shared memory are padded by 8 elements, so that
// ldmatrix is conflict-free for every width.  Value widths above 256 are cut into slices (grid.z).
#include <algorithm>
#include <climits>

#include "layered_ops.h"
#include "span_core.cuh"

namespace hb {

namespace {
constexpr int kThreads = 128;
constexpr int kWarps = 4;
constexpr int kRows = 64;      // query rows of a tile
constexpr int kKeys = 64;      // keys of a tile step
constexpr int kSlice = 256;    // widest value slice
constexpr int kRing = 3;       // 16-key stages of a warp (token kernel)
constexpr int kMaxSplits = 64; // of a row
constexpr int kMaxCluster = 8; // splits of a row that sum up in a cluster
}  // namespace

// NV: 16-column pairs of n-tiles, i.e. the value slice is at most 16 * NV wide.  DK > 0: keys are DK and
// values 16 * NV wide exactly, known to the compiler.
template <int NV, bool EXT, int DK>
__global__ void __launch_bounds__(kThreads)
span_attention_tiles_kernel(const SpanAttention a, const RowRange* __restrict__ tiles, int stages) {
  extern __shared__ __align__(16) uint8_t smem[];
  const HeadSlice hs(a, blockIdx.y);
  constexpr bool FIX = DK > 0;
  const int R = hs.n, D = FIX ? DK : a.dim, DP = pad16(D), KS = DP + 8;
  const bool tied = EXT && !a.vc;                       // one tile is keys and values
  const int v0 = FIX ? 0 : blockIdx.z * kSlice, VW = FIX ? 16 * NV : min(kSlice, a.vdim - v0), VP = pad16(VW), VS = tied ? KS : VP + 8;
  __nv_bfloat16* s_q = (__nv_bfloat16*)smem;           // [64][KS]
  __nv_bfloat16* s_k = s_q + kRows * KS;               // [stages][64][KS]
  __nv_bfloat16* s_v = tied ? s_k : s_k + stages * kKeys * KS;               // [stages][64][VS]
  float* s_ks = (float*)(s_k + stages * kKeys * KS);   // tied: [stages][64] scales of the keys
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gi = lane >> 2, t = lane & 3, kvh = hs.kvh;
  // padding columns stay zero
  for (int i = tid; i < (kRows + stages * kKeys) * KS / 8; i += kThreads)
    if (i % (KS / 8) * 8 >= D) reinterpret_cast<uint4*>(s_q)[i] = make_uint4(0, 0, 0, 0);
  if (!tied)
    for (int i = tid; i < stages * kKeys * VS / 8; i += kThreads)
      if (i % (VS / 8) * 8 >= VW) reinterpret_cast<uint4*>(s_v)[i] = make_uint4(0, 0, 0, 0);
  pdl_grid_wait();
  const RowRange tile = tiles[gridDim.x - 1 - blockIdx.x];  // later positions see more: they go first
  const int first_pos = a.pos[tile.row0], last_pos = first_pos + tile.n - 1;
  const BlockRuns runs = block_runs(first_pos, last_pos, a);
  const int32_t* table = a.tables + (a.linear ? (int64_t)tile.seg : (int64_t)tile.seg * a.max_blocks);
  const int n_rows = tile.n * R, n_steps = (runs.n + kKeys / kBS - 1) / (kKeys / kBS);

  const __nv_bfloat16* q = (const __nv_bfloat16*)a.q + (int64_t)hs.first * D;
  for (int i = tid; i < kRows * (D / 8); i += kThreads) {
    const int m = i / (D / 8), c = i % (D / 8) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (m < n_rows) v = *reinterpret_cast<const uint4*>(q + (int64_t)(tile.row0 + m / R) * a.ld_q + (m % R) * D + c);
    *reinterpret_cast<uint4*>(s_q + m * KS + c) = v;
  }
  const int DH = D - a.tail;  // channels of a key that are its head's own
  const BlockCopy copy_k(DH, lane), copy_v(VW, lane), copy_t(max(a.tail, 8), lane);
  auto load = [&](int step) {  // every warp one block of 16 keys
    const int s = step % stages;
    // past the last block: any block will do, its keys are masked (positions beyond the row's)
    const int lb = runs.block(min(step * kWarps + warp, runs.n - 1));
    int64_t phys = lb < a.max_blocks ? (a.linear ? table[0] + lb : table[lb]) : 0;
    if (phys < 0 || phys >= a.num_blocks) phys = 0;  // never outside the pool
    const uint32_t k_dst = smem_u32(s_k + (s * kKeys + warp * kBS) * KS);
    copy_k(k_dst, KS * 2, (const __nv_bfloat16*)a.kc + phys * a.k_step.block + kvh * a.k_step.head, a.k_step.token);
    if (a.tail) copy_t(k_dst + DH * 2, KS * 2, (const __nv_bfloat16*)a.kt + phys * kBS * a.ld_kt, a.ld_kt);
    if (!tied)
      copy_v(smem_u32(s_v + (s * kKeys + warp * kBS) * VS), VS * 2,
             (const __nv_bfloat16*)a.vc + phys * a.v_step.block + kvh * a.v_step.head + v0, a.v_step.token);
    else if (a.key_scale && lane < 4) cp_async_16(smem_u32(s_ks + s * kKeys + warp * kBS + lane * 4), a.key_scale + phys * kBS + lane * 4);
    cp_async_commit();
  };
  load(0);

  const int r0 = warp * 16 + gi, r1 = r0 + 8;
  const int p0 = first_pos + r0 / R, p1 = first_pos + r1 / R;
  const int lo0 = a.first_seen(p0), lo1 = a.first_seen(p1);
  const bool live = warp * 16 < n_rows;  // warps without rows only help to load
  float o[2 * NV][4];
#pragma unroll
  for (int i = 0; i < 2 * NV; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  const float sc = a.scale * kLog2e;               // scores in units of log2
  const bool sc_ok = !EXT && sc > 0.f;
  const float es = sc_ok ? sc : 1.f;               // what the exponential still multiplies by
  const int warp_first = first_pos + warp * 16 / R, warp_last = min(first_pos + (warp * 16 + 15) / R, last_pos);
  const int warp_lo = a.first_seen(warp_last);
  const float cap = EXT ? a.softcap * kLog2e : 0.f, cap_k = cap > 0.f ? 2.f / a.softcap : 0.f;
  const float *bias0 = nullptr, *bias1 = nullptr;  // of the rows' heads, by distance
  float far0 = 0.f, far1 = 0.f;                    // from distance dist_len - 1 on, in units of log2
  if (EXT && a.dist_bias) {
    bias0 = a.dist_bias + (int64_t)(hs.first + r0 % R) * a.dist_len;
    bias1 = a.dist_bias + (int64_t)(hs.first + r1 % R) * a.dist_len;
    far0 = __ldg(bias0 + a.dist_len - 1) * kLog2e;
    far1 = __ldg(bias1 + a.dist_len - 1) * kLog2e;
  }
  const uint32_t q_addr = smem_u32(s_q + (warp * 16 + (lane & 15)) * KS + (lane >> 4) * 8);

  for (int step = 0; step < n_steps; ++step) {
    if (stages > 1 && step + 1 < n_steps) {
      load(step + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (live) {
      const __nv_bfloat16* kt = s_k + step % stages * kKeys * KS;
      const __nv_bfloat16* vt = s_v + step % stages * kKeys * VS;
      float s[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
      // lanes 0-7 / 8-15 / 16-23 / 24-31 address keys 0-7 k-low, 0-7 k-high, 8-15 k-low, 8-15 k-high
      const uint32_t k_addr = smem_u32(kt + ((lane & 7) + (lane >> 4) * 8) * KS + ((lane >> 3) & 1) * 8);
#pragma unroll(FIX ? DK / 16 : 1)
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t qa[4];
        ldsm_x4(q_addr + ks * 32, qa[0], qa[1], qa[2], qa[3]);
#pragma unroll
        for (int nk = 0; nk < 4; ++nk) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(k_addr + (nk * 16 * KS + ks * 16) * 2, b0, b1, b2, b3);
          mma_bf16_16816(s[2 * nk], qa, b0, b1);
          mma_bf16_16816(s[2 * nk + 1], qa, b2, b3);
        }
      }
      // scores stay unscaled: sc > 0 is applied inside the exponential (sc <= 0: scaled here)
      bool full = sc_ok || EXT;
      int last_key = 0;
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        const int vb = step * (kKeys / kBS) + b;
        full = full && vb < runs.n && all_visible(runs.block(vb) * kBS, warp_first, warp_lo, a.keep_first);
        last_key = max(last_key, vb < runs.n ? runs.block(vb) * kBS + kBS - 1 : INT_MAX / 2);
      }
      if (EXT) {
        // scale per key and bias by distance; from the table's last distance on the bias is one number
        const bool far = !bias0 || warp_first - last_key >= a.dist_len - 1;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          float2 f = make_float2(sc, sc);
          if (a.key_scale) {
            f = *reinterpret_cast<const float2*>(s_ks + step % stages * kKeys + i * 8 + 2 * t);
            f.x *= sc;
            f.y *= sc;
          }
          if (cap > 0.f) {
            s[i][0] = capped(s[i][0] * f.x, cap, cap_k); s[i][1] = capped(s[i][1] * f.y, cap, cap_k);
            s[i][2] = capped(s[i][2] * f.x, cap, cap_k); s[i][3] = capped(s[i][3] * f.y, cap, cap_k);
            f = make_float2(1.f, 1.f);
          }
          if (far) {
            s[i][0] = fmaf(s[i][0], f.x, far0); s[i][1] = fmaf(s[i][1], f.y, far0);
            s[i][2] = fmaf(s[i][2], f.x, far1); s[i][3] = fmaf(s[i][3], f.y, far1);
          } else {
            const int vb = step * (kKeys / kBS) + i / 2, top = a.dist_len - 1;
            const int key = (vb < runs.n ? runs.block(vb) * kBS : 0) + (i & 1) * 8 + 2 * t;
            s[i][0] = fmaf(s[i][0], f.x, __ldg(bias0 + min(max(p0 - key, 0), top)) * kLog2e);
            s[i][1] = fmaf(s[i][1], f.y, __ldg(bias0 + min(max(p0 - key - 1, 0), top)) * kLog2e);
            s[i][2] = fmaf(s[i][2], f.x, __ldg(bias1 + min(max(p1 - key, 0), top)) * kLog2e);
            s[i][3] = fmaf(s[i][3], f.y, __ldg(bias1 + min(max(p1 - key - 1, 0), top)) * kLog2e);
          }
        }
      }
      if (!full) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int vb = step * (kKeys / kBS) + i / 2;
          const int key = vb < runs.n ? runs.block(vb) * kBS + (i & 1) * 8 + 2 * t : INT_MAX - 1;
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const bool scaled = EXT || sc_ok;
            s[i][c] = visible(key + c, p0, lo0, a.keep_first) ? (scaled ? s[i][c] : s[i][c] * sc) : -INFINITY;
            s[i][2 + c] = visible(key + c, p1, lo1, a.keep_first) ? (scaled ? s[i][2 + c] : s[i][2 + c] * sc) : -INFINITY;
          }
        }
      }
      float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        x0 = fmaxf(x0, fmaxf(s[i][0], s[i][1]));
        x1 = fmaxf(x1, fmaxf(s[i][2], s[i][3]));
      }
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
      const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);
      const float e0 = n0 == -INFINITY ? 0.f : n0, e1 = n1 == -INFINITY ? 0.f : n1;  // nothing visible yet
      if (__any_sync(0xffffffffu, n0 != m0 || n1 != m1)) {
        const float al0 = ex2((m0 - e0) * es), al1 = ex2((m1 - e1) * es);
        m0 = n0; m1 = n1;
        l0 *= al0; l1 *= al1;
#pragma unroll
        for (int i = 0; i < 2 * NV; ++i) { o[i][0] *= al0; o[i][1] *= al0; o[i][2] *= al1; o[i][3] *= al1; }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        s[i][0] = ex2((s[i][0] - e0) * es); s[i][1] = ex2((s[i][1] - e0) * es);
        s[i][2] = ex2((s[i][2] - e1) * es); s[i][3] = ex2((s[i][3] - e1) * es);
        l0 += s[i][0] + s[i][1];
        l1 += s[i][2] + s[i][3];
      }
      const uint32_t v_addr = smem_u32(vt + (lane & 15) * VS + (lane >> 4) * 8 + (tied ? v0 : 0));
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t hi[4], lo[4];
        split_bf16(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
        split_bf16(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
        split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
        split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int nv = 0; nv < NV; ++nv) {
          if (nv * 16 < VP) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4_trans(v_addr + (kk * 16 * VS + nv * 16) * 2, b0, b1, b2, b3);
            mma_bf16_16816(o[2 * nv], hi, b0, b1);
            mma_bf16_16816(o[2 * nv + 1], hi, b2, b3);
            mma_bf16_16816(o[2 * nv], lo, b0, b1);
            mma_bf16_16816(o[2 * nv + 1], lo, b2, b3);
          }
        }
      }
    }
    __syncthreads();
    if (stages == 1 && step + 1 < n_steps) load(step + 1);
  }
  pdl_trigger();
  if (!live) return;
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  float i0 = 1.f / l0, i1 = 1.f / l1;
  if (a.sink) {  // one more member of the softmax, without a value
    const float k0 = a.sink[hs.first + r0 % R] * kLog2e, k1 = a.sink[hs.first + r1 % R] * kLog2e;
    const float t0 = fmaxf(m0 * es, k0), t1 = fmaxf(m1 * es, k1), f0 = ex2(m0 * es - t0), f1 = ex2(m1 * es - t1);
    i0 = f0 / fmaf(l0, f0, ex2(k0 - t0));
    i1 = f1 / fmaf(l1, f1, ex2(k1 - t1));
  }
  const __nv_bfloat16 *g0 = nullptr, *g1 = nullptr;
  if (a.gate) {
    const __nv_bfloat16* gate = (const __nv_bfloat16*)a.gate;
    g0 = gate + a.gate_at(tile.row0 + r0 / R, hs.first + r0 % R, v0);
    g1 = gate + a.gate_at(tile.row0 + r1 / R, hs.first + r1 % R, v0);
    if (a.gate_per_head) {
      if (r0 < n_rows) i0 *= sigmoid_of(*reinterpret_cast<const uint16_t*>(g0));
      if (r1 < n_rows) i1 *= sigmoid_of(*reinterpret_cast<const uint16_t*>(g1));
    }
  }
  __nv_bfloat16* out = (__nv_bfloat16*)a.out + (int64_t)hs.first * a.vdim + v0;
  __nv_bfloat16* w0 = out + (int64_t)(tile.row0 + r0 / R) * a.ld_out + (r0 % R) * a.vdim;
  __nv_bfloat16* w1 = out + (int64_t)(tile.row0 + r1 / R) * a.ld_out + (r1 % R) * a.vdim;
#pragma unroll
  for (int i = 0; i < 2 * NV; ++i) {
    const int c = i * 8 + 2 * t;
    if (c < VW) {
      float x[4] = {o[i][0] * i0, o[i][1] * i0, o[i][2] * i1, o[i][3] * i1};
      if (a.gate && !a.gate_per_head) {
        const uint32_t z0 = r0 < n_rows ? *reinterpret_cast<const uint32_t*>(g0 + c) : 0u;
        const uint32_t z1 = r1 < n_rows ? *reinterpret_cast<const uint32_t*>(g1 + c) : 0u;
        x[0] *= sigmoid_of(z0 & 0xffffu); x[1] *= sigmoid_of(z0 >> 16);
        x[2] *= sigmoid_of(z1 & 0xffffu); x[3] *= sigmoid_of(z1 >> 16);
      }
      if (r0 < n_rows) *reinterpret_cast<uint32_t*>(w0 + c) = pack_bf16(x[0], x[1]);
      if (r1 < n_rows) *reinterpret_cast<uint32_t*>(w1 + c) = pack_bf16(x[2], x[3]);
    }
  }
}

// n_splits > 1: every CTA takes its share of the row's blocks.  The CTAs of a row and kv head form a
// thread-block cluster (`clustered`) and sum up through each other's shared memory, or, more than
// fit one, write (m, l, O) partials that a second kernel sums up.
//
// The products are turned over, so that the few query heads are the narrow MMA side:
// S^T[16 keys, 8 NT heads] = K Q^T and O^T[values, heads] += V^T P^T (P transposed in registers).
// MT: 16-column tiles of the value slice, NT: groups of 8 query heads.
// FIX: keys and values are 16 * MT wide exactly, known to the compiler.
template <int MT, int NT, bool EXT, bool FIX>
__global__ void __launch_bounds__(kThreads)
span_attention_tokens_kernel(const SpanAttention a, const int32_t* __restrict__ rows, int n_splits, int clustered,
                             float* __restrict__ part) {
  extern __shared__ __align__(16) uint8_t smem[];
  const HeadSlice hs(a, blockIdx.y);
  const int R = hs.n, D = FIX ? 16 * MT : a.dim, DP = pad16(D), KS = DP + 8;
  const bool tied = EXT && !a.vc;                   // one tile is keys and values; their scales lie behind it
  const int v0 = FIX ? 0 : (int)(blockIdx.z / n_splits) * kSlice, VW = FIX ? 16 * MT : min(kSlice, a.vdim - v0), VP = pad16(VW), VS = VP + 8;
  const int split = blockIdx.z % n_splits;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, gi = lane >> 2, t = lane & 3, kvh = hs.kvh;
  const int stage_elems = tied ? kBS * (KS + 2) : kBS * (KS + VS);
  __nv_bfloat16* s_q = (__nv_bfloat16*)smem;                                  // [16][KS]
  __nv_bfloat16* ring = s_q + 16 * KS + (size_t)warp * kRing * stage_elems;   // [kRing][K 16 x KS | V 16 x VS]
  if (D % 16 || VW % 16) {  // padding columns stay zero
    for (int s = 0; s < kRing; ++s)
      for (int i = lane; i < kBS; i += 32) {
        for (int c = D; c < DP; c += 8) *reinterpret_cast<uint4*>(ring + s * stage_elems + i * KS + c) = make_uint4(0, 0, 0, 0);
        for (int c = VW; c < VP && !tied; c += 8)
          *reinterpret_cast<uint4*>(ring + s * stage_elems + kBS * KS + i * VS + c) = make_uint4(0, 0, 0, 0);
      }
  }
  pdl_grid_wait();
  const int64_t row = rows[blockIdx.x];
  const int pos = a.pos[row];
  const int32_t* table = a.tables + (int64_t)a.row_seg[row] * a.max_blocks;
  const int lo = a.first_seen(pos);
  const BlockRuns runs = block_runs(pos, pos, a);
  const int per = (runs.n + n_splits - 1) / n_splits, s_lo = split * per, s_hi = min(runs.n, s_lo + per);
  const int n_w = s_hi - s_lo > warp ? (s_hi - s_lo - warp + kWarps - 1) / kWarps : 0;  // this warp's blocks

  int tab_base = 0, tab = 0;
  auto load_tab = [&](int base) {  // block table entries of this warp, 32 at a time, one per lane
    tab_base = base;
    const int i = base + lane;
    const int lb = i < n_w ? runs.block(s_lo + warp + kWarps * i) : 0;
    tab = lb < a.max_blocks ? table[lb] : 0;
    if (tab < 0 || tab >= a.num_blocks) tab = 0;  // never outside the pool
  };
  const BlockCopy copy_k(D, lane), copy_v(VW, lane);
  const uint32_t ring_u = smem_u32(ring);
  int stage_in = 0;  // stage the next load fills
  auto load = [&](int i) {
    if (i < n_w) {
      if (i >= tab_base + 32) load_tab(i);
      const int64_t phys = __shfl_sync(0xffffffffu, tab, i - tab_base), slot = (phys * a.kv_heads + kvh) * kBS;
      const uint32_t dst = ring_u + stage_in * stage_elems * 2;
      copy_k(dst, KS * 2, (const __nv_bfloat16*)a.kc + slot * D, D);
      if (!tied) copy_v(dst + kBS * KS * 2, VS * 2, (const __nv_bfloat16*)a.vc + slot * a.vdim + v0, a.vdim);
      else if (a.key_scale && lane < 4) cp_async_16(dst + kBS * KS * 2 + lane * 16, a.key_scale + phys * kBS + lane * 4);
    }
    cp_async_commit();
    stage_in = stage_in + 1 == kRing ? 0 : stage_in + 1;
  };
  load_tab(0);
  for (int i = 0; i < kRing - 1; ++i) load(i);
  const __nv_bfloat16* q = (const __nv_bfloat16*)a.q + row * a.ld_q + (int64_t)hs.first * D;
  for (int i = tid; i < 16 * (KS / 8); i += kThreads) {
    const int m = i / (KS / 8), c = i % (KS / 8) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (m < R && c < D) v = *reinterpret_cast<const uint4*>(q + m * D + c);
    *reinterpret_cast<uint4*>(s_q + m * KS + c) = v;
  }
  __syncthreads();
  float o[NT][MT][4], m[NT][2], l[NT][2];  // heads 8n + 2t, 8n + 2t + 1; o: value columns gi, gi + 8 of a tile
#pragma unroll
  for (int n = 0; n < NT; ++n) {
#pragma unroll
    for (int i = 0; i < MT; ++i) o[n][i][0] = o[n][i][1] = o[n][i][2] = o[n][i][3] = 0.f;
    m[n][0] = m[n][1] = -INFINITY;
    l[n][0] = l[n][1] = 0.f;
  }
  const float sc = a.scale * kLog2e;  // scores in units of log2
  const float cap = EXT ? a.softcap * kLog2e : 0.f, cap_k = cap > 0.f ? 2.f / a.softcap : 0.f;
  float far[NT][2];                   // bias from distance dist_len - 1 on
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int head = min(n * 8 + 2 * t + c, R - 1);
      far[n][c] = EXT && a.dist_bias ? __ldg(a.dist_bias + (int64_t)(hs.first + head + 1) * a.dist_len - 1) * kLog2e : 0.f;
    }
  const uint32_t q_addr = smem_u32(s_q + (lane & 7) * KS + (lane >> 3) * 8);  // B fragments of two 16-channel steps
  const uint32_t k_off = (uint32_t)(((lane & 15) * KS + (lane >> 4) * 8) * 2);
  const uint32_t v_off = (uint32_t)(((tied ? v0 : kBS * KS) + ((lane & 7) + (lane >> 4) * 8) * (tied ? KS : VS) +
                                     ((lane >> 3) & 1) * 8) * 2);
  int stage = 0;
  for (int i = 0; i < n_w; ++i) {
    load(i + kRing - 1);
    cp_async_wait<kRing - 1>();
    __syncwarp();
    const uint32_t base = ring_u + stage * stage_elems * 2;
    const __nv_bfloat16* stage_ptr = ring + stage * stage_elems;
    stage = stage + 1 == kRing ? 0 : stage + 1;
    float s[NT][2][4];  // two partial sums, so that neighbouring steps do not wait for each other
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][0][e] = s[n][1][e] = 0.f;
#pragma unroll(FIX ? (MT + 1) / 2 : 4)
    for (int ks = 0; ks < DP / 16; ks += 2) {
      uint32_t k0[4], k1[4];
      ldsm_x4(base + k_off + ks * 32, k0[0], k0[1], k0[2], k0[3]);
      const bool two = ks + 1 < DP / 16;
      if (two) ldsm_x4(base + k_off + ks * 32 + 32, k1[0], k1[1], k1[2], k1[3]);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        uint32_t b0, b1, b2, b3;
        // (a lone last step also reads the 16 elements behind it, into the ring at most: unused)
        ldsm_x4(q_addr + (n * 8 * KS + ks * 16) * 2, b0, b1, b2, b3);
        mma_bf16_16816(s[n][0], k0, b0, b1);
        if (two) mma_bf16_16816(s[n][1], k1, b2, b3);
      }
    }
    const int key0 = runs.block(s_lo + warp + kWarps * i) * kBS;
    const bool full = all_visible(key0, pos, lo, a.keep_first);
    const bool see0 = full || visible(key0 + gi, pos, lo, a.keep_first);
    const bool see1 = full || visible(key0 + gi + 8, pos, lo, a.keep_first);
    float f0 = sc, f1 = sc;  // scales of keys gi and gi + 8
    if (EXT && a.key_scale) {
      const float* ks = reinterpret_cast<const float*>(stage_ptr + kBS * KS);
      f0 *= ks[gi];
      f1 *= ks[gi + 8];
    }
    const bool near = EXT && a.dist_bias && pos - (key0 + kBS - 1) < a.dist_len - 1;
    const int d0 = near ? min(max(pos - key0 - gi, 0), a.dist_len - 1) : 0;
    const int d1 = near ? min(max(pos - key0 - gi - 8, 0), a.dist_len - 1) : 0;
    uint32_t ph[NT][2], plo[NT][2];
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      float p[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float b = far[n][e & 1];
        if (near) {
          const int head = min(n * 8 + 2 * t + (e & 1), R - 1);
          b = __ldg(a.dist_bias + (int64_t)(hs.first + head) * a.dist_len + (e < 2 ? d0 : d1)) * kLog2e;
        }
        float x = s[n][0][e] + s[n][1][e];
        if (EXT) {
          x *= e < 2 ? f0 : f1;
          if (cap > 0.f) x = capped(x, cap, cap_k);
        }
        p[e] = (e < 2 ? see0 : see1) ? (EXT ? x + b : x * sc) : -INFINITY;
      }
      float x0 = fmaxf(p[0], p[2]), x1 = fmaxf(p[1], p[3]);
#pragma unroll
      for (int w = 4; w < 32; w <<= 1) {
        x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, w));
        x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, w));
      }
      const float n0 = fmaxf(m[n][0], x0), n1 = fmaxf(m[n][1], x1);
      const float e0 = n0 == -INFINITY ? 0.f : n0, e1 = n1 == -INFINITY ? 0.f : n1;
      if (__any_sync(0xffffffffu, n0 != m[n][0] || n1 != m[n][1])) {
        const float al0 = ex2(m[n][0] - e0), al1 = ex2(m[n][1] - e1);
        m[n][0] = n0; m[n][1] = n1;
        l[n][0] *= al0; l[n][1] *= al1;
#pragma unroll
        for (int k = 0; k < MT; ++k) { o[n][k][0] *= al0; o[n][k][1] *= al1; o[n][k][2] *= al0; o[n][k][3] *= al1; }
      }
      p[0] = ex2(p[0] - e0); p[1] = ex2(p[1] - e1);
      p[2] = ex2(p[2] - e0); p[3] = ex2(p[3] - e1);
      l[n][0] += p[0] + p[2];
      l[n][1] += p[1] + p[3];
      uint32_t h0, g0, h1, g1;
      split_bf16(p[0], p[1], h0, g0);
      split_bf16(p[2], p[3], h1, g1);
      ph[n][0] = transpose_8x8(h0); ph[n][1] = transpose_8x8(h1);
      plo[n][0] = transpose_8x8(g0); plo[n][1] = transpose_8x8(g1);
    }
#pragma unroll
    for (int k = 0; k < MT; ++k) {
      if (k * 16 < VP) {
        uint32_t va[4];
        ldsm_x4_trans(base + v_off + k * 32, va[0], va[1], va[2], va[3]);
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          mma_bf16_16816(o[n][k], va, ph[n][0], ph[n][1]);
          mma_bf16_16816(o[n][k], va, plo[n][0], plo[n][1]);
        }
      }
    }
    __syncwarp();  // the stage is refilled by the next iteration's load
  }
  cp_async_wait<0>();
  pdl_trigger();
  // the warps' results meet in shared memory (the rings are idle now)
  __syncthreads();
  const int OS = VP + 2;
  float* s_o = (float*)(s_q + 16 * KS);          // [kWarps][R][OS]
  float* s_ml = s_o + (size_t)kWarps * R * OS;   // [kWarps][R][2]
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      float ll = l[n][c];
#pragma unroll
      for (int w = 4; w < 32; w <<= 1) ll += __shfl_xor_sync(0xffffffffu, ll, w);
      const int head = n * 8 + 2 * t + c;
      if (head < R) {
        float* dst = s_o + ((size_t)warp * R + head) * OS;
#pragma unroll
        for (int k = 0; k < MT; ++k)
          if (k * 16 < VP) { dst[k * 16 + gi] = o[n][k][c]; dst[k * 16 + gi + 8] = o[n][k][2 + c]; }
        if (gi == 0) { s_ml[(warp * R + head) * 2] = m[n][c]; s_ml[(warp * R + head) * 2 + 1] = ll; }
      }
    }
  __syncthreads();
  for (int h = warp; h < R; h += kWarps) {
    float mx = -INFINITY, ls = 0.f, f[kWarps];
#pragma unroll
    for (int w = 0; w < kWarps; ++w) mx = fmaxf(mx, s_ml[(w * R + h) * 2]);
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float mw = s_ml[(w * R + h) * 2];
      f[w] = mw == -INFINITY ? 0.f : ex2(mw - mx);
      ls = fmaf(f[w], s_ml[(w * R + h) * 2 + 1], ls);
    }
    const int64_t head = hs.first + h;
    float inv = 1.f / ls;
    if (a.sink && n_splits == 1) {
      const float k = a.sink[head] * kLog2e, top = fmaxf(mx, k), f = ex2(mx - top);
      inv = f / fmaf(ls, f, ex2(k - top));
    }
    float* p = n_splits > 1 && !clustered ? part + (((int64_t)blockIdx.x * a.heads + head) * n_splits + split) * (a.vdim + 2) : nullptr;
    for (int c = lane; c < VW; c += 32) {
      float acc = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) acc = fmaf(f[w], s_o[((size_t)w * R + h) * OS + c], acc);
      if (n_splits == 1) {
        acc *= inv;
        if (a.gate) acc *= sigmoid_of(((const uint16_t*)a.gate)[a.gate_at(row, head, v0 + c)]);
        ((__nv_bfloat16*)a.out)[row * a.ld_out + head * a.vdim + v0 + c] = __float2bfloat16_rn(acc);
      } else if (clustered) {
        s_o[(size_t)h * OS + c] = acc;  // the place of warp 0, read by this lane above
      } else {
        p[v0 + c] = acc;
      }
    }
    if (clustered) {
      __syncwarp();
      if (lane == 0) { s_ml[h * 2] = mx; s_ml[h * 2 + 1] = ls; }
    } else if (n_splits > 1 && lane == 0 && v0 == 0) {
      p[a.vdim] = mx;
      p[a.vdim + 1] = ls;
    }
  }
  if (!clustered) return;
  cluster_sync_all();
  const uint32_t o_addr = smem_u32(s_o), ml_addr = smem_u32(s_ml);
  for (int i = split * kThreads + tid; i < R * VW; i += n_splits * kThreads) {
    const int h = i / VW, c = i % VW;
    const int64_t head = hs.first + h;
    const float k = a.sink ? a.sink[head] * kLog2e : -INFINITY;
    float mx = k, ls = 0.f, acc = 0.f, mw[kMaxCluster];
#pragma unroll
    for (int s = 0; s < kMaxCluster; ++s) {
      mw[s] = s < n_splits ? ld_cluster_f32(cluster_map(ml_addr + h * 8, s)) : -INFINITY;
      mx = fmaxf(mx, mw[s]);
    }
    if (a.sink) ls = ex2(k - mx);
#pragma unroll
    for (int s = 0; s < kMaxCluster; ++s) {
      if (s < n_splits) {
        const float f = mw[s] == -INFINITY ? 0.f : ex2(mw[s] - mx);
        ls = fmaf(f, ld_cluster_f32(cluster_map(ml_addr + h * 8 + 4, s)), ls);
        acc = fmaf(f, ld_cluster_f32(cluster_map(o_addr + (uint32_t)(h * OS + c) * 4, s)), acc);
      }
    }
    acc /= ls;
    if (a.gate) acc *= sigmoid_of(((const uint16_t*)a.gate)[a.gate_at(row, head, v0 + c)]);
    ((__nv_bfloat16*)a.out)[row * a.ld_out + head * a.vdim + v0 + c] = __float2bfloat16_rn(acc);
  }
  cluster_sync_all();  // nobody leaves while a partner still reads its shared memory
}

// Sum of a row's split partials, weighted by their maxima.
__global__ void __launch_bounds__(kThreads)
span_attention_merge_kernel(const SpanAttention a, const int32_t* __restrict__ rows, int n_splits, const float* __restrict__ part) {
  pdl_trigger();
  pdl_grid_wait();
  __shared__ float s_f[kMaxSplits], s_scale;
  const int64_t row = rows[blockIdx.x];
  const int head = blockIdx.y, tid = threadIdx.x, ld = a.vdim + 2;
  const float* p = part + ((int64_t)blockIdx.x * a.heads + head) * n_splits * ld;
  if (tid < 32) {  // the splits' factors, by one warp
    const float k = a.sink ? a.sink[head] * kLog2e : -INFINITY;
    float mx = k, l = 0.f, m[kMaxSplits / 32];
#pragma unroll
    for (int i = 0; i < kMaxSplits / 32; ++i) {
      m[i] = tid + 32 * i < n_splits ? p[(tid + 32 * i) * ld + a.vdim] : -INFINITY;
      mx = fmaxf(mx, m[i]);
    }
    mx = warp_max(mx);
#pragma unroll
    for (int i = 0; i < kMaxSplits / 32; ++i) {
      if (tid + 32 * i >= n_splits) continue;
      const float f = m[i] == -INFINITY ? 0.f : ex2(m[i] - mx);
      s_f[tid + 32 * i] = f;
      if (f > 0.f) l = fmaf(f, p[(tid + 32 * i) * ld + a.vdim + 1], l);
    }
    l = warp_sum(l);
    if (tid == 0) s_scale = 1.f / (a.sink ? l + ex2(k - mx) : l);
  }
  __syncthreads();
  for (int c = tid; c < a.vdim; c += kThreads) {
    float acc = 0.f;
#pragma unroll 8
    for (int s = 0; s < n_splits; ++s) {
      const float f = s_f[s];
      acc = f > 0.f ? fmaf(f, p[s * ld + c], acc) : acc;
    }
    acc *= s_scale;
    if (a.gate) acc *= sigmoid_of(((const uint16_t*)a.gate)[a.gate_at(row, head, c)]);
    ((__nv_bfloat16*)a.out)[row * a.ld_out + (int64_t)head * a.vdim + c] = __float2bfloat16_rn(acc);
  }
}

static SpanAttention sliced(const SpanAttention& args, int most) {
  SpanAttention a = args;
  a.cut(most);
  return a;
}
static bool is_ext(const SpanAttention& a) { return !a.vc || a.dist_bias || a.softcap > 0.f; }
static size_t tiles_smem(const SpanAttention& a, int stages) {
  const int KS = pad16(a.dim) + 8, VS = pad16(std::min(a.vdim, kSlice)) + 8;
  return (size_t)(kRows * KS + stages * kKeys * (KS + (a.vc ? VS : 2))) * 2;
}
static size_t tokens_smem(const SpanAttention& a) {
  const int R = sliced(a, 16).slice, KS = pad16(a.dim) + 8, VP = pad16(std::min(a.vdim, kSlice)), VS = VP + 8;
  const size_t ring = (size_t)kWarps * kRing * kBS * (KS + (a.vc ? VS : 2)) * 2;
  const size_t merge = (size_t)kWarps * R * (VP + 4) * sizeof(float);
  return (size_t)16 * KS * 2 + std::max(ring, merge);
}
bool span_attention_mma_ok(const SpanAttention& a, hb_dtype dtype) {
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  static const bool simt = [] { const char* e = getenv("HB_ATTN"); return e && e[0] == 's'; }();
  return !simt && dtype == HB_BF16 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ld_q % 8 == 0 && a.ld_out % 2 == 0 && al(a.q) &&
         al(a.out) && (!a.gate || a.gate_per_head || (a.ld_gate % 2 == 0 && (reinterpret_cast<uintptr_t>(a.gate) & 3) == 0)) &&
         (a.vc || a.vdim <= a.dim) && (!a.key_scale || (a.dim == a.vdim && !a.vc && al(a.key_scale)));
}

int span_attention_tile_positions(const SpanAttention& a, hb_dtype dtype) {
  if (!span_attention_mma_ok(a, dtype) || tiles_smem(a, 1) > kSmemCap) return 0;
  return kRows / sliced(a, kRows).slice;
}
int span_attention_tokens_slots(const SpanAttention& a) {
  constexpr int kSms = 148;
  if (latent_tokens_supported(a, HB_BF16)) return kSms;
  return kSms * (int)std::max<size_t>(1, std::min<size_t>(8, (size_t)227 * 1024 / (tokens_smem(a) + 1024)));
}
bool span_attention_tokens_supported(const SpanAttention& a, hb_dtype dtype) {
  return latent_tokens_supported(a, dtype) || (span_attention_mma_ok(a, dtype) && tokens_smem(a) <= kSmemCap);
}

template <typename K>
static int opt_in(K kernel, size_t smem) {
  if (smem > 48 * 1024) HB_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemCap));
  return HB_OK;
}

int span_attention_token_units(const SpanAttention& a) {
  if (latent_tokens_supported(a, HB_BF16)) return latent_tokens_units(a);
  return a.kv_heads * sliced(a, 16).slices();
}

int span_attention_tiles(cudaStream_t st, const SpanAttention& args, const RowRange* tiles, int n_tiles) {
  if (n_tiles == 0) return HB_OK;
  SpanAttention a = sliced(args, kRows);
  auto pool = [&](SpanAttention::Steps& s, int width) {
    if (!s.token) s = {(int64_t)a.kv_heads * kBS * width, (int64_t)kBS * width, width};
  };
  pool(a.k_step, a.dim);
  pool(a.v_step, a.vdim);
  if (a.tail % 8 || a.k_step.token % 8 || a.v_step.token % 8 || a.k_step.head % 8 || a.v_step.head % 8 || a.ld_kt % 8)
    return fail(HB_ERR_INVALID_ARG, "span attention: keys and values must lie on 16-byte boundaries");
  const int stages = tiles_smem(a, 2) <= kSmemCap ? 2 : 1;
  const size_t smem = tiles_smem(a, stages);
  const dim3 grid((unsigned)n_tiles, (unsigned)(a.kv_heads * a.slices()), (unsigned)((a.vdim + kSlice - 1) / kSlice));
  auto launch = [&](auto* k) -> int {
    int rc = opt_in(k, smem);
    if (rc) return rc;
    HB_CUDA_CHECK(launch_pdl(k, grid, dim3(kThreads), smem, st, a, tiles, stages));
    return HB_OK;
  };
  const int vw = std::min(a.vdim, kSlice);
  const bool ext = is_ext(a);
#define HB_TILES(NV)                                                                                          \
  return a.dim == 16 * NV && a.vdim == 16 * NV                                                                \
             ? (ext ? launch(span_attention_tiles_kernel<NV, true, 16 * NV>) : launch(span_attention_tiles_kernel<NV, false, 16 * NV>)) \
             : (ext ? launch(span_attention_tiles_kernel<NV, true, 0>) : launch(span_attention_tiles_kernel<NV, false, 0>))
  if (a.dim == 192 && a.vdim == 128 && !ext) return launch(span_attention_tiles_kernel<8, false, 192>);  // expanded latents
  if (vw <= 64) HB_TILES(4);
  if (vw <= 128) HB_TILES(8);
  if (vw <= 192) HB_TILES(12);
  HB_TILES(16);
#undef HB_TILES
}

int span_attention_tokens(cudaStream_t st, const SpanAttention& args, const int32_t* rows, int n_rows, int n_splits, float* part) {
  if (n_rows == 0) return HB_OK;
  if (latent_tokens_supported(args, HB_BF16)) return latent_tokens(st, args, rows, n_rows, n_splits, part);
  const SpanAttention a = sliced(args, 16);
  const size_t smem = tokens_smem(a);
  const int slices = (a.vdim + kSlice - 1) / kSlice;
  const bool clustered = n_splits > 1 && n_splits <= kMaxCluster;
  const dim3 grid((unsigned)n_rows, (unsigned)(a.kv_heads * a.slices()), (unsigned)(slices * n_splits));
  auto launch = [&](auto* k) -> int {
    int rc = opt_in(k, smem);
    if (rc) return rc;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = dim3(kThreads);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (pdl_enabled()) {
      attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
      attr[n++].val.programmaticStreamSerializationAllowed = 1;
    }
    if (clustered) {
      attr[n].id = cudaLaunchAttributeClusterDimension;
      attr[n].val.clusterDim.x = attr[n].val.clusterDim.y = 1;
      attr[n++].val.clusterDim.z = (unsigned)n_splits;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    HB_CUDA_CHECK(cudaLaunchKernelEx(&cfg, k, a, rows, n_splits, clustered ? 1 : 0, part));
    return HB_OK;
  };
  const int vw = std::min(a.vdim, kSlice);
  int rc;
  const bool wide = a.slice > 8;
  const bool ext = is_ext(a);
#define HB_TOKENS_OF(MT, FIX)                                                                                      \
  rc = ext ? (wide ? launch(span_attention_tokens_kernel<MT, 2, true, FIX>) : launch(span_attention_tokens_kernel<MT, 1, true, FIX>)) \
           : (wide ? launch(span_attention_tokens_kernel<MT, 2, false, FIX>) : launch(span_attention_tokens_kernel<MT, 1, false, FIX>))
#define HB_TOKENS(MT)                                            \
  do {                                                           \
    if (a.dim == 16 * MT && a.vdim == 16 * MT) HB_TOKENS_OF(MT, true); \
    else HB_TOKENS_OF(MT, false);                                \
  } while (0)
  if (vw <= 64) HB_TOKENS(4);
  else if (vw <= 128) HB_TOKENS(8);
  else HB_TOKENS(16);
#undef HB_TOKENS
#undef HB_TOKENS_OF
  return rc || n_splits == 1 || clustered ? rc : span_attention_merge(st, a, rows, n_rows, n_splits, part);
}

int span_attention_merge(cudaStream_t st, const SpanAttention& a, const int32_t* rows, int n_rows, int n_splits, const float* part) {
  HB_CUDA_CHECK(launch_pdl(span_attention_merge_kernel, dim3((unsigned)n_rows, (unsigned)a.heads), dim3(kThreads), 0, st, a, rows,
                           n_splits, part));
  return HB_OK;
}

}  // namespace hb
