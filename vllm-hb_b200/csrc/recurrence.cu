// Gated linear recurrences with a matrix state per head:
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t        (S fp32 [dim, vdim])
// The decay a_t is a constant per head or, per key channel, sigmoid(z)^(1/tau) with z from a
// low-rank projection, or follows a step per token (selective state space), which also scales the key;
// q, k and v may pass through SiLU and q carries a scale.
#include "layered_ops.h"

namespace hb {

constexpr int kRecThreads = 256;
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// log(sigmoid(z)) without cancellation on either side
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// log of the decay of key channel c = head * dim + d, from the row's low-rank input t
template <typename T>
__device__ __forceinline__ float low_rank_log_decay(const Recurrence& a, const T* t, int c) {
  float z = a.a2_bias[c];
  const float* w = a.a2 + (int64_t)c * a.rank;
#pragma unroll 8
  for (int r = 0; r < a.rank; ++r) z = fmaf(w[r], to_f32<T>(t[r]), z);
  return log_sigmoid(z) * a.inv_tau;
}

// step of a row and head
template <typename T>
__device__ __forceinline__ float step_of(const Recurrence& a, int64_t row, int h) {
  const float z = to_f32<T>(((const T*)a.dt)[row * a.ld_dt + h]) + a.dt_bias[h];
  return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
}

// CTA = (segment, head, COLS state columns).  A thread owns VEC neighbouring columns of every
// DG-th state row, so its part of the state never meets another thread's; only the output needs
// a sum over the row groups.  RPT > 0: the thread's rows stay in registers for the whole segment.
template <typename T, int COLS, int VEC, int RPT>
__global__ void __launch_bounds__(kRecThreads, RPT > 0 ? 4 : 1)
recurrence_tokens_kernel(const Recurrence a, const int32_t* __restrict__ list) {
  constexpr int LANES = COLS / VEC, DG = kRecThreads / LANES;
  extern __shared__ float sm[];
  const int D = a.dim, VD = a.vdim;
  float* s_q = sm;               // [D]
  float* s_k = s_q + D;          // [D]
  float* s_a = s_k + D;          // [D]
  __shared__ float s_v[COLS];
  __shared__ float s_o[DG][COLS];
  const int tid = threadIdx.x, col = tid % LANES * VEC, dg = tid / LANES, h = blockIdx.y;
  const int v0 = blockIdx.z * COLS;
  pdl_grid_wait();
  const SegInfo seg = a.segs[list[blockIdx.x]];
  float* state = a.state + ((int64_t)seg.slot * a.heads + h) * D * VD + v0 + col;
  const bool live = v0 + col < VD;
  float s[RPT > 0 ? RPT : 1][VEC];
  auto load = [&](float (&f)[VEC], int d) {
    if (VEC == 4) {
      const float4 v = *reinterpret_cast<const float4*>(state + (int64_t)d * VD);
      f[0] = v.x; f[1 % VEC] = v.y; f[2 % VEC] = v.z; f[3 % VEC] = v.w;
    } else {
      f[0] = state[(int64_t)d * VD];
    }
  };
  auto store = [&](const float (&f)[VEC], int d) {
    if (VEC == 4) *reinterpret_cast<float4*>(state + (int64_t)d * VD) = make_float4(f[0], f[1 % VEC], f[2 % VEC], f[3 % VEC]);
    else state[(int64_t)d * VD] = f[0];
  };
  if (RPT > 0) {
#pragma unroll
    for (int i = 0; i < (RPT > 0 ? RPT : 1); ++i) {
      const int d = dg + i * DG;
#pragma unroll
      for (int j = 0; j < VEC; ++j) s[i][j] = 0.f;
      if (seg.pos0 > 0 && live && d < D) load(s[i], d);  // a new sequence starts from zero
    }
  }
  for (int t = 0; t < seg.n; ++t) {
    const int64_t row = seg.row0 + t;
    const T* p = (const T*)a.p + row * a.ld;
    // every kind of input has threads of its own: decays, then q and k, then v
    for (int i = tid; i < 2 * D + COLS; i += kRecThreads) {
      if (i < D) {
        if (a.dt) s_a[i] = expf(-expf(a.a_log[h]) * step_of<T>(a, row, h));
        else s_a[i] = a.decay ? a.decay[h] : expf(low_rank_log_decay<T>(a, p + a.off_a1, h * D + i));
      } else if (i < 2 * D) {
        const int d = i - D;
        float q = to_f32<T>(p[a.off_q + a.qk(h) * D + d]), k = to_f32<T>(p[a.off_k + a.qk(h) * D + d]);
        if (a.silu_qkv) { q = silu_f(q); k = silu_f(k); }
        s_q[d] = q * a.q_scale;
        s_k[d] = a.dt ? k * step_of<T>(a, row, h) : k;
      } else {
        const int c = i - 2 * D;
        const float v = v0 + c < VD ? to_f32<T>(p[a.off_v + h * VD + v0 + c]) : 0.f;
        s_v[c] = a.silu_qkv ? silu_f(v) : v;
      }
    }
    __syncthreads();
    float vv[VEC], acc[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) { vv[j] = s_v[col + j]; acc[j] = 0.f; }
    if (RPT > 0) {
#pragma unroll
      for (int i = 0; i < (RPT > 0 ? RPT : 1); ++i) {
        const int d = dg + i * DG;
        if (d < D) {
          const float al = s_a[d], kd = s_k[d], qd = s_q[d];
#pragma unroll
          for (int j = 0; j < VEC; ++j) {
            s[i][j] = fmaf(al, s[i][j], kd * vv[j]);
            acc[j] = fmaf(qd, s[i][j], acc[j]);
          }
        }
      }
    } else if (live) {
      const bool zero = seg.pos0 == 0 && t == 0;
      for (int d = dg; d < D; d += DG) {
        float f[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) f[j] = 0.f;
        if (!zero) load(f, d);
        const float al = s_a[d], kd = s_k[d], qd = s_q[d];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          f[j] = fmaf(al, f[j], kd * vv[j]);
          acc[j] = fmaf(qd, f[j], acc[j]);
        }
        store(f, d);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) s_o[dg][col + j] = acc[j];
    __syncthreads();
    for (int i = tid; i < COLS; i += kRecThreads) {
      float o = 0.f;
#pragma unroll
      for (int g = 0; g < DG; ++g) o += s_o[g][i];
      if (a.skip) o = fmaf(a.skip[h], s_v[i], o);
      if (v0 + i < VD) a.o[row * a.ld_o + (int64_t)h * VD + v0 + i] = o;
    }
    __syncthreads();
  }
  pdl_trigger();
  if (RPT > 0 && live) {
#pragma unroll
    for (int i = 0; i < (RPT > 0 ? RPT : 1); ++i) {
      const int d = dg + i * DG;
      if (d < D) store(s[i], d);
    }
  }
}

int recurrence_tokens(cudaStream_t st, const Recurrence& a, const int32_t* list, int n_list, hb_dtype dtype) {
  if (n_list == 0) return HB_OK;
  const size_t smem = (size_t)3 * a.dim * sizeof(float);
  auto launch = [&](auto* kernel, int cols) -> int {
    const dim3 grid((unsigned)n_list, (unsigned)a.heads, (unsigned)((a.vdim + cols - 1) / cols));
    HB_CUDA_CHECK(launch_pdl(kernel, grid, dim3(kRecThreads), smem, st, a, list));
    return HB_OK;
  };
  // about 32 KB of state per CTA in registers: enough loads in flight to stream it
  const bool vec = a.vdim % 4 == 0;
  if (dtype == HB_F32) {
    if (!vec) return launch(recurrence_tokens_kernel<float, 64, 1, 0>, 64);
    return a.dim <= 128 ? launch(recurrence_tokens_kernel<float, 64, 4, 8>, 64) : launch(recurrence_tokens_kernel<float, 64, 4, 0>, 64);
  }
  if (dtype == HB_BF16) {
    if (!vec) return launch(recurrence_tokens_kernel<__nv_bfloat16, 64, 1, 0>, 64);
    if (a.dim <= 64 && a.vdim > 64) return launch(recurrence_tokens_kernel<__nv_bfloat16, 128, 4, 8>, 128);
    return a.dim <= 128 ? launch(recurrence_tokens_kernel<__nv_bfloat16, 64, 4, 8>, 64)
                        : launch(recurrence_tokens_kernel<__nv_bfloat16, 64, 4, 0>, 64);
  }
  return fail(HB_ERR_UNSUPPORTED_DTYPE, "recurrence runs in bf16 or f32");
}

}  // namespace hb
