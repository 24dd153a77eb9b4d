// Internal GEMM interface: Y[M,N] = X[M,K] . W[N,K]^T (+ fused epilogues).
#pragma once

#include <cuda.h>

#include <cmath>

#include "common.h"

namespace hb {

// CUDA-core kernel, any dtype/shape.
int gemm_simt(cudaStream_t st, void* Y, const void* X, const void* W, int64_t M, int64_t N,
              int64_t K, hb_dtype dtype, bool out_f32);

// Gated activation of a feed-forward: with g clipped from above and u to both sides at `limit`,
//   act(g, u) = g * sigmoid(slope * (g + cubic * g^3)) * (u + shift)         (kLogistic)
//               g * (1 + erf(g / sqrt(2))) / 2 * (u + shift)                 (kErf).
// The defaults are SiLU; gelu in its tanh form is slope = 2 sqrt(2 / pi), cubic = 0.044715, because
// (1 + tanh(z)) / 2 = sigmoid(2 z).  Without a gate (`single`) there is no u and its factor is 1; such a
// form may also be limit * tanh(g / limit) (kTanh).
struct GatedAct {
  enum Form : int { kLogistic = 0, kErf = 1, kTanh = 2 };
  float slope = 1.f, cubic = 0.f, limit = INFINITY, shift = 0.f;
  int form = kLogistic;
  int single = 0;
  bool silu() const {
    return slope == 1.f && cubic == 0.f && limit == INFINITY && shift == 0.f && form == kLogistic && !single;
  }
};
// out[m, i] = act(gate_up[m, i] + gate_bias[i], gate_up[m, inter + i] + up_bias[i]); rows of out have
// stride inter, the biases may be null.  (single: rows of inter numbers.)
int gated_act(cudaStream_t st, void* out, const void* gate_up, int64_t M, int64_t inter, const GatedAct& act, hb_dtype dtype,
              const float* gate_bias = nullptr, const float* up_bias = nullptr);

// Rows of a GEMM sorted by group (mixture of experts): every batch tile of `m_pad` rows belongs to
// one group, whose weights start at row group * (weight rows of one group); tile_group[i] < 0: no
// such tile.  The number of tiles is only known on the device; `max_tiles` bounds it, `likely_tiles`
// steers the split of K.  One further group, number `groups`, may have a [shared_n, shared_k] matrix
// and an activation of its own (the expert every token passes through); rows of X and Y have
// strides of ldx and ldy elements, so that groups of different K and N share them.
struct TcGroups {
  int groups = 0;
  int m_pad = 0;
  int max_tiles = 0, likely_tiles = 0;
  const void* shared_w = nullptr;
  int64_t shared_n = 0, shared_k = 0;
  GatedAct shared_act;
  int64_t ldx = 0, ldy = 0;  // 0: K, N
};
// CUDA-core form: Y[r] = X[r] . W[group of r]^T, tiles of m_pad rows (a multiple of 8).
int gemm_simt_grouped(cudaStream_t st, void* Y, const void* X, const void* W, int64_t N, int64_t K, hb_dtype dtype, bool out_f32,
                      const TcGroups& groups, const int32_t* tile_group);
// Independent products side by side, one per head: Y_h = X_h . W_h^T with the [N, K] matrices of all
// heads one after another in W, X_h = X + h * x_step (rows of ldx elements) and Y_h = Y + h * y_step
// (rows of ldy elements, y_step >= N).
struct TcHeads {
  int heads = 0;
  int64_t ldx = 0, x_step = 0, ldy = 0, y_step = 0;
};
// CUDA-core form.
int gemm_simt_heads(cudaStream_t st, void* Y, const void* X, const void* W, int64_t M, int64_t N, int64_t K, hb_dtype dtype,
                    bool out_f32, const TcHeads& heads);
// Sizes and steps that gemm_tc_plan takes with heads (bf16).
bool gemm_tc_heads_supported(int64_t N, int64_t K, bool out_f32, const TcHeads& heads);
// gated_act over the rows of a grouped GEMM: gate | up rows of stride ld_gu, out rows of stride ld_out;
// inter and act of the groups, and of the further one.
int gated_act_grouped(cudaStream_t st, void* out, int64_t ld_out, const void* gate_up, int64_t ld_gu, int64_t inter,
                      const GatedAct& act, hb_dtype dtype, const TcGroups& groups, const int32_t* tile_group);

// What the tensor-core kernel does with the finished fp32 tile.
enum TcEpilogue : int {
  kEpiStore = 0,     // Y = acc (bf16, or f32 when out_f32)
  kEpiSwiGLU = 1,    // W rows are [gate tile | up tile] pairs: Y = act(gate, up) (GatedAct), N_out = N/2
  kEpiResidual = 2,  // deferred RMSNorm producer (cluster plans only), see TcNormLink
  kEpiPush = 3,      // row-parallel partial pushed into the reducing ranks' staging, see TcNormLink
  kEpiAct = 4,       // Y = act(acc), a GatedAct without a gate
};

// Deferred RMSNorm between two GEMMs of a single-rank decode step.  Instead of a separate
// add + norm kernel between a row-parallel projection P and the projection C that consumes
// the normalised activations, P's epilogue (kEpiResidual) writes
//     h  = resid + Y                      (the new residual, in place in `resid`)
//     Y' = h * norm_w                     (what C reads as its X operand)
//     rowsq[m][tile] = sum over the tile's 128 features of h[m]^2
// and C multiplies batch row m of its accumulator by rsqrt(sum_tiles rowsq[m][.] / n + eps)
// before its own epilogue:  (h * r * w) . W^T == r * ((h * w) . W^T).  The only numerical
// difference from normalising first is where the single bf16 rounding of the activations
// falls (h*w instead of h*r*w).
struct TcNormLink {
  // producer side (kEpiResidual)
  void* resid = nullptr;           // [M, N] bf16, read and overwritten with h
  const void* norm_w = nullptr;    // [N] bf16
  float* rowsq_out = nullptr;      // [M, rowsq_stride] fp32
  // consumer side
  const float* rowsq_in = nullptr; // [M, rowsq_stride] fp32 written by the producer
  int rowsq_tiles = 0;             // entries to sum per row = producer's N / 128
  int rowsq_stride = 0;
  float n = 1.f, eps = 0.f;        // mean over n features
  // independent of the norm: scale of batch row m after the activation, per group of output
  // tiles (mixture of experts: group = expert, post_scale[m * post_groups + group])
  const float* post_scale = nullptr;
  int post_groups = 0, post_tiles_per_group = 0;
  // independent of the norm: RoPE and the paged KV write in the epilogue of the q|k|v
  // projection (cluster plans, bf16, head_dim 128 so that an output tile is one head).
  // Query heads are rotated and stored to Y as usual; key heads are rotated and written to
  // slot kv_slots[m] of k_cache, value heads copied to v_cache, and neither is stored to Y.
  // rope_cs[m * 64 + i] = (cos, sin) of row m's position times frequency i, rounded to bf16
  // (rope_table() in ops.h); caches are [num_blocks, n_kv_heads, 16, 128].
  const float2* rope_cs = nullptr;
  const int64_t* kv_slots = nullptr;
  void* k_cache = nullptr;
  void* v_cache = nullptr;
  int n_q_heads = 0, n_kv_heads = 0;
  int64_t num_blocks = 0;
  // kEpiPush (cluster plans, bf16): the first hop of the all-reduce that follows a
  // row-parallel projection happens here.  Rank q of push_ranks reduces the q-th column slice
  // of the [M, N] result; a CTA that has staged its [rows][128] tile writes it with 16-byte
  // stores straight into rank q's staging (peer memory over NVLink, or this rank's own) and
  // raises the tile's arrival flag there with a system-scope release.  Nothing is written to
  // Y.  The consumer is world_ar_add_norm(..., staged) in ar_norm.cu.  push_peers are the
  // staging bases of all ranks (hb_world::peer), push_spin the poll limit of the one wait
  // (peers done with the previous exchange).
  void* const* push_peers = nullptr;
  int push_ranks = 0, push_rank = 0;
  uint32_t push_spin = 0;
  // independent of everything above: the GEMM announces its own completion to all ranks (the
  // exchange through the NVLink switch, ar_multimem.cu, then starts without an arrival hop of
  // its own).  The CTA that finishes last — counted in ready_ctas, which wraps back to zero —
  // increments ready_calls (local, read by the exchange kernel as the number of calls so far)
  // and adds 1 to the arrival counter of every rank through its multicast address.
  uint32_t* ready_mc = nullptr;
  uint32_t* ready_calls = nullptr;
  uint32_t* ready_ctas = nullptr;
};

// A launch plan for one (M, N, K) problem: tensor maps are encoded once and passed by
// value to the kernel, so a plan can be replayed inside a CUDA graph.
struct TcGemmPlan {
  CUtensorMap tm_w;  // A operand: W [N, K], box 128 x 64
  CUtensorMap tm_x;  // B operand: X [M, K], box m_pad x 64
  int64_t M = 0, N = 0, K = 0;
  int m_pad = 0;      // UMMA N (multiple of 16, <= 256)
  int m_tiles = 0;    // ceil(M / m_pad)
  int n_tiles = 0;    // ceil(N / 128)
  int splits = 1;     // split-K factor
  bool cluster = false;  // the splits of a tile form a thread-block cluster (on-chip reduction)
  bool recv_dedicated = false;  // cluster: the exchange's receive area lies behind the pipeline buffers
  int stages = 0;
  int tmem_cols = 0;
  size_t smem_bytes = 0;
  int epilogue = kEpiStore;
  GatedAct act;          // kEpiSwiGLU, kEpiAct
  const float *gate_bias = nullptr, *up_bias = nullptr;  // kEpiSwiGLU: [N], added before the activation
  TcHeads heads;         // heads > 0: TcHeads form
  int groups = 0;        // > 0: TcGroups form; rows of the batch operand are sorted by group
  int group_rows = 0;    // weight rows of one group (or head)
  CUtensorMap tm_w2;     // further group: its weights, features, K and activation
  int64_t N2 = 0, K2 = 0;
  GatedAct act2;
  int64_t ldx = 0, ldy = 0;
  bool out_f32 = false;
  bool tma_store = false;  // output rows are 16-byte multiples: bulk tensor stores
  // scratch layout inside the caller's workspace
  size_t ws_partials_bytes = 0;  // fp32 [m_tiles*n_tiles*splits][m_pad][128]
  size_t ws_counters_bytes = 0;  // int32 [m_tiles*n_tiles] (zero between calls)
  size_t workspace_bytes() const { return ws_partials_bytes + ws_counters_bytes + 16; }
};

bool gemm_tc_supported(int64_t M, int64_t N, int64_t K, hb_dtype dtype);
// X and W must be 16-byte aligned device pointers; they are baked into the plan.
int gemm_tc_plan(TcGemmPlan* plan, const void* X, const void* W, int64_t M, int64_t N, int64_t K,
                 int epilogue, bool out_f32, int device, int force_splits = 0, const TcGroups* groups = nullptr,
                 const TcHeads* heads = nullptr);
// groups: W holds the [N, K] matrices of all groups one after another, M is the row capacity of the
// sorted batch operand; gemm_tc_run then needs tile_group (device, max_tiles entries).
// Y row stride ldy in elements.  workspace: plan.workspace_bytes(), zeroed once.
// err_flag (device int, may be null) is set non-zero when a bounded wait ran out.
// True when `plan` can carry the RoPE + KV-write epilogue of TcNormLink.
bool gemm_tc_rope_epilogue_ok(const TcGemmPlan& plan);
// Batch rows per arrival flag of a kEpiPush plan (the PushGeometry::row_block its consumer
// needs): the rows a cluster partner owns, or the whole batch tile of an unsplit plan; 0 when
// the plan cannot push.
int gemm_tc_push_row_block(const TcGemmPlan& plan);
int gemm_tc_run(const TcGemmPlan& plan, cudaStream_t st, void* Y, int64_t ldy, void* workspace,
                int* err_flag, const TcNormLink* link = nullptr, const int32_t* tile_group = nullptr);

}  // namespace hb
