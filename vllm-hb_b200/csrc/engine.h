// The engine object shared by every model family: sequences and their block tables, the
// paged KV pool, state slots, step inputs, plans and graphs.  A family (ModelFamily) says how a
// config.json becomes weights and which kernels one step issues; the step itself — validation,
// inputs, graph or stream, results, status — is run_step() in engine.cu for all of them.
#pragma once

#include <cmath>
#include <deque>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "comm.h"
#include "common.h"
#include "gemm.h"
#include "json.h"
#include "layered.h"
#include "ops.h"
#include "rowpar.h"
#include "safetensors.h"

struct hb_seq {
  uint64_t id = 0;
  std::vector<int64_t> blocks;  // physical block ids, table[pos / 16]
  int64_t len = 0;              // tokens whose K/V (and recurrent state) the engine holds
  int state_slot = -1;          // slot of the recurrent-state pool, taken at the first step (-1: none)
};

namespace hb {

struct LayerWeights {
  void* wqkv = nullptr;   // [(hq_l + 2*hkv_l) * hd, H]   rows: q | k | v (column-parallel)
  void* wo = nullptr;     // [H, hq_l * hd]               (row-parallel)
  // Dense FFN: E = 1.  Mixture of experts: the experts' weights are concatenated, gate
  // (w1) rows of all experts first, then their up (w3) rows; down (w2) along K.
  void* wgu = nullptr;    // [2 * E * I_l, H]             rows: gate_0..gate_{E-1} | up_0..up_{E-1}
  void* wdown = nullptr;  // [H, E * I_l]                 columns: expert e at [e * I_l, (e+1) * I_l)
  void* wgate = nullptr;  // [E, H] router (replicated), null for a dense FFN
  void* norm_in = nullptr;
  void* norm_post = nullptr;
};

struct NamedTensor {
  void* ptr;
  int64_t rows, cols;
  int64_t ld = 0;   // row stride in elements (0 = cols): expert down-projections are column blocks
  int dtype = -1;   // hb_dtype of the stored elements (-1 = the engine's)
};

enum GemmKind { kQkv = 0, kO = 1, kGateUp = 2, kDown = 3, kLmHead = 4 };
constexpr int kPairCap = 1024;  // block pairs per copy launch

struct StepPlans {
  std::vector<TcGemmPlan> layer;  // [L * 4]
  TcGemmPlan lm_head;
  int attn_splits = 1;
  int q_group = 1;          // prefill chunks: consecutive positions that share an attention CTA
  bool defer_norm = false;  // add + norm folded into the GEMM epilogues (TcNormLink)
  bool mm = false;          // exchange through the NVLink switch (multicast window of the world)
  const void* mm_window = nullptr;  // the window the plans (and the captured graph) were made for
  bool rope_epi = false;    // RoPE + KV write folded into the q|k|v GEMM epilogue (TcNormLink)
  bool push = false;        // o_proj / down_proj epilogues push their partials to the reducing ranks (kEpiPush)
  PushGeometry geo_o, geo_down;
  int64_t launches = 0;  // kernels in one step (fixed per batch size)
  cudaGraphExec_t graph = nullptr;
};

// ---- one step, as every family sees it
// A run of consecutive tokens of one sequence: a decoded token or a portion of a prompt.
struct StepSeg {
  const int64_t* blocks = nullptr;  // the sequence's block table (ids into the KV pool), table[pos / 16]
  size_t n_blocks = 0;
  int64_t pos0 = 0;                 // position of the first token
  const uint32_t* tokens = nullptr;
  int n = 0;
  int row0 = 0;                     // first batch row
  int state_slot = -1;
};
struct StepBatch {
  std::vector<StepSeg> segs;
  int rows = 0;
  std::vector<int32_t> want;  // batch rows whose logits (and arg-max) are asked for, ascending
  void add(const int64_t* blocks, size_t n_blocks, int64_t pos0, const uint32_t* tokens, int n, int slot = -1) {
    StepSeg s;
    s.blocks = blocks; s.n_blocks = n_blocks; s.pos0 = pos0; s.tokens = tokens; s.n = n; s.row0 = rows; s.state_slot = slot;
    segs.push_back(s);
    rows += n;
  }
};
// What a family's prepare() decided for the step.
struct StepExec {
  int rows = 0;
  size_t input_bytes = 0;               // prefix of the pinned input block to upload
  cudaGraphExec_t* graph = nullptr;     // where the captured step lives; null: issued on the stream
  int64_t* graph_launches = nullptr;
  bool logits_compact = false;          // logits row i belongs to want[i] (else to batch row want[i])
  StepPlans* plans = nullptr;           // Llama family
  LayeredStep layered;                  // layered family
};

// Where a family reads its weights: a checkpoint folder, or a generator on the device.
class TensorSource;

struct ModelFamily {
  const char* name;
  bool (*serves)(const Json& config);
  int (*configure)(hb_engine* e, const Json& config);                  // shapes and checks
  int (*load)(hb_engine* e, TensorSource& src);                        // allocate and fill the weights
  int (*alloc_runtime)(hb_engine* e, const hb_model_config* cfg);      // pools and step buffers
  int (*prepare)(hb_engine* e, const StepBatch& batch, StepExec* x);   // pinned inputs and plans of a step
  int (*issue)(hb_engine* e, const StepExec& x);                       // every kernel of the step
  double (*step_bytes)(const hb_engine* e, const int32_t* ctx_lens, int64_t n_seqs);
  double (*gemm_bytes)(const hb_engine* e, int64_t rows);
};
extern const ModelFamily kLlamaFamily;    // engine.cu
extern const ModelFamily kLayeredFamily;  // layered.cu

}  // namespace hb

struct hb_engine {
  const hb::ModelFamily* family = &hb::kLlamaFamily;
  int device = 0;
  cudaStream_t stream = nullptr;
  hb_world* world = nullptr;
  int rank = 0, ws = 1;
  hb_dtype dtype = HB_BF16;
  size_t es = 2;
  // shape
  int64_t H = 0, I = 0, L = 0, hq = 0, hkv = 0, hd = 0, V = 0;
  double eps = 1e-5, theta = 10000.0;
  int64_t hq_l = 0, hkv_l = 0, I_l = 0, qkv_rows = 0;
  // mixture of experts (mixtral.rs:40-57): E experts, top-k routing, sliding window; I_e = E * I_l
  int64_t E = 1, topk = 1, window = 0, I_e = 0;
  bool moe = false;
  float* d_scale = nullptr;  // [max_batch, E] routing weights of the step
  float* d_rowsq = nullptr;  // [max_batch, rowsq_stride] row sums of the deferred norm
  float2* d_rope_cs = nullptr;  // [max_batch, hd/2] (cos, sin) of the step's positions
  int rowsq_stride = 0;
  // weights
  void* embed = nullptr;
  void* lm_head = nullptr;
  void* final_norm = nullptr;
  std::vector<hb::LayerWeights> layers;
  std::unique_ptr<hb::LayeredModel> lm;  // layered family: its mixers, weights and buffers
  std::map<std::string, hb::NamedTensor> named;
  std::vector<void*> allocations;
  // KV pool: one K and one V pool per attention layer, all addressed by the same block ids
  int64_t num_blocks = 0;
  std::vector<void*> kc, vc;
  std::vector<size_t> k_block_bytes, v_block_bytes;  // per pool
  std::deque<int64_t> free_blocks;  // FIFO: pop front / push back (block_manager.rs:58,63-83)
  // recurrent state: slots of the layered family's state pool (0 = the model keeps none)
  int num_state_slots = 0;
  std::deque<int> free_slots;
  uint64_t next_seq_id = 0;
  // step buffers
  int max_batch = 0;
  int max_logits_rows = 0;   // most rows one step can return logits for
  int64_t max_blocks_per_seq = 0;
  int64_t max_positions = 0; // longest sequence the model itself allows (0 = any)
  uint8_t* d_inputs = nullptr;  // Llama family: [ids | positions | ctx | pad | slots | tables]
  uint8_t* h_inputs = nullptr;  // pinned mirror
  size_t inputs_bytes = 0;
  size_t off_ids = 0, off_pos = 0, off_ctx = 0, off_slots = 0, off_tables = 0;
  void *d_h = nullptr, *d_x = nullptr, *d_qkv = nullptr, *d_attn = nullptr, *d_gu = nullptr,
       *d_act = nullptr, *d_proj = nullptr;
  float* d_logits = nullptr;
  std::vector<int> last_rows;  // rows of d_logits the last step filled for its caller, in order
  uint32_t* d_next = nullptr;
  uint32_t* h_next = nullptr;  // pinned
  float* d_inv_freq = nullptr;
  void* d_attn_ws = nullptr;
  size_t attn_ws_bytes = 0;
  void* d_gemm_ws = nullptr;
  size_t gemm_ws_bytes = 0;
  int* d_err = nullptr;
  int64_t* d_pairs = nullptr;   // (src, dst) block ids of a copy request, kPairCap pairs at a time
  uint8_t* h_swap = nullptr;    // pinned CPU block pool [cpu_blocks][L][K|V][block bytes] (hb_engine_reserve_cpu_blocks)
  int64_t cpu_blocks = 0;
  // device scratch of hb_engine_sample
  float *d_probs = nullptr, *d_picked = nullptr;
  uint64_t* d_seeds = nullptr;
  uint32_t* d_sampled = nullptr;
  int sample_rows = 0;
  bool use_tc = false, use_graph = true, fused_swiglu = true;
  std::map<int, hb::StepPlans> plans;
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  float last_ms = -1.f;
  int64_t last_launches = 0;
  // per-kernel-kind timing of one eager step (hb_engine_profile_step)
  bool profiling = false;
  bool prof_capture = false;  // the profiled step is being captured: events become graph nodes
  std::vector<cudaEvent_t> prof_events;
  std::vector<int> prof_cats;
  size_t prof_used = 0;
  float prof_ms[16] = {0};
};

namespace hb {

// kCatGemm is the QKV projection; the other projections have kinds of their own
enum ProfCat { kCatGemm = 0, kCatAttention = 1, kCatRopeKv = 2, kCatNorm = 3, kCatOther = 4, kCatComm = 5,
               kCatGemmO = 6, kCatGemmGateUp = 7, kCatGemmDown = 8, kCatGemmLmHead = 9, kCatRecurrence = 10,
               kCatRouting = 11, kCatExpertsUp = 12, kCatExpertsDown = 13, kCatLatent = 14, kCatConv = 15, kNumCats = 16 };

// While profiling, every call opens a timed segment of kind `cat` on the stream.
void prof_mark(hb_engine* e, int cat);

// Device memory owned by the engine; `zero` clears it.
int dev_alloc(hb_engine* e, void** p, size_t bytes, bool zero = false);
// Grows the GEMM scratch to `bytes` (zeroed) before a step of a new size is captured or issued.
int ensure_gemm_workspace(hb_engine* e, size_t bytes);

class TensorSource {
 public:
  virtual ~TensorSource() = default;
  // Shape of a named tensor (empty when the source has no opinion, i.e. a generator).
  virtual std::vector<int64_t> shape(const std::string& name) const = 0;
  virtual bool has(const std::string& name) const = 0;
  virtual bool generated() const { return false; }  // random weights: vectors take neutral values
  // rows [r0, r0+nr) x columns [c0, c0+nc) of the [rows, cols] tensor `name` (rows == 1: a vector)
  // to device memory at dst (row stride dst_ld elements, 0 = nc) as `dst_dtype`.
  virtual int fetch(const std::string& name, int64_t rows, int64_t cols, int64_t r0, int64_t nr, int64_t c0, int64_t nc,
                    void* dst, hb_dtype dst_dtype, int64_t dst_ld) = 0;
  int fetch_all(const std::string& name, int64_t rows, int64_t cols, void* dst, hb_dtype dst_dtype, int64_t dst_ld = 0) {
    return fetch(name, rows, cols, 0, rows, 0, cols, dst, dst_dtype, dst_ld);
  }
};

}  // namespace hb
