// The decode-step engine behind hb_engine_* / hb_seq_* / hb_forward / hb_decode_batch.
//
// It stands where Engine (src/engine/loader.rs:66-339) -> Backend
// (src/engine/arch/mod.rs:33-118) -> TpLlamaBackend (src/engine/arch/llama_tp.rs) stand
// in the reference, with these differences of structure:
//   - one engine object per rank (the reference loops over ranks inside one process,
//     llama_tp.rs:506-576); with a multi-rank hb_world every rank runs the same step
//     and the row-parallel partials meet in the peer-memory all-reduce;
//   - B sequences per step through batched GEMMs and a paged KV pool, each sequence with
//     a real block table (the reference decodes sequence by sequence over one shared,
//     cat-grown cache: src/worker/mod.rs:280-293, llama_tp.rs:245-259);
//   - no allocation and no host round trip inside a step: all buffers are created at
//     load, the step is captured once per batch size into a CUDA graph and replayed.
#include "engine.h"

namespace hb {

// ------------------------------------------------------------------ host helpers
int dev_alloc(hb_engine* e, void** p, size_t bytes, bool zero) {
  HB_CUDA_CHECK(cudaMalloc(p, bytes ? bytes : 16));
  e->allocations.push_back(*p);
  if (zero) HB_CUDA_CHECK(cudaMemsetAsync(*p, 0, bytes ? bytes : 16, e->stream));
  return HB_OK;
}

static bool same_dtype(const std::string& s, hb_dtype d) {
  return (s == "F32" && d == HB_F32) || (s == "F16" && d == HB_F16) || (s == "BF16" && d == HB_BF16);
}

static hb_dtype st_dtype(const std::string& s) { return s == "F32" ? HB_F32 : s == "F16" ? HB_F16 : HB_BF16; }

// Rows [r0, r0+nr) x cols [c0, c0+nc) of a [rows, cols] tensor of the memory-mapped
// checkpoint go to device memory at dst (row-major [nr, nc], row stride dst_ld elements) in
// `dst_dtype` (the engine's for matrices) — the narrow() of column_shard / row_shard (src/parallel/shard.rs:46-74)
// followed by to_device, without the reference's full CPU copy in the target dtype
// (llama_tp.rs:367-377): only this rank's slice leaves the page cache, as one strided copy
// straight from the mapping, and a checkpoint in another dtype is converted on the device.
// `stage` is a device buffer that grows to the largest slice that needs converting.
struct UploadStage {
  void* buf = nullptr;
  size_t bytes = 0;
  ~UploadStage() { if (buf) cudaFree(buf); }
};

static int upload_slice(hb_engine* e, void* dst, hb_dtype dst_dtype, const StTensor& t, int64_t cols, int64_t r0,
                        int64_t nr, int64_t c0, int64_t nc, UploadStage* stage, int64_t dst_ld = 0) {
  const size_t src_es = t.dtype == "F32" ? 4 : 2;
  const uint8_t* src = t.data + ((size_t)r0 * cols + c0) * src_es;
  if (dst_ld <= 0) dst_ld = nc;
  // every copy and conversion is ordered on the engine's stream; hb_engine_load synchronises it
  // before the mapping goes away
  if (same_dtype(t.dtype, dst_dtype)) {
    HB_CUDA_CHECK(cudaMemcpy2DAsync(dst, (size_t)dst_ld * src_es, src, (size_t)cols * src_es, (size_t)nc * src_es,
                                    (size_t)nr, cudaMemcpyHostToDevice, e->stream));
    return HB_OK;
  }
  const size_t need = (size_t)nr * nc * src_es;
  if (need > stage->bytes) {
    HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
    if (stage->buf) cudaFree(stage->buf);
    stage->buf = nullptr;
    stage->bytes = 0;
    HB_CUDA_CHECK(cudaMalloc(&stage->buf, need));
    stage->bytes = need;
  }
  HB_CUDA_CHECK(cudaMemcpy2DAsync(stage->buf, (size_t)nc * src_es, src, (size_t)cols * src_es, (size_t)nc * src_es,
                                  (size_t)nr, cudaMemcpyHostToDevice, e->stream));
  int rc = convert_2d(e->stream, dst, dst_dtype, dst_ld, stage->buf, st_dtype(t.dtype), nr, nc);
  if (rc) return rc;
  HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));  // the stage is reused by the next slice
  return HB_OK;
}

// The *.safetensors shards of a model folder, memory-mapped.
class CheckpointSource : public TensorSource {
 public:
  explicit CheckpointSource(hb_engine* e) : e_(e) {}
  int open(const std::string& dir) {
    std::vector<std::string> files;
    int rc = list_safetensors(dir, &files);
    if (rc) return rc;
    for (auto& f : files) {
      shards_.emplace_back(new SafetensorsFile);
      if ((rc = shards_.back()->open(f))) return rc;
      for (auto& kv : shards_.back()->tensors()) all_[kv.first] = &kv.second;
    }
    return HB_OK;
  }
  bool has(const std::string& name) const override { return all_.count(name) != 0; }
  std::vector<int64_t> shape(const std::string& name) const override {
    auto it = all_.find(name);
    return it == all_.end() ? std::vector<int64_t>() : it->second->shape;
  }
  int fetch(const std::string& name, int64_t rows, int64_t cols, int64_t r0, int64_t nr, int64_t c0, int64_t nc, void* dst,
            hb_dtype dst_dtype, int64_t dst_ld) override {
    auto it = all_.find(name);
    if (it == all_.end()) return fail(HB_ERR_IO, "Weight not found: %s", name.c_str());  // llama_tp.rs:380-385
    const StTensor* s = it->second;
    if (s->dtype != "F32" && s->dtype != "F16" && s->dtype != "BF16")
      return fail(HB_ERR_UNSUPPORTED_DTYPE, "%s has dtype %s", name.c_str(), s->dtype.c_str());
    // the shape itself, not only the element count: a transposed matrix must not be sharded
    const bool shape_ok = (s->shape.size() == 2 && s->shape[0] == rows && s->shape[1] == cols) ||
                          (rows == 1 && s->shape.size() == 1 && s->shape[0] == cols);
    if (!shape_ok)
      return fail(HB_ERR_IO, "%s has %lld elements in a shape other than the expected [%lld, %lld]", name.c_str(),
                  (long long)s->numel(), (long long)rows, (long long)cols);
    const size_t src_es = s->dtype == "F32" ? 4 : 2;
    if (s->nbytes != (size_t)(rows * cols) * src_es)
      return fail(HB_ERR_IO, "%s holds %zu bytes, [%lld, %lld] of %s needs %zu", name.c_str(), s->nbytes,
                  (long long)rows, (long long)cols, s->dtype.c_str(), (size_t)(rows * cols) * src_es);
    return upload_slice(e_, dst, dst_dtype, *s, cols, r0, nr, c0, nc, &stage_, dst_ld);
  }

 private:
  hb_engine* e_;
  UploadStage stage_;
  std::vector<std::unique_ptr<SafetensorsFile>> shards_;
  std::map<std::string, const StTensor*> all_;
};

// Weights drawn on the device: N(0, std), every tensor from a stream keyed by its name.
class RandomSource : public TensorSource {
 public:
  RandomSource(hb_engine* e, uint64_t seed, float std) : e_(e), seed_(seed), std_(std) {}
  bool has(const std::string&) const override { return true; }
  std::vector<int64_t> shape(const std::string&) const override { return {}; }
  bool generated() const override { return true; }
  int fetch(const std::string& name, int64_t rows, int64_t cols, int64_t r0, int64_t nr, int64_t c0, int64_t nc, void* dst,
            hb_dtype dst_dtype, int64_t dst_ld) override {
    uint64_t id = 1469598103934665603ull;
    for (char c : name) id = (id ^ (uint8_t)c) * 1099511628211ull;
    return fill_normal(e_->stream, dst, dst_dtype, nr, nc, r0, c0, cols, seed_, id, std_, dst_ld);
  }

 private:
  hb_engine* e_;
  uint64_t seed_;
  float std_;
};

static int check_divisibility(const hb_engine* e) {
  // TpLlamaBackend::load (src/engine/arch/llama_tp.rs:407-427)
  const int n = e->ws;
  if (e->hq % n)
    return fail(HB_ERR_NOT_DIVISIBLE,
                "num_attention_heads (%lld) must be divisible by tensor_parallel_size (%d)",
                (long long)e->hq, n);
  if (e->hkv % n)
    return fail(HB_ERR_NOT_DIVISIBLE,
                "num_key_value_heads (%lld) must be divisible by tensor_parallel_size (%d)",
                (long long)e->hkv, n);
  if (e->I % n)
    return fail(HB_ERR_NOT_DIVISIBLE,
                "intermediate_size (%lld) must be divisible by tensor_parallel_size (%d)",
                (long long)e->I, n);
  return HB_OK;
}

static int setup_common(hb_engine* e, const hb_model_config* cfg, hb_world* world) {
  const int tp = cfg->tensor_parallel_size > 0 ? cfg->tensor_parallel_size : 1;
  e->world = world;
  e->ws = world ? world->ws : 1;
  e->rank = world ? world->rank : 0;
  if (tp != e->ws)
    return fail(HB_ERR_INVALID_ARG,
                "tensor_parallel_size=%d but the world handed to the engine has %d rank(s)", tp, e->ws);
  if (world) e->device = world->device;
  else HB_CUDA_CHECK(cudaGetDevice(&e->device));
  HB_CUDA_CHECK(cudaSetDevice(e->device));
  e->dtype = cfg->force_f32 ? HB_F32 : (cfg->bf16 ? HB_BF16 : HB_F16);  // src/engine/dtype.rs:22-28
  e->es = dtype_size(e->dtype);
  HB_CUDA_CHECK(cudaStreamCreateWithFlags(&e->stream, cudaStreamNonBlocking));
  HB_CUDA_CHECK(cudaEventCreate(&e->ev0));
  HB_CUDA_CHECK(cudaEventCreate(&e->ev1));
  const char* g = getenv("HB_NO_GRAPH");
  e->use_graph = !(g && g[0] == '1');
  return HB_OK;
}

static int setup_shape(hb_engine* e, const hb_model_shape& s) {
  e->H = s.hidden_size; e->I = s.intermediate_size; e->L = s.num_hidden_layers;
  e->hq = s.num_attention_heads;
  e->hkv = s.num_key_value_heads == 0 ? s.num_attention_heads : s.num_key_value_heads;  // llama_tp.rs:81-87
  e->V = s.vocab_size;
  e->eps = s.rms_norm_eps; e->theta = s.rope_theta;
  if (e->H <= 0 || e->I <= 0 || e->L <= 0 || e->hq <= 0 || e->V <= 0 || e->H % e->hq)
    return fail(HB_ERR_INVALID_ARG, "bad model shape");
  e->hd = e->H / e->hq;  // llama_tp.rs:77-79
  int rc = check_divisibility(e);
  if (rc) return rc;
  e->hq_l = e->hq / e->ws; e->hkv_l = e->hkv / e->ws; e->I_l = e->I / e->ws;
  e->moe = s.num_local_experts > 0;
  e->E = e->moe ? s.num_local_experts : 1;
  e->topk = e->moe ? (s.num_experts_per_tok > 0 ? s.num_experts_per_tok : 2) : 1;
  e->window = s.sliding_window > 0 ? s.sliding_window : 0;
  if (e->E > 64) return fail(HB_ERR_INVALID_ARG, "num_local_experts %lld unsupported (<= 64)", (long long)e->E);
  e->I_e = e->E * e->I_l;
  e->qkv_rows = (e->hq_l + 2 * e->hkv_l) * e->hd;
  const char* g = getenv("HB_GEMM");
  const bool want_simt = g && std::string(g) == "simt";
  e->use_tc = !want_simt && e->dtype == HB_BF16 && e->H % 64 == 0 && (e->hq_l * e->hd) % 64 == 0 &&
              e->I_l % 64 == 0;
  // expert boundaries must fall on 128-feature tiles of the SwiGLU GEMM
  if (e->moe && e->I_l % 128 != 0) e->use_tc = false;
  return HB_OK;
}

static int alloc_weights(hb_engine* e) {
  const size_t es = e->es;
  int rc;
  if ((rc = dev_alloc(e, &e->embed, (size_t)e->V * e->H * es))) return rc;
  if ((rc = dev_alloc(e, &e->lm_head, (size_t)e->V * e->H * es))) return rc;
  if ((rc = dev_alloc(e, &e->final_norm, (size_t)e->H * es))) return rc;
  e->layers.resize(e->L);
  for (auto& l : e->layers) {
    if ((rc = dev_alloc(e, &l.wqkv, (size_t)e->qkv_rows * e->H * es))) return rc;
    if ((rc = dev_alloc(e, &l.wo, (size_t)e->H * e->hq_l * e->hd * es))) return rc;
    if ((rc = dev_alloc(e, &l.wgu, (size_t)2 * e->I_e * e->H * es))) return rc;
    if ((rc = dev_alloc(e, &l.wdown, (size_t)e->H * e->I_e * es))) return rc;
    if (e->moe && (rc = dev_alloc(e, &l.wgate, (size_t)e->E * e->H * es))) return rc;
    if ((rc = dev_alloc(e, &l.norm_in, (size_t)e->H * es))) return rc;
    if ((rc = dev_alloc(e, &l.norm_post, (size_t)e->H * es))) return rc;
  }
  // names as the reference looks them up (llama_tp.rs:451-462,482-488), sharded shapes
  e->named["model.embed_tokens.weight"] = {e->embed, e->V, e->H};
  e->named["lm_head.weight"] = {e->lm_head, e->V, e->H};
  e->named["model.norm.weight"] = {e->final_norm, 1, e->H};
  for (int64_t i = 0; i < e->L; ++i) {
    const std::string pf = "model.layers." + std::to_string(i);
    auto& l = e->layers[i];
    uint8_t* qkv = (uint8_t*)l.wqkv;
    const size_t rowb = (size_t)e->H * es;
    e->named[pf + ".self_attn.q_proj.weight"] = {qkv, e->hq_l * e->hd, e->H};
    e->named[pf + ".self_attn.k_proj.weight"] = {qkv + (size_t)e->hq_l * e->hd * rowb, e->hkv_l * e->hd, e->H};
    e->named[pf + ".self_attn.v_proj.weight"] = {qkv + (size_t)(e->hq_l + e->hkv_l) * e->hd * rowb, e->hkv_l * e->hd, e->H};
    e->named[pf + ".self_attn.o_proj.weight"] = {l.wo, e->H, e->hq_l * e->hd};
    if (!e->moe) {
      e->named[pf + ".mlp.gate_proj.weight"] = {l.wgu, e->I_l, e->H};
      e->named[pf + ".mlp.up_proj.weight"] = {(uint8_t*)l.wgu + (size_t)e->I_l * rowb, e->I_l, e->H};
      e->named[pf + ".mlp.down_proj.weight"] = {l.wdown, e->H, e->I_l};
    } else {
      // names of mixtral.rs:330-333,354-363
      e->named[pf + ".block_sparse_moe.gate.weight"] = {l.wgate, e->E, e->H};
      for (int64_t x = 0; x < e->E; ++x) {
        const std::string ex = pf + ".block_sparse_moe.experts." + std::to_string(x);
        e->named[ex + ".w1.weight"] = {(uint8_t*)l.wgu + (size_t)(x * e->I_l) * rowb, e->I_l, e->H};
        e->named[ex + ".w3.weight"] = {(uint8_t*)l.wgu + (size_t)(e->I_e + x * e->I_l) * rowb, e->I_l, e->H};
        e->named[ex + ".w2.weight"] = {(uint8_t*)l.wdown + (size_t)(x * e->I_l) * es, e->H, e->I_l, e->I_e};
      }
    }
    e->named[pf + ".input_layernorm.weight"] = {l.norm_in, 1, e->H};
    e->named[pf + ".post_attention_layernorm.weight"] = {l.norm_post, 1, e->H};
  }
  return HB_OK;
}

static int alloc_runtime(hb_engine* e, const hb_model_config* cfg) {
  int rc;
  e->max_batch = cfg->max_batch > 0 ? cfg->max_batch : 256;
  const int64_t max_seq = cfg->max_seq_len > 0 ? (int64_t)cfg->max_seq_len : 2048;
  e->max_blocks_per_seq = (max_seq + HB_BLOCK_SIZE - 1) / HB_BLOCK_SIZE;
  e->num_blocks = cfg->num_kv_blocks > 0 ? cfg->num_kv_blocks : e->max_blocks_per_seq * e->max_batch;
  const size_t blk_bytes = (size_t)e->hkv_l * HB_BLOCK_SIZE * e->hd * e->es;
  e->kc.resize(e->L); e->vc.resize(e->L);
  for (int64_t l = 0; l < e->L; ++l) {
    if ((rc = dev_alloc(e, &e->kc[l], blk_bytes * e->num_blocks))) return rc;
    if ((rc = dev_alloc(e, &e->vc[l], blk_bytes * e->num_blocks))) return rc;
    // unwritten slots are read (and masked) by the attention kernel: keep them finite
    HB_CUDA_CHECK(cudaMemset(e->kc[l], 0, blk_bytes * e->num_blocks));
    HB_CUDA_CHECK(cudaMemset(e->vc[l], 0, blk_bytes * e->num_blocks));
  }
  e->k_block_bytes.assign(e->L, blk_bytes);
  e->v_block_bytes.assign(e->L, blk_bytes);
  for (int64_t b = 0; b < e->num_blocks; ++b) e->free_blocks.push_back(b);
  e->max_logits_rows = e->max_batch;

  const int B = e->max_batch;
  auto align16 = [](size_t v) { return (v + 15) / 16 * 16; };
  e->off_ids = 0;
  e->off_pos = align16(e->off_ids + (size_t)B * 4);
  e->off_ctx = align16(e->off_pos + (size_t)B * 4);
  e->off_slots = align16(e->off_ctx + (size_t)B * 4);
  e->off_tables = align16(e->off_slots + (size_t)B * 8);
  e->inputs_bytes = align16(e->off_tables + (size_t)B * e->max_blocks_per_seq * 4);
  if ((rc = dev_alloc(e, (void**)&e->d_inputs, e->inputs_bytes))) return rc;
  HB_CUDA_CHECK(cudaMallocHost((void**)&e->h_inputs, e->inputs_bytes));
  HB_CUDA_CHECK(cudaMallocHost((void**)&e->h_next, (size_t)B * 4));
  const size_t es = e->es;
  if ((rc = dev_alloc(e, &e->d_h, (size_t)B * e->H * es))) return rc;
  if ((rc = dev_alloc(e, &e->d_x, (size_t)B * e->H * es))) return rc;
  if ((rc = dev_alloc(e, &e->d_qkv, (size_t)B * e->qkv_rows * es))) return rc;
  if ((rc = dev_alloc(e, &e->d_attn, (size_t)B * e->hq_l * e->hd * es))) return rc;
  if ((rc = dev_alloc(e, &e->d_gu, (size_t)B * 2 * e->I_e * es))) return rc;
  if ((rc = dev_alloc(e, &e->d_act, (size_t)B * e->I_e * es))) return rc;
  if (e->moe && (rc = dev_alloc(e, (void**)&e->d_scale, (size_t)B * e->E * 4))) return rc;
  e->rowsq_stride = (int)(((e->H + 127) / 128 + 3) / 4 * 4);
  if ((rc = dev_alloc(e, (void**)&e->d_rowsq, (size_t)B * e->rowsq_stride * 4))) return rc;
  HB_CUDA_CHECK(cudaMemset(e->d_rowsq, 0, (size_t)B * e->rowsq_stride * 4));
  if ((rc = dev_alloc(e, (void**)&e->d_rope_cs, (size_t)B * (e->hd / 2 + 1) * sizeof(float2)))) return rc;
  if ((rc = dev_alloc(e, &e->d_proj, (size_t)B * e->H * es))) return rc;
  if ((rc = dev_alloc(e, (void**)&e->d_logits, (size_t)B * e->V * 4))) return rc;
  if ((rc = dev_alloc(e, (void**)&e->d_next, (size_t)B * 4))) return rc;
  if ((rc = dev_alloc(e, (void**)&e->d_err, 16))) return rc;
  HB_CUDA_CHECK(cudaMemset(e->d_err, 0, 16));
  if ((rc = dev_alloc(e, (void**)&e->d_pairs, (size_t)kPairCap * 2 * sizeof(int64_t)))) return rc;
  std::vector<float> inv(e->hd / 2);
  if ((rc = hb_rope_inv_freq((float)e->theta, (int)e->hd, inv.data()))) return rc;
  if ((rc = dev_alloc(e, (void**)&e->d_inv_freq, inv.size() * 4))) return rc;
  HB_CUDA_CHECK(cudaMemcpy(e->d_inv_freq, inv.data(), inv.size() * 4, cudaMemcpyHostToDevice));
  if ((rc = paged_attention_mma_prepare())) return rc;
  e->attn_ws_bytes = hb_attention_workspace_bytes(B, (int)e->hq_l, (int)e->hd, 16);
  if ((rc = dev_alloc(e, &e->d_attn_ws, e->attn_ws_bytes))) return rc;
  return HB_OK;
}

// ------------------------------------------------------------------ step
int ensure_gemm_workspace(hb_engine* e, size_t ws) {
  if (ws <= e->gemm_ws_bytes) return HB_OK;
  // grows only when a new batch size needs more; never inside a captured step
  void* p = nullptr;
  HB_CUDA_CHECK(cudaMalloc(&p, ws));
  HB_CUDA_CHECK(cudaMemset(p, 0, ws));
  e->allocations.push_back(p);
  e->d_gemm_ws = p;
  e->gemm_ws_bytes = ws;
  // graphs captured with the old scratch are dropped (it stays allocated until the engine goes)
  for (auto& kv : e->plans)
    if (kv.second.graph) { cudaGraphExecDestroy(kv.second.graph); kv.second.graph = nullptr; }
  if (e->lm)
    for (auto& kv : e->lm->graphs)
      if (kv.second.exec) { cudaGraphExecDestroy(kv.second.exec); kv.second.exec = nullptr; }
  return HB_OK;
}

static int pick_attn_splits(const hb_engine* e, int B) {
  DeviceInfo di;
  if (device_info(e->device, &di)) return 1;
  // A split costs a partial write and the merge kernel: only worth it when the
  // (sequence, kv head) units alone leave most SMs idle (measured).
  const int64_t units = (int64_t)B * e->hkv_l;
  if (units * 3 >= 2 * (int64_t)di.sm_count) return 1;
  int s = (int)(((int64_t)di.sm_count + units - 1) / units);
  return std::max(1, std::min(s, 16));
}

// Plans (and the captured graph) of a step of B rows; `chunk`: the rows are consecutive
// positions of one sequence (a prefill chunk), which lets the attention kernel share the K/V
// stream among them.
static int ensure_plans(hb_engine* e, int B, bool chunk, StepPlans** out) {
  const int key = B | (chunk ? 1 << 20 : 0);
  auto it = e->plans.find(key);
  const void* window = e->world ? e->world->mc_base : nullptr;
  if (it != e->plans.end()) {
    if (it->second.mm_window == window) { *out = &it->second; return HB_OK; }
    // the world's multicast window was attached, detached or replaced since: the captured graph
    // addresses the old one
    if (it->second.graph) cudaGraphExecDestroy(it->second.graph);
    e->plans.erase(it);
  }
  StepPlans sp;
  sp.mm_window = window;
  sp.attn_splits = pick_attn_splits(e, B);
  if (chunk && B > 1) {
    const int nrep = (int)(e->hq_l / e->hkv_l);
    const bool tc_attn = !getenv("HB_ATTN") &&
                         paged_attention_mma_supported(e->d_qkv, e->qkv_rows, e->kc[0], e->vc[0], nrep, (int)e->hd,
                                                       e->num_blocks, (int)e->hkv_l, e->dtype);
    if (tc_attn && nrep <= 8) {
      sp.q_group = 16 / nrep;   // 16 MMA rows = q_group positions x nrep heads
      sp.attn_splits = 1;
    }
  }
  size_t ws = 0;
  if (e->use_tc) {
    sp.layer.resize(e->L * 4);
    int rc;
    // Single rank: residual add and RMSNorm ride in the GEMM epilogues (HB_DEFER_NORM=0:
    // separate add+norm kernels) when o_proj and down_proj get cluster plans.
    static const bool no_defer = [] { const char* v = getenv("HB_DEFER_NORM"); return v && v[0] == '0'; }();
    sp.defer_norm = e->ws == 1 && !no_defer && e->H % 128 == 0 && !e->moe;  // the router reads normalised x
    if (sp.defer_norm) {
      TcGemmPlan probe_o, probe_d;
      auto& w0 = e->layers[0];
      if ((rc = gemm_tc_plan(&probe_o, e->d_attn, w0.wo, B, e->H, e->hq_l * e->hd, kEpiResidual, false, e->device))) return rc;
      if ((rc = gemm_tc_plan(&probe_d, e->d_act, w0.wdown, B, e->H, e->I_e, kEpiResidual, false, e->device))) return rc;
      sp.defer_norm = probe_o.cluster && probe_d.cluster && probe_o.m_tiles == 1 && probe_d.m_tiles == 1;
    }
    // Several ranks: the row-parallel GEMMs push their partial tiles straight into the
    // reducing ranks' staging (the first hop of the all-reduce rides in the GEMM epilogue)
    // when the batch is large enough for the two-hop exchange (HB_PUSH=0: GEMM, then the
    // exchange kernel reads the partial back; HB_PUSH=1: push at every batch size).
    // A world with a multicast window lets the switch form the sum instead (HB_MULTIMEM=0: not).
    {
      static const bool mm_off = [] { const char* v = getenv("HB_MULTIMEM"); return v && v[0] == '0'; }();
      sp.mm = e->ws > 1 && !mm_off && mm_ar_add_norm_supported(e->world, B, e->H, e->dtype);
      const char* pe = getenv("HB_PUSH");
      const bool off = pe && pe[0] == '0', always = pe && pe[0] == '1';
      const bool two_hop = exchange_two_hops(e->ws, (size_t)B * e->H * e->es);
      sp.push = e->ws > 1 && !sp.mm && !off && (always || two_hop) && push_exchange_supported(e->world, B, e->H, e->dtype);
      if (sp.push) {
        TcGemmPlan probe_o, probe_d;
        auto& w0 = e->layers[0];
        if ((rc = gemm_tc_plan(&probe_o, e->d_attn, w0.wo, B, e->H, e->hq_l * e->hd, kEpiPush, false, e->device))) return rc;
        if ((rc = gemm_tc_plan(&probe_d, e->d_act, w0.wdown, B, e->H, e->I_e, kEpiPush, false, e->device))) return rc;
        const int tiles = (int)(e->H / 128 / e->ws);
        sp.geo_o = {gemm_tc_push_row_block(probe_o), tiles};
        sp.geo_down = {gemm_tc_push_row_block(probe_d), tiles};
        sp.push = sp.geo_o.row_block > 0 && sp.geo_down.row_block > 0;
      }
    }
    const int row_epi = sp.defer_norm ? kEpiResidual : (sp.push ? kEpiPush : kEpiStore);
    for (int64_t l = 0; l < e->L; ++l) {
      auto& w = e->layers[l];
      if ((rc = gemm_tc_plan(&sp.layer[l * 4 + kQkv], e->d_x, w.wqkv, B, e->qkv_rows, e->H, kEpiStore, false, e->device))) return rc;
      if ((rc = gemm_tc_plan(&sp.layer[l * 4 + kO], e->d_attn, w.wo, B, e->H, e->hq_l * e->hd, row_epi, false, e->device))) return rc;
      if (e->fused_swiglu) {
        if ((rc = gemm_tc_plan(&sp.layer[l * 4 + kGateUp], e->d_x, w.wgu, B, 2 * e->I_e, e->H, kEpiSwiGLU, false, e->device))) return rc;
      } else {
        if ((rc = gemm_tc_plan(&sp.layer[l * 4 + kGateUp], e->d_x, w.wgu, B, 2 * e->I_e, e->H, kEpiStore, false, e->device))) return rc;
      }
      if ((rc = gemm_tc_plan(&sp.layer[l * 4 + kDown], e->d_act, w.wdown, B, e->H, e->I_e, row_epi, false, e->device))) return rc;
      for (int k = 0; k < 4; ++k) ws = std::max(ws, sp.layer[l * 4 + k].workspace_bytes());
    }
    if ((rc = gemm_tc_plan(&sp.lm_head, e->d_x, e->lm_head, B, e->V, e->H, kEpiStore, true, e->device))) return rc;
    ws = std::max(ws, sp.lm_head.workspace_bytes());
    // RoPE and the KV write ride in the q|k|v GEMM epilogue when its output tile is one head
    // (HB_ROPE_EPI=0: the separate kernel)
    const char* re_env = getenv("HB_ROPE_EPI");  // read per plan, so that tests can compare both forms
    const bool no_rope_epi = re_env && re_env[0] == '0';
    sp.rope_epi = !no_rope_epi && e->dtype == HB_BF16 && e->hd == 128 && e->L > 0 &&
                  gemm_tc_rope_epilogue_ok(sp.layer[kQkv]);
    if (sp.defer_norm) {
      auto can_scale = [](const TcGemmPlan& pl) { return pl.tma_store && (pl.cluster || pl.splits == 1) && pl.m_tiles == 1; };
      bool ok = can_scale(sp.lm_head);
      for (int64_t l = 0; l < e->L && ok; ++l)
        ok = can_scale(sp.layer[l * 4 + kQkv]) && can_scale(sp.layer[l * 4 + kGateUp]) && e->fused_swiglu;
      if (!ok) {  // re-plan the row-parallel projections with the plain epilogue
        sp.defer_norm = false;
        for (int64_t l = 0; l < e->L; ++l) {
          auto& w = e->layers[l];
          if ((rc = gemm_tc_plan(&sp.layer[l * 4 + kO], e->d_attn, w.wo, B, e->H, e->hq_l * e->hd, kEpiStore, false, e->device))) return rc;
          if ((rc = gemm_tc_plan(&sp.layer[l * 4 + kDown], e->d_act, w.wdown, B, e->H, e->I_e, kEpiStore, false, e->device))) return rc;
        }
      }
    }
  }
  {
    const int rc = ensure_gemm_workspace(e, ws);
    if (rc) return rc;
  }
  auto ins = e->plans.emplace(key, std::move(sp));
  *out = &ins.first->second;
  return HB_OK;
}

static int run_gemm(hb_engine* e, StepPlans* sp, int64_t l, int kind, void* Y, const void* X,
                    const void* W, int B, int64_t N, int64_t K, bool out_f32, const TcNormLink* link = nullptr) {
  ++e->last_launches;
  if (e->use_tc) {
    const TcGemmPlan& pl = (kind == kLmHead) ? sp->lm_head : sp->layer[l * 4 + kind];
    return gemm_tc_run(pl, e->stream, Y, pl.N, e->d_gemm_ws, e->d_err, link);
  }
  return gemm_simt(e->stream, Y, X, W, B, N, K, e->dtype, out_f32);
}

// While profiling, every call opens a timed segment of kind `cat` on the stream.
void prof_mark(hb_engine* e, int cat) {
  if (!e->profiling) return;
  if (e->prof_used == e->prof_events.size()) {
    cudaEvent_t ev = nullptr;
    cudaEventCreate(&ev);
    e->prof_events.push_back(ev);
  }
  if (e->prof_capture) cudaEventRecordWithFlags(e->prof_events[e->prof_used++], e->stream, cudaEventRecordExternal);
  else cudaEventRecord(e->prof_events[e->prof_used++], e->stream);
  e->prof_cats.push_back(cat);
}

// h += SUM_ranks d_proj; x = norm(h; norm_w): one kernel over peer memory when the world has
// several ranks (shapes the kernel does not take: all-reduce kernel, then add+norm), add+norm alone otherwise.
static int reduce_add_norm(hb_engine* e, void* x_out, const void* norm_w, int B, bool mm = false,
                           bool gemm_signals = false) {
  int rc;
  cudaStream_t st = e->stream;
  const float eps = (float)e->eps;
  if (e->ws > 1) {
    prof_mark(e, kCatComm);
    if (mm) {
      // the projection left its partial in the world's multicast window: the switch sums it
      if ((rc = world_mm_ar_add_norm(e->world, st, x_out, e->d_h, mm_partial_ptr(e->world), e->d_h, norm_w, B, e->H, eps,
                                     e->dtype, gemm_signals))) return rc;
      ++e->last_launches;
      return HB_OK;
    }
    if (ar_add_norm_supported(e->world, B, e->H, e->dtype)) {
      if ((rc = world_ar_add_norm(e->world, st, x_out, e->d_h, e->d_proj, e->d_h, norm_w, B, e->H, eps, e->dtype,
                                  HB_ALGO_AUTO))) return rc;
      ++e->last_launches;
      return HB_OK;
    }
    if ((rc = world_all_reduce(e->world, st, e->d_proj, (size_t)B * e->H, e->dtype, HB_ALGO_AUTO))) return rc;
    ++e->last_launches;
  }
  prof_mark(e, kCatNorm);
  if ((rc = hb_add_rms_norm(st, x_out, e->d_h, e->d_proj, e->d_h, norm_w, B, e->H, eps, e->dtype))) return rc;
  ++e->last_launches;
  return HB_OK;
}

// Issues every kernel of one decode step on e->stream (captured or direct).
static int issue_step(hb_engine* e, StepPlans* sp, int B) {
  int rc;
  cudaStream_t st = e->stream;
  const uint32_t* d_ids = (const uint32_t*)(e->d_inputs + e->off_ids);
  const int32_t* d_pos = (const int32_t*)(e->d_inputs + e->off_pos);
  const int32_t* d_ctx = (const int32_t*)(e->d_inputs + e->off_ctx);
  const int64_t* d_slots = (const int64_t*)(e->d_inputs + e->off_slots);
  const int32_t* d_tables = (const int32_t*)(e->d_inputs + e->off_tables);
  const float eps = (float)e->eps;
  e->last_launches = 0;

  // h = embed[ids]; x = norm(h; w_in[0])                       llama_tp.rs:508-522
  prof_mark(e, kCatOther);
  if ((rc = hb_embed(st, e->d_h, e->embed, d_ids, B, e->H, e->V, e->dtype))) return rc;
  prof_mark(e, kCatNorm);
  if ((rc = hb_rms_norm(st, e->d_x, e->d_h, e->layers[0].norm_in, B, e->H, eps, e->dtype))) return rc;
  e->last_launches += 2;
  // deferred norm: the GEMM after a row-parallel projection scales its rows (TcNormLink)
  const bool defer = e->use_tc && sp->defer_norm;
  TcNormLink consume;
  consume.rowsq_in = e->d_rowsq;
  consume.rowsq_tiles = (int)(e->H / 128);
  consume.rowsq_stride = e->rowsq_stride;
  consume.n = (float)e->H;
  consume.eps = eps;
  // Rows of one step are different sequences (decode: one new token each) or consecutive
  // positions of one sequence (prefill chunk): at most B tokens at the end of any context are
  // written by this step, everything older in the pool is final: the attention kernel may
  // fetch it before the q|k|v projection has completed (measured 4.70 -> 4.64 ms per step).
  const int attn_fresh = B;
  const bool rope_epi = e->use_tc && sp->rope_epi;
  TcNormLink push_link;
  if (sp->push) {
    push_link.push_peers = e->world->peer;
    push_link.push_ranks = e->ws;
    push_link.push_rank = e->rank;
    push_link.push_spin = e->world->wait_limit;
  }
  // exchange through the switch: the row-parallel GEMMs announce their completion themselves
  // (HB_MM_SIGNAL=0: the exchange kernel does, with an arrival hop of its own)
  static const bool mm_sig_off = [] { const char* v = getenv("HB_MM_SIGNAL"); return v && v[0] == '0'; }();
  const bool mm_sig = sp->mm && e->use_tc && !mm_sig_off;
  TcNormLink mm_link;
  if (mm_sig) mm_gemm_signal(e->world, &mm_link.ready_mc, &mm_link.ready_calls, &mm_link.ready_ctas);
  if (rope_epi) {
    // the step's (cos, sin) table, shared by the q|k|v epilogues of every layer
    prof_mark(e, kCatRopeKv);
    if ((rc = rope_table(st, e->d_rope_cs, d_pos, e->d_inv_freq, B, (int)e->hd, e->dtype))) return rc;
    ++e->last_launches;
  }
  for (int64_t l = 0; l < e->L; ++l) {
    auto& w = e->layers[l];
    // q|k|v = x . Wqkv^T                                      llama_tp.rs:232-234
    prof_mark(e, kCatGemm);
    TcNormLink qkv_link;
    if (defer && l > 0) qkv_link = consume;
    if (rope_epi) {
      // RoPE + KV append in the epilogue                      llama_tp.rs:242-259
      qkv_link.rope_cs = e->d_rope_cs;
      qkv_link.kv_slots = d_slots;
      qkv_link.k_cache = e->kc[l];
      qkv_link.v_cache = e->vc[l];
      qkv_link.n_q_heads = (int)e->hq_l;
      qkv_link.n_kv_heads = (int)e->hkv_l;
      qkv_link.num_blocks = e->num_blocks;
    }
    if ((rc = run_gemm(e, sp, l, kQkv, e->d_qkv, e->d_x, w.wqkv, B, e->qkv_rows, e->H, false,
                       ((defer && l > 0) || rope_epi) ? &qkv_link : nullptr))) return rc;
    // RoPE + KV append                                        llama_tp.rs:242-259
    if (!rope_epi) {
      prof_mark(e, kCatRopeKv);
      if ((rc = rope_kv_write(st, e->d_qkv, e->kc[l], e->vc[l], d_pos, d_slots, e->d_inv_freq, B,
                              (int)e->hq_l, (int)e->hkv_l, (int)e->hd, e->num_blocks, e->dtype))) return rc;
      ++e->last_launches;
    }
    // softmax(q k^T / sqrt d) v over the block table          llama_tp.rs:264-324
    prof_mark(e, kCatAttention);
    if ((rc = paged_attention(st, e->d_attn, e->d_qkv, e->qkv_rows, e->kc[l], e->vc[l], d_tables,
                              d_ctx, B, (int)e->hq_l, (int)e->hkv_l, (int)e->hd,
                              e->max_blocks_per_seq, e->num_blocks, sp->attn_splits, e->d_attn_ws,
                              e->dtype, e->d_err, (int)e->window, attn_fresh, sp->q_group))) return rc;
    e->last_launches += 1 + (sp->attn_splits > 1 ? 1 : 0);
    // o_proj partial, sum over ranks, residual, post-attention norm   llama_tp.rs:327,533-552
    prof_mark(e, kCatGemmO);
    if (sp->push) {
      // the GEMM epilogue pushes each tile to the rank that reduces its column slice; the
      // exchange kernel starts at the wait                      llama_tp.rs:327,533-552
      if ((rc = run_gemm(e, sp, l, kO, nullptr, e->d_attn, w.wo, B, e->H, e->hq_l * e->hd, false, &push_link))) return rc;
      prof_mark(e, kCatComm);
      if ((rc = world_ar_add_norm(e->world, st, e->d_x, e->d_h, nullptr, e->d_h, w.norm_post, B, e->H, eps, e->dtype,
                                  HB_ALGO_TWO_SHOT, &sp->geo_o))) return rc;
      ++e->last_launches;
    } else if (defer) {
      // h += o_proj(attn); x' = h * w_post; row sums for the gate|up GEMM
      TcNormLink produce;
      produce.resid = e->d_h; produce.norm_w = w.norm_post; produce.rowsq_out = e->d_rowsq;
      produce.rowsq_stride = e->rowsq_stride;
      if ((rc = run_gemm(e, sp, l, kO, e->d_x, e->d_attn, w.wo, B, e->H, e->hq_l * e->hd, false, &produce))) return rc;
    } else {
      void* proj = sp->mm ? mm_partial_ptr(e->world) : e->d_proj;
      if ((rc = run_gemm(e, sp, l, kO, proj, e->d_attn, w.wo, B, e->H, e->hq_l * e->hd, false, mm_sig ? &mm_link : nullptr))) return rc;
      if ((rc = reduce_add_norm(e, e->d_x, w.norm_post, B, sp->mm, mm_sig))) return rc;
    }
    // mixture of experts: routing weights of every token       mixtral.rs:371-412
    if (e->moe) {
      prof_mark(e, kCatOther);
      if ((rc = moe_route(st, e->d_scale, e->d_x, w.wgate, B, e->H, (int)e->E, (int)e->topk, e->dtype))) return rc;
      ++e->last_launches;
    }
    // down( silu(gate x) * up x ) partial                     llama_tp.rs:333-339
    prof_mark(e, kCatGemmGateUp);
    bool moe_scaled = false;
    if (e->use_tc && e->fused_swiglu) {
      TcNormLink moe_link;
      const TcGemmPlan& gpl = sp->layer[l * 4 + kGateUp];
      if (e->moe && gpl.tma_store && (gpl.cluster || gpl.splits == 1) && gpl.m_tiles == 1) {
        // the routing weight of (token, expert) multiplies the expert's activations in the
        // epilogue of the gate|up GEMM (expert = output tile / tiles per expert)
        moe_link.post_scale = e->d_scale;
        moe_link.post_groups = (int)e->E;
        moe_link.post_tiles_per_group = (int)(e->I_l / 128);
        moe_scaled = true;
      }
      if ((rc = run_gemm(e, sp, l, kGateUp, e->d_act, e->d_x, w.wgu, B, 2 * e->I_e, e->H, false,
                         defer ? &consume : (moe_scaled ? &moe_link : nullptr)))) return rc;
    } else {
      if ((rc = run_gemm(e, sp, l, kGateUp, e->d_gu, e->d_x, w.wgu, B, 2 * e->I_e, e->H, false))) return rc;
      prof_mark(e, kCatOther);
      if ((rc = hb_silu_mul(st, e->d_act, e->d_gu, B, e->I_e, e->dtype))) return rc;
      ++e->last_launches;
    }
    if (e->moe && !moe_scaled) {
      // every expert ran on every token; the ones a token did not choose get weight 0,
      // the chosen ones their renormalised probability                 mixtral.rs:404-427
      prof_mark(e, kCatOther);
      if ((rc = moe_scale_act(st, e->d_act, e->d_scale, B, e->I_l, (int)e->E, e->dtype))) return rc;
      ++e->last_launches;
    }
    // residual + the next layer's input norm (or the final norm)   llama_tp.rs:566-571,517-522,349-351
    const void* nw = (l + 1 < e->L) ? e->layers[l + 1].norm_in : e->final_norm;
    prof_mark(e, kCatGemmDown);
    if (sp->push) {
      if ((rc = run_gemm(e, sp, l, kDown, nullptr, e->d_act, w.wdown, B, e->H, e->I_e, false, &push_link))) return rc;
      prof_mark(e, kCatComm);
      if ((rc = world_ar_add_norm(e->world, st, e->d_x, e->d_h, nullptr, e->d_h, nw, B, e->H, eps, e->dtype,
                                  HB_ALGO_TWO_SHOT, &sp->geo_down))) return rc;
      ++e->last_launches;
    } else if (defer) {
      TcNormLink produce;
      produce.resid = e->d_h; produce.norm_w = nw; produce.rowsq_out = e->d_rowsq;
      produce.rowsq_stride = e->rowsq_stride;
      if ((rc = run_gemm(e, sp, l, kDown, e->d_x, e->d_act, w.wdown, B, e->H, e->I_e, false, &produce))) return rc;
    } else {
      void* proj = sp->mm ? mm_partial_ptr(e->world) : e->d_proj;
      if ((rc = run_gemm(e, sp, l, kDown, proj, e->d_act, w.wdown, B, e->H, e->I_e, false, mm_sig ? &mm_link : nullptr))) return rc;
      if ((rc = reduce_add_norm(e, e->d_x, nw, B, sp->mm, mm_sig))) return rc;
    }
  }
  // logits = x . lm_head^T (fp32 out), greedy argmax            llama_tp.rs:352-355, sampling/mod.rs:105-107
  prof_mark(e, kCatGemmLmHead);
  if ((rc = run_gemm(e, sp, 0, kLmHead, e->d_logits, e->d_x, e->lm_head, B, e->V, e->H, true,
                     defer ? &consume : nullptr))) return rc;
  prof_mark(e, kCatOther);
  if ((rc = hb_argmax(st, e->d_next, e->d_logits, B, e->V, HB_F32))) return rc;
  ++e->last_launches;
  prof_mark(e, -1);  // closes the last segment
  return HB_OK;
}

static int seq_ensure_block(hb_engine* e, hb_seq* s, int64_t pos) {
  while ((int64_t)s->blocks.size() * HB_BLOCK_SIZE <= pos) {
    if (e->free_blocks.empty())
      return fail(HB_ERR_OOM_BLOCKS, "no free KV blocks (pool of %lld)", (long long)e->num_blocks);
    if ((int64_t)s->blocks.size() >= e->max_blocks_per_seq)
      return fail(HB_ERR_OOM_BLOCKS, "sequence exceeds max_seq_len (%lld tokens)",
                  (long long)(e->max_blocks_per_seq * HB_BLOCK_SIZE));
    s->blocks.push_back(e->free_blocks.front());
    e->free_blocks.pop_front();
  }
  return HB_OK;
}

// Blocks (and, for a model with recurrent state, the state slot) that the next `n` tokens of a
// sequence need.
static int seq_reserve(hb_engine* e, hb_seq* s, int64_t n) {
  if (e->max_positions > 0 && s->len + n > e->max_positions)
    return fail(HB_ERR_INVALID_ARG, "sequence of %lld tokens exceeds the model's %lld positions", (long long)(s->len + n),
                (long long)e->max_positions);
  int rc = seq_ensure_block(e, s, s->len + n - 1);
  if (rc) return rc;
  if (e->num_state_slots > 0 && s->state_slot < 0) {
    if (e->free_slots.empty())
      return fail(HB_ERR_OOM_BLOCKS, "no free state slot (%d sequences may be live)", e->num_state_slots);
    s->state_slot = e->free_slots.front();
    e->free_slots.pop_front();
  }
  return HB_OK;
}

static int run_step(hb_engine* e, const StepBatch& batch, uint32_t* next_tokens, float* logits_out);

static int decode_step(hb_engine* e, hb_seq* const* seqs, int B, const uint32_t* tokens,
                       uint32_t* next_tokens, float* logits_out /* host [B, V] or null */) {
  if (B <= 0 || B > e->max_batch)
    return fail(HB_ERR_INVALID_ARG, "batch %d outside [1, %d]", B, e->max_batch);
  for (int b = 0; b < B; ++b) {
    hb_seq* s = seqs[b];
    if (!s) return fail(HB_ERR_INVALID_ARG, "null sequence at index %d", b);
    for (int j = 0; j < b; ++j)
      if (seqs[j] == s) return fail(HB_ERR_INVALID_ARG, "sequence repeated in one batch");
  }
  int rc;
  StepBatch batch;
  batch.segs.reserve((size_t)B);
  batch.want.resize((size_t)B);
  for (int b = 0; b < B; ++b)
    if ((rc = seq_reserve(e, seqs[b], 1))) return rc;
  for (int b = 0; b < B; ++b) {
    batch.add(seqs[b]->blocks.data(), seqs[b]->blocks.size(), seqs[b]->len, tokens + b, 1, seqs[b]->state_slot);
    batch.want[b] = b;
  }
  if ((rc = run_step(e, batch, next_tokens, logits_out))) return rc;
  for (int b = 0; b < B; ++b) seqs[b]->len += 1;
  return HB_OK;
}

// Prefill of `n` prompt tokens of one sequence in chunks of up to max_batch rows; the
// logits of the last token go to logits_out (host [V]) when it is not null.
static int prefill(hb_engine* e, hb_seq* s, const uint32_t* ids, size_t n, float* logits_out,
                   bool all_positions = false) {
  size_t done = 0;
  const size_t cap = (size_t)(all_positions ? std::min(e->max_batch, e->max_logits_rows) : e->max_batch);
  while (done < n) {
    const int c = (int)std::min<size_t>(n - done, cap);
    int rc;
    if ((rc = seq_reserve(e, s, c))) return rc;
    StepBatch batch;
    batch.add(s->blocks.data(), s->blocks.size(), s->len, ids + done, c, s->state_slot);
    const bool last = done + (size_t)c == n;
    if (all_positions) for (int i = 0; i < c; ++i) batch.want.push_back(i);
    else if (last && logits_out) batch.want.push_back(c - 1);
    if ((rc = run_step(e, batch, nullptr, all_positions ? logits_out + done * (size_t)e->V : logits_out))) return rc;
    s->len += c;
    done += (size_t)c;
  }
  return HB_OK;
}

// Llama family: every batch row has its own position, context length, KV slot and block table.
static int llama_prepare(hb_engine* e, const StepBatch& batch, StepExec* x) {
  uint32_t* h_ids = (uint32_t*)(e->h_inputs + e->off_ids);
  int32_t* h_pos = (int32_t*)(e->h_inputs + e->off_pos);
  int32_t* h_ctx = (int32_t*)(e->h_inputs + e->off_ctx);
  int64_t* h_slots = (int64_t*)(e->h_inputs + e->off_slots);
  int32_t* h_tables = (int32_t*)(e->h_inputs + e->off_tables);
  for (const StepSeg& g : batch.segs)
    for (int i = 0; i < g.n; ++i) {
      const int b = g.row0 + i;
      const int64_t pos = g.pos0 + i, need = pos / HB_BLOCK_SIZE + 1;
      h_ids[b] = g.tokens[i];
      h_pos[b] = (int32_t)pos;
      h_ctx[b] = (int32_t)(pos + 1);
      h_slots[b] = g.blocks[pos / HB_BLOCK_SIZE] * HB_BLOCK_SIZE + pos % HB_BLOCK_SIZE;
      int32_t* row = h_tables + (size_t)b * e->max_blocks_per_seq;
      for (int64_t k = 0; k < need; ++k) row[k] = (int32_t)g.blocks[k];
    }
  // rows that are consecutive positions of ONE sequence may share the attention's K/V stream
  const bool chunk = batch.segs.size() == 1 && batch.rows > 1;
  int rc = ensure_plans(e, batch.rows, chunk, &x->plans);
  if (rc) return rc;
  x->rows = batch.rows;
  // only the used prefix of each region matters; one copy of the whole block is simplest
  x->input_bytes = e->inputs_bytes;
  x->graph = &x->plans->graph;
  x->graph_launches = &x->plans->launches;
  x->logits_compact = false;
  return HB_OK;
}

static int llama_issue(hb_engine* e, const StepExec& x) { return issue_step(e, x.plans, x.rows); }

// One step of any model family: the batch is checked, its inputs are uploaded in one copy, the
// kernels replay from a graph (or are issued on the stream), the wanted rows come back.
static int run_step(hb_engine* e, const StepBatch& batch, uint32_t* next_tokens, float* logits_out) {
  HB_CUDA_CHECK(cudaSetDevice(e->device));
  int rc;
  const int n_want = (int)batch.want.size();
  if (batch.rows < 1 || batch.rows > e->max_batch)
    return fail(HB_ERR_INVALID_ARG, "batch %d outside [1, %d]", batch.rows, e->max_batch);
  if (n_want > e->max_logits_rows)
    return fail(HB_ERR_INVALID_ARG, "logits of %d rows asked for, %d at most", n_want, e->max_logits_rows);
  for (const StepSeg& g : batch.segs) {
    for (int i = 0; i < g.n; ++i)
      // the reference's embedding lookup fails on an id outside the vocabulary
      // (index_select, llama_tp.rs:213-216); so does this
      if ((int64_t)g.tokens[i] >= e->V)
        return fail(HB_ERR_INVALID_ARG, "token id %u at row %d is outside the vocabulary of %lld", g.tokens[i], g.row0 + i,
                    (long long)e->V);
    const int64_t last = g.pos0 + g.n - 1, need = last / HB_BLOCK_SIZE + 1;
    if (g.pos0 < 0 || (int64_t)g.n_blocks < need || need > e->max_blocks_per_seq)
      return fail(HB_ERR_INVALID_ARG, "row %d: a block table of %zu block(s) does not cover position %lld", g.row0 + g.n - 1,
                  g.n_blocks, (long long)last);
    for (int64_t i = 0; i < need; ++i)
      if (g.blocks[i] < 0 || g.blocks[i] >= e->num_blocks)
        return fail(HB_ERR_INVALID_ARG, "row %d: block id %lld outside the pool of %lld", g.row0, (long long)g.blocks[i],
                    (long long)e->num_blocks);
    if (e->num_state_slots > 0 && (g.state_slot < 0 || g.state_slot >= e->num_state_slots))
      return fail(HB_ERR_INVALID_ARG, "row %d: this model keeps recurrent state; its sequences need engine handles", g.row0);
  }
  StepExec x;
  if ((rc = e->family->prepare(e, batch, &x))) return rc;
  HB_CUDA_CHECK(cudaMemcpyAsync(e->d_inputs, e->h_inputs, x.input_bytes, cudaMemcpyHostToDevice, e->stream));
  if (e->use_graph && !e->profiling && x.graph) {
    if (!*x.graph) {
      cudaGraph_t g = nullptr;
      HB_CUDA_CHECK(cudaStreamBeginCapture(e->stream, cudaStreamCaptureModeThreadLocal));
      e->last_launches = 0;
      rc = e->family->issue(e, x);
      *x.graph_launches = e->last_launches;
      cudaError_t ce = cudaStreamEndCapture(e->stream, &g);
      if (rc) { if (g) cudaGraphDestroy(g); return rc; }
      if (ce != cudaSuccess) return fail(HB_ERR_CUDA, "graph capture failed: %s", cudaGetErrorString(ce));
      ce = cudaGraphInstantiate(x.graph, g, 0);
      cudaGraphDestroy(g);
      if (ce != cudaSuccess) return fail(HB_ERR_CUDA, "graph instantiate failed: %s", cudaGetErrorString(ce));
    }
    e->last_launches = *x.graph_launches;
    HB_CUDA_CHECK(cudaEventRecord(e->ev0, e->stream));
    HB_CUDA_CHECK(cudaGraphLaunch(*x.graph, e->stream));
    HB_CUDA_CHECK(cudaEventRecord(e->ev1, e->stream));
  } else {
    // Profiling.  With graphs enabled the step is captured once more with an event-record
    // node between the kernels and replayed, so that the per-kind times are those of the
    // kernels inside a graph (a failed capture: kernel by kernel
    // on the stream, which adds the launch gaps).
    bool done = false;
    e->last_launches = 0;
    if (e->profiling && e->use_graph) {
      cudaGraph_t g = nullptr;
      cudaGraphExec_t ge = nullptr;
      if (cudaStreamBeginCapture(e->stream, cudaStreamCaptureModeThreadLocal) == cudaSuccess) {
        e->prof_capture = true;
        rc = e->family->issue(e, x);
        e->prof_capture = false;
        cudaError_t ce = cudaStreamEndCapture(e->stream, &g);
        if (!rc && ce == cudaSuccess && cudaGraphInstantiate(&ge, g, 0) == cudaSuccess) {
          HB_CUDA_CHECK(cudaEventRecord(e->ev0, e->stream));
          ce = cudaGraphLaunch(ge, e->stream);
          HB_CUDA_CHECK(cudaEventRecord(e->ev1, e->stream));
          HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
          done = ce == cudaSuccess;
        }
        if (ge) cudaGraphExecDestroy(ge);
        if (g) cudaGraphDestroy(g);
        cudaGetLastError();
      }
      if (!done) { e->prof_used = 0; e->prof_cats.clear(); e->last_launches = 0; }
    }
    if (!done) {
      HB_CUDA_CHECK(cudaEventRecord(e->ev0, e->stream));
      if ((rc = e->family->issue(e, x))) return rc;
      HB_CUDA_CHECK(cudaEventRecord(e->ev1, e->stream));
    }
  }
  // wanted rows back to the host: runs of neighbouring logits rows go as one copy
  auto row_of = [&](int i) { return x.logits_compact ? i : batch.want[i]; };
  e->last_rows.clear();
  if (n_want > 0) {
    const int n_rows = x.logits_compact ? n_want : batch.rows;
    if (next_tokens)
      HB_CUDA_CHECK(cudaMemcpyAsync(e->h_next, e->d_next, (size_t)n_rows * 4, cudaMemcpyDeviceToHost, e->stream));
    if (logits_out)
      for (int i = 0; i < n_want;) {
        int j = i + 1;
        while (j < n_want && row_of(j) == row_of(j - 1) + 1) ++j;
        HB_CUDA_CHECK(cudaMemcpyAsync(logits_out + (size_t)i * e->V, e->d_logits + (size_t)row_of(i) * e->V,
                                      (size_t)(j - i) * e->V * 4, cudaMemcpyDeviceToHost, e->stream));
        i = j;
      }
  }
  int h_err = 0;
  HB_CUDA_CHECK(cudaMemcpyAsync(&h_err, e->d_err, 4, cudaMemcpyDeviceToHost, e->stream));
  HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
  HB_CUDA_CHECK(cudaEventElapsedTime(&e->last_ms, e->ev0, e->ev1));
  if (e->profiling) {
    for (int c = 0; c < kNumCats; ++c) e->prof_ms[c] = 0.f;
    for (size_t i = 0; i + 1 < e->prof_used; ++i) {
      float ms = 0.f;
      cudaEventElapsedTime(&ms, e->prof_events[i], e->prof_events[i + 1]);
      if (e->prof_cats[i] >= 0 && e->prof_cats[i] < kNumCats) e->prof_ms[e->prof_cats[i]] += ms;
    }
    e->prof_used = 0;
    e->prof_cats.clear();
  }
  if (h_err) {
    cudaMemsetAsync(e->d_err, 0, 4, e->stream);
    return fail(HB_ERR_TIMEOUT, "a bounded device-side wait ran out during the decode step");
  }
  if (e->world && e->ws > 1) {
    const int stw = hb_world_status(e->world);
    if (stw) return fail(stw, "a peer did not arrive in the all-reduce of the decode step");
  }
  if (next_tokens)
    for (int i = 0; i < n_want; ++i) next_tokens[i] = e->h_next[row_of(i)];
  for (int i = 0; i < n_want; ++i) e->last_rows.push_back(row_of(i));
  return HB_OK;
}

// Any mix of prompt portions and decoded tokens, one entry per sequence.  Entries whose rows (or
// wanted rows) exceed what one step can hold are cut; everything else is one batch.
static int mixed_step(hb_engine* e, const hb_step_entry* entries, size_t n, uint32_t* next_tokens, float* logits_out) {
  for (size_t i = 0; i < n; ++i) {
    const hb_step_entry& t = entries[i];
    if (!t.seq || !t.tokens) return fail(HB_ERR_INVALID_ARG, "hb_step: null sequence or tokens at entry %zu", i);
    if (t.n_tokens == 0) return fail(HB_ERR_EMPTY, "hb_step: entry %zu brings no tokens", i);
    for (size_t j = 0; j < i; ++j)
      if (entries[j].seq == t.seq) return fail(HB_ERR_INVALID_ARG, "hb_step: sequence repeated in one step");
    for (size_t k = 0; k < t.n_want; ++k)
      if (t.want[k] >= t.n_tokens || (k && t.want[k] <= t.want[k - 1]))
        return fail(HB_ERR_INVALID_ARG, "hb_step: wanted places of entry %zu must ascend below %zu", i, t.n_tokens);
    for (size_t k = 0; k < t.n_tokens; ++k)
      if ((int64_t)t.tokens[k] >= e->V)
        return fail(HB_ERR_INVALID_ARG, "token id %u of entry %zu is outside the vocabulary of %lld", t.tokens[k], i,
                    (long long)e->V);
  }
  size_t i = 0, off = 0, w = 0, out = 0;  // entry, its next token, its next wanted place, results so far
  while (i < n) {
    StepBatch batch;
    std::vector<std::pair<hb_seq*, int>> fed;
    const size_t out0 = out;
    while (i < n && batch.rows < e->max_batch && (int)batch.segs.size() < e->max_batch) {
      const hb_step_entry& t = entries[i];
      int64_t c = std::min<int64_t>((int64_t)(t.n_tokens - off), e->max_batch - batch.rows);
      // no more wanted rows than the logits buffer holds
      const size_t room = (size_t)e->max_logits_rows - batch.want.size();
      if (w + room < t.n_want) c = std::min<int64_t>(c, (int64_t)t.want[w + room] - (int64_t)off);
      if (c <= 0) break;
      int rc = seq_reserve(e, t.seq, c);
      if (rc) return rc;
      for (; w < t.n_want && t.want[w] < off + (size_t)c; ++w, ++out)
        batch.want.push_back(batch.rows + (int)(t.want[w] - off));
      batch.add(t.seq->blocks.data(), t.seq->blocks.size(), t.seq->len, t.tokens + off, (int)c, t.seq->state_slot);
      fed.emplace_back(t.seq, (int)c);
      off += (size_t)c;
      if (off < t.n_tokens) break;
      ++i;
      off = w = 0;
    }
    int rc = run_step(e, batch, next_tokens ? next_tokens + out0 : nullptr,
                      logits_out ? logits_out + out0 * (size_t)e->V : nullptr);
    if (rc) return rc;
    for (auto& f : fed) f.first->len += f.second;
  }
  return HB_OK;
}

static double llama_step_bytes(const hb_engine* e, const int32_t* ctx_lens, int64_t n_seqs) {
  const double es = (double)e->es;
  double w = 0.0;
  w += (double)e->L * ((double)e->qkv_rows * e->H + (double)e->H * e->hq_l * e->hd +
                       3.0 * (double)e->I_e * e->H + (e->moe ? (double)e->E * e->H : 0.0) + 2.0 * e->H) * es;
  w += ((double)e->V * e->H + e->H) * es;    // lm_head + final norm
  w += (double)n_seqs * e->H * es;            // embedding rows
  double kv = 0.0;
  for (int64_t i = 0; i < n_seqs; ++i)
    kv += (double)(ctx_lens ? ctx_lens[i] : 0) * e->L * 2.0 * e->hkv_l * e->hd * es;  // read
  kv += (double)n_seqs * e->L * 2.0 * e->hkv_l * e->hd * es;                           // write
  return w + kv;
}

static double llama_gemm_bytes(const hb_engine* e, int64_t B) {
  const double es = (double)e->es, b = (double)B;
  const double qkv = (double)e->qkv_rows, o_in = (double)e->hq_l * e->hd, H = (double)e->H,
               Il = (double)e->I_e, V = (double)e->V;
  double per_layer = (qkv * H + b * H + b * qkv) * es        // q|k|v projection
                     + (H * o_in + b * o_in + b * H) * es    // o_proj
                     + (2 * Il * H + b * H + b * Il) * es    // gate|up with the SwiGLU epilogue
                     + (H * Il + b * Il + b * H) * es;       // down_proj
  return (double)e->L * per_layer + (V * H + b * H) * es + b * V * 4.0;  // + lm_head, fp32 logits
}

// ------------------------------------------------------------------ Llama family: load
static bool llama_serves(const Json& root) { return !root.get("architecture"); }

static int llama_configure(hb_engine* e, const Json& root) {
  const std::string mt = root.string_or("model_type", "llama");
  if (mt != "llama" && mt != "mistral" && mt != "mixtral")
    return fail(HB_ERR_INVALID_ARG, "model_type '%s' is not served by this path (llama, mistral, mixtral)",
                    mt.c_str());
  const bool mixtral = mt == "mixtral";
  hb_model_shape sh;
  memset(&sh, 0, sizeof(sh));
  sh.hidden_size = (int64_t)root.number_or("hidden_size", 0);
  sh.intermediate_size = (int64_t)root.number_or("intermediate_size", 0);
  sh.num_hidden_layers = (int64_t)root.number_or("num_hidden_layers", 0);
  sh.num_attention_heads = (int64_t)root.number_or("num_attention_heads", 0);
  sh.num_key_value_heads = (int64_t)root.number_or("num_key_value_heads", 0);
  sh.vocab_size = (int64_t)root.number_or("vocab_size", 0);
  sh.rms_norm_eps = root.number_or("rms_norm_eps", 1e-5);     // llama_tp.rs:68-70
  sh.rope_theta = root.number_or("rope_theta", mixtral ? 1000000.0 : 10000.0);  // llama_tp.rs:71-73, mixtral.rs:56-58
  if (mixtral) {  // mixtral.rs:40-57
    sh.num_local_experts = (int64_t)root.number_or("num_local_experts", 0);
    sh.num_experts_per_tok = (int64_t)root.number_or("num_experts_per_tok", 0);
    sh.sliding_window = (int64_t)root.number_or("sliding_window", 4096);
    if (sh.num_local_experts < 1 || sh.num_experts_per_tok < 1)
      return fail(HB_ERR_INVALID_ARG, "mixtral config.json needs num_local_experts and num_experts_per_tok");
  }
  return setup_shape(e, sh);
}

static int llama_load(hb_engine* g, TensorSource& src) {
  int rc = alloc_weights(g);
  if (rc) return rc;
  const hb_dtype dt = g->dtype;
  const int r = g->rank;
  if ((rc = src.fetch("model.embed_tokens.weight", g->V, g->H, 0, g->V, 0, g->H, g->embed, dt, 0))) return rc;
  if ((rc = src.fetch("lm_head.weight", g->V, g->H, 0, g->V, 0, g->H, g->lm_head, dt, 0))) return rc;  // no tied-embedding fallback (llama_tp.rs:488)
  if ((rc = src.fetch("model.norm.weight", 1, g->H, 0, 1, 0, g->H, g->final_norm, dt, 0))) return rc;
  const size_t rowb = (size_t)g->H * g->es;
  for (int64_t l = 0; l < g->L; ++l) {
    const std::string pf = "model.layers." + std::to_string(l);
    auto& w = g->layers[l];
    const int64_t qr = g->hq_l * g->hd, kr = g->hkv_l * g->hd, qd = g->hq * g->hd;
    uint8_t* qkv = (uint8_t*)w.wqkv;
    if ((rc = src.fetch(pf + ".self_attn.q_proj.weight", qd, g->H, r * qr, qr, 0, g->H, qkv, dt, 0))) return rc;
    if ((rc = src.fetch(pf + ".self_attn.k_proj.weight", g->hkv * g->hd, g->H, r * kr, kr, 0, g->H, qkv + (size_t)qr * rowb, dt, 0))) return rc;
    if ((rc = src.fetch(pf + ".self_attn.v_proj.weight", g->hkv * g->hd, g->H, r * kr, kr, 0, g->H, qkv + (size_t)(qr + kr) * rowb, dt, 0))) return rc;
    if ((rc = src.fetch(pf + ".self_attn.o_proj.weight", g->H, qd, 0, g->H, r * qr, qr, w.wo, dt, 0))) return rc;
    if (!g->moe) {
      if ((rc = src.fetch(pf + ".mlp.gate_proj.weight", g->I, g->H, r * g->I_l, g->I_l, 0, g->H, w.wgu, dt, 0))) return rc;
      if ((rc = src.fetch(pf + ".mlp.up_proj.weight", g->I, g->H, r * g->I_l, g->I_l, 0, g->H, (uint8_t*)w.wgu + (size_t)g->I_l * rowb, dt, 0))) return rc;
      if ((rc = src.fetch(pf + ".mlp.down_proj.weight", g->H, g->I, 0, g->H, r * g->I_l, g->I_l, w.wdown, dt, 0))) return rc;
    } else {
      // mixtral.rs:330-333,354-363: w1 (gate) and w3 (up) column-parallel, w2 (down)
      // row-parallel over the expert's intermediate size; the router is replicated
      if ((rc = src.fetch(pf + ".block_sparse_moe.gate.weight", g->E, g->H, 0, g->E, 0, g->H, w.wgate, dt, 0))) return rc;
      for (int64_t x = 0; x < g->E; ++x) {
        const std::string ex = pf + ".block_sparse_moe.experts." + std::to_string(x);
        uint8_t* w1 = (uint8_t*)w.wgu + (size_t)(x * g->I_l) * rowb;
        uint8_t* w3 = (uint8_t*)w.wgu + (size_t)(g->I_e + x * g->I_l) * rowb;
        uint8_t* w2 = (uint8_t*)w.wdown + (size_t)(x * g->I_l) * g->es;
        if ((rc = src.fetch(ex + ".w1.weight", g->I, g->H, r * g->I_l, g->I_l, 0, g->H, w1, dt, 0))) return rc;
        if ((rc = src.fetch(ex + ".w3.weight", g->I, g->H, r * g->I_l, g->I_l, 0, g->H, w3, dt, 0))) return rc;
        if ((rc = src.fetch(ex + ".w2.weight", g->H, g->I, 0, g->H, r * g->I_l, g->I_l, w2, dt, g->I_e))) return rc;
      }
    }
    if ((rc = src.fetch(pf + ".input_layernorm.weight", 1, g->H, 0, 1, 0, g->H, w.norm_in, dt, 0))) return rc;
    if ((rc = src.fetch(pf + ".post_attention_layernorm.weight", 1, g->H, 0, 1, 0, g->H, w.norm_post, dt, 0))) return rc;
  }
  return HB_OK;
}

const ModelFamily kLlamaFamily = {"llama", llama_serves, llama_configure, llama_load, alloc_runtime,
                                  llama_prepare, llama_issue, llama_step_bytes, llama_gemm_bytes};

// The registry: the first family that serves a config.json loads it.
static const ModelFamily* const kFamilies[] = {&kLlamaFamily, &kLayeredFamily};

}  // namespace hb

// ------------------------------------------------------------------------- C ABI
extern "C" {

int hb_engine_free(hb_engine* e) {
  if (!e) return HB_OK;
  cudaSetDevice(e->device);
  if (e->stream) cudaStreamSynchronize(e->stream);
  for (auto& kv : e->plans)
    if (kv.second.graph) cudaGraphExecDestroy(kv.second.graph);
  for (void* p : e->allocations) cudaFree(p);
  if (e->h_swap) cudaFreeHost(e->h_swap);
  if (e->h_inputs) cudaFreeHost(e->h_inputs);
  if (e->h_next) cudaFreeHost(e->h_next);
  if (e->ev0) cudaEventDestroy(e->ev0);
  if (e->ev1) cudaEventDestroy(e->ev1);
  if (e->stream) cudaStreamDestroy(e->stream);
  delete e;
  return HB_OK;
}

int hb_engine_create_random(const hb_model_shape* shape, const hb_model_config* cfg,
                            hb_world* world, uint64_t seed, float std, int norm_ones,
                            hb_engine** out) {
  HB_CHECK_ARG(shape && cfg && out, "hb_engine_create_random: null argument");
  std::unique_ptr<hb_engine, int (*)(hb_engine*)> e(new hb_engine, hb_engine_free);
  int rc;
  if ((rc = hb::setup_common(e.get(), cfg, world))) return rc;
  if ((rc = hb::setup_shape(e.get(), *shape))) return rc;
  if ((rc = hb::alloc_weights(e.get()))) return rc;
  hb_engine* g = e.get();
  cudaStream_t st = g->stream;
  const int r = g->rank;
  // tensor ids: 0 embed, 1 lm_head, 2 final norm, 16 + 16*layer + k for layer tensors.
  // Each rank draws its slice of the global tensor: rows for column-parallel weights,
  // columns for row-parallel ones (src/parallel/shard.rs:46-74).
  if ((rc = hb::fill_normal(st, g->embed, g->dtype, g->V, g->H, 0, 0, g->H, seed, 0, std))) return rc;
  if ((rc = hb::fill_normal(st, g->lm_head, g->dtype, g->V, g->H, 0, 0, g->H, seed, 1, std))) return rc;
  auto fill_norm = [&](void* p, uint64_t tid) {
    return norm_ones ? hb::fill_const(st, p, g->dtype, g->H, 1.0f)
                     : hb::fill_normal(st, p, g->dtype, 1, g->H, 0, 0, g->H, seed, tid, std);
  };
  if ((rc = fill_norm(g->final_norm, 2))) return rc;
  const size_t rowb = (size_t)g->H * g->es;
  for (int64_t l = 0; l < g->L; ++l) {
    auto& w = g->layers[l];
    const uint64_t t0 = 16 + 16 * (uint64_t)l;
    const int64_t qr = g->hq_l * g->hd, kr = g->hkv_l * g->hd;
    uint8_t* qkv = (uint8_t*)w.wqkv;
    if ((rc = hb::fill_normal(st, qkv, g->dtype, qr, g->H, r * qr, 0, g->H, seed, t0 + 0, std))) return rc;
    if ((rc = hb::fill_normal(st, qkv + (size_t)qr * rowb, g->dtype, kr, g->H, r * kr, 0, g->H, seed, t0 + 1, std))) return rc;
    if ((rc = hb::fill_normal(st, qkv + (size_t)(qr + kr) * rowb, g->dtype, kr, g->H, r * kr, 0, g->H, seed, t0 + 2, std))) return rc;
    if ((rc = hb::fill_normal(st, w.wo, g->dtype, g->H, qr, 0, r * qr, g->hq * g->hd, seed, t0 + 3, std))) return rc;
    if (!g->moe) {
      if ((rc = hb::fill_normal(st, w.wgu, g->dtype, g->I_l, g->H, r * g->I_l, 0, g->H, seed, t0 + 4, std))) return rc;
      if ((rc = hb::fill_normal(st, (uint8_t*)w.wgu + (size_t)g->I_l * rowb, g->dtype, g->I_l, g->H, r * g->I_l, 0, g->H, seed, t0 + 5, std))) return rc;
      if ((rc = hb::fill_normal(st, w.wdown, g->dtype, g->H, g->I_l, 0, r * g->I_l, g->I, seed, t0 + 6, std))) return rc;
    } else {
      // tensor ids of expert x: 1024 + 4096*layer + 4*x + {0: w1, 1: w3, 2: w2}; router: t0 + 9
      if ((rc = hb::fill_normal(st, w.wgate, g->dtype, g->E, g->H, 0, 0, g->H, seed, t0 + 9, std))) return rc;
      for (int64_t x = 0; x < g->E; ++x) {
        const uint64_t tx = 1024 + 4096 * (uint64_t)l + 4 * (uint64_t)x;
        uint8_t* w1 = (uint8_t*)w.wgu + (size_t)(x * g->I_l) * rowb;
        uint8_t* w3 = (uint8_t*)w.wgu + (size_t)(g->I_e + x * g->I_l) * rowb;
        uint8_t* w2 = (uint8_t*)w.wdown + (size_t)(x * g->I_l) * g->es;
        if ((rc = hb::fill_normal(st, w1, g->dtype, g->I_l, g->H, r * g->I_l, 0, g->H, seed, tx + 0, std))) return rc;
        if ((rc = hb::fill_normal(st, w3, g->dtype, g->I_l, g->H, r * g->I_l, 0, g->H, seed, tx + 1, std))) return rc;
        if ((rc = hb::fill_normal(st, w2, g->dtype, g->H, g->I_l, 0, r * g->I_l, g->I, seed, tx + 2, std, g->I_e))) return rc;
      }
    }
    if ((rc = fill_norm(w.norm_in, t0 + 7))) return rc;
    if ((rc = fill_norm(w.norm_post, t0 + 8))) return rc;
  }
  HB_CUDA_CHECK(cudaStreamSynchronize(st));
  if ((rc = hb::alloc_runtime(g, cfg))) return rc;
  *out = e.release();
  return HB_OK;
}

// The family that serves the parsed config.json, its shapes and checks.
static int configure_family(hb_engine* e, const hb::Json& root) {
  for (const hb::ModelFamily* f : hb::kFamilies)
    if (f->serves(root)) {
      e->family = f;
      return f->configure(e, root);
    }
  return hb::fail(HB_ERR_INVALID_ARG, "architecture '%s' is not served by this library",
                  root.string_or("architecture", "").c_str());
}

int hb_engine_load(const hb_model_config* cfg, hb_world* world, hb_engine** out) {
  HB_CHECK_ARG(cfg && out && cfg->model_path, "hb_engine_load: null argument");
  std::unique_ptr<hb_engine, int (*)(hb_engine*)> e(new hb_engine, hb_engine_free);
  int rc;
  if ((rc = hb::setup_common(e.get(), cfg, world))) return rc;
  const std::string dir = cfg->model_path;
  std::string text;
  if ((rc = hb::read_text_file(dir + "/config.json", &text))) return rc;
  hb::Json root;
  std::string err;
  hb::JsonParser jp(text.data(), text.size());
  if (!jp.parse(&root, &err)) return hb::fail(HB_ERR_IO, "config.json: %s", err.c_str());
  if ((rc = configure_family(e.get(), root))) return rc;
  hb::CheckpointSource ckpt(e.get());
  if ((rc = ckpt.open(dir))) return rc;
  if ((rc = e->family->load(e.get(), ckpt))) return rc;
  HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));  // the mapped files are closed when this function returns
  if ((rc = e->family->alloc_runtime(e.get(), cfg))) return rc;
  HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
  *out = e.release();
  return HB_OK;
}

int hb_engine_create_random_config(const char* config_json, const hb_model_config* cfg, uint64_t seed, float std,
                                   hb_engine** out) {
  HB_CHECK_ARG(config_json && cfg && out, "hb_engine_create_random_config: null argument");
  std::unique_ptr<hb_engine, int (*)(hb_engine*)> e(new hb_engine, hb_engine_free);
  int rc;
  if ((rc = hb::setup_common(e.get(), cfg, nullptr))) return rc;
  hb::Json root;
  std::string err;
  hb::JsonParser jp(config_json, strlen(config_json));
  if (!jp.parse(&root, &err)) return hb::fail(HB_ERR_IO, "config: %s", err.c_str());
  if ((rc = configure_family(e.get(), root))) return rc;
  hb::RandomSource src(e.get(), seed, std);
  if ((rc = e->family->load(e.get(), src))) return rc;
  if ((rc = e->family->alloc_runtime(e.get(), cfg))) return rc;
  HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
  *out = e.release();
  return HB_OK;
}

int64_t hb_engine_num_layers(const hb_engine* e) { return e ? e->L : -1; }
int64_t hb_engine_vocab_size(const hb_engine* e) { return e ? e->V : -1; }
int64_t hb_engine_hidden_size(const hb_engine* e) { return e ? e->H : -1; }
int64_t hb_engine_param_count(const hb_engine* e) {
  if (!e) return -1;
  if (e->lm) return e->lm->params;
  // Engine::param_count (src/engine/loader.rs:323-329)
  const int64_t attn = 4 * e->H * e->H, ffn = 3 * e->H * e->I;
  return e->V * e->H + e->L * (attn + ffn) + e->V * e->H;
}
int64_t hb_engine_num_free_blocks(const hb_engine* e) { return e ? (int64_t)e->free_blocks.size() : -1; }
void* hb_engine_stream(hb_engine* e) { return e ? (void*)e->stream : nullptr; }
float hb_engine_last_step_ms(hb_engine* e) { return e ? e->last_ms : -1.f; }
int64_t hb_engine_last_step_launches(const hb_engine* e) { return e ? e->last_launches : -1; }

double hb_engine_step_bytes(const hb_engine* e, const int32_t* ctx_lens, int64_t n_seqs) {
  return e ? e->family->step_bytes(e, ctx_lens, n_seqs) : -1.0;
}

int64_t hb_engine_get_tensor(hb_engine* e, const char* name, float* out, int64_t cap) {
  if (!e || !name) return HB_ERR_INVALID_ARG;
  auto it = e->named.find(name);
  if (it == e->named.end()) return hb::fail(HB_ERR_INVALID_ARG, "no tensor named %s", name);
  const int64_t n = it->second.rows * it->second.cols;
  if (!out) return n;
  if (cap < n) return hb::fail(HB_ERR_INVALID_ARG, "buffer of %lld floats too small for %lld", (long long)cap, (long long)n);
  cudaSetDevice(e->device);
  float* tmp = nullptr;
  if (cudaMalloc((void**)&tmp, (size_t)n * 4) != cudaSuccess) return hb::fail(HB_ERR_CUDA, "cudaMalloc failed");
  const hb_dtype dt = it->second.dtype >= 0 ? (hb_dtype)it->second.dtype : e->dtype;
  int rc = hb::to_f32(e->stream, tmp, it->second.ptr, dt, n, it->second.cols, it->second.ld);
  if (!rc && cudaMemcpyAsync(out, tmp, (size_t)n * 4, cudaMemcpyDeviceToHost, e->stream) != cudaSuccess) rc = HB_ERR_CUDA;
  cudaStreamSynchronize(e->stream);
  cudaFree(tmp);
  return rc ? rc : n;
}

int hb_seq_create(hb_engine* e, hb_seq** out) {
  HB_CHECK_ARG(e && out, "hb_seq_create: null argument");
  hb_seq* s = new hb_seq;
  s->id = e->next_seq_id++;
  *out = s;
  return HB_OK;
}

int hb_seq_free(hb_engine* e, hb_seq* s) {
  if (!s) return HB_OK;
  HB_CHECK_ARG(e, "hb_seq_free: null engine");
  for (int64_t b : s->blocks) e->free_blocks.push_back(b);
  if (s->state_slot >= 0) e->free_slots.push_back(s->state_slot);
  delete s;
  return HB_OK;
}

int64_t hb_seq_len(const hb_seq* s) { return s ? s->len : -1; }

int hb_seq_truncate(hb_engine* e, hb_seq* s, int64_t new_len) {
  HB_CHECK_ARG(e && s, "hb_seq_truncate: null argument");
  HB_CHECK_ARG(new_len >= 0 && new_len <= s->len, "hb_seq_truncate: length %lld outside [0, %lld]", (long long)new_len,
               (long long)s->len);
  // a recurrent state cannot be wound back; forgetting everything is always possible
  HB_CHECK_ARG(e->num_state_slots == 0 || new_len == 0 || new_len == s->len,
               "hb_seq_truncate: the model's recurrent state cannot be cut to %lld of %lld tokens", (long long)new_len,
               (long long)s->len);
  s->len = new_len;
  // blocks that hold no token any more go back to the free list (FIFO, as freed blocks do)
  const size_t keep = (size_t)((new_len + HB_BLOCK_SIZE - 1) / HB_BLOCK_SIZE);
  while (s->blocks.size() > keep) {
    e->free_blocks.push_back(s->blocks.back());
    s->blocks.pop_back();
  }
  return HB_OK;
}

int hb_forward_all_positions(hb_engine* e, hb_seq* s, const uint32_t* ids, size_t n, size_t seq_pos,
                             float* logits_out) {
  if (n == 0) return hb::fail(HB_ERR_EMPTY, "hb_forward_all_positions: token list is empty");
  HB_CHECK_ARG(e && s && ids && logits_out, "hb_forward_all_positions: null argument");
  if ((int64_t)seq_pos != s->len)
    return hb::fail(HB_ERR_INVALID_ARG, "hb_forward_all_positions: seq_pos %zu but the sequence holds %lld tokens",
                    seq_pos, (long long)s->len);
  return hb::prefill(e, s, ids, n, logits_out, true);
}

int64_t hb_seq_block_table(const hb_seq* s, int64_t* out, int64_t cap) {
  if (!s) return HB_ERR_INVALID_ARG;
  for (size_t i = 0; i < s->blocks.size() && (int64_t)i < cap && out; ++i) out[i] = s->blocks[i];
  return (int64_t)s->blocks.size();
}

int hb_decode_batch(hb_engine* e, hb_seq* const* seqs, size_t B, const uint32_t* last_tokens,
                    uint32_t* next_tokens, float* logits_opt) {
  HB_CHECK_ARG(e && seqs && last_tokens, "hb_decode_batch: null argument");
  return hb::decode_step(e, seqs, (int)B, last_tokens, next_tokens, logits_opt);
}

// ---- the same step driven by a scheduler's own block tables (src/scheduler/mod.rs:40-61,
// 203-208 emits them, with copy-on-write pairs and swap lists; src/worker/mod.rs:250-305
// never consumes them)
int hb_kv_copy_blocks(hb_engine* e, const int64_t* pairs, size_t n_pairs) {
  HB_CHECK_ARG(e && (pairs || n_pairs == 0), "hb_kv_copy_blocks: null argument");
  HB_CUDA_CHECK(cudaSetDevice(e->device));
  HB_CHECK_ARG(e->num_state_slots == 0, "hb_kv_copy_blocks: this model keeps recurrent state besides its blocks");
  for (size_t i = 0; i < 2 * n_pairs; ++i)
    if (pairs[i] < 0 || pairs[i] >= e->num_blocks)
      return hb::fail(HB_ERR_INVALID_ARG, "hb_kv_copy_blocks: block id %lld outside the pool of %lld",
                      (long long)pairs[i], (long long)e->num_blocks);
  for (size_t done = 0; done < n_pairs; done += hb::kPairCap) {
    const size_t n = std::min<size_t>(hb::kPairCap, n_pairs - done);
    HB_CUDA_CHECK(cudaMemcpyAsync(e->d_pairs, pairs + 2 * done, n * 2 * sizeof(int64_t), cudaMemcpyHostToDevice, e->stream));
    for (size_t l = 0; l < e->kc.size(); ++l) {
      int rc = hb::kv_copy_blocks(e->stream, e->kc[l], e->vc[l], e->d_pairs, (int64_t)n, (int64_t)e->k_block_bytes[l],
                                  (int64_t)e->v_block_bytes[l], e->num_blocks);
      if (rc) return rc;
    }
    HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));  // `pairs` and d_pairs may be reused
  }
  return HB_OK;
}

int hb_engine_reserve_cpu_blocks(hb_engine* e, int64_t n_blocks) {
  HB_CHECK_ARG(e && n_blocks >= 0, "hb_engine_reserve_cpu_blocks: bad argument");
  HB_CUDA_CHECK(cudaSetDevice(e->device));
  if (e->h_swap) { cudaFreeHost(e->h_swap); e->h_swap = nullptr; e->cpu_blocks = 0; }
  if (n_blocks == 0) return HB_OK;
  HB_CHECK_ARG(e->num_state_slots == 0, "hb_engine_reserve_cpu_blocks: this model keeps recurrent state besides its blocks");
  size_t per_block = 0;
  for (size_t l = 0; l < e->kc.size(); ++l) per_block += e->k_block_bytes[l] + e->v_block_bytes[l];
  HB_CUDA_CHECK(cudaMallocHost((void**)&e->h_swap, (size_t)n_blocks * per_block));
  e->cpu_blocks = n_blocks;
  return HB_OK;
}

int hb_kv_swap_blocks(hb_engine* e, const int64_t* pairs, size_t n_pairs, int to_cpu) {
  HB_CHECK_ARG(e && (pairs || n_pairs == 0), "hb_kv_swap_blocks: null argument");
  HB_CUDA_CHECK(cudaSetDevice(e->device));
  for (size_t i = 0; i < n_pairs; ++i) {
    // swap_out pairs are (gpu, cpu), swap_in pairs (cpu, gpu): block_manager.rs:359-406
    const int64_t g = to_cpu ? pairs[2 * i] : pairs[2 * i + 1], c = to_cpu ? pairs[2 * i + 1] : pairs[2 * i];
    if (g < 0 || g >= e->num_blocks || c < 0 || c >= e->cpu_blocks)
      return hb::fail(HB_ERR_INVALID_ARG, "hb_kv_swap_blocks: pair %zu (gpu %lld, cpu %lld) outside the pools (%lld, %lld)",
                      i, (long long)g, (long long)c, (long long)e->num_blocks, (long long)e->cpu_blocks);
  }
  for (size_t i = 0; i < n_pairs; ++i) {
    const int64_t g = to_cpu ? pairs[2 * i] : pairs[2 * i + 1], c = to_cpu ? pairs[2 * i + 1] : pairs[2 * i];
    size_t per_block = 0;
    for (size_t l = 0; l < e->kc.size(); ++l) per_block += e->k_block_bytes[l] + e->v_block_bytes[l];
    uint8_t* host = e->h_swap + (size_t)c * per_block;
    for (size_t l = 0; l < e->kc.size(); ++l)
      for (int kv = 0; kv < 2; ++kv) {
        const size_t block_bytes = kv ? e->v_block_bytes[l] : e->k_block_bytes[l];
        if (!block_bytes) continue;  // a layer of one pool
        uint8_t* dev = (uint8_t*)(kv ? e->vc[l] : e->kc[l]) + (size_t)g * block_bytes;
        if (to_cpu) HB_CUDA_CHECK(cudaMemcpyAsync(host, dev, block_bytes, cudaMemcpyDeviceToHost, e->stream));
        else HB_CUDA_CHECK(cudaMemcpyAsync(dev, host, block_bytes, cudaMemcpyHostToDevice, e->stream));
        host += block_bytes;
      }
  }
  HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
  return HB_OK;
}

int hb_decode_batch_tables(hb_engine* e, size_t B, const uint32_t* last_tokens, const int64_t* positions,
                           const int64_t* block_tables, size_t table_stride, const int64_t* copy_pairs,
                           size_t n_copies, uint32_t* next_tokens, float* logits_opt) {
  HB_CHECK_ARG(e && last_tokens && positions && block_tables, "hb_decode_batch_tables: null argument");
  if (B == 0 || (int)B > e->max_batch)
    return hb::fail(HB_ERR_INVALID_ARG, "batch %zu outside [1, %d]", B, e->max_batch);
  int rc;
  // blocks_to_copy first: a sequence that shared its last block writes into its own copy
  if (n_copies && (rc = hb_kv_copy_blocks(e, copy_pairs, n_copies))) return rc;
  hb::StepBatch batch;
  for (size_t b = 0; b < B; ++b) {
    if (positions[b] < 0) return hb::fail(HB_ERR_INVALID_ARG, "row %zu: negative position", b);
    const size_t covered = std::min<size_t>(table_stride, (size_t)(positions[b] / HB_BLOCK_SIZE + 1));
    batch.add(block_tables + b * table_stride, covered, positions[b], last_tokens + b, 1);
    batch.want.push_back((int32_t)b);
  }
  // two rows of one decode step are two sequences: they never write the same KV slot
  auto slot_of = [](const hb::StepSeg& g, int64_t* slot) {
    if (g.n_blocks * HB_BLOCK_SIZE <= (size_t)g.pos0) return false;  // reported by run_step
    *slot = g.blocks[g.pos0 / HB_BLOCK_SIZE] * HB_BLOCK_SIZE + g.pos0 % HB_BLOCK_SIZE;
    return true;
  };
  for (size_t b = 0; b < B; ++b) {
    int64_t slot = 0, other = 0;
    if (!slot_of(batch.segs[b], &slot)) continue;
    for (size_t j = 0; j < b; ++j)
      if (slot_of(batch.segs[j], &other) && other == slot)
        return hb::fail(HB_ERR_INVALID_ARG, "rows %zu and %zu write the same KV slot %lld", j, b, (long long)slot);
  }
  return hb::run_step(e, batch, next_tokens, logits_opt);
}

int hb_forward_tables(hb_engine* e, const uint32_t* ids, size_t n, size_t seq_pos, const int64_t* block_table,
                      size_t table_len, float* logits_out) {
  if (n == 0) return hb::fail(HB_ERR_EMPTY, "hb_forward_tables: token list is empty");
  HB_CHECK_ARG(e && ids && block_table && logits_out, "hb_forward_tables: null argument");
  // chunks of consecutive positions, as hb_forward; positions below seq_pos must already hold
  // this sequence's K/V in the table's blocks (a prefix-cache hit: block_manager.rs:213-234)
  size_t done = 0;
  while (done < n) {
    const int c = (int)std::min<size_t>(n - done, (size_t)e->max_batch);
    hb::StepBatch batch;
    batch.add(block_table, table_len, (int64_t)(seq_pos + done), ids + done, c);
    if (done + (size_t)c == n) batch.want.push_back(c - 1);
    int rc = hb::run_step(e, batch, nullptr, logits_out);
    if (rc) return rc;
    done += (size_t)c;
  }
  return HB_OK;
}

int hb_step(hb_engine* e, const hb_step_entry* entries, size_t n, uint32_t* next_tokens, float* logits_out) {
  HB_CHECK_ARG(e && (entries || n == 0), "hb_step: null argument");
  return hb::mixed_step(e, entries, n, next_tokens, logits_out);
}

int hb_engine_sample(hb_engine* e, size_t n, const uint64_t* seeds, float temperature, float top_p, uint32_t* tokens) {
  HB_CHECK_ARG(e && seeds && tokens, "hb_engine_sample: null argument");
  HB_CHECK_ARG(n > 0 && n <= e->last_rows.size(), "hb_engine_sample: %zu rows asked for, the last step left %zu", n,
               e->last_rows.size());
  HB_CUDA_CHECK(cudaSetDevice(e->device));
  if ((int)n > e->sample_rows) {
    const int rows = std::min(e->max_logits_rows, std::max((int)n, 2 * e->sample_rows));
    int rc;
    if ((rc = hb::dev_alloc(e, (void**)&e->d_probs, (size_t)rows * e->V * 4))) return rc;
    if ((rc = hb::dev_alloc(e, (void**)&e->d_picked, (size_t)rows * e->V * 4))) return rc;
    if ((rc = hb::dev_alloc(e, (void**)&e->d_seeds, (size_t)rows * 8))) return rc;
    if ((rc = hb::dev_alloc(e, (void**)&e->d_sampled, (size_t)rows * 4))) return rc;
    e->sample_rows = rows;
  }
  HB_CUDA_CHECK(cudaMemcpyAsync(e->d_seeds, seeds, n * 8, cudaMemcpyHostToDevice, e->stream));
  // wanted rows that lie apart (Llama family: one logits row per batch row) are gathered first
  const float* logits = e->d_logits;
  bool in_place = true;
  for (size_t i = 0; i < n && in_place; ++i) in_place = e->last_rows[i] == (int)i;
  if (!in_place) {
    for (size_t i = 0; i < n; ++i)
      HB_CUDA_CHECK(cudaMemcpyAsync(e->d_picked + i * e->V, e->d_logits + (size_t)e->last_rows[i] * e->V, (size_t)e->V * 4,
                                    cudaMemcpyDeviceToDevice, e->stream));
    logits = e->d_picked;
  }
  int rc = hb_sample(e->stream, e->d_sampled, e->d_probs, logits, nullptr, e->d_seeds, (int64_t)n, e->V, temperature,
                     top_p, 0.f, 0.f);
  if (rc) return rc;
  HB_CUDA_CHECK(cudaMemcpyAsync(tokens, e->d_sampled, n * 4, cudaMemcpyDeviceToHost, e->stream));
  HB_CUDA_CHECK(cudaStreamSynchronize(e->stream));
  return HB_OK;
}

int hb_engine_num_free_state_slots(const hb_engine* e) { return e ? (int)e->free_slots.size() : -1; }

int hb_engine_profile_step(hb_engine* e, hb_seq* const* seqs, size_t B, const uint32_t* last_tokens,
                           uint32_t* next_tokens, float* ms_by_kind) {
  HB_CHECK_ARG(e && seqs && last_tokens && ms_by_kind, "hb_engine_profile_step: null argument");
  e->profiling = true;
  int rc = hb::decode_step(e, seqs, (int)B, last_tokens, next_tokens, nullptr);
  e->profiling = false;
  if (rc) return rc;
  for (int c = 0; c < HB_PROFILE_KINDS; ++c) ms_by_kind[c] = e->prof_ms[c];
  return HB_OK;
}

int hb_engine_set_profiling(hb_engine* e, int on) {
  HB_CHECK_ARG(e, "hb_engine_set_profiling: null engine");
  e->profiling = on != 0;
  return HB_OK;
}

int hb_engine_profile_ms(const hb_engine* e, float* ms_by_kind) {
  HB_CHECK_ARG(e && ms_by_kind, "hb_engine_profile_ms: null argument");
  for (int c = 0; c < HB_PROFILE_KINDS; ++c) ms_by_kind[c] = e->prof_ms[c];
  return HB_OK;
}

double hb_engine_gemm_bytes(const hb_engine* e, int64_t B) { return e ? e->family->gemm_bytes(e, B) : -1.0; }

int hb_forward(hb_engine* e, hb_seq* s, const uint32_t* ids, size_t n, size_t seq_pos,
               float* logits_out) {
  if (n == 0) return hb::fail(HB_ERR_EMPTY, "hb_forward: token list is empty");
  HB_CHECK_ARG(e && s && ids && logits_out, "hb_forward: null argument");
  if ((int64_t)seq_pos != s->len)
    return hb::fail(HB_ERR_INVALID_ARG, "hb_forward: seq_pos %zu but the sequence holds %lld tokens",
                    seq_pos, (long long)s->len);
  // Prefill runs through the decode kernels in chunks whose rows are consecutive positions
  // of this sequence: causal attention over the growing cache equals the masked prefill of
  // llama_tp.rs:313-316.
  {
    int rc = hb::prefill(e, s, ids, n, logits_out);
    if (rc) return rc;
  }
  return HB_OK;
}

}  // extern "C"
