// The engine behind the C ABI: what it owns, and the pieces of it that more than one source file works on.
#pragma once

#include <map>
#include <string>
#include <tuple>
#include <vector>

#include "common.cuh"

namespace cmld {

struct LayerW {
  Weight proj[7];  // q k v o gate up down
  float *attn_norm = nullptr, *ffn_norm = nullptr;
  bool dense_set = false;
  // Mixtral
  float *router = nullptr;
  Weight exps[3];  // gate, up, down slabs: rows = n_experts * rows_per_expert
  bool moe_set = false;
};

struct LayeredModel;  // layered.cu: a design described layer by layer, in place of the llama-shaped fields

}  // namespace cmld

using namespace cmld;

struct cmld_engine {
  cmld_config cfg{};   // dimensions of THIS rank: n_heads, n_kv_heads and ffn_dim are the tensor-parallel shares
  cmld_config full{};  // the model's dimensions as given to cmld_engine_create
  int32_t tp = 1, ep = 1, shard_rank = 0;
  int32_t vocab_local = 0;  // rows of the output matrix held here
  void *comm = nullptr;     // NCCL communicator of a sharded engine
  unsigned long long *am_keys = nullptr;  // packed (value, index) per row for the sharded argmax
  float *logits_gather = nullptr, *logits_full = nullptr;
  // Peer-memory link of a tensor-parallel group: one region per rank, mapped into every rank.
  //   parts: [2 slots][rank][kPeerRows][hidden] f32, then arrival words [2 slots][rank] u32
  struct PeerLink {
    bool ready = false;
    uint8_t *region[kMaxPeers] = {};  // [shard_rank] is this rank's own allocation
    uint32_t *local = nullptr;        // epochs[2], tickets[2]
    unsigned long long timeout_ns = 0;
  } peer;
  float *mma_scratch = nullptr;  // per-chunk partial sums of the batched tensor-core matvec
  uint8_t *kq8 = nullptr, *vq8 = nullptr;  // CMLD_FLAG_KV_Q8_0: the KV cache as Q8_0 blocks, [layer][slot][kv_head][max_pos][hd/32] x 34 B
  int64_t kv_q8_bytes = 0;                 // bytes of one layer of one side
  uint32_t *tree_mask = nullptr;  // [kTreeMaxNodes] ancestor masks of a draft tree (one word: at most 32 nodes)
  std::vector<float> rope_freq;  // per-pair angular frequency of the engine-owned RoPE table (rope_pair_frequency)
  uint8_t *tc5_pack = nullptr;   // packed activation records of the tcgen05 batched matvec
  int64_t tc5_pack_bytes = 0;
  int64_t mma_scratch_floats = 0;
  unsigned long long *trace = nullptr;  // matvec timeline (environment CMLD_TRACE=<file>), dumped at destroy
  unsigned long long *attn_phases = nullptr;  // with CMLD_TRACE: the last attention launch's phase clocks (8 words)
  std::string trace_path;
  std::map<int32_t, bool> peer_fit;   // rows -> every matvec of a step fits the staged kernel in one pass
  int device = 0;
  cudaStream_t stream = nullptr;
  int32_t max_rows = 0;  // scratch rows (sequences per step)
  int32_t n_splits = 1, sm_count = 148;
  int32_t q_width = 0, kv_width = 0;
  std::vector<LayerW> layers;
  Weight output, token_embd;
  float *final_norm = nullptr;
  bool has_output = false, has_embd = false;
  __half *kcache = nullptr, *vcache = nullptr;
  int64_t kv_layer_elems = 0;  // halfs per layer per side
  float *cos_all = nullptr, *sin_all = nullptr, *cos_step = nullptr, *sin_step = nullptr;
  float *h = nullptr, *normed = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *attn = nullptr, *gate = nullptr,
        *up = nullptr, *logits = nullptr, *taps = nullptr;
  uint8_t *act_k = nullptr, *act_0 = nullptr;  // Q8_K and Q8_0 operand buffers (widest row)
  float *attn_part = nullptr;
  uint32_t *attn_tickets = nullptr;
  float *am_val = nullptr;
  int32_t *am_idx = nullptr;
  uint32_t *am_ticket = nullptr;  // [2*max_rows]: tickets, then history lengths
  int32_t *out_idx = nullptr, *d_tokens = nullptr, *d_positions = nullptr, *d_slots = nullptr, *d_history = nullptr;
  int64_t history_cap = 0;
  int32_t *moe_sel_idx = nullptr, *moe_counts = nullptr, *moe_lists = nullptr;
  float *moe_sel_w = nullptr, *moe_g = nullptr, *moe_u = nullptr, *moe_act = nullptr, *moe_down = nullptr;
  // tensor-core expert path: three Q8_K rows per assignment, `moe_cap` rows per local expert
  int32_t *moe_pos = nullptr;
  int32_t moe_cap = 0, moe_pass_rows = 0;
  uint8_t *moe_act3_h = nullptr, *moe_act3_f = nullptr;
  float *moe_g3 = nullptr, *moe_u3 = nullptr, *moe_d3 = nullptr, *moe_scratch = nullptr;
  int64_t moe_scratch_floats = 0;
  int32_t *d_status = nullptr;  // set by a kernel whose bounded wait gave up
  int64_t filled = 0;
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  float last_ms = 0.0f;
  int64_t last_launches = 0, launches = 0;
  LayeredModel *lay = nullptr;  // set: this engine runs a layered design
  int32_t logit_rows = 0;       // rows of `logits` (llama-shaped: max_rows)
  int32_t last_logit_row = 0;   // the row of `logits` that the last call's final token left
  std::vector<void *> allocs;
  // CUDA graphs of whole steps, keyed by (rows, option bits, score-scale bits).  A key's first
  // step runs as plain launches (it also sets kernel attributes); its second is captured.
  struct StepGraph {
    cudaGraphExec_t exec = nullptr;
    int64_t launches = 0;
    int uses = 0;
  };
  std::map<std::tuple<int64_t, uint32_t, uint32_t>, StepGraph> graphs;
  bool graphs_off = false;
};

namespace cmld {

struct DeviceGuard {
  int prev = -1;
  bool ok = true;
  explicit DeviceGuard(int dev) {
    if (cudaGetDevice(&prev) != cudaSuccess) ok = false;
    if (ok && prev != dev && cudaSetDevice(dev) != cudaSuccess) ok = false;
  }
  ~DeviceGuard() {
    if (prev >= 0) cudaSetDevice(prev);
  }
};

#define CMLD_ENGINE_ENTER(e)                                              \
  if (!(e)) return fail(CMLD_ERR_INVALID, "engine handle is null");       \
  DeviceGuard guard__((e)->device);                                       \
  if (!guard__.ok) return fail(CMLD_ERR_CUDA, "cannot select CUDA device %d", (e)->device)

template <typename T>
inline int32_t dev_alloc(cmld_engine *e, T **p, int64_t count, bool zero = true) {
  void *raw = nullptr;
  const size_t bytes = (size_t)std::max<int64_t>(count, 1) * sizeof(T);
  CMLD_CUDA(cudaMalloc(&raw, bytes));
  e->allocs.push_back(raw);
  if (zero) CMLD_CUDA(cudaMemsetAsync(raw, 0, bytes, e->stream));
  *p = static_cast<T *>(raw);
  return CMLD_OK;
}

struct StepOpts {
  int32_t batch = 1;
  bool from_tokens = false;    // gather embeddings of d_tokens, else h holds them
  bool rope_by_position = true;  // index the engine's all-position table, else cos_step/sin_step rows
  float scale = 0.0f;
  bool logits = true;
  bool argmax = true;
  bool feed_back = false;  // argmax writes next token / position / history
  bool taps = false;
  int32_t layer_begin = 0, layer_end = -1;  // layers to run; -1 = through the last
  bool attn_cluster = false;  // short contexts, few rows: attention ranges as a thread-block cluster (host-side choice)
  int32_t attn_cap = 0;       // bound on the context length of every row of this step (a bucket: 1024, 2048, 4096, 8192), 0 = unknown
  const uint32_t *tree_mask = nullptr;  // tree verification: per-row ancestor masks (device), nodes at cache rows tree_base..
  int32_t tree_base = 0, tree_words = 0;
  bool shared_slots = false;  // several rows of this step belong to one sequence (prefill, verify): row b
                              // reads K/V that rows < b write, so the KV append must be a kernel of its own
  // layered designs, rows that are consecutive tokens of one sequence (shared_slots):
  int64_t seq_start = 0;      // position of row 0
  int32_t seq_slot = 0;
  int32_t n_want = -1;        // logits only for this many rows, listed in the engine's row map; -1 = every row
  float *taps_out = nullptr;  // device: residual stream after every layer run, [runs][batch][width]
};

// engine.cu
int32_t weight_alloc(Weight &w, int32_t qt, int64_t rows, int64_t cols);
void weight_free(Weight &w);
int32_t run_step(cmld_engine *e, const StepOpts &o);
int32_t finish(cmld_engine *e, const char *what);
int32_t stage_rows(cmld_engine *e, int32_t n, const int32_t *tokens, const int32_t *positions, const int32_t *slots);
int32_t attn_cap_for(int64_t max_position);
int32_t engine_open(cmld_engine *e, int32_t device);  // device, stream, events
int32_t init_rows(cmld_engine *e, int64_t rows, int64_t logit_rows, int64_t vocab_local);  // token, position, logits and argmax buffers

// layered.cu
void layered_free(cmld_engine *e);
int32_t layered_ready(const cmld_engine *e, bool report);  // 1: every tensor is set; `report`: leave an error message if not
int32_t layered_step(cmld_engine *e, const StepOpts &o);
int32_t layered_claim(cmld_engine *e, int32_t n, const int32_t *seqs, const int64_t *positions);
void layered_advance(cmld_engine *e, int32_t n, const int32_t *seqs, const int64_t *positions, int64_t steps);
int32_t layered_extend(cmld_engine *e, int32_t seq, const int32_t *tokens, int64_t n, int64_t start, const int32_t *want, int32_t n_want,
                       float *logits_out, float *taps_out);

}  // namespace cmld
