// Runtime objects shared by the model families: a loaded model, its cache (paged keys and values, step state,
// workspaces) and the helpers every family's host code uses. Internal to the library.
#pragma once
#include <cuda_runtime.h>

#include <cstdlib>
#include <cstring>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "common.h"
#include "kernels.cuh"

namespace pg {

#define PG_CUDA_TRY(expr)                                                                      \
  do {                                                                                         \
    cudaError_t _e = (expr);                                                                   \
    if (_e != cudaSuccess)                                                                     \
      return set_error(PG_CUDA, std::string("CUDA error: ") + cudaGetErrorString(_e) + " at " + \
                                    __FILE__ + ":" + std::to_string(__LINE__) + " (" #expr ")"); \
  } while (0)

struct LayerWeights {
  float *ln1_g, *ln1_b, *w_qkv, *b_qkv, *w_proj, *b_proj, *ln2_g, *ln2_b, *w_fc, *b_fc, *w_proj2, *b_proj2;
  // copies in the tiled layout of the tensor-core decode kernel (nullptr in fp32 mode)
  float *t_qkv = nullptr, *t_proj = nullptr, *t_fc = nullptr, *t_proj2 = nullptr;
  // lo parts (w - hi(w), hi = the upper 19 bits a TF32 tensor core reads) of the four matrices, [out, in] row-major:
  // second operand of the FP32-grade prefill GEMM (nullptr in fp32 mode)
  float *l_qkv = nullptr, *l_proj = nullptr, *l_fc = nullptr, *l_proj2 = nullptr;
  // packed copies for the single-kernel decode step (BF16 or row-quantised int8 weights), [out, in] rows, and,
  // for int8, one scale per output row
  void *p_qkv = nullptr, *p_proj = nullptr, *p_fc = nullptr, *p_proj2 = nullptr;
  float *s_qkv = nullptr, *s_proj = nullptr, *s_fc = nullptr, *s_proj2 = nullptr;
};

inline bool env_flag(const char* name) {
  const char* v = getenv(name);
  return v && *v && strcmp(v, "0") != 0;
}

constexpr int MAX_SPLITS = 16;
constexpr int MAX_TOPK = 64;

// Per-operation device timing of one decode step: the buckets of Gpt2OperationProfile
// (rust.rs:336-347). Events around every launch serialise the step, so this is a profiling mode.
enum Bucket { B_LAYER_NORM = 0, B_QKV, B_ATTN, B_ATTN_PROJ, B_MLP_FC, B_MLP_PROJ, B_LOGITS, B_OTHER, B_COUNT };
struct StepProfiler {
  std::vector<cudaEvent_t> ev;
  std::vector<int> bucket;
  int chain_event = -1;  // index of the event pair around the persistent chain kernel, if it ran
  cudaError_t mark(cudaStream_t s, int b) {
    cudaEvent_t e;
    cudaError_t r = cudaEventCreate(&e);
    if (r != cudaSuccess) return r;
    ev.push_back(e);
    bucket.push_back(b);
    return cudaEventRecord(e, s);
  }
  ~StepProfiler() {
    for (auto e : ev) cudaEventDestroy(e);
  }
};

// Page table of one group of attention layers. Layers whose keys stay visible for the whole context index it by
// position (span = max context); layers whose keys die at a fixed boundary index it by position modulo `span`, so a
// sequence never holds more than ceil(span / page_tokens) pages of them.
struct PageTable {
  int span = 0;             // cache index of position p = p % span
  int page_tokens = 32, pages_per_seq = 0, num_pages = 0;
  std::vector<int> free_pages;
  std::vector<int> h_table;  // [max_batch][pages_per_seq], -1 = unassigned
  int* d_table = nullptr;
  bool dirty = true;
};

int ensure_device(int device);
int page_table_init(PageTable* t, int max_batch, int span, int page_tokens, cudaStream_t s);

// A layered model (layered.cu) and its per-cache state; opaque to the GPT-2 code.
struct LayeredModel;
struct LayeredCache;

}  // namespace pg

using namespace pg;  // the C ABI's handle types live in the global namespace

// ------------------------------------------------------------------ model
struct pg_model {
  pg_gpt2_config cfg{};
  pg_backend_config backend{};
  int device = 0;
  int num_sms = 148;
  float* arena = nullptr;  // every weight tensor lives in this one allocation
  float* tiled_arena = nullptr;  // second copy of the dense matrices, tiled for TMA (tensor-core modes)
  size_t tiled_floats = 0;
  float* t_wte = nullptr;
  float* lo_arena = nullptr;
  size_t arena_floats = 0;
  int stream_weight_type = STREAM_W_F32;  // what the single-kernel decode step streams
  unsigned char* packed_arena = nullptr;  // BF16 / int8 copies of the dense matrices and of wte
  float* scale_arena = nullptr;           // int8: row scales
  void* p_wte = nullptr;
  float* s_wte = nullptr;
  float* head_w = nullptr;      // FP32 rows of the lm_head: wte itself, or (int8) its dequantised copy
  float* head_deq = nullptr;    // owned storage of that copy
  float *wte = nullptr, *wpe = nullptr, *lnf_g = nullptr, *lnf_b = nullptr;
  std::vector<LayerWeights> layers;
  bool fused_ok = false;  // LayerNorm/argmax fusion needs n_embd % 4 == 0 and n_embd <= 2048
  bool use_pdl = true;
  std::shared_ptr<LayeredModel> layered;  // set for models described layer by layer; everything GPT-2 above is then unused

  int c() const { return (int)cfg.n_embd; }
  int f() const { return (int)cfg.n_inner; }
  int v() const { return (int)cfg.vocab_size; }
  int heads() const { return (int)cfg.n_head; }
  int head_dim() const { return (int)(cfg.n_embd / cfg.n_head); }
  int layers_n() const { return (int)cfg.n_layer; }
  int positions() const { return (int)cfg.n_positions; }

  ~pg_model();
};

// ------------------------------------------------------------------ cache
struct pg_cache {
  const pg_model* model = nullptr;
  int max_batch = 0;
  cudaStream_t stream = nullptr;
  KvLayout kv{};
  size_t page_floats = 0;  // floats of one page of one layer
  std::vector<PageTable> tables;  // GPT-2: one; layered models: one per distinct key lifetime
  float* kv_pool = nullptr;    // [layer][page][2][head][page_tokens][head_dim]
  std::vector<int> seq_len;    // host mirror of d_pos
  int *d_ids = nullptr, *d_pos = nullptr, *d_argmax = nullptr, *d_token_log = nullptr;
  float *x = nullptr, *norm = nullptr, *qkv = nullptr, *attn = nullptr, *hbuf = nullptr, *logits = nullptr;
  float* part_val = nullptr;
  int* part_idx = nullptr;
  int part_stride = 0;
  float* attn_part = nullptr;
  unsigned* attn_counters = nullptr;
  float* topk_vals = nullptr;
  int* topk_idx = nullptr;
  // tensor-core decode path (9..64 sequences): TF32 hi/lo pairs of the GEMM inputs, split-K scratch
  float *norm_lo = nullptr, *attn_lo = nullptr, *h_lo = nullptr;
  int* d_error = nullptr;
  // persistent chain kernel of the tensor-core decode path: partial tiles, grid-barrier word
  float* chain_partials = nullptr;
  unsigned* d_chain_barrier = nullptr;
  unsigned long long* d_chain_best = nullptr;  // row arg-max accumulators of the lm_head phase
  unsigned long long* d_chain_trace = nullptr;  // developer aid: only allocated in builds with -DPG_DEV_TRACE
  int chain_ctas = 0;
  int chain_min_batch = 9;  // smallest batch whose decode step runs as the chain kernel in the tensor-core modes (measured on
                            // B200, GPT-2 medium, 8 sequences: 1.34 ms as the chain kernel, 1.09 ms as one kernel per operation)
  struct ChainProgram {  // whole-step phase list of the persistent chain kernel for one batch size
    ChainPhase* dev = nullptr;            // in device memory (nullptr: this batch size is not supported)
    ChainPhase* dev_argmax_only = nullptr;  // the same list whose lm_head reduce phase keeps the row arg-max but stores no logits
    int n = 0;
    std::vector<int> bucket;              // profile bucket of every phase
    unsigned long long* d_times = nullptr;  // n + 1 time stamps, written in profiling runs
  };
  std::map<int, ChainProgram> chain_programs;
  bool step_wants_logits = true;  // false: the caller of this step only reads the arg-max (greedy decoding)
  // single-kernel decode step (at most 8 sequences): layer table, tagged exchange buffers, tag counter
  unsigned long long* d_stream_ll = nullptr;  // ll_x | ll_qkv | ll_attn | ll_h | ll_part | ll_best
  unsigned* d_stream_epoch = nullptr;
  int stream_grid = 0;
  unsigned dbg_spin_limit = 0, dbg_poison = 0;  // pg_cache_debug_expire_next_wait: consumed by the next decode step
#ifdef PG_DEV_TRACE
  unsigned long long* d_stream_trace = nullptr;
#endif
  int *h_ids = nullptr, *h_out = nullptr;  // pinned staging
  // prefill workspace (grow-only)
  size_t pre_rows = 0;
  float *px = nullptr, *pnorm = nullptr, *pqkv = nullptr, *pattn = nullptr, *ph = nullptr, *plo = nullptr;
  int* prow = nullptr;  // [4][pre_rows]: ids, pos, slot, (batch+1 seq_start / last rows)
  std::map<std::pair<int, int>, cudaGraphExec_t> graphs;  // (batch, splits) -> decode-step graph
  std::map<std::pair<int, int>, uint64_t> graphs_launches;  // kernel nodes in each graph
  uint64_t decode_launches = 0;  // kernels launched by decode steps (for gpu_launches accounting)
  cudaEvent_t t0 = nullptr, t1 = nullptr;  // pg_cache_time_begin / pg_cache_time_end

  std::shared_ptr<LayeredCache> layered;

  float* layer_pool(int l) const { return kv_pool + (size_t)l * tables[0].num_pages * page_floats; }

  ~pg_cache();
};

