// Models described layer by layer (see design.h): device weights, per-cache state (key / value pages, recurrent
// states), the decode step and the pass over portions of prompts. Every layer is
//   x += LayerNorm(mixer(LayerNorm(x)));  x += LayerNorm(down(gelu(up(LayerNorm(x)))))   (the second one optional)
// where the mixer is one branch or the scaled sum of several. All branches of a layer share one input projection (their
// weight rows are concatenated) and one output projection (their columns are concatenated, the branch scales applied
// to the columns before it).
#include <algorithm>
#include <cmath>
#include <cstdio>

#include "layered.h"
#include "layered_kernels.cuh"

namespace pg {

namespace {

int align_to(int n, int a) { return (n + a - 1) / a * a; }
constexpr int K_ALIGN = 64;  // input columns of every product: one TMA box of BF16
constexpr int N_ALIGN = 8;
constexpr int MAX_ROWS_LINEAR = 8;
// tokens per segment of a recurrence over a long portion: many enough to fill the chip, few enough to combine quickly
int segment_tokens(int max_len) { return max_len >= 4096 ? 256 : 128; }

struct Matrix {  // [np, kp] row-major in the storage type, zero outside [n, k]
  void* w = nullptr;
  void* tiled = nullptr;  // BF16: the second copy that batches of decode rows stream
  int n = 0, k = 0, np = 0, kp = 0;
};
struct Norm {
  float *g = nullptr, *b = nullptr;
};

struct DevBranch {
  int kind = 0, y_off = 0;
  AttentionLayer attn{};
  RecurrenceLayer rec{};
  int pool = -1;       // attention: index of the key / value pool and ...
  int table = -1;      // ... of the page table (by distinct span)
  int state = -1;      // recurrence: index of the state array
};
struct DevLayer {
  Norm norm1, norm1b, norm2, norm2b;
  Matrix in, out, up, down;
  std::vector<DevBranch> branches;
  bool ff = false;
};

}  // namespace

struct LayeredModel {
  LayeredConfig cfg;
  bool bf16 = false;
  int widthp = 0;  // row pitch of the residual stream and of normed rows
  Matrix embed;    // token embedding and output projection
  Norm final_norm;
  double* freq = nullptr;
  std::vector<DevLayer> layers;
  int max_in = 0, max_y = 0, max_ff = 0, max_rec = 0;  // widest projection, mixer output, hidden row, heads * dim ...
  int max_rec_out = 0, max_rec_heads = 0;                  // ... heads * vdim and heads of a recurrence
  int n_pools = 0, n_states = 0;
  std::vector<int> spans;  // one page table each
  std::vector<void*> allocations;
  uint64_t weight_bytes = 0;
  int device = 0;
  size_t elem() const { return bf16 ? 2 : 4; }
  ~LayeredModel() {
    if (allocations.empty()) return;
    cudaSetDevice(device);
    for (void* p : allocations) cudaFree(p);
  }
};

struct LayeredRows {  // activations of one pass, all [rows, pitch]
  size_t rows = 0;
  float *x[2] = {nullptr, nullptr};  // residual stream, used in turns
  float *p = nullptr;                // input projection
  float *yo = nullptr;               // sublayer output
  void *h = nullptr, *y = nullptr, *ff = nullptr;  // storage type
  float *h32 = nullptr, *y32 = nullptr, *ff32 = nullptr;  // decode with at most 8 BF16 rows: FP32 product inputs
};

struct LayeredCache {
  std::vector<void*> pools;
  std::vector<float*> states;
  LayeredRows step, portion;
  float* attn_part = nullptr;
  unsigned* attn_counters = nullptr;
  // portion workspaces (grow-only)
  float *decay = nullptr, *unit = nullptr, *rate = nullptr, *unit_next = nullptr, *pair = nullptr, *out_raw = nullptr, *segments = nullptr;
  void *q = nullptr, *k = nullptr, *v = nullptr;
  int* meta = nullptr;
  float* logits = nullptr;
  size_t q_rows = 0, k_rows = 0, seg_floats = 0, meta_ints = 0, logit_rows = 0, gate_rows = 0;
  ~LayeredCache() {
    for (void* p : pools) cudaFree(p);
    for (float* p : states) cudaFree(p);
    for (LayeredRows* r : {&step, &portion})
      for (void* p : {(void*)r->x[0], (void*)r->x[1], (void*)r->p, (void*)r->yo, r->h, r->y, r->ff, (void*)r->h32, (void*)r->y32, (void*)r->ff32})
        if (p) cudaFree(p);
    for (void* p : {(void*)attn_part, (void*)attn_counters, (void*)decay, (void*)unit, (void*)rate, (void*)unit_next, (void*)pair, (void*)out_raw, (void*)segments, q, k, v,
                    (void*)meta, (void*)logits})
      if (p) cudaFree(p);
  }
};

namespace {

// ------------------------------------------------------------------ weights
struct Builder {
  LayeredModel* m;
  const SafeTensorsFile& file;

  int alloc(size_t bytes, void** out) {
    PG_CUDA_TRY(cudaMalloc(out, std::max<size_t>(bytes, 16)));
    m->allocations.push_back(*out);
    PG_CUDA_TRY(cudaMemset(*out, 0, std::max<size_t>(bytes, 16)));
    return PG_OK;
  }
  int upload(const std::vector<float>& v, size_t padded, float** out) {
    if (int r = alloc(std::max(padded, v.size()) * sizeof(float), (void**)out)) return r;
    PG_CUDA_TRY(cudaMemcpy(*out, v.data(), v.size() * sizeof(float), cudaMemcpyHostToDevice));
    m->weight_bytes += v.size() * sizeof(float);
    return PG_OK;
  }
  int vec(const std::string& name, size_t padded, float** out) { return upload(tensor_f32(file, name), padded, out); }
  int norm(const std::string& name, Norm* n) {
    if (int r = vec(name, m->widthp, &n->g)) return r;
    return vec(name + ".b", m->widthp, &n->b);
  }
  // [n, k] row-major FP32 on the host
  int matrix(const std::vector<float>& v, int n, int k, int n_align, Matrix* out) {
    out->n = n;
    out->k = k;
    out->np = align_to(n, n_align);
    out->kp = align_to(k, K_ALIGN);
    if (int r = alloc((size_t)out->np * out->kp * m->elem(), &out->w)) return r;
    m->weight_bytes += (uint64_t)n * k * m->elem();
    if (m->bf16) {
      float* tmp = nullptr;
      PG_CUDA_TRY(cudaMalloc(&tmp, v.size() * sizeof(float)));
      cudaError_t e = cudaMemcpy(tmp, v.data(), v.size() * sizeof(float), cudaMemcpyHostToDevice);
      if (e == cudaSuccess) e = launch_pack_bf16(tmp, out->w, n, k, out->np, out->kp, 0);
      if (e == cudaSuccess) e = cudaDeviceSynchronize();
      cudaFree(tmp);
      PG_CUDA_TRY(e);
      if (int r = alloc(tiled_bf16_elems(out->np, out->kp) * 2, &out->tiled)) return r;
      PG_CUDA_TRY(launch_tile_bf16(out->w, out->tiled, out->np, out->kp, 0));
    } else {
      PG_CUDA_TRY(cudaMemcpy2D(out->w, (size_t)out->kp * 4, v.data(), (size_t)k * 4, (size_t)k * 4, n, cudaMemcpyHostToDevice));
    }
    return PG_OK;
  }
  int matrix(const std::string& name, int n, int k, int n_align, Matrix* out) { return matrix(tensor_f32(file, name), n, k, n_align, out); }
  // [n, r] -> [r, n]
  int transposed(const std::string& name, int n, int r, float** out) {
    const std::vector<float> v = tensor_f32(file, name);
    std::vector<float> t(v.size());
    for (int i = 0; i < n; ++i)
      for (int j = 0; j < r; ++j) t[(size_t)j * n + i] = v[(size_t)i * r + j];
    return upload(t, 0, out);
  }
};

int build_layer(Builder& b, const LayerSpec& spec, const std::string& p, int page_tokens, int max_context, DevLayer* d) {
  LayeredModel* m = b.m;
  const int W = m->cfg.width;
  const float eps = m->cfg.norm_eps;
  if (int r = b.norm(p + "norm1", &d->norm1)) return r;
  if (int r = b.norm(p + "norm1b", &d->norm1b)) return r;
  std::vector<float> in;
  int rows = 0, y_cols = 0;
  auto part = [&](const std::string& name, int n) {  // appends weight rows; every part starts at a multiple of 4 columns
    const int at = rows;
    const std::vector<float> v = tensor_f32(b.file, name);
    in.insert(in.end(), v.begin(), v.end());
    rows += n;
    const int pad = align_to(rows, 4) - rows;
    in.insert(in.end(), (size_t)pad * W, 0.f);
    rows += pad;
    return at;
  };
  for (const BranchSpec& bs : spec.branches) {
    const std::string t = p + bs.prefix + ".";
    DevBranch br;
    br.kind = bs.kind;
    br.y_off = y_cols;
    y_cols += bs.out_dim();
    if (bs.kind == BranchSpec::ATTENTION) {
      const AttentionSpec& s = bs.attn;
      AttentionLayer& a = br.attn;
      a.heads = s.heads; a.kv_heads = s.kv_heads; a.dim = s.dim; a.vdim = s.vdim;
      a.dimp = align_to(s.dim, 8); a.vdimp = align_to(s.vdim, 8);
      a.span = s.chunk > 0 ? std::min(s.chunk, max_context) : max_context;
      a.off_q = part(t + "q", s.heads * s.dim);
      a.off_k = part(t + "k", s.kv_heads * s.dim);
      a.off_v = part(t + "v", s.kv_heads * s.vdim);
      if (s.qk_norm) {
        float* g = nullptr;
        if (int r = b.vec(t + "q.norm", 0, &g)) return r;
        a.q_norm = g;
        if (int r = b.vec(t + "k.norm", 0, &g)) return r;
        a.k_norm = g;
      }
      a.v_norm = s.v_norm ? 1 : 0;
      a.scale = s.scale; a.eps = eps; a.out_scale = bs.scale;
      a.page_tokens = page_tokens;
      a.pages_per_seq = (a.span + page_tokens - 1) / page_tokens;
      auto it = std::find(m->spans.begin(), m->spans.end(), a.span);
      br.table = (int)(it - m->spans.begin());
      if (it == m->spans.end()) m->spans.push_back(a.span);
      br.pool = m->n_pools++;
      if (!attention_supported(a))
        return set_error(PG_INVALID_CONFIG, p + bs.prefix + ": " + std::to_string(s.heads / s.kv_heads) + " query heads per key head of size " +
                                                std::to_string(s.dim) + " exceed what the decode kernel holds");
    } else {
      const RecurrenceSpec& s = bs.rec;
      RecurrenceLayer& a = br.rec;
      const int K = s.heads * s.dim, V = s.heads * s.vdim;
      const bool delta = s.kind == RECUR_DELTA;
      a.kind = s.kind; a.heads = s.heads; a.dim = s.dim; a.vdim = s.vdim; a.dvp = align_to(s.vdim, 4); a.rank = s.rank;
      a.off_q = part(t + (delta ? "r" : "q"), K);
      a.off_k = part(t + "k", K);
      a.off_v = part(t + "v", V);
      a.off_g = part(t + "g", V);
      if (delta) a.off_a = part(t + "a", K);
      a.off_t = part(t + (delta ? "w1" : "a1"), s.rank);
      float* f = nullptr;
      if (int r = b.transposed(t + (delta ? "w2" : "a2"), K, s.rank, &f)) return r;
      a.w2 = f;
      if (int r = b.vec(t + (delta ? "w0" : "a2.b"), 0, &f)) return r;
      a.b2 = f;
      if (delta) {
        if (int r = b.vec(t + "a.b", 0, &f)) return r;
        a.a_bias = f;
      }
      if (int r = b.vec(t + "norm", 0, &f)) return r;
      a.norm = f;
      a.q_scale = delta ? 1.f : (float)(1.0 / std::sqrt((double)s.dim));
      a.inv_tau = (float)(1.0 / (double)s.tau);
      a.eps = eps;
      a.out_scale = bs.scale;
      br.state = m->n_states++;
      m->max_rec = std::max(m->max_rec, K);
      m->max_rec_out = std::max(m->max_rec_out, V);
      m->max_rec_heads = std::max(m->max_rec_heads, s.heads);
    }
    d->branches.push_back(br);
  }
  if (int r = b.matrix(in, rows, W, N_ALIGN, &d->in)) return r;
  in.clear();
  in.shrink_to_fit();
  // output projections of the branches side by side: [W, sum of the branches' columns]
  std::vector<float> out((size_t)W * y_cols);
  for (size_t i = 0; i < spec.branches.size(); ++i) {
    const int n = spec.branches[i].out_dim(), off = d->branches[i].y_off;
    const std::vector<float> v = tensor_f32(b.file, p + spec.branches[i].prefix + ".o");
    for (int r = 0; r < W; ++r) std::copy(v.begin() + (size_t)r * n, v.begin() + (size_t)(r + 1) * n, out.begin() + (size_t)r * y_cols + off);
  }
  if (int r = b.matrix(out, W, y_cols, K_ALIGN, &d->out)) return r;
  m->max_in = std::max(m->max_in, d->in.np);
  m->max_y = std::max(m->max_y, d->out.kp);
  if (spec.ff > 0) {
    d->ff = true;
    if (int r = b.norm(p + "norm2", &d->norm2)) return r;
    if (int r = b.norm(p + "norm2b", &d->norm2b)) return r;
    if (int r = b.matrix(p + "mlp.up", spec.ff, W, K_ALIGN, &d->up)) return r;
    if (int r = b.matrix(p + "mlp.down", W, spec.ff, K_ALIGN, &d->down)) return r;
    m->max_ff = std::max(m->max_ff, d->down.kp);
  }
  return PG_OK;
}

int alloc_rows(const LayeredModel* m, LayeredRows* r, size_t rows, bool step) {
  if (rows <= r->rows) return PG_OK;
  void** bufs[] = {(void**)&r->x[0], (void**)&r->x[1], (void**)&r->p, (void**)&r->yo, &r->h, &r->y, &r->ff,
                   (void**)&r->h32, (void**)&r->y32, (void**)&r->ff32};
  for (void** p : bufs) {
    if (*p) cudaFree(*p);
    *p = nullptr;
  }
  r->rows = 0;
  // padding columns are read by the products (against zero weights): they must hold finite numbers
  auto get = [&](void** p, size_t bytes) -> int {
    PG_CUDA_TRY(cudaMalloc(p, std::max<size_t>(bytes, 16)));
    PG_CUDA_TRY(cudaMemset(*p, 0, std::max<size_t>(bytes, 16)));
    return PG_OK;
  };
  const size_t wp = m->widthp, e = m->elem();
  for (int i = 0; i < 2; ++i)
    if (int q = get((void**)&r->x[i], rows * wp * 4)) return q;
  if (int q = get((void**)&r->p, rows * m->max_in * 4)) return q;
  if (int q = get((void**)&r->yo, rows * wp * 4)) return q;
  if (int q = get(&r->h, rows * wp * e)) return q;
  if (int q = get(&r->y, rows * m->max_y * e)) return q;
  if (int q = get(&r->ff, rows * std::max(m->max_ff, 1) * e)) return q;
  if (step && m->bf16) {
    const size_t n = std::min<size_t>(rows, MAX_ROWS_LINEAR);
    if (int q = get((void**)&r->h32, n * wp * 4)) return q;
    if (int q = get((void**)&r->y32, n * m->max_y * 4)) return q;
    if (int q = get((void**)&r->ff32, n * std::max(m->max_ff, 1) * 4)) return q;
  }
  PG_CUDA_TRY(cudaDeviceSynchronize());
  r->rows = rows;
  return PG_OK;
}

template <typename P>
int grow(P** p, size_t* have, size_t want, size_t bytes_each) {
  if (want <= *have) return PG_OK;
  if (*p) cudaFree((void*)*p);
  *p = nullptr;
  *have = 0;
  PG_CUDA_TRY(cudaMalloc((void**)p, want * bytes_each));
  PG_CUDA_TRY(cudaMemset((void*)*p, 0, want * bytes_each));
  PG_CUDA_TRY(cudaDeviceSynchronize());
  *have = want;
  return PG_OK;
}

}  // namespace

int build_layered_model(const LayeredConfig& cfg, const SafeTensorsFile& file, const pg_backend_config* backend, pg_model** out) {
  pg_backend_config be{};
  if (backend) be = *backend;
  if (be.page_tokens == 0) be.page_tokens = 32;
  if (be.page_tokens != 16 && be.page_tokens != 32 && be.page_tokens != 64)
    return set_error(PG_INVALID_CONFIG, "cuda page_tokens must be 16, 32 or 64");
  if (be.math_mode != PG_MATH_FP32 && be.math_mode != PG_MATH_BF16)
    return set_error(PG_INVALID_CONFIG, "cuda math_mode of a " + cfg.architecture + " model must be fp32 or bf16");
  if (be.quantized_weights) return set_error(PG_INVALID_CONFIG, "cuda quantized_weights is not available for " + cfg.architecture + " models");
  if (be.attn_splits < 0 || be.attn_splits > MAX_SPLITS) return set_error(PG_INVALID_CONFIG, "cuda attn_splits must be in 0..16");
  if (be.max_context < 0 || be.max_context > (1 << 24)) return set_error(PG_INVALID_CONFIG, "cuda max_context must be in 0..16777216");
  if (be.max_context == 0) be.max_context = 32768;
  if (int r = ensure_device(be.device)) return r;

  auto model = std::make_unique<pg_model>();
  auto m = std::make_shared<LayeredModel>();
  model->backend = be;
  model->device = m->device = be.device;
  PG_CUDA_TRY(cudaDeviceGetAttribute(&model->num_sms, cudaDevAttrMultiProcessorCount, be.device));
  model->use_pdl = !env_flag("PG_NO_PDL");
  model->cfg.vocab_size = cfg.vocab;
  model->cfg.n_positions = be.max_context;
  model->cfg.n_embd = cfg.width;
  model->cfg.n_layer = cfg.layers.size();
  model->cfg.n_head = 1;
  model->cfg.n_inner = 1;
  model->cfg.layer_norm_epsilon = cfg.norm_eps;
  model->layered = m;
  m->cfg = cfg;
  m->bf16 = be.math_mode == PG_MATH_BF16;
  m->widthp = align_to(cfg.width, K_ALIGN);
  Builder b{m.get(), file};
  if (int r = b.matrix("embed", cfg.vocab, cfg.width, 1, &m->embed)) return r;
  if (int r = b.norm("final.norm", &m->final_norm)) return r;
  std::vector<double> freq((cfg.width + 1) / 2 + 2);
  for (size_t i = 0; i < freq.size(); ++i) freq[i] = std::pow(10000.0, -2.0 * (double)i / (double)cfg.width);
  if (int r = b.alloc(freq.size() * sizeof(double), (void**)&m->freq)) return r;
  PG_CUDA_TRY(cudaMemcpy(m->freq, freq.data(), freq.size() * sizeof(double), cudaMemcpyHostToDevice));
  m->layers.resize(cfg.layers.size());
  for (size_t i = 0; i < cfg.layers.size(); ++i)
    if (int r = build_layer(b, cfg.layers[i], "l" + std::to_string(i) + ".", be.page_tokens, be.max_context, &m->layers[i])) return r;
  PG_CUDA_TRY(cudaDeviceSynchronize());
  *out = model.release();
  return PG_OK;
}

const LayeredConfig& layered_config(const pg_model* m) { return m->layered->cfg; }

uint64_t layered_weight_bytes_per_step(const pg_model* m) { return m->layered->weight_bytes; }

uint64_t layered_state_bytes_per_sequence(const pg_model* m) {
  uint64_t n = 0;
  for (const DevLayer& l : m->layered->layers)
    for (const DevBranch& b : l.branches)
      if (b.kind == BranchSpec::RECURRENCE) n += recurrence_state_floats(b.rec) * sizeof(float);
  return n;
}

// ------------------------------------------------------------------ cache
int layered_cache_init(pg_cache* c) {
  const LayeredModel* m = c->model->layered.get();
  auto lc = std::make_shared<LayeredCache>();
  const size_t B = c->max_batch;
  c->tables.resize(m->spans.size());
  for (size_t i = 0; i < m->spans.size(); ++i)
    if (int r = page_table_init(&c->tables[i], c->max_batch, m->spans[i], c->model->backend.page_tokens, c->stream)) return r;
  lc->pools.assign(m->n_pools, nullptr);
  lc->states.assign(m->n_states, nullptr);
  size_t part = 0, counters = 0;
  for (const DevLayer& l : m->layers)
    for (const DevBranch& b : l.branches) {
      if (b.kind == BranchSpec::ATTENTION) {
        const size_t bytes = (size_t)c->tables[b.table].num_pages * attention_page_elems(b.attn) * m->elem();
        PG_CUDA_TRY(cudaMalloc(&lc->pools[b.pool], bytes));
        PG_CUDA_TRY(cudaMemsetAsync(lc->pools[b.pool], 0, bytes, c->stream));
        part = std::max(part, B * b.attn.heads * MAX_SPLITS * (b.attn.vdim + 2));
        counters = std::max(counters, B * b.attn.kv_heads);
      } else {
        const size_t bytes = B * recurrence_state_floats(b.rec) * sizeof(float);
        PG_CUDA_TRY(cudaMalloc(&lc->states[b.state], bytes));
        PG_CUDA_TRY(cudaMemsetAsync(lc->states[b.state], 0, bytes, c->stream));
      }
    }
  if (part) {
    PG_CUDA_TRY(cudaMalloc(&lc->attn_part, part * sizeof(float)));
    PG_CUDA_TRY(cudaMalloc(&lc->attn_counters, counters * sizeof(unsigned)));
    PG_CUDA_TRY(cudaMemsetAsync(lc->attn_counters, 0, counters * sizeof(unsigned), c->stream));
  }
  if (int r = alloc_rows(m, &lc->step, B, true)) return r;
  c->layered = lc;
  return PG_OK;
}

int layered_choose_splits(const pg_cache* c, int batch, int max_len) {
  const pg_model* m = c->model;
  if (m->backend.attn_splits > 0) return std::min(m->backend.attn_splits, MAX_SPLITS);
  // by the longest key range any layer can have at this length, in powers of two (a step graph per value)
  int span = 0, kv = 1 << 30;
  for (const DevLayer& l : m->layered->layers)
    for (const DevBranch& b : l.branches)
      if (b.kind == BranchSpec::ATTENTION) {
        span = std::max(span, std::min(b.attn.span, max_len));
        kv = std::min(kv, b.attn.kv_heads);
      }
  if (!span) return 1;
  const int by_fill = (2 * m->num_sms + batch * kv - 1) / (batch * kv), by_len = (span + 127) / 128;
  int s = 1;
  while (s * 2 <= std::min(std::min(by_fill, by_len), 8)) s *= 2;
  return s;
}

namespace {

#define PG_L(bucket_, expr)                                                    \
  do {                                                                         \
    if (prof && (e = prof->mark(s, bucket_)) != cudaSuccess) return e;         \
    e = (expr);                                                                \
    ++n;                                                                       \
    if (e != cudaSuccess) return e;                                            \
    if (prof && (e = prof->mark(s, -1)) != cudaSuccess) return e;              \
  } while (0)

NormStepArgs norm_args(const LayeredModel* m) {
  NormStepArgs a{};
  a.ldx = a.ldh = a.ld_embed = m->widthp;
  a.width = m->cfg.width;
  a.eps = m->cfg.norm_eps;
  a.embed = m->embed.w;
  a.freq = m->freq;
  return a;
}

// out[rows, ldo] = x . w^T over rows in the storage type; gelu: exact gelu, result in the storage type
cudaError_t product(const LayeredModel* m, const Matrix& w, const void* x, float* out, void* out_h, int ldo, int n_out, int rows, bool gelu,
                    int* error_flag, bool pdl, cudaStream_t s) {
  if (m->bf16) {
    Bf16GemmArgs a{};
    a.x = x; a.w = w.w; a.w_tiled = w.tiled; a.out = out; a.out_h = out_h; a.ldo = ldo; a.error_flag = error_flag;
    a.m = rows; a.n = n_out; a.k = w.kp; a.gelu_erf = gelu ? 1 : 0;
    return launch_tc_gemm_bf16(a, pdl, s);
  }
  LinearArgs a{};
  a.w = static_cast<const float*>(w.w); a.x = static_cast<const float*>(x); a.out = out ? out : static_cast<float*>(out_h);
  a.m = rows; a.n = n_out; a.k = w.kp;
  if (ldo != n_out) return cudaErrorInvalidValue;  // the FP32 products store packed rows
  cudaError_t e = rows <= 16 ? launch_linear_decode(a, EPI_NONE, false, s, nullptr) : launch_gemm_f32(a, EPI_NONE, s);
  if (e == cudaSuccess && gelu) e = launch_gelu_erf(a.out, (size_t)rows * n_out, false, s);
  return e;
}

}  // namespace

cudaError_t layered_enqueue_decode(pg_cache* c, int batch, int splits, cudaStream_t s, uint64_t* launches, StepProfiler* prof) {
  const pg_model* pm = c->model;
  const LayeredModel* m = pm->layered.get();
  LayeredCache* lc = c->layered.get();
  LayeredRows& r = lc->step;
  const int V = m->cfg.vocab, wp = m->widthp;
  // at most eight BF16 rows: products that stream the weights and make their own input rows; else row kernels and
  // tensor-core products (BF16) or FP32 products
  bool rows_path = m->bf16 && batch <= MAX_ROWS_LINEAR && rows_linear_supported(batch, m->max_y, false, 0) &&
                   rows_linear_supported(batch, m->embed.kp, true, 0) && (m->max_ff == 0 || rows_linear_supported(batch, m->max_ff, false, 0));
  const bool pdl = pm->use_pdl && (rows_path || m->bf16);
  const bool y_bf16 = m->bf16 && !rows_path;
  void* y = rows_path ? (void*)r.y32 : r.y;
  cudaError_t e;
  uint64_t n = 0;
  int cur = 0;               // x[cur] is the residual stream before the pending sublayer output
  const Norm* post = nullptr;  // norm of the pending sublayer output in r.yo (nullptr: none pending)
  bool embed = true;         // the residual stream is still the embedding of the step's tokens

  auto step_norm = [&](const Norm& pre) {
    NormStepArgs a = norm_args(m);
    if (embed) { a.ids = c->d_ids; a.pos = c->d_pos; }
    else a.x_in = r.x[cur];
    if (post) { a.y = r.yo; a.post_g = post->g; a.post_b = post->b; }
    if (embed || post) a.x_out = r.x[cur ^ 1];
    a.pre_g = pre.g; a.pre_b = pre.b;
    a.h = r.h;
    return a;
  };
  auto advanced = [&] {  // what step_norm wrote is the stream now
    if (embed || post) cur ^= 1;
    embed = false;
    post = nullptr;
  };
  // With a few rows every block of a product makes the normed rows itself; with more of them one row kernel is cheaper.
  const bool fuse_norm = batch <= 4;
  auto rows_linear = [&](const Matrix& w, const float* x, const NormStepArgs* norm, float* out, int ldo, int n_out, int epi, float* pv, int* pi,
                         int* grid) -> cudaError_t {
    RowsLinearArgs a{};
    a.w = w.w; a.x = x; a.ldx = w.kp; a.out = out; a.ldo = ldo; a.m = batch; a.n = n_out; a.k = w.kp; a.epilogue = epi;
    if (norm && fuse_norm) {
      a.fuse_norm = 1;
      a.norm = *norm;
    } else if (norm) {
      NormStepArgs na = *norm;
      na.h32 = r.h32;
      if ((e = launch_norm_step(na, batch, true, pdl, s)) != cudaSuccess) return e;
      ++n;
      a.x = r.h32;
    }
    a.part_val = pv; a.part_idx = pi;
    return launch_rows_linear(a, pdl, s, grid);
  };

  for (const DevLayer& l : m->layers) {
    if (rows_path) {
      const NormStepArgs a = step_norm(l.norm1);
      PG_L(B_QKV, rows_linear(l.in, nullptr, &a, r.p, l.in.np, l.in.np, ROWS_NONE, nullptr, nullptr, nullptr));
    } else {
      PG_L(B_LAYER_NORM, launch_norm_step(step_norm(l.norm1), batch, m->bf16, pdl, s));
      PG_L(B_QKV, product(m, l.in, r.h, r.p, nullptr, l.in.np, l.in.np, batch, false, c->d_error, pdl, s));
    }
    advanced();
    for (const DevBranch& b : l.branches) {
      const size_t off = (size_t)b.y_off * (y_bf16 ? 2 : 4);
      if (b.kind == BranchSpec::ATTENTION) {
        AttentionStepArgs a{};
        a.l = b.attn; a.p = r.p; a.ldp = l.in.np; a.pool = lc->pools[b.pool]; a.page_table = c->tables[b.table].d_table;
        a.pos = c->d_pos; a.part = lc->attn_part; a.counters = lc->attn_counters;
        a.y = static_cast<char*>(y) + off; a.ldy = l.out.kp; a.batch = batch; a.splits = splits;
        PG_L(B_ATTN, launch_attention_step(a, m->bf16, y_bf16, pdl, s));
      } else {
        RecurrenceStepArgs a{};
        a.l = b.rec; a.p = r.p; a.ldp = l.in.np; a.state = lc->states[b.state]; a.pos = c->d_pos;
        a.y = static_cast<char*>(y) + off; a.ldy = l.out.kp; a.batch = batch;
        PG_L(B_ATTN, launch_recurrence_step(a, y_bf16, pdl, s));
      }
    }
    if (rows_path) PG_L(B_ATTN_PROJ, rows_linear(l.out, r.y32, nullptr, r.yo, wp, wp, ROWS_NONE, nullptr, nullptr, nullptr));
    else PG_L(B_ATTN_PROJ, product(m, l.out, r.y, r.yo, nullptr, wp, wp, batch, false, c->d_error, pdl, s));
    post = &l.norm1b;
    if (!l.ff) continue;
    if (rows_path) {
      const NormStepArgs a = step_norm(l.norm2);
      PG_L(B_MLP_FC, rows_linear(l.up, nullptr, &a, r.ff32, l.down.kp, l.up.np, ROWS_GELU_ERF, nullptr, nullptr, nullptr));
      advanced();
      PG_L(B_MLP_PROJ, rows_linear(l.down, r.ff32, nullptr, r.yo, wp, wp, ROWS_NONE, nullptr, nullptr, nullptr));
    } else {
      PG_L(B_LAYER_NORM, launch_norm_step(step_norm(l.norm2), batch, m->bf16, pdl, s));
      advanced();
      PG_L(B_MLP_FC, product(m, l.up, r.h, nullptr, r.ff, l.down.kp, l.up.np, batch, true, c->d_error, pdl, s));
      PG_L(B_MLP_PROJ, product(m, l.down, r.ff, r.yo, nullptr, wp, wp, batch, false, c->d_error, pdl, s));
    }
    post = &l.norm2b;
  }
  FinalizeArgs fa{};
  fa.m = batch; fa.argmax_out = c->d_argmax; fa.next_ids = c->d_ids; fa.pos = c->d_pos;
  fa.token_log = c->d_token_log; fa.n_positions = pm->positions();
  if (rows_path && rows_linear_grid(batch, V, m->embed.kp) <= c->part_stride) {
    const NormStepArgs a = step_norm(m->final_norm);
    int grid = 0;
    PG_L(B_LOGITS, rows_linear(m->embed, nullptr, &a, c->step_wants_logits || prof ? c->logits : nullptr, V, V, ROWS_NONE, c->part_val,
                               c->part_idx, &grid));
    fa.part_val = c->part_val; fa.part_idx = c->part_idx; fa.parts = grid;
  } else {
    PG_L(B_LAYER_NORM, launch_norm_step(step_norm(m->final_norm), batch, m->bf16, pdl, s));
    PG_L(B_LOGITS, product(m, m->embed, r.h, c->logits, nullptr, V, V, batch, false, c->d_error, pdl, s));
    PG_L(B_LOGITS, launch_argmax_rows(c->logits, batch, V, c->d_argmax, s));
  }
  PG_L(B_OTHER, launch_finalize(fa, pdl, s));
  if (launches) *launches = n;
  return cudaSuccess;
}

// ------------------------------------------------------------------ portions
int layered_logits_buffer(pg_cache* c, size_t rows, float** out) {
  LayeredCache* lc = c->layered.get();
  if (int r = grow(&lc->logits, &lc->logit_rows, rows, (size_t)c->model->v() * sizeof(float))) return r;
  *out = lc->logits;
  return PG_OK;
}

namespace {

struct PortionDevice {
  const int *ids, *pos, *row_seq, *seq_start, *slot, *start_pos, *out_rows;
  std::vector<const int*> key_start;  // per page table
  std::vector<int> krows;
};

cudaError_t enqueue_portions(pg_cache* c, const PortionPlan& plan, const PortionDevice& d, float* logits, StepProfiler* prof, uint64_t* launches) {
  const LayeredModel* m = c->model->layered.get();
  LayeredCache* lc = c->layered.get();
  LayeredRows& r = lc->portion;
  cudaStream_t s = c->stream;
  const int rows = plan.rows(), wp = m->widthp, V = m->cfg.vocab;
  cudaError_t e;
  uint64_t n = 0;
  float* x = r.x[0];
  bool first = true;
  const Norm* post = nullptr;
  auto norm = [&](const Norm* pre) {
    NormStepArgs a = norm_args(m);
    if (first) { a.ids = d.ids; a.pos = d.pos; }
    else a.x_in = x;
    if (post) { a.y = r.yo; a.post_g = post->g; a.post_b = post->b; }
    if (first || post) a.x_out = x;
    if (pre) { a.pre_g = pre->g; a.pre_b = pre->b; a.h = r.h; }
    first = false;
    post = nullptr;
    return launch_norm_step(a, rows, m->bf16, false, s);
  };
  const int max_segs = (plan.max_len + segment_tokens(plan.max_len) - 1) / segment_tokens(plan.max_len);
  for (const DevLayer& l : m->layers) {
    PG_L(B_LAYER_NORM, norm(&l.norm1));
    PG_L(B_QKV, product(m, l.in, r.h, r.p, nullptr, l.in.np, l.in.np, rows, false, c->d_error, false, s));
    for (const DevBranch& b : l.branches) {
      void* y = static_cast<char*>(r.y) + (size_t)b.y_off * m->elem();
      if (b.kind == BranchSpec::ATTENTION) {
        AttentionPortionArgs a{};
        a.l = b.attn; a.p = r.p; a.ldp = l.in.np; a.rows = rows; a.nseq = plan.n(); a.max_len = plan.max_len; a.krows = d.krows[b.table];
        a.seq_start = d.seq_start; a.key_start = d.key_start[b.table]; a.seq_slot = d.slot; a.seq_pos = d.start_pos; a.row_seq = d.row_seq;
        a.pool = lc->pools[b.pool]; a.page_table = c->tables[b.table].d_table;
        a.q = lc->q; a.k = lc->k; a.v = lc->v; a.error_flag = c->d_error; a.y = y; a.ldy = l.out.kp;
        PG_L(B_ATTN, launch_attention_portion(a, m->bf16, s));
      } else {
        RecurrenceScanArgs a{};
        a.l = b.rec; a.p = r.p; a.ldp = l.in.np; a.rows = rows; a.nseq = plan.n();
        a.seq_start = d.seq_start; a.seq_slot = d.slot; a.seq_pos = d.start_pos; a.state = lc->states[b.state];
        a.decay = lc->decay; a.unit = lc->unit; a.rate = lc->rate; a.unit_next = lc->unit_next; a.pair = lc->pair;
        a.out_raw = lc->out_raw; a.error_flag = c->d_error;
        a.segments = lc->segments; a.seg_tokens = segment_tokens(plan.max_len);
        a.max_segs = recurrence_use_segments(b.rec, plan.n(), plan.max_len, max_segs) ? max_segs : 0;
        a.y = y; a.ldy = l.out.kp;
        PG_L(B_ATTN, launch_recurrence_scan(a, m->bf16, s));
      }
    }
    PG_L(B_ATTN_PROJ, product(m, l.out, r.y, r.yo, nullptr, wp, wp, rows, false, c->d_error, false, s));
    post = &l.norm1b;
    if (!l.ff) continue;
    PG_L(B_LAYER_NORM, norm(&l.norm2));
    PG_L(B_MLP_FC, product(m, l.up, r.h, nullptr, r.ff, l.down.kp, l.up.np, rows, true, c->d_error, false, s));
    PG_L(B_MLP_PROJ, product(m, l.down, r.ff, r.yo, nullptr, wp, wp, rows, false, c->d_error, false, s));
    post = &l.norm2b;
  }
  const int outs = (int)plan.out_rows.size();
  if (outs > 0) {
    PG_L(B_LAYER_NORM, norm(nullptr));
    NormStepArgs a = norm_args(m);
    a.x_in = x; a.row_index = d.out_rows; a.pre_g = m->final_norm.g; a.pre_b = m->final_norm.b; a.h = r.h;
    PG_L(B_LAYER_NORM, launch_norm_step(a, outs, m->bf16, false, s));
    PG_L(B_LOGITS, product(m, m->embed, r.h, logits, nullptr, V, V, outs, false, c->d_error, false, s));
  }
  if (launches) *launches = n;
  return cudaSuccess;
}

}  // namespace

int layered_run_portions(pg_cache* c, const PortionPlan& plan, float* logits, StepProfiler* prof) {
  const LayeredModel* m = c->model->layered.get();
  LayeredCache* lc = c->layered.get();
  const int rows = plan.rows(), ns = plan.n();
  PG_CUDA_TRY(cudaStreamSynchronize(c->stream));  // workspaces may be replaced below
  if (int r = alloc_rows(m, &lc->portion, std::max<size_t>(rows, 64), false)) return r;
  // key / value workspace rows per page table: the cached keys a sequence still sees, then its own
  PortionDevice d;
  std::vector<int> meta;
  auto put = [&](const std::vector<int>& v) {
    const size_t at = meta.size();
    meta.insert(meta.end(), v.begin(), v.end());
    return at;
  };
  const size_t o_ids = put(plan.ids), o_pos = put(plan.pos), o_rs = put(plan.row_seq), o_ss = put(plan.seq_start), o_sl = put(plan.slot),
               o_sp = put(plan.start_pos), o_or = put(plan.out_rows);
  std::vector<size_t> o_ks;
  size_t max_krows = rows;
  for (const PageTable& t : c->tables) {
    std::vector<int> ks(1, 0);
    for (int i = 0; i < ns; ++i) ks.push_back(ks.back() + plan.start_pos[i] % t.span + (plan.seq_start[i + 1] - plan.seq_start[i]));
    o_ks.push_back(put(ks));
    d.krows.push_back(ks.back());
    max_krows = std::max<size_t>(max_krows, ks.back());
  }
  if (int r = grow(&lc->meta, &lc->meta_ints, meta.size(), sizeof(int))) return r;
  size_t qe = 0, ke = 0, ve = 0, seg = 0;
  const int max_segs = (plan.max_len + segment_tokens(plan.max_len) - 1) / segment_tokens(plan.max_len);
  for (const DevLayer& l : m->layers)
    for (const DevBranch& b : l.branches) {
      if (b.kind == BranchSpec::ATTENTION) {
        qe = std::max<size_t>(qe, (size_t)b.attn.heads * b.attn.dimp);
        ke = std::max<size_t>(ke, (size_t)b.attn.kv_heads * b.attn.dimp);
        ve = std::max<size_t>(ve, (size_t)b.attn.kv_heads * b.attn.vdimp);
      } else if (recurrence_use_segments(b.rec, ns, plan.max_len, max_segs)) {
        seg = std::max(seg, recurrence_segment_floats(b.rec, ns, max_segs));
      }
    }
  if (qe) {
    if (int r = grow(&lc->q, &lc->q_rows, rows, qe * m->elem())) return r;
    if (max_krows > lc->k_rows) {
      size_t kr = lc->k_rows;
      if (int r = grow(&lc->k, &kr, max_krows, ke * m->elem())) return r;
      if (int r = grow(&lc->v, &lc->k_rows, max_krows, ve * m->elem())) return r;
    }
  }
  if (m->max_rec && (size_t)rows > lc->gate_rows) {
    size_t g = lc->gate_rows, h = g, o = g, x = g, y = g;
    if (int r = grow(&lc->unit_next, &x, rows, m->max_rec * sizeof(float))) return r;
    if (int r = grow(&lc->pair, &y, rows, m->max_rec_heads * 4 * sizeof(float))) return r;
    if (int r = grow(&lc->out_raw, &o, rows, m->max_rec_out * sizeof(float))) return r;
    if (int r = grow(&lc->decay, &g, rows, m->max_rec * sizeof(float))) return r;
    if (int r = grow(&lc->unit, &h, rows, m->max_rec * sizeof(float))) return r;
    if (int r = grow(&lc->rate, &lc->gate_rows, rows, m->max_rec * sizeof(float))) return r;
  }
  if (seg)
    if (int r = grow(&lc->segments, &lc->seg_floats, seg, sizeof(float))) return r;
  PG_CUDA_TRY(cudaMemcpyAsync(lc->meta, meta.data(), meta.size() * sizeof(int), cudaMemcpyHostToDevice, c->stream));
  PG_CUDA_TRY(cudaStreamSynchronize(c->stream));  // `meta` is a pageable temporary
  d.ids = lc->meta + o_ids; d.pos = lc->meta + o_pos; d.row_seq = lc->meta + o_rs; d.seq_start = lc->meta + o_ss;
  d.slot = lc->meta + o_sl; d.start_pos = lc->meta + o_sp; d.out_rows = lc->meta + o_or;
  for (size_t o : o_ks) d.key_start.push_back(lc->meta + o);
  PG_CUDA_TRY(enqueue_portions(c, plan, d, logits, prof, nullptr));
  return PG_OK;
}

}  // namespace pg
