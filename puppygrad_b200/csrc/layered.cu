// Models described layer by layer (see design.h): device weights, per-cache state (key / value pages, recurrent
// states), the decode step and the pass over portions of prompts. A layer is one of
//   x += post(mixer(norm(x)));  x += post(down(act(up(norm(x)))))     (post: another norm, or nothing)
//   h = norm(x);  x += mixer(h) + down(act(up(h)))
// the feed-forward being optional, where the mixer is one branch or the scaled sum of several. All branches of a layer share one
// input projection (their weight rows are concatenated) and one output projection (their columns are concatenated, the branch
// scales applied to the columns before it); where the feed-forward reads the same normed rows, its rows and columns are part of
// the two as well.
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
  AttentionLayer attn{};  // latent attention: the heads against the latent rows
  RecurrenceLayer rec{};
  int pool = -1;       // attention: index of the key / value pool and ...
  int table = -1;      // ... of the page table (by distinct key lifetime)
  int state = -1;      // recurrence: index of the state array (and of the convolution inputs)
  int rot = -1, v_rot = -1;  // indices of the rotations
  bool heads_step = false;   // decode: all heads of a sequence in one block ...
  bool heads_tc = false;     // ... on the tensor cores
  // second step of two-step projections, over columns mid_off.. of the first ones' result (normed where mid_norm is set)
  Matrix mid;
  int mid_off = 0, mid_cols = 0;
  float* mid_norm = nullptr;
  // latent attention: the heads' own keys and values of a portion, and the two products per head that replace them in a step
  AttentionLayer full{};
  Matrix up_kv;
  void *to_latent = nullptr, *from_latent = nullptr;  // [heads][dim][attn.dimp], [heads][kv_rank][full.vdimp]
  Matrix to_latent_rows, from_latent_rows;            // the same for the tensor cores, 128 rows and their multiples per head
};
struct DevLayer {
  Norm norm1, norm1b, norm2, norm2b;
  Matrix in, out, up, down;
  std::vector<DevBranch> branches;
  bool ff = false;
  ActArgs act{};
  // feed-forward beside the mixer: `up` is the rows of `in` from in_mixer on, its result columns ff_off.. of the out product's input
  bool parallel = false;
  int in_mixer = 0, ff_off = 0;
  int ldp = 0;  // row pitch of the input projection
};
struct Rotation {
  int dims = 0;
  double base = 0;
  double* freq = nullptr;
};

}  // namespace

struct LayeredModel {
  LayeredConfig cfg;
  bool bf16 = false;
  int widthp = 0;  // row pitch of the residual stream and of normed rows
  Matrix embed, head;  // token embedding, output projection (the same where they are tied)
  Norm final_norm;
  double* freq = nullptr;
  std::vector<DevLayer> layers;
  int max_in = 0, max_y = 0, max_ff = 0, max_rec = 0;  // widest projection, mixer output, hidden row, heads * dim ...
  int max_rec_out = 0, max_rec_heads = 0;                  // ... heads * vdim and heads of a recurrence
  int max_mid_k = 0, max_mid = 0, max_latent = 0, max_wide = 0;  // widest second-step input and output; heads * latent row, heads * query
  int n_pools = 0, n_states = 0;
  bool tc_rotations = false;  // a step needs the angles of its rows
  bool channel_rules = false;  // some recurrence is a channel delta rule
  std::vector<KeyLife> lives;  // one page table each
  std::vector<Rotation> rotations;
  std::vector<void*> allocations;
  uint64_t weight_bytes = 0;
  int device = 0;
  size_t elem() const { return bf16 ? 2 : 4; }
  size_t rotation_pairs() const {
    size_t n = 0;
    for (const Rotation& r : rotations) n += r.dims / 2;
    return n;
  }
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
  float *h32 = nullptr, *y32 = nullptr, *ff32 = nullptr, *t32 = nullptr;  // decode with at most 8 BF16 rows: FP32 product inputs
  void* t = nullptr;                                // second-step input, storage type
  float* z = nullptr;                               // ... and output
  float *q_latent = nullptr, *o_latent = nullptr;   // decode: queries against wide key rows, sums of latent rows
  float2* angles = nullptr;                         // decode: (cos, sin) of every rotation, one after the other
  std::vector<void**> buffers() {
    return {(void**)&x[0], (void**)&x[1], (void**)&p,   (void**)&yo, &h, &y, &ff, (void**)&h32, (void**)&y32, (void**)&ff32,
            (void**)&t32,  &t,            (void**)&z,   (void**)&q_latent, (void**)&o_latent, (void**)&angles};
  }
};

struct LayeredCache {
  std::vector<void*> pools;
  std::vector<float*> states, taps;
  LayeredRows step, portion;
  float* attn_part = nullptr;
  unsigned* attn_counters = nullptr;
  // portion workspaces (grow-only)
  float *decay = nullptr, *unit = nullptr, *rate = nullptr, *unit_next = nullptr, *pair = nullptr, *out_raw = nullptr, *segments = nullptr, *vals = nullptr, *writes = nullptr, *quad_decay = nullptr,
        *quads = nullptr;
  float2* angles = nullptr;
  void *q = nullptr, *k = nullptr, *v = nullptr;
  int* meta = nullptr;
  float* logits = nullptr;
  size_t q_rows = 0, k_rows = 0, seg_floats = 0, meta_ints = 0, logit_rows = 0, gate_rows = 0, angle_rows = 0, channel_rows = 0, quad_rows = 0;
  ~LayeredCache() {
    for (void* p : pools) cudaFree(p);
    for (float* p : states) cudaFree(p);
    for (float* p : taps)
      if (p) cudaFree(p);
    for (LayeredRows* r : {&step, &portion})
      for (void** p : r->buffers())
        if (*p) cudaFree(*p);
    for (void* p : {(void*)attn_part, (void*)attn_counters, (void*)decay, (void*)unit, (void*)rate, (void*)unit_next, (void*)pair, (void*)out_raw, (void*)segments, (void*)vals, (void*)writes, (void*)quad_decay, (void*)quads, (void*)angles, q, k, v,
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
    return m->cfg.norm_kind == NORM_LAYER ? vec(name + ".b", m->widthp, &n->b) : PG_OK;
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
  // [rows, cols] in the storage type with rows of ld, no tiled copy
  int packed(const std::vector<float>& v, int rows, int cols, int ld, void** out) {
    if (int r = alloc((size_t)rows * ld * m->elem(), out)) return r;
    m->weight_bytes += (uint64_t)rows * cols * m->elem();
    if (!m->bf16) {
      PG_CUDA_TRY(cudaMemcpy2D(*out, (size_t)ld * 4, v.data(), (size_t)cols * 4, (size_t)cols * 4, rows, cudaMemcpyHostToDevice));
      return PG_OK;
    }
    float* tmp = nullptr;
    PG_CUDA_TRY(cudaMalloc(&tmp, v.size() * sizeof(float)));
    cudaError_t e = cudaMemcpy(tmp, v.data(), v.size() * sizeof(float), cudaMemcpyHostToDevice);
    if (e == cudaSuccess) e = launch_pack_bf16(tmp, *out, rows, cols, rows, ld, 0);
    if (e == cudaSuccess) e = cudaDeviceSynchronize();
    cudaFree(tmp);
    PG_CUDA_TRY(e);
    return PG_OK;
  }
  // Index of a rotation of the first `dims` entries of a row.
  int rotation(int dims, double base, int* index) {
    *index = -1;
    if (dims < 2) return PG_OK;
    for (size_t i = 0; i < m->rotations.size(); ++i)
      if (m->rotations[i].dims == dims && m->rotations[i].base == base) *index = (int)i;
    if (*index >= 0) return PG_OK;
    Rotation r{dims, base, nullptr};
    std::vector<double> f(dims / 2);
    for (size_t i = 0; i < f.size(); ++i) f[i] = std::pow(base, -2.0 * (double)i / (double)dims);
    if (int e = alloc(f.size() * sizeof(double), (void**)&r.freq)) return e;
    PG_CUDA_TRY(cudaMemcpy(r.freq, f.data(), f.size() * sizeof(double), cudaMemcpyHostToDevice));
    *index = (int)m->rotations.size();
    m->rotations.push_back(r);
    return PG_OK;
  }
  int table(const KeyLife& life) {
    auto it = std::find(m->lives.begin(), m->lives.end(), life);
    const int i = (int)(it - m->lives.begin());
    if (it == m->lives.end()) m->lives.push_back(life);
    return i;
  }
  // [n, r] -> [r, n]
  int transposed(const std::string& name, int n, int r, float** out) {
    const std::vector<float> v = tensor_f32(file, name);
    std::vector<float> t(v.size());
    for (int i = 0; i < n; ++i)
      for (int j = 0; j < r; ++j) t[(size_t)j * n + i] = v[(size_t)i * r + j];
    return upload(t, 0, out);
  }
};

// Rows of `heads` blocks of n, each block padded to np rows of zeros.
std::vector<float> pad_heads(const std::vector<float>& v, int heads, int n, int np, int cols) {
  std::vector<float> out((size_t)heads * np * cols, 0.f);
  for (int h = 0; h < heads; ++h)
    std::copy(v.begin() + (size_t)h * n * cols, v.begin() + (size_t)(h + 1) * n * cols, out.begin() + (size_t)h * np * cols);
  return out;
}

int build_layer(Builder& b, const LayerSpec& spec, const std::string& p, int page_tokens, int max_context, DevLayer* d) {
  LayeredModel* m = b.m;
  const int W = m->cfg.width;
  const float eps = m->cfg.norm_eps;
  if (int r = b.norm(p + "norm1", &d->norm1)) return r;
  if (m->cfg.post_norms)
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
      a.dimp = align_to(s.dim, 8); a.vdimp = a.vrow = align_to(s.vdim, 8);
      a.life.span = s.chunk > 0 ? std::min(s.chunk, max_context) : max_context;
      if (s.window > 0) {
        a.life.window = s.window;
        a.life.keep = std::min(s.keep_first, max_context);
        a.life.span = (int)std::min<long long>((long long)a.life.keep + s.window, max_context);
      }
      a.off_gate = -1;
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
      float* f = nullptr;
      auto optional = [&](bool has, const char* name, const float** out) -> int {
        if (!has) return PG_OK;
        const int r = b.vec(t + name, 0, &f);
        *out = f;
        return r;
      };
      if (int r = optional(s.bias, "q.b", &a.q_bias)) return r;
      if (int r = optional(s.bias, "k.b", &a.k_bias)) return r;
      if (int r = optional(s.bias, "v.b", &a.v_bias)) return r;
      if (int r = optional(s.head_mix, "talk", &a.mix)) return r;
      if (int r = optional(s.sink, "sink", &a.sink)) return r;
      if (int r = b.rotation(s.rot_dims, s.rot_base, &br.rot)) return r;
      if (br.rot >= 0) {
        a.rot_dims = s.rot_dims;
        a.rot_freq = m->rotations[br.rot].freq;
      }
      if (s.v_rot) {
        if (int r = b.rotation(s.vdim, s.rot_base, &br.v_rot)) return r;
        a.v_rot = 1;
        a.v_freq = m->rotations[br.v_rot].freq;
      }
      br.heads_step = a.life.window > 0 || a.mix || a.sink || a.q_bias || a.rot_dims || a.v_rot;
      a.wide = br.heads_step ? 1 : 0;
      a.scale = s.scale; a.eps = eps; a.out_scale = bs.scale;
      a.page_tokens = page_tokens;
      a.pages_per_seq = (a.life.span + page_tokens - 1) / page_tokens;
      br.table = b.table(a.life);
      m->max_wide = std::max(m->max_wide, s.heads * attention_q_width(a));
      br.pool = m->n_pools++;
      br.heads_tc = m->bf16 && br.heads_step && attention_heads_tc_supported(a);
      m->tc_rotations = m->tc_rotations || (br.heads_tc && (br.rot >= 0 || br.v_rot >= 0));
      if (br.heads_step ? !attention_heads_supported(a) : !attention_supported(a))
        return set_error(PG_INVALID_CONFIG, p + bs.prefix + ": " + std::to_string(s.heads / s.kv_heads) + " query heads per key head of size " +
                                                std::to_string(s.dim) + " exceed what the decode kernel holds");
    } else if (bs.kind == BranchSpec::LATENT) {
      const AttentionSpec& s = bs.attn;
      AttentionLayer &a = br.attn, &e = br.full;
      const int H = s.heads;
      a.heads = H; a.kv_heads = 1; a.dim = a.vdim = s.kv_rank;
      a.dimp = a.vdimp = align_to(s.kv_rank, K_ALIGN);  // a latent row is the input of a product
      a.life.span = max_context;
      a.off_q = part(t + "dq", s.q_rank);
      a.off_k = part(t + "dkv", s.kv_rank);
      a.off_gate = s.head_gate ? part(t + "g", H) : -1;
      float* f = nullptr;
      if (int r = b.vec(t + "dkv.norm", a.dimp, &f)) return r;
      a.k_norm = f;
      a.scale = s.scale; a.eps = eps; a.out_scale = bs.scale;
      a.page_tokens = page_tokens;
      a.pages_per_seq = (a.life.span + page_tokens - 1) / page_tokens;
      br.table = b.table(a.life);
      br.pool = m->n_pools++;
      br.heads_step = true;
      a.wide = 1;
      br.heads_tc = m->bf16 && attention_heads_tc_supported(a);
      e = a;
      e.kv_heads = H; e.dim = s.dim; e.vdim = s.vdim;
      e.dimp = align_to(s.dim, 8); e.vdimp = e.vrow = align_to(s.vdim, 8);
      br.mid_off = a.off_q; br.mid_cols = s.q_rank;
      if (int r = b.vec(t + "dq.norm", align_to(s.q_rank, K_ALIGN), &br.mid_norm)) return r;
      if (int r = b.matrix(pad_heads(tensor_f32(b.file, t + "uq"), H, s.dim, e.dimp, s.q_rank), H * e.dimp, s.q_rank, N_ALIGN, &br.mid)) return r;
      const std::vector<float> uk = tensor_f32(b.file, t + "uk"), uv = tensor_f32(b.file, t + "uv");
      if (int r = b.packed(uk, H * s.dim, s.kv_rank, a.dimp, &br.to_latent)) return r;
      std::vector<float> uvt((size_t)H * s.kv_rank * s.vdim);
      for (int h = 0; h < H; ++h)
        for (int c = 0; c < s.vdim; ++c)
          for (int j = 0; j < s.kv_rank; ++j) uvt[((size_t)h * s.kv_rank + j) * s.vdim + c] = uv[((size_t)h * s.vdim + c) * s.kv_rank + j];
      if (int r = b.packed(uvt, H * s.kv_rank, s.vdim, e.vdimp, &br.from_latent)) return r;
      std::vector<float> kv = pad_heads(uk, H, s.dim, e.dimp, s.kv_rank), v = pad_heads(uv, H, s.vdim, e.vdimp, s.kv_rank);
      kv.insert(kv.end(), v.begin(), v.end());
      const uint64_t bytes = m->weight_bytes;  // a step does not read the copy for prompts
      if (int r = b.matrix(kv, H * (e.dimp + e.vdimp), s.kv_rank, N_ALIGN, &br.up_kv)) return r;
      if (m->bf16) {
        std::vector<float> ukt((size_t)H * s.kv_rank * s.dim);
        for (int h = 0; h < H; ++h)
          for (int c = 0; c < s.dim; ++c)
            for (int j = 0; j < s.kv_rank; ++j) ukt[((size_t)h * s.kv_rank + j) * s.dim + c] = uk[((size_t)h * s.dim + c) * s.kv_rank + j];
        const int kn = align_to(a.dimp, 128), vn = align_to(s.vdim, 128);
        if (int r = b.matrix(pad_heads(ukt, H, s.kv_rank, kn, s.dim), H * kn, s.dim, 128, &br.to_latent_rows)) return r;
        if (int r = b.matrix(pad_heads(uv, H, s.vdim, vn, s.kv_rank), H * vn, s.kv_rank, 128, &br.from_latent_rows)) return r;
      }
      m->weight_bytes = bytes;
      m->max_latent = std::max(m->max_latent, H * a.dimp);
      m->max_wide = std::max(m->max_wide, H * a.dimp);
      if (!attention_heads_supported(a))
        return set_error(PG_INVALID_CONFIG, p + bs.prefix + ": " + std::to_string(H) + " heads with latent rows of " + std::to_string(s.kv_rank) +
                                                " exceed what the decode kernel holds");
    } else if (bs.rec.kind == RECUR_CHANNEL) {
      const RecurrenceSpec& s = bs.rec;
      RecurrenceLayer& a = br.rec;
      const int K = s.heads * s.dim, V = s.heads * s.vdim, Q = s.kv_heads * s.dim;
      a.kind = s.kind; a.heads = s.heads; a.kv_heads = s.kv_heads; a.dim = s.dim; a.vdim = s.vdim; a.dvp = align_to(s.vdim, 4);
      a.off_q = part(t + "q", Q);
      a.off_k = part(t + "k", Q);
      a.off_v = part(t + "v", V);
      a.taps = s.conv;
      a.channels = a.off_v + align_to(V, 4) - a.off_q;
      std::vector<float> conv((size_t)s.conv * a.channels, 0.f);
      const struct { const char* name; int off, n; } parts[] = {{"q.conv", a.off_q, Q}, {"k.conv", a.off_k, Q}, {"v.conv", a.off_v, V}};
      for (const auto& c : parts) {
        const std::vector<float> w = tensor_f32(b.file, t + c.name);
        for (int i = 0; i < c.n; ++i)
          for (int j = 0; j < s.conv; ++j) conv[(size_t)j * a.channels + c.off - a.off_q + i] = w[(size_t)i * s.conv + j];
      }
      float* f = nullptr;
      if (int r = b.upload(conv, 0, &f)) return r;
      a.conv = f;
      a.off_b = part(t + "b", s.heads);
      std::vector<float> log = tensor_f32(b.file, t + "A_log");
      for (float& v : log) v = (float)-std::exp((double)v);
      if (int r = b.upload(log, 0, &f)) return r;
      a.neg_a = f;
      if (int r = b.vec(t + "dt_bias", 0, &f)) return r;
      a.b2 = f;
      if (int r = b.vec(t + "norm", 0, &f)) return r;
      a.norm = f;
      a.q_scale = (float)(1.0 / std::sqrt((double)s.dim));
      a.eps = eps;
      a.out_scale = bs.scale;
      // second steps of decay and gate as one product: their matrices on the diagonal
      br.mid_off = part(t + "a1", s.rank);
      br.mid_cols = part(t + "g1", s.rank2) + s.rank2 - br.mid_off;
      const std::vector<float> a2 = tensor_f32(b.file, t + "a2"), g2 = tensor_f32(b.file, t + "g2");
      std::vector<float> mid((size_t)(K + V) * br.mid_cols, 0.f);
      for (int i = 0; i < K; ++i) std::copy(a2.begin() + (size_t)i * s.rank, a2.begin() + (size_t)(i + 1) * s.rank, mid.begin() + (size_t)i * br.mid_cols);
      for (int i = 0; i < V; ++i)
        std::copy(g2.begin() + (size_t)i * s.rank2, g2.begin() + (size_t)(i + 1) * s.rank2,
                  mid.begin() + (size_t)(K + i) * br.mid_cols + br.mid_cols - s.rank2);
      if (int r = b.matrix(mid, K + V, br.mid_cols, N_ALIGN, &br.mid)) return r;
      m->channel_rules = true;
      br.state = m->n_states++;
      m->max_rec = std::max(m->max_rec, K);
      m->max_rec_out = std::max(m->max_rec_out, V);
      m->max_rec_heads = std::max(m->max_rec_heads, s.heads);
    } else {
      const RecurrenceSpec& s = bs.rec;
      RecurrenceLayer& a = br.rec;
      const int K = s.heads * s.dim, V = s.heads * s.vdim;
      const bool delta = s.kind == RECUR_DELTA;
      a.kind = s.kind; a.heads = a.kv_heads = s.heads; a.dim = s.dim; a.vdim = s.vdim; a.dvp = align_to(s.vdim, 4); a.rank = s.rank;
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
  for (const DevBranch& br : d->branches) {
    m->max_mid_k = std::max(m->max_mid_k, br.mid.kp);
    m->max_mid = std::max(m->max_mid, br.mid.np);
  }
  d->parallel = m->cfg.parallel_ff && spec.ff > 0;
  d->act.kind = m->cfg.activation;
  if (spec.ff > 0 && m->cfg.activation == ACT_XIELU) {
    const std::vector<float> pq = tensor_f32(b.file, p + "mlp.act");
    auto softplus = [](double z) { return std::max(z, 0.0) + std::log1p(std::exp(-std::fabs(z))); };
    d->act.a = (float)softplus(pq[0]);
    d->act.b = (float)(0.5 + softplus(pq[1]));
  }
  d->in_mixer = align_to(rows, N_ALIGN);
  if (d->parallel) {
    in.resize((size_t)d->in_mixer * W, 0.f);
    const std::vector<float> up = tensor_f32(b.file, p + "mlp.up");
    in.insert(in.end(), up.begin(), up.end());
    rows = d->in_mixer + spec.ff;
  }
  if (int r = b.matrix(in, rows, W, N_ALIGN, &d->in)) return r;
  in.clear();
  in.shrink_to_fit();
  d->ldp = d->parallel && m->bf16 ? d->in_mixer : d->in.np;
  if (d->parallel) {  // the same weights, seen as two matrices
    d->up = d->in;
    d->up.w = static_cast<char*>(d->in.w) + (size_t)d->in_mixer * d->in.kp * m->elem();
    d->up.tiled = nullptr;
    d->up.n = spec.ff;
    d->up.np = d->in.np - d->in_mixer;
  }
  // output projections of the branches (and the feed-forward's) side by side: [W, sum of the columns]
  d->ff_off = align_to(y_cols, K_ALIGN);
  const int cols = d->parallel ? d->ff_off + spec.ff : y_cols;
  std::vector<float> out((size_t)W * cols, 0.f);
  auto columns = [&](const std::string& name, int n, int off) {
    const std::vector<float> v = tensor_f32(b.file, name);
    for (int r = 0; r < W; ++r) std::copy(v.begin() + (size_t)r * n, v.begin() + (size_t)(r + 1) * n, out.begin() + (size_t)r * cols + off);
  };
  for (size_t i = 0; i < spec.branches.size(); ++i)
    columns(p + spec.branches[i].prefix + ".o", spec.branches[i].out_dim(), d->branches[i].y_off);
  if (d->parallel) columns(p + "mlp.down", spec.ff, d->ff_off);
  if (int r = b.matrix(out, W, cols, K_ALIGN, &d->out)) return r;
  m->max_in = std::max(m->max_in, d->ldp);
  m->max_y = std::max(m->max_y, d->out.kp);
  if (spec.ff > 0 && !d->parallel) {
    d->ff = true;
    if (int r = b.norm(p + "norm2", &d->norm2)) return r;
    if (m->cfg.post_norms)
      if (int r = b.norm(p + "norm2b", &d->norm2b)) return r;
    if (int r = b.matrix(p + "mlp.up", spec.ff, W, K_ALIGN, &d->up)) return r;
    if (int r = b.matrix(p + "mlp.down", W, spec.ff, K_ALIGN, &d->down)) return r;
    m->max_ff = std::max(m->max_ff, d->down.kp);
  }
  return PG_OK;
}

int alloc_rows(const LayeredModel* m, LayeredRows* r, size_t rows, bool step) {
  if (rows <= r->rows) return PG_OK;
  for (void** p : r->buffers()) {
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
  if (m->max_mid) {
    if (int q = get(&r->t, rows * m->max_mid_k * e)) return q;
    if (int q = get((void**)&r->z, rows * m->max_mid * 4)) return q;
  }
  if (step && m->max_wide)
    if (int q = get((void**)&r->q_latent, rows * m->max_wide * 4)) return q;
  if (step && m->rotation_pairs())
    if (int q = get((void**)&r->angles, rows * m->rotation_pairs() * sizeof(float2))) return q;
  if (step && m->max_latent) {
    if (int q = get((void**)&r->o_latent, rows * m->max_latent * 4)) return q;
  }
  if (step && m->bf16) {
    const size_t n = std::min<size_t>(rows, MAX_ROWS_LINEAR);
    if (int q = get((void**)&r->h32, n * wp * 4)) return q;
    if (int q = get((void**)&r->y32, n * m->max_y * 4)) return q;
    if (int q = get((void**)&r->ff32, n * std::max(m->max_ff, 1) * 4)) return q;
    if (int q = get((void**)&r->t32, n * std::max(m->max_mid_k, 1) * 4)) return q;
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
  m->head = m->embed;
  if (!cfg.tied_head) {
    m->weight_bytes = 0;  // a step reads a few rows of the embedding
    if (int r = b.matrix("head", cfg.vocab, cfg.width, 1, &m->head)) return r;
  }
  if (int r = b.norm("final.norm", &m->final_norm)) return r;
  if (cfg.sinusoids) {
    std::vector<double> freq((cfg.width + 1) / 2 + 2);
    for (size_t i = 0; i < freq.size(); ++i) freq[i] = std::pow(10000.0, -2.0 * (double)i / (double)cfg.width);
    if (int r = b.alloc(freq.size() * sizeof(double), (void**)&m->freq)) return r;
    PG_CUDA_TRY(cudaMemcpy(m->freq, freq.data(), freq.size() * sizeof(double), cudaMemcpyHostToDevice));
  }
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
      if (b.kind == BranchSpec::RECURRENCE) n += (recurrence_state_floats(b.rec) + recurrence_tap_floats(b.rec)) * sizeof(float);
  return n;
}

// ------------------------------------------------------------------ cache
int layered_cache_init(pg_cache* c) {
  const LayeredModel* m = c->model->layered.get();
  auto lc = std::make_shared<LayeredCache>();
  const size_t B = c->max_batch;
  c->tables.resize(m->lives.size());
  for (size_t i = 0; i < m->lives.size(); ++i)
    if (int r = page_table_init(&c->tables[i], c->max_batch, m->lives[i].span, c->model->backend.page_tokens, c->stream)) return r;
  lc->pools.assign(m->n_pools, nullptr);
  lc->states.assign(m->n_states, nullptr);
  lc->taps.assign(m->n_states, nullptr);
  size_t part = 0, counters = 0;
  for (const DevLayer& l : m->layers)
    for (const DevBranch& b : l.branches) {
      if (b.kind != BranchSpec::RECURRENCE) {
        const size_t bytes = (size_t)c->tables[b.table].num_pages * attention_page_elems(b.attn) * m->elem();
        PG_CUDA_TRY(cudaMalloc(&lc->pools[b.pool], bytes));
        PG_CUDA_TRY(cudaMemsetAsync(lc->pools[b.pool], 0, bytes, c->stream));
        part = std::max(part, B * b.attn.heads * MAX_SPLITS * attention_part_floats(b.attn));
        counters = std::max(counters, B * std::max(b.attn.kv_heads, b.attn.heads));
      } else {
        const size_t bytes = B * recurrence_state_floats(b.rec) * sizeof(float);
        PG_CUDA_TRY(cudaMalloc(&lc->states[b.state], bytes));
        PG_CUDA_TRY(cudaMemsetAsync(lc->states[b.state], 0, bytes, c->stream));
        if (const size_t taps = B * recurrence_tap_floats(b.rec) * sizeof(float)) {
          PG_CUDA_TRY(cudaMalloc(&lc->taps[b.state], taps));
          PG_CUDA_TRY(cudaMemsetAsync(lc->taps[b.state], 0, taps, c->stream));
        }
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
  int span = 0, kv = 1 << 30, piece = 128, most = 8;
  bool tc = false;
  for (const DevLayer& l : m->layered->layers)
    for (const DevBranch& b : l.branches)
      if (b.kind != BranchSpec::RECURRENCE) {
        span = std::max(span, std::min(b.attn.life.span, max_len));
        kv = std::min(kv, b.heads_step ? 1 : b.attn.kv_heads);
        tc = tc || b.heads_tc;
        if (b.heads_step) {  // one block would hold all heads: shorter parts, more of them
          piece = 32;
          most = MAX_SPLITS;
        }
      }
  if (!span) return 1;
  int s = 1;
  if (tc) {  // tiles of keys; every layer chooses its parts from them (branch_splits)
    while (s * 128 < span) s *= 2;
    return s;
  }
  const int by_fill = (2 * m->num_sms + batch * kv - 1) / (batch * kv), by_len = (span + piece - 1) / piece;
  while (s * 2 <= std::min(std::min(by_fill, by_len), most)) s *= 2;
  return s;
}

namespace {

// The parts of a branch's keys in a step, from what layered_choose_splits returned.
int branch_splits(const pg_model* m, const DevBranch& b, int batch, int chosen) {
  if (m->backend.attn_splits > 0) return chosen;
  if (!b.heads_tc) return std::min(chosen, MAX_SPLITS);
  return attention_heads_tc_splits(b.attn, batch, std::min(chosen, (b.attn.life.span + 127) / 128), m->num_sms);
}

}  // namespace

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
  a.ldx = a.ldh = a.ld_in = a.ld_embed = m->widthp;
  a.width = m->cfg.width;
  a.eps = m->cfg.norm_eps;
  a.embed = m->embed.w;
  a.embed_scale = m->cfg.embed_scale;
  a.freq = m->freq;
  a.norm = m->cfg.norm_kind;
  return a;
}

// The input rows of a branch's second-step product: columns of the first one's result, normed or as they are.
NormStepArgs mid_args(const LayeredModel* m, const DevLayer& l, const DevBranch& b, const float* p) {
  NormStepArgs a{};
  a.x_in = p + b.mid_off;
  a.ld_in = l.ldp;
  a.ldx = a.ldh = b.mid.kp;
  a.width = b.mid_cols;
  a.eps = m->cfg.norm_eps;
  a.pre_g = b.mid_norm;
  a.norm = b.mid_norm ? (int)NORM_RMS : NORM_COPY;
  return a;
}

// out[rows, ldo] = x . w^T over rows in the storage type; act: activation, result in the storage type
cudaError_t product(const LayeredModel* m, const Matrix& w, const void* x, float* out, void* out_h, int ldo, int n_out, int rows, const ActArgs* act,
                    int* error_flag, bool pdl, cudaStream_t s) {
  if (m->bf16) {
    Bf16GemmArgs a{};
    a.x = x; a.w = w.w; a.w_tiled = w.tiled; a.out = out; a.out_h = out_h; a.ldo = ldo; a.error_flag = error_flag;
    a.m = rows; a.n = n_out; a.k = w.kp;
    if (act) a.act = *act;
    return launch_tc_gemm_bf16(a, pdl, s);
  }
  LinearArgs a{};
  a.w = static_cast<const float*>(w.w); a.x = static_cast<const float*>(x); a.out = out ? out : static_cast<float*>(out_h);
  a.m = rows; a.n = n_out; a.k = w.kp;
  if (ldo != n_out) return cudaErrorInvalidValue;  // the FP32 products store packed rows
  cudaError_t e = rows <= 16 ? launch_linear_decode(a, EPI_NONE, false, s, nullptr) : launch_gemm_f32(a, EPI_NONE, s);
  if (e == cudaSuccess && act) e = launch_activation(a.out, ldo, a.out, ldo, rows, n_out, *act, false, s);
  return e;
}

// The input projection of a layer over rows in the storage type; where the feed-forward is part of it, its hidden row goes
// to y (the out product's input).
cudaError_t in_product(const LayeredModel* m, const DevLayer& l, const void* h, float* p, void* y, int rows, int* error_flag, bool pdl, cudaStream_t s,
                       uint64_t* n) {
  if (!l.parallel) return product(m, l.in, h, p, nullptr, l.ldp, l.in.np, rows, nullptr, error_flag, pdl, s);
  cudaError_t e;
  void* hidden = static_cast<char*>(y) + (size_t)l.ff_off * m->elem();
  if (!m->bf16) {
    e = product(m, l.in, h, p, nullptr, l.ldp, l.in.np, rows, nullptr, error_flag, pdl, s);
    ++*n;
    return e != cudaSuccess ? e : launch_activation(p + l.in_mixer, l.ldp, static_cast<float*>(hidden), l.out.kp, rows, l.up.n, l.act, false, s);
  }
  if (gemm_bf16_rows_kernel(rows, l.in.kp)) {
    Bf16GemmArgs a{};
    a.x = h; a.w = l.in.w; a.w_tiled = l.in.tiled; a.out = p; a.ldo = l.ldp; a.error_flag = error_flag;
    a.m = rows; a.n = l.in.n; a.k = l.in.kp;
    a.act = l.act; a.act_from = l.in_mixer; a.out_act = hidden; a.ldo_act = l.out.kp;
    return launch_tc_gemm_bf16(a, pdl, s);
  }
  if ((e = product(m, l.in, h, p, nullptr, l.ldp, l.in_mixer, rows, nullptr, error_flag, pdl, s)) != cudaSuccess) return e;
  ++*n;
  return product(m, l.up, h, nullptr, hidden, l.out.kp, l.up.n, rows, &l.act, error_flag, pdl, s);
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
                   rows_linear_supported(batch, m->head.kp, true, 0) && (m->max_mid == 0 || rows_linear_supported(batch, m->max_mid_k, true, 0)) &&
                   (m->max_ff == 0 || rows_linear_supported(batch, m->max_ff, false, 0));
  const bool pdl = pm->use_pdl && (rows_path || m->bf16);
  const bool y_bf16 = m->bf16 && !rows_path;
  void* y = rows_path ? (void*)r.y32 : r.y;
  cudaError_t e;
  uint64_t n = 0;
  int cur = 0;               // x[cur] is the residual stream before the pending sublayer output
  const Norm* post = nullptr;  // norm of the pending sublayer output in r.yo (without weights: added as it is); nullptr: none pending
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
  auto run_rows = [&](RowsLinearArgs& a, const Matrix& w, const float* x, int ldx, int kx, const NormStepArgs* norm, float* rows32, int* grid) -> cudaError_t {
    a.w = w.w; a.m = batch; a.k = w.kp; a.x = x; a.ldx = ldx; a.kx = kx;
    if (norm && fuse_norm) {
      a.fuse_norm = 1;
      a.norm = *norm;
    } else if (norm) {
      NormStepArgs na = *norm;
      na.h32 = rows32;
      if ((e = launch_norm_step(na, batch, true, pdl, s)) != cudaSuccess) return e;
      ++n;
      a.x = rows32;
      a.ldx = a.kx = w.kp;
    }
    return launch_rows_linear(a, pdl, s, grid);
  };
  auto rows_linear = [&](const Matrix& w, const float* x, const NormStepArgs* norm, float* out, int ldo, int n_out, const ActArgs* act, float* pv, int* pi,
                         int* grid) -> cudaError_t {
    RowsLinearArgs a{};
    a.out = out; a.ldo = ldo; a.n = n_out; a.act_from = n_out;
    if (act) { a.act = *act; a.act_from = 0; a.out_act = out; a.ldo_act = ldo; }
    a.part_val = pv; a.part_idx = pi;
    return run_rows(a, w, x, w.kp, w.kp, norm, r.h32, grid);
  };
  // second-step product of a branch, into r.z
  auto mid_product = [&](const DevLayer& l, const DevBranch& b) -> cudaError_t {
    NormStepArgs na = mid_args(m, l, b, r.p);
    if (rows_path) {
      RowsLinearArgs a{};
      a.out = r.z; a.ldo = a.n = a.act_from = b.mid.np;
      return run_rows(a, b.mid, r.p + b.mid_off, l.ldp, b.mid_cols, b.mid_norm ? &na : nullptr, r.t32, nullptr);
    }
    na.h = r.t;
    if ((e = launch_norm_step(na, batch, m->bf16, pdl, s)) != cudaSuccess) return e;
    ++n;
    const bool half = b.kind == BranchSpec::LATENT && b.heads_tc;  // straight into the next product
    return product(m, b.mid, r.t, half ? nullptr : r.z, half ? r.z : nullptr, b.mid.np, b.mid.np, batch, nullptr, c->d_error, pdl, s);
  };

  if (m->tc_rotations) {
    float2* at = r.angles;
    for (const Rotation& rot : m->rotations) {
      PG_L(B_OTHER, launch_angles(c->d_pos, rot.freq, at, batch, rot.dims / 2, pdl, s));
      at += (size_t)batch * (rot.dims / 2);
    }
  }
  auto angles_of = [&](int rotation) {
    const float2* at = r.angles;
    for (int i = 0; i < rotation; ++i) at += (size_t)batch * (m->rotations[i].dims / 2);
    return at;
  };
  // Attention of a step on the tensor cores: queries and the new token's row, the products over the cached rows, the merge.
  auto heads_tc_step = [&](const DevLayer& l, const DevBranch& b, AttentionStepArgs a, void* yb) -> cudaError_t {
    AttentionPortionArgs pa{};
    pa.l = b.attn; pa.p = r.p; pa.ldp = l.ldp; pa.rows = batch; pa.step_pos = c->d_pos; pa.pool = a.pool; pa.page_table = a.page_table;
    pa.q = r.q_latent;
    a.q16 = r.q_latent;
    const float2* v_rot = b.v_rot >= 0 ? angles_of(b.v_rot) : nullptr;
    if (b.kind == BranchSpec::ATTENTION) {
      if (b.rot >= 0) pa.rot = angles_of(b.rot);
      pa.v_rot = v_rot;
      PG_L(B_ATTN, launch_attention_rotate(pa, true, s, pdl));
      PG_L(B_ATTN, launch_attention_heads_tc(a, pdl, s));
      PG_L(B_ATTN, launch_attention_merge(a, v_rot, y_bf16, pdl, s));
      return cudaSuccess;
    }
    const int H = b.attn.heads;
    PG_L(B_ATTN, launch_attention_latent(pa, true, s, pdl));
    if (rows_path) {
      HeadProductArgs hp{};
      hp.w = b.to_latent; hp.x = r.z; hp.ldx = b.mid.np; hp.ldxh = b.full.dimp;
      hp.out = r.q_latent; hp.ldo = H * b.attn.dimp; hp.ldh = b.attn.dimp;
      hp.batch = batch; hp.heads = H; hp.k = b.full.dim; hp.n = hp.np = b.attn.dimp;
      PG_L(B_ATTN, launch_head_product(hp, true, true, pdl, s));
      PG_L(B_ATTN, launch_attention_heads_tc(a, pdl, s));
      a.y = r.o_latent; a.ldy = H * b.attn.dimp; a.ldyh = b.attn.dimp;
      PG_L(B_ATTN, launch_attention_merge(a, nullptr, false, pdl, s));
      hp.w = b.from_latent; hp.x = r.o_latent; hp.ldx = a.ldy; hp.ldxh = a.ldyh;
      hp.out = yb; hp.ldo = l.out.kp; hp.ldh = b.full.vdim;
      hp.k = b.attn.vdim; hp.n = b.full.vdim; hp.np = b.full.vdimp;
      PG_L(B_ATTN, launch_head_product(hp, true, false, pdl, s));
      return cudaSuccess;
    }
    // a product per head: the kernel takes 64 rows at a time
    auto per_head = [&](Bf16GemmArgs g) -> cudaError_t {
      const char *x = static_cast<const char*>(g.x), *out = static_cast<const char*>(g.out_h);
      for (int r0 = 0; r0 < batch; r0 += 64) {
        g.x = x + (size_t)r0 * g.ldx * 2;
        g.out_h = const_cast<char*>(out) + (size_t)r0 * g.ldo * 2;
        g.m = std::min(64, batch - r0);
        PG_L(B_ATTN, launch_tc_gemm_bf16(g, pdl, s));
      }
      return cudaSuccess;
    };
    Bf16GemmArgs g{};
    g.w = b.to_latent_rows.w; g.w_tiled = b.to_latent_rows.tiled; g.k = b.to_latent_rows.kp;
    g.x = r.z; g.ldx = b.mid.np; g.x_head = b.full.dimp; g.heads = H; g.m = batch; g.error_flag = c->d_error;
    g.out_h = r.q_latent; g.ldo = H * b.attn.dimp; g.out_head = b.attn.dimp; g.n = b.attn.dimp;
    if ((e = per_head(g)) != cudaSuccess) return e;
    PG_L(B_ATTN, launch_attention_heads_tc(a, pdl, s));
    a.y = r.o_latent; a.ldy = H * b.attn.dimp; a.ldyh = b.attn.dimp;
    PG_L(B_ATTN, launch_attention_merge(a, nullptr, true, pdl, s));
    g.w = b.from_latent_rows.w; g.w_tiled = b.from_latent_rows.tiled; g.k = b.from_latent_rows.kp;
    g.x = r.o_latent; g.ldx = a.ldy; g.x_head = a.ldyh;
    g.out_h = yb; g.ldo = l.out.kp; g.out_head = b.full.vdim; g.n = b.full.vdim;
    return per_head(g);
  };

  for (const DevLayer& l : m->layers) {
    if (rows_path) {
      const NormStepArgs na = step_norm(l.norm1);
      RowsLinearArgs a{};
      a.out = r.p; a.ldo = l.ldp; a.n = a.act_from = l.in.np;
      if (l.parallel) {
        a.n = l.in.n;
        a.act = l.act; a.act_from = l.in_mixer; a.out_act = r.y32 + l.ff_off; a.ldo_act = l.out.kp;
      }
      PG_L(B_QKV, run_rows(a, l.in, nullptr, 0, 0, &na, r.h32, nullptr));
    } else {
      PG_L(B_LAYER_NORM, launch_norm_step(step_norm(l.norm1), batch, m->bf16, pdl, s));
      PG_L(B_QKV, in_product(m, l, r.h, r.p, r.y, batch, c->d_error, pdl, s, &n));
    }
    advanced();
    for (const DevBranch& b : l.branches) {
      void* yb = static_cast<char*>(y) + (size_t)b.y_off * (y_bf16 ? 2 : 4);
      if (b.mid.w) PG_L(B_QKV, mid_product(l, b));
      if (b.kind != BranchSpec::RECURRENCE) {
        AttentionStepArgs a{};
        a.l = b.attn; a.p = r.p; a.ldp = l.ldp; a.pool = lc->pools[b.pool]; a.page_table = c->tables[b.table].d_table;
        a.pos = c->d_pos; a.part = lc->attn_part; a.counters = lc->attn_counters; a.num_pages = c->tables[b.table].num_pages;
        a.y = yb; a.ldy = l.out.kp; a.ldyh = b.attn.vdim; a.batch = batch; a.splits = branch_splits(pm, b, batch, splits);
        a.error_flag = c->d_error;
        if (b.heads_tc) {
          if ((e = heads_tc_step(l, b, a, yb)) != cudaSuccess) return e;
        } else if (b.kind == BranchSpec::ATTENTION) {
          PG_L(B_ATTN, b.heads_step ? launch_attention_heads_step(a, m->bf16, y_bf16, pdl, s) : launch_attention_step(a, m->bf16, y_bf16, pdl, s));
        } else {  // queries to the latent space, attention over latent rows, values back from it
          HeadProductArgs hp{};
          hp.w = b.to_latent; hp.x = r.z; hp.ldx = b.mid.np; hp.ldxh = b.full.dimp;
          hp.out = r.q_latent; hp.ldo = b.attn.heads * b.attn.dimp; hp.ldh = b.attn.dimp;
          hp.batch = batch; hp.heads = b.attn.heads; hp.k = b.full.dim; hp.n = hp.np = b.attn.dimp;
          PG_L(B_ATTN, launch_head_product(hp, m->bf16, false, pdl, s));
          a.q = r.q_latent; a.y = r.o_latent; a.ldy = b.attn.heads * b.attn.vdim; a.ldyh = b.attn.vdim;
          PG_L(B_ATTN, launch_attention_heads_step(a, m->bf16, false, pdl, s));
          hp.w = b.from_latent; hp.x = r.o_latent; hp.ldx = a.ldy; hp.ldxh = b.attn.vdim;
          hp.out = yb; hp.ldo = l.out.kp; hp.ldh = b.full.vdim;
          hp.k = b.attn.vdim; hp.n = b.full.vdim; hp.np = b.full.vdimp;
          PG_L(B_ATTN, launch_head_product(hp, m->bf16, y_bf16, pdl, s));
        }
      } else {
        RecurrenceStepArgs a{};
        a.l = b.rec; a.p = r.p; a.ldp = l.ldp; a.z = r.z; a.ldz = b.mid.np; a.state = lc->states[b.state]; a.taps = lc->taps[b.state]; a.pos = c->d_pos;
        a.y = yb; a.ldy = l.out.kp; a.batch = batch;
        PG_L(B_ATTN, launch_recurrence_step(a, y_bf16, pdl, s));
      }
    }
    if (rows_path) PG_L(B_ATTN_PROJ, rows_linear(l.out, r.y32, nullptr, r.yo, wp, wp, nullptr, nullptr, nullptr, nullptr));
    else PG_L(B_ATTN_PROJ, product(m, l.out, r.y, r.yo, nullptr, wp, wp, batch, nullptr, c->d_error, pdl, s));
    post = &l.norm1b;
    if (!l.ff) continue;
    if (rows_path) {
      const NormStepArgs a = step_norm(l.norm2);
      PG_L(B_MLP_FC, rows_linear(l.up, nullptr, &a, r.ff32, l.down.kp, l.up.np, &l.act, nullptr, nullptr, nullptr));
      advanced();
      PG_L(B_MLP_PROJ, rows_linear(l.down, r.ff32, nullptr, r.yo, wp, wp, nullptr, nullptr, nullptr, nullptr));
    } else {
      PG_L(B_LAYER_NORM, launch_norm_step(step_norm(l.norm2), batch, m->bf16, pdl, s));
      advanced();
      PG_L(B_MLP_FC, product(m, l.up, r.h, nullptr, r.ff, l.down.kp, l.up.np, batch, &l.act, c->d_error, pdl, s));
      PG_L(B_MLP_PROJ, product(m, l.down, r.ff, r.yo, nullptr, wp, wp, batch, nullptr, c->d_error, pdl, s));
    }
    post = &l.norm2b;
  }
  FinalizeArgs fa{};
  fa.m = batch; fa.argmax_out = c->d_argmax; fa.next_ids = c->d_ids; fa.pos = c->d_pos;
  fa.token_log = c->d_token_log; fa.n_positions = pm->positions();
  if (rows_path && rows_linear_grid(batch, V, m->head.kp) <= c->part_stride) {
    const NormStepArgs a = step_norm(m->final_norm);
    int grid = 0;
    PG_L(B_LOGITS, rows_linear(m->head, nullptr, &a, c->step_wants_logits || prof ? c->logits : nullptr, V, V, nullptr, c->part_val,
                               c->part_idx, &grid));
    fa.part_val = c->part_val; fa.part_idx = c->part_idx; fa.parts = grid;
  } else {
    PG_L(B_LAYER_NORM, launch_norm_step(step_norm(m->final_norm), batch, m->bf16, pdl, s));
    PG_L(B_LOGITS, product(m, m->head, r.h, c->logits, nullptr, V, V, batch, nullptr, c->d_error, pdl, s));
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
  std::vector<const float2*> angles;  // per rotation
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
    PG_L(B_QKV, in_product(m, l, r.h, r.p, r.y, rows, c->d_error, false, s, &n));
    for (const DevBranch& b : l.branches) {
      void* y = static_cast<char*>(r.y) + (size_t)b.y_off * m->elem();
      if (b.mid.w) {  // second step of two-step projections; latent attention: straight to the queries
        NormStepArgs na = mid_args(m, l, b, r.p);
        na.h = r.t;
        PG_L(B_QKV, launch_norm_step(na, rows, m->bf16, false, s));
        const bool query = b.kind == BranchSpec::LATENT;
        PG_L(B_QKV, product(m, b.mid, r.t, query ? nullptr : r.z, query ? lc->q : nullptr, b.mid.np, b.mid.np, rows, nullptr, c->d_error, false, s));
      }
      if (b.kind != BranchSpec::RECURRENCE) {
        AttentionPortionArgs a{};
        a.l = b.attn; a.p = r.p; a.ldp = l.ldp; a.rows = rows; a.nseq = plan.n(); a.max_len = plan.max_len; a.krows = d.krows[b.table];
        a.seq_start = d.seq_start; a.key_start = d.key_start[b.table]; a.seq_slot = d.slot; a.seq_pos = d.start_pos; a.row_seq = d.row_seq;
        a.pool = lc->pools[b.pool]; a.page_table = c->tables[b.table].d_table;
        a.q = lc->q; a.k = lc->k; a.v = lc->v; a.error_flag = c->d_error; a.y = y; a.ldy = l.out.kp;
        a.ldk = b.attn.kv_heads * b.attn.dimp; a.ldv = b.attn.kv_heads * b.attn.vdimp;
        if (b.rot >= 0) a.rot = d.angles[b.rot];
        if (b.v_rot >= 0) a.v_rot = d.angles[b.v_rot];
        if (b.kind == BranchSpec::ATTENTION) {
          PG_L(B_ATTN, launch_attention_portion(a, m->bf16, s));
        } else {  // latent rows, new and cached, then the heads' own keys and values from them
          PG_L(B_ATTN, launch_attention_latent(a, m->bf16, s));
          PG_L(B_ATTN, launch_attention_context(a, m->bf16, s));
          PG_L(B_ATTN, launch_attention_store(a, m->bf16, s));
          PG_L(B_ATTN, product(m, b.up_kv, lc->k, nullptr, lc->v, b.up_kv.np, b.up_kv.np, a.krows, nullptr, c->d_error, false, s));
          a.l = b.full;
          a.k = lc->v;
          a.v = static_cast<char*>(lc->v) + (size_t)b.full.heads * b.full.dimp * m->elem();
          a.ldk = a.ldv = b.up_kv.np;
          PG_L(B_ATTN, launch_attention_core(a, m->bf16, s));
        }
      } else {
        RecurrenceScanArgs a{};
        a.l = b.rec; a.p = r.p; a.ldp = l.ldp; a.rows = rows; a.nseq = plan.n(); a.row_seq = d.row_seq;
        a.z = r.z; a.ldz = b.mid.np; a.taps = lc->taps[b.state]; a.vals = lc->vals;
        a.max_len = plan.max_len; a.writes = lc->writes; a.quad_decay = lc->quad_decay; a.quads = lc->quads;
        a.seq_start = d.seq_start; a.seq_slot = d.slot; a.seq_pos = d.start_pos; a.state = lc->states[b.state];
        a.decay = lc->decay; a.unit = lc->unit; a.rate = lc->rate; a.unit_next = lc->unit_next; a.pair = lc->pair;
        a.out_raw = lc->out_raw; a.error_flag = c->d_error;
        a.segments = lc->segments; a.seg_tokens = segment_tokens(plan.max_len);
        a.max_segs = recurrence_use_segments(b.rec, plan.n(), plan.max_len, max_segs) ? max_segs : 0;
        a.y = y; a.ldy = l.out.kp;
        PG_L(B_ATTN, launch_recurrence_scan(a, m->bf16, s));
      }
    }
    PG_L(B_ATTN_PROJ, product(m, l.out, r.y, r.yo, nullptr, wp, wp, rows, nullptr, c->d_error, false, s));
    post = &l.norm1b;
    if (!l.ff) continue;
    PG_L(B_LAYER_NORM, norm(&l.norm2));
    PG_L(B_MLP_FC, product(m, l.up, r.h, nullptr, r.ff, l.down.kp, l.up.np, rows, &l.act, c->d_error, false, s));
    PG_L(B_MLP_PROJ, product(m, l.down, r.ff, r.yo, nullptr, wp, wp, rows, nullptr, c->d_error, false, s));
    post = &l.norm2b;
  }
  const int outs = (int)plan.out_rows.size();
  if (outs > 0) {
    PG_L(B_LAYER_NORM, norm(nullptr));
    NormStepArgs a = norm_args(m);
    a.x_in = x; a.row_index = d.out_rows; a.pre_g = m->final_norm.g; a.pre_b = m->final_norm.b; a.h = r.h;
    PG_L(B_LAYER_NORM, launch_norm_step(a, outs, m->bf16, false, s));
    PG_L(B_LOGITS, product(m, m->head, r.h, logits, nullptr, V, V, outs, nullptr, c->d_error, false, s));
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
  for (const KeyLife& life : m->lives) {
    std::vector<int> ks(1, 0);
    for (int i = 0; i < ns; ++i) ks.push_back(ks.back() + life.context(plan.start_pos[i]) + (plan.seq_start[i + 1] - plan.seq_start[i]));
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
        qe = std::max<size_t>(qe, (size_t)b.attn.heads * attention_q_width(b.attn));
        ke = std::max<size_t>(ke, (size_t)b.attn.kv_heads * b.attn.dimp);
        ve = std::max<size_t>(ve, (size_t)b.attn.kv_heads * b.attn.vdimp);
      } else if (b.kind == BranchSpec::LATENT) {
        qe = std::max<size_t>(qe, b.mid.np);
        ke = std::max<size_t>(ke, b.attn.dimp);
        ve = std::max<size_t>(ve, b.up_kv.np);
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
  if (m->channel_rules) {
    if ((size_t)rows > lc->channel_rows) {
      size_t v = lc->channel_rows;
      if (int r = grow(&lc->vals, &v, rows, m->max_rec_out * sizeof(float))) return r;
      if (int r = grow(&lc->writes, &lc->channel_rows, rows, m->max_rec * sizeof(float))) return r;
    }
    const size_t quads = recurrence_quads(rows, ns);
    if (quads > lc->quad_rows) {
      size_t d = lc->quad_rows;
      if (int r = grow(&lc->quad_decay, &d, quads, m->max_rec * sizeof(float))) return r;
      if (int r = grow(&lc->quads, &lc->quad_rows, quads, (size_t)m->max_rec_heads * 20 * sizeof(float))) return r;
    }
  }
  if (seg)
    if (int r = grow(&lc->segments, &lc->seg_floats, seg, sizeof(float))) return r;
  PG_CUDA_TRY(cudaMemcpyAsync(lc->meta, meta.data(), meta.size() * sizeof(int), cudaMemcpyHostToDevice, c->stream));
  PG_CUDA_TRY(cudaStreamSynchronize(c->stream));  // `meta` is a pageable temporary
  d.ids = lc->meta + o_ids; d.pos = lc->meta + o_pos; d.row_seq = lc->meta + o_rs; d.seq_start = lc->meta + o_ss;
  d.slot = lc->meta + o_sl; d.start_pos = lc->meta + o_sp; d.out_rows = lc->meta + o_or;
  for (size_t o : o_ks) d.key_start.push_back(lc->meta + o);
  size_t half = 0;
  for (const Rotation& r : m->rotations) half += r.dims / 2;
  if (half)
    if (int r = grow(&lc->angles, &lc->angle_rows, rows, half * sizeof(float2))) return r;
  float2* at = lc->angles;
  for (const Rotation& r : m->rotations) {  // this pass's angles, shared by the layers
    PG_CUDA_TRY(launch_angles(d.pos, r.freq, at, rows, r.dims / 2, false, c->stream));
    d.angles.push_back(at);
    at += (size_t)rows * (r.dims / 2);
  }
  PG_CUDA_TRY(enqueue_portions(c, plan, d, logits, prof, nullptr));
  return PG_OK;
}

}  // namespace pg
