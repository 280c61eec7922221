// Design registry, configuration reader and tensor checks of the layered models (host only).
#include "design.h"

#include <cmath>
#include <cstring>
#include <functional>

namespace pg {

namespace {

// Largest sizes the kernels take (per head: shared-memory rows and registers; per model: 32-bit indexing).
constexpr int MAX_WIDTH = 16384, MAX_HEAD_DIM = 256, MAX_HEADS = 1024, MAX_RANK = 512, MAX_LATENT = 1024, MAX_TAPS = 64;

struct Reader {
  std::string path;
  int fail(const std::string& what) const {
    return set_error(PG_INVALID_CONFIG, "config file " + path + ": " + what);
  }
  const Json* object(const Json& j, const char* key) const {
    const Json* f = j.get(key);
    return f && f->kind == Json::Object ? f : nullptr;
  }
  int integer(const Json& j, const std::string& where, const char* key, int lo, int hi, int* out) const {
    const Json* f = j.get(key);
    if (!f || f->kind != Json::Number || f->num != std::floor(f->num))
      return fail(where + ": missing or invalid integer `" + key + "`");
    if (f->num < lo || f->num > hi)
      return fail(where + ": `" + key + "` " + std::to_string((long long)f->num) + " must be in " + std::to_string(lo) + ".." + std::to_string(hi));
    *out = (int)f->num;
    return PG_OK;
  }
  int number(const Json& j, const std::string& where, const char* key, float* out) const {
    const Json* f = j.get(key);
    if (!f || f->kind != Json::Number || !std::isfinite(f->num)) return fail(where + ": missing or invalid number `" + key + "`");
    *out = (float)f->num;
    return PG_OK;
  }
  int number(const Json& j, const std::string& where, const char* key, double* out) const {
    float f = 0.f;
    if (int e = number(j, where, key, &f)) return e;
    *out = j.get(key)->num;
    return PG_OK;
  }
};

int heads_divide(const Reader& r, const std::string& where, int heads, int kv_heads) {
  if (heads % kv_heads == 0) return PG_OK;
  return r.fail(where + ": heads " + std::to_string(heads) + " must be divisible by kv_heads " + std::to_string(kv_heads));
}

// heads, kv_heads, dim, vdim, scale of grouped-head attention.
int read_head_sizes(const Reader& r, const Json& m, const std::string& where, AttentionSpec* a) {
  if (int e = r.integer(m, where, "heads", 1, MAX_HEADS, &a->heads)) return e;
  if (int e = r.integer(m, where, "kv_heads", 1, MAX_HEADS, &a->kv_heads)) return e;
  if (int e = r.integer(m, where, "dim", 1, MAX_HEAD_DIM, &a->dim)) return e;
  if (int e = r.integer(m, where, "vdim", 1, MAX_HEAD_DIM, &a->vdim)) return e;
  if (int e = r.number(m, where, "scale", &a->scale)) return e;
  return heads_divide(r, where, a->heads, a->kv_heads);
}

// Grouped-head attention: heads, kv_heads, dim, vdim, scale and an optional mask {size}.
int read_attention(const Reader& r, const Json& m, const std::string& where, BranchSpec* b) {
  b->kind = BranchSpec::ATTENTION;
  AttentionSpec& a = b->attn;
  if (int e = read_head_sizes(r, m, where, &a)) return e;
  const Json* mask = m.get("mask");
  if (mask && mask->kind == Json::Object) {
    if (int e = r.integer(*mask, where + ".mask", "size", 1, 1 << 30, &a.chunk)) return e;
  } else if (mask && mask->kind != Json::Null) {
    return r.fail(where + ": invalid `mask`");
  }
  return PG_OK;
}

int read_gla(const Reader& r, const Json& m, const std::string& where, BranchSpec* b) {
  b->kind = BranchSpec::RECURRENCE;
  RecurrenceSpec& s = b->rec;
  s.kind = RECUR_GLA;
  if (int e = r.integer(m, where, "heads", 1, MAX_HEADS, &s.heads)) return e;
  if (int e = r.integer(m, where, "dim", 1, MAX_HEAD_DIM, &s.dim)) return e;
  if (int e = r.integer(m, where, "vdim", 1, MAX_HEAD_DIM, &s.vdim)) return e;
  if (int e = r.number(m, where, "tau", &s.tau)) return e;
  if (!(s.tau > 0.f)) return r.fail(where + ": tau must be > 0");
  return PG_OK;
}

int read_delta(const Reader& r, const Json& m, const std::string& where, BranchSpec* b) {
  b->kind = BranchSpec::RECURRENCE;
  RecurrenceSpec& s = b->rec;
  s.kind = RECUR_DELTA;
  if (int e = r.integer(m, where, "heads", 1, MAX_HEADS, &s.heads)) return e;
  if (int e = r.integer(m, where, "dim", 1, MAX_HEAD_DIM, &s.dim)) return e;
  s.vdim = s.dim;
  return PG_OK;
}

// Sizes, eps and the list of layers, each with an optional dense feed-forward; `mixer(type, entry, where, layer, known)` fills in
// the branches of a layer.
int read_layers(const Reader& r, const Json& root, LayeredConfig* out,
                const std::function<int(const std::string&, const Json&, const std::string&, LayerSpec*, bool*)>& mixer) {
  if (int e = r.integer(root, "model", "vocab", 1, 1 << 24, &out->vocab)) return e;
  if (int e = r.integer(root, "model", "width", 1, MAX_WIDTH, &out->width)) return e;
  const Json* norm = r.object(root, "norm");
  if (!norm) return r.fail("model: missing `norm`");
  if (int e = r.number(*norm, "norm", "eps", &out->norm_eps)) return e;
  if (!(out->norm_eps > 0.f)) return r.fail("norm: eps must be > 0");
  const Json* layers = root.get("layers");
  if (!layers || layers->kind != Json::Array || layers->arr.empty()) return r.fail("model: missing `layers`");
  for (size_t i = 0; i < layers->arr.size(); ++i) {
    const Json& j = layers->arr[i];
    const std::string where = "layers[" + std::to_string(i) + "]";
    const Json *type = j.get("type"), *mix = r.object(j, "mixer");
    if (!type || type->kind != Json::String) return r.fail(where + ": missing `type`");
    if (!mix) return r.fail(where + ": missing `mixer`");
    LayerSpec l;
    l.type = type->str;
    bool known = true;
    if (int e = mixer(l.type, *mix, where + ".mixer", &l, &known)) return e;
    if (!known) return r.fail(where + ": unknown type \"" + l.type + "\"");
    const Json* mlp = j.get("mlp");
    if (mlp && mlp->kind == Json::Object) {
      const Json* kind = mlp->get("kind");
      if (!kind || kind->kind != Json::String || kind->str != "dense") return r.fail(where + ".mlp: unknown kind");
      if (int e = r.integer(*mlp, where + ".mlp", "ff", 1, 1 << 20, &l.ff)) return e;
    } else if (mlp && mlp->kind != Json::Null) {
      return r.fail(where + ": invalid `mlp`");
    }
    out->layers.push_back(std::move(l));
  }
  return PG_OK;
}

// Dirurax: layers of type "gla" (gated linear attention) and "parallel" (chunked attention with normed queries, keys
// and values beside a generalized delta rule), each with an optional dense feed-forward.
int parse_dirurax(const Json& root, const std::string& path, LayeredConfig* out) {
  Reader r{path};
  return read_layers(r, root, out, [&](const std::string& type, const Json& mixer, const std::string& where, LayerSpec* l, bool* known) -> int {
    if (type == "gla") {
      BranchSpec b;
      b.prefix = "mix";
      if (int e = read_gla(r, mixer, where, &b)) return e;
      l->branches.push_back(b);
    } else if (type == "parallel") {
      const Json *left = r.object(mixer, "left"), *right = r.object(mixer, "right");
      if (!left || !right) return r.fail(where + ": missing `left` or `right`");
      BranchSpec a, d;
      a.prefix = "mix.left";
      d.prefix = "mix.right";
      if (int e = read_attention(r, *left, where + ".left", &a)) return e;
      a.attn.qk_norm = a.attn.v_norm = true;
      if (int e = read_delta(r, *right, where + ".right", &d)) return e;
      if (int e = r.number(mixer, where, "left_scale", &a.scale)) return e;
      if (int e = r.number(mixer, where, "right_scale", &d.scale)) return e;
      l->branches.push_back(a);
      l->branches.push_back(d);
    } else {
      *known = false;
    }
    return PG_OK;
  });
}

// Rotated attention with mixed heads, a sink and a window that keeps the first tokens.
int read_window_attention(const Reader& r, const Json& m, const std::string& where, BranchSpec* b) {
  b->kind = BranchSpec::ATTENTION;
  AttentionSpec& a = b->attn;
  if (int e = read_head_sizes(r, m, where, &a)) return e;
  const Json *rot = r.object(m, "rot"), *mask = r.object(m, "mask");
  if (!rot) return r.fail(where + ": missing `rot`");
  if (!mask) return r.fail(where + ": missing `mask`");
  if (int e = r.integer(*mask, where + ".mask", "size", 1, 1 << 30, &a.window)) return e;
  if (int e = r.integer(*mask, where + ".mask", "keep_first", 0, 1 << 30, &a.keep_first)) return e;
  if (int e = r.integer(*rot, where + ".rot", "dims", 0, a.dim, &a.rot_dims)) return e;
  if (int e = r.number(*rot, where + ".rot", "base", &a.rot_base)) return e;
  if (!(a.rot_base > 0)) return r.fail(where + ".rot: base must be > 0");
  if (a.rot_dims % 2 != 0 || a.vdim % 2 != 0) return r.fail(where + ": rot.dims and vdim must be even");
  a.bias = a.v_rot = a.head_mix = a.sink = true;
  return PG_OK;
}

int read_latent_attention(const Reader& r, const Json& m, const std::string& where, BranchSpec* b) {
  b->kind = BranchSpec::LATENT;
  AttentionSpec& a = b->attn;
  if (int e = r.integer(m, where, "heads", 1, MAX_HEADS, &a.heads)) return e;
  if (int e = r.integer(m, where, "dim", 1, MAX_HEAD_DIM, &a.dim)) return e;
  if (int e = r.integer(m, where, "vdim", 1, MAX_HEAD_DIM, &a.vdim)) return e;
  if (int e = r.integer(m, where, "kv_rank", 1, MAX_LATENT, &a.kv_rank)) return e;
  if (int e = r.integer(m, where, "q_rank", 1, MAX_WIDTH, &a.q_rank)) return e;
  if (int e = r.number(m, where, "scale", &a.scale)) return e;
  a.kv_heads = 1;
  a.head_gate = true;
  return PG_OK;
}

int read_channel_delta(const Reader& r, const Json& m, const std::string& where, BranchSpec* b) {
  b->kind = BranchSpec::RECURRENCE;
  RecurrenceSpec& s = b->rec;
  s.kind = RECUR_CHANNEL;
  if (int e = r.integer(m, where, "heads", 1, MAX_HEADS, &s.heads)) return e;
  if (int e = r.integer(m, where, "kv_heads", 1, MAX_HEADS, &s.kv_heads)) return e;
  if (int e = r.integer(m, where, "dim", 1, MAX_HEAD_DIM, &s.dim)) return e;
  if (int e = r.integer(m, where, "vdim", 1, MAX_HEAD_DIM, &s.vdim)) return e;
  if (int e = r.integer(m, where, "conv", 1, MAX_TAPS, &s.conv)) return e;
  return heads_divide(r, where, s.heads, s.kv_heads);
}

// Sanesun: layers of type "attention", "channel_delta" and "latent_attention", each beside an optional dense feed-forward
// that reads the same normed input; RMS norms, no position vectors, a head of its own.
int parse_sanesun(const Json& root, const std::string& path, LayeredConfig* out) {
  Reader r{path};
  out->norm_kind = NORM_RMS;
  out->activation = ACT_XIELU;
  out->post_norms = out->sinusoids = out->tied_head = false;
  out->parallel_ff = true;
  const Json* embedding = r.object(root, "embedding");
  if (!embedding) return r.fail("model: missing `embedding`");
  if (int e = r.number(*embedding, "embedding", "scale", &out->embed_scale)) return e;
  return read_layers(r, root, out, [&](const std::string& type, const Json& mixer, const std::string& where, LayerSpec* l, bool* known) -> int {
    BranchSpec b;
    b.prefix = "mix";
    int e = PG_OK;
    if (type == "attention") e = read_window_attention(r, mixer, where, &b);
    else if (type == "channel_delta") e = read_channel_delta(r, mixer, where, &b);
    else if (type == "latent_attention") e = read_latent_attention(r, mixer, where, &b);
    else *known = false;
    l->branches.push_back(b);
    return e;
  });
}

const Design kDesigns[] = {{"Dirurax", parse_dirurax}, {"Sanesun", parse_sanesun}};

}  // namespace

const Design* find_design(const std::string& name) {
  for (const Design& d : kDesigns)
    if (name == d.name) return &d;
  return nullptr;
}

std::string registered_designs() {
  std::string s = "gpt2";
  for (const Design& d : kDesigns) s += std::string(", ") + d.name;
  return s;
}

int load_design_config(const std::string& path, bool* layered, LayeredConfig* out) {
  std::vector<uint8_t> bytes;
  std::string err;
  Json root;
  *layered = false;
  if (!read_file(path, &bytes, &err)) return set_error(PG_ASSET, "failed to read config file " + path + ": " + err);
  if (!parse_json((const char*)bytes.data(), bytes.size(), &root, &err) || root.kind != Json::Object)
    return set_error(PG_ASSET, "failed to parse config file " + path + ": " + (err.empty() ? "not an object" : err));
  const Json* a = root.get("architecture");
  if (!a || a->kind != Json::String || a->str == "gpt2") return PG_OK;
  const Design* d = find_design(a->str);
  if (!d)
    return set_error(PG_INVALID_CONFIG, "config file " + path + ": unknown architecture \"" + a->str + "\" (known: " + registered_designs() + ")");
  out->architecture = d->name;
  if (int r = d->parse(root, path, out)) return r;
  *layered = true;
  return PG_OK;
}

// ------------------------------------------------------------------ tensors
int check_layered_tensors(const SafeTensorsFile& file, const std::string& path, LayeredConfig* cfg) {
  auto shape_text = [](const std::vector<int64_t>& s) {
    std::string o = "[";
    for (size_t i = 0; i < s.size(); ++i) o += (i ? ", " : "") + (s[i] < 0 ? std::string("?") : std::to_string(s[i]));
    return o + "]";
  };
  // `rank`: where a -1 in the wanted shape is read from, or checked against once known
  auto want = [&](const std::string& name, const std::vector<int64_t>& shape, int* rank = nullptr) -> int {
    auto it = file.tensors.find(name);
    if (it == file.tensors.end()) return set_error(PG_ASSET, "tensor " + name + " not found in " + path);
    const TensorEntry& e = it->second;
    if (e.dtype != "BF16" && e.dtype != "F32")
      return set_error(PG_ASSET, "tensor " + name + " has dtype " + e.dtype + ", expected BF16 or F32");
    bool ok = e.shape.size() == shape.size();
    for (size_t i = 0; ok && i < shape.size(); ++i) {
      if (shape[i] >= 0) ok = e.shape[i] == (uint64_t)shape[i];
      else if (*rank == 0) *rank = (int)std::min<uint64_t>(e.shape[i], MAX_RANK + 1);
      else ok = e.shape[i] == (uint64_t)*rank;
    }
    if (!ok)
      return set_error(PG_INVALID_WEIGHTS, "tensor " + name + " shape " + shape_text(std::vector<int64_t>(e.shape.begin(), e.shape.end())) +
                                               " does not match expected " + shape_text(shape));
    return PG_OK;
  };
  const int64_t W = cfg->width;
  auto norm = [&](const std::string& name) -> int {
    if (int r = want(name, {W})) return r;
    return cfg->norm_kind == NORM_LAYER ? want(name + ".b", {W}) : PG_OK;
  };
  if (int r = want("embed", {cfg->vocab, W})) return r;
  if (!cfg->tied_head)
    if (int r = want("head", {cfg->vocab, W})) return r;
  if (int r = norm("final.norm")) return r;
  for (size_t i = 0; i < cfg->layers.size(); ++i) {
    LayerSpec& l = cfg->layers[i];
    const std::string p = "l" + std::to_string(i) + ".";
    if (int r = norm(p + "norm1")) return r;
    if (cfg->post_norms)
      if (int r = norm(p + "norm1b")) return r;
    for (BranchSpec& b : l.branches) {
      const std::string m = p + b.prefix + ".";
      std::vector<std::pair<std::string, std::vector<int64_t>>> t, t2;  // t2: tensors of the second unknown size
      int *rank = nullptr, *rank2 = nullptr;
      if (b.kind == BranchSpec::ATTENTION) {
        const AttentionSpec& a = b.attn;
        const int64_t H = a.heads, G = a.kv_heads;
        t = {{"q", {H * a.dim, W}}, {"k", {G * a.dim, W}}, {"v", {G * a.vdim, W}}, {"o", {W, H * a.vdim}}};
        if (a.qk_norm) t.insert(t.end(), {{"q.norm", {a.dim}}, {"k.norm", {a.dim}}});
        if (a.bias) t.insert(t.end(), {{"q.b", {H * a.dim}}, {"k.b", {G * a.dim}}, {"v.b", {G * a.vdim}}});
        if (a.head_mix) t.push_back({"talk", {H, H}});
        if (a.sink) t.push_back({"sink", {H}});
      } else if (b.kind == BranchSpec::LATENT) {
        const AttentionSpec& a = b.attn;
        const int64_t H = a.heads;
        t = {{"dq", {a.q_rank, W}}, {"dq.norm", {a.q_rank}}, {"uq", {H * a.dim, a.q_rank}}, {"dkv", {a.kv_rank, W}},
             {"dkv.norm", {a.kv_rank}}, {"uk", {H * a.dim, a.kv_rank}}, {"uv", {H * a.vdim, a.kv_rank}}, {"o", {W, H * a.vdim}}};
        if (a.head_gate) t.push_back({"g", {H, W}});
      } else {
        RecurrenceSpec& s = b.rec;
        rank = &s.rank;
        const int64_t K = (int64_t)s.heads * s.dim, V = (int64_t)s.heads * s.vdim, Q = (int64_t)s.kv_heads * s.dim;
        if (s.kind == RECUR_GLA) {
          t = {{"q", {K, W}}, {"k", {K, W}}, {"v", {V, W}}, {"g", {V, W}}, {"o", {W, V}}, {"norm", {s.vdim}},
               {"a1", {-1, W}}, {"a2", {K, -1}}, {"a2.b", {K}}};
        } else if (s.kind == RECUR_DELTA) {
          t = {{"r", {K, W}}, {"k", {K, W}}, {"v", {V, W}}, {"g", {V, W}}, {"o", {W, V}}, {"norm", {V}},
               {"a", {K, W}}, {"a.b", {K}}, {"w1", {-1, W}}, {"w2", {K, -1}}, {"w0", {K}}};
        } else {
          t = {{"q", {Q, W}}, {"k", {Q, W}}, {"v", {V, W}}, {"q.conv", {Q, s.conv}}, {"k.conv", {Q, s.conv}}, {"v.conv", {V, s.conv}},
               {"b", {s.heads, W}}, {"A_log", {s.heads}}, {"norm", {s.vdim}}, {"o", {W, V}}, {"dt_bias", {K}},
               {"a1", {-1, W}}, {"a2", {K, -1}}};
          t2 = {{"g1", {-1, W}}, {"g2", {V, -1}}};
          rank2 = &s.rank2;
        }
      }
      for (auto& e : t)
        if (int r = want(m + e.first, e.second, rank)) return r;
      for (auto& e : t2)
        if (int r = want(m + e.first, e.second, rank2)) return r;
      for (const int* n : {rank, rank2})
        if (n && (*n < 1 || *n > MAX_RANK))
          return set_error(PG_INVALID_WEIGHTS, m + "* has a decay or gate rank outside 1.." + std::to_string(MAX_RANK));
    }
    if (l.ff > 0) {
      if (!cfg->parallel_ff)
        if (int r = norm(p + "norm2")) return r;
      if (cfg->post_norms)
        if (int r = norm(p + "norm2b")) return r;
      if (cfg->activation == ACT_XIELU)
        if (int r = want(p + "mlp.act", {2})) return r;
      if (int r = want(p + "mlp.up", {l.ff, W})) return r;
      if (int r = want(p + "mlp.down", {W, l.ff})) return r;
    }
  }
  return PG_OK;
}

std::vector<float> tensor_f32(const SafeTensorsFile& file, const std::string& name) {
  const TensorEntry& e = file.tensors.at(name);
  const uint8_t* p = file.data(e);
  if (e.dtype == "F32") {
    std::vector<float> v((e.end - e.begin) / 4);
    memcpy(v.data(), p, v.size() * 4);
    return v;
  }
  std::vector<float> v((e.end - e.begin) / 2);
  for (size_t i = 0; i < v.size(); ++i) {
    const uint32_t u = ((uint32_t)p[2 * i] | ((uint32_t)p[2 * i + 1] << 8)) << 16;
    memcpy(&v[i], &u, 4);
  }
  return v;
}

}  // namespace pg
