// Design registry, configuration reader and tensor checks of the layered models (host only).
#include "design.h"

#include <cmath>
#include <cstring>
#include <functional>

namespace pg {

namespace {

// Largest sizes the kernels take (per head: shared-memory rows and registers; per model: 32-bit indexing).
constexpr int MAX_WIDTH = 16384, MAX_HEAD_DIM = 256, MAX_HEADS = 1024, MAX_RANK = 512;

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
};

// Grouped-head attention: heads, kv_heads, dim, vdim, scale and an optional mask {size}.
int read_attention(const Reader& r, const Json& m, const std::string& where, BranchSpec* b) {
  b->kind = BranchSpec::ATTENTION;
  AttentionSpec& a = b->attn;
  if (int e = r.integer(m, where, "heads", 1, MAX_HEADS, &a.heads)) return e;
  if (int e = r.integer(m, where, "kv_heads", 1, MAX_HEADS, &a.kv_heads)) return e;
  if (int e = r.integer(m, where, "dim", 1, MAX_HEAD_DIM, &a.dim)) return e;
  if (int e = r.integer(m, where, "vdim", 1, MAX_HEAD_DIM, &a.vdim)) return e;
  if (int e = r.number(m, where, "scale", &a.scale)) return e;
  if (a.heads % a.kv_heads != 0)
    return r.fail(where + ": heads " + std::to_string(a.heads) + " must be divisible by kv_heads " + std::to_string(a.kv_heads));
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

// Dirurax: layers of type "gla" (gated linear attention) and "parallel" (chunked attention with normed queries, keys
// and values beside a generalized delta rule), each with an optional dense feed-forward.
int parse_dirurax(const Json& root, const std::string& path, LayeredConfig* out) {
  Reader r{path};
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
    const Json* type = j.get("type");
    const Json* mixer = r.object(j, "mixer");
    if (!type || type->kind != Json::String) return r.fail(where + ": missing `type`");
    if (!mixer) return r.fail(where + ": missing `mixer`");
    LayerSpec l;
    l.type = type->str;
    if (l.type == "gla") {
      BranchSpec b;
      b.prefix = "mix";
      if (int e = read_gla(r, *mixer, where + ".mixer", &b)) return e;
      l.branches.push_back(b);
    } else if (l.type == "parallel") {
      const Json *left = r.object(*mixer, "left"), *right = r.object(*mixer, "right");
      if (!left || !right) return r.fail(where + ".mixer: missing `left` or `right`");
      BranchSpec a, d;
      a.prefix = "mix.left";
      d.prefix = "mix.right";
      if (int e = read_attention(r, *left, where + ".mixer.left", &a)) return e;
      a.attn.qk_norm = a.attn.v_norm = true;
      if (int e = read_delta(r, *right, where + ".mixer.right", &d)) return e;
      if (int e = r.number(*mixer, where + ".mixer", "left_scale", &a.scale)) return e;
      if (int e = r.number(*mixer, where + ".mixer", "right_scale", &d.scale)) return e;
      l.branches.push_back(a);
      l.branches.push_back(d);
    } else {
      return r.fail(where + ": unknown type \"" + l.type + "\"");
    }
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

const Design kDesigns[] = {{"Dirurax", parse_dirurax}};

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
    return want(name + ".b", {W});
  };
  if (int r = want("embed", {cfg->vocab, W})) return r;
  if (int r = norm("final.norm")) return r;
  for (size_t i = 0; i < cfg->layers.size(); ++i) {
    LayerSpec& l = cfg->layers[i];
    const std::string p = "l" + std::to_string(i) + ".";
    if (int r = norm(p + "norm1")) return r;
    if (int r = norm(p + "norm1b")) return r;
    for (BranchSpec& b : l.branches) {
      const std::string m = p + b.prefix + ".";
      std::vector<std::pair<std::string, std::vector<int64_t>>> t;
      int* rank = nullptr;
      if (b.kind == BranchSpec::ATTENTION) {
        const AttentionSpec& a = b.attn;
        const int64_t H = a.heads, G = a.kv_heads;
        t = {{"q", {H * a.dim, W}}, {"k", {G * a.dim, W}}, {"v", {G * a.vdim, W}}, {"o", {W, H * a.vdim}}};
        if (a.qk_norm) t.insert(t.end(), {{"q.norm", {a.dim}}, {"k.norm", {a.dim}}});
      } else {
        RecurrenceSpec& s = b.rec;
        rank = &s.rank;
        const int64_t K = (int64_t)s.heads * s.dim, V = (int64_t)s.heads * s.vdim;
        if (s.kind == RECUR_GLA)
          t = {{"q", {K, W}}, {"k", {K, W}}, {"v", {V, W}}, {"g", {V, W}}, {"o", {W, V}}, {"norm", {s.vdim}},
               {"a1", {-1, W}}, {"a2", {K, -1}}, {"a2.b", {K}}};
        else
          t = {{"r", {K, W}}, {"k", {K, W}}, {"v", {V, W}}, {"g", {V, W}}, {"o", {W, V}}, {"norm", {V}},
               {"a", {K, W}}, {"a.b", {K}}, {"w1", {-1, W}}, {"w2", {K, -1}}, {"w0", {K}}};
      }
      for (auto& e : t)
        if (int r = want(m + e.first, e.second, rank)) return r;
      if (rank && (*rank < 1 || *rank > MAX_RANK))
        return set_error(PG_INVALID_WEIGHTS, m + "* has a decay rank outside 1.." + std::to_string(MAX_RANK));
    }
    if (l.ff > 0) {
      if (int r = norm(p + "norm2")) return r;
      if (int r = norm(p + "norm2b")) return r;
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
