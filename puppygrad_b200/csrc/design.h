// Models described layer by layer: the design registry, the parsed configuration and the list of tensors it implies.
// Host only. A design is a name (config.json "architecture") with a reader that turns its configuration file into a
// LayeredConfig; everything after that (loading, cache, step, sampling) is common to all designs.
#pragma once
#include <cstdint>
#include <string>
#include <vector>

#include "common.h"

namespace pg {

// Softmax attention with grouped heads: query head h reads key / value head h / (heads / kv_heads).
struct AttentionSpec {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  float scale = 1.f;       // score = (q . k) * scale
  bool qk_norm = false;    // per-head RMS norm of q and k with a shared weight of size dim
  bool v_norm = false;     // each head's value divided by its root mean square
  int chunk = 0;           // > 0: position i sees j only inside the same block of `chunk` positions; 0: every j <= i
};

// A recurrence over tokens whose state is one [dim, vdim] FP32 matrix per head.
//  RECUR_GLA    S = diag(alpha) S + k v^T, alpha = sigmoid(A2 (A1 h) + b)^(1/tau); out = S^T (q / sqrt(dim)); the
//               per-head RMS norm has a weight of size vdim shared by the heads, the gate is silu
//  RECUR_DELTA  S = diag(w) S - (a * u) (u^T S) + k v^T, w = exp(-e^-1/2 * sigmoid(W2 tanh(W1 h) + w0)),
//               a = sigmoid(W_a h + b), u = k / sqrt(|k|^2 + 1e-6); out = S^T r; the per-head RMS norm has no weight of
//               its own, the concatenation is multiplied by a weight of all heads' size and the gate is sigmoid
enum RecurrenceKind { RECUR_GLA = 0, RECUR_DELTA = 1 };
struct RecurrenceSpec {
  int kind = RECUR_GLA;
  int heads = 0, dim = 0, vdim = 0;
  float tau = 1.f;
  int rank = 0;  // inner size of the two-step decay projection, from the tensors' shapes
};

// One branch of a layer's mixer; branches read the same input and their results are added, each times its scale.
struct BranchSpec {
  enum Kind { ATTENTION = 0, RECURRENCE = 1 } kind = ATTENTION;
  AttentionSpec attn;
  RecurrenceSpec rec;
  float scale = 1.f;
  std::string prefix;  // tensors of this branch: "<layer prefix>.<prefix>.<name>"
  int out_dim() const { return kind == ATTENTION ? attn.heads * attn.vdim : rec.heads * rec.vdim; }
};

struct LayerSpec {
  std::string type;
  std::vector<BranchSpec> branches;
  int ff = 0;  // 0: no feed-forward; else W_down gelu(W_up h) with the exact (erf) gelu
};

struct LayeredConfig {
  std::string architecture;
  int vocab = 0, width = 0;
  float norm_eps = 1e-5f;  // layer norms before and after every sublayer, head norms, query / key / value norms
  std::vector<LayerSpec> layers;
};

struct Design {
  const char* name;
  int (*parse)(const Json& root, const std::string& path, LayeredConfig* out);
};
// nullptr when no design of that name is registered.
const Design* find_design(const std::string& name);
std::string registered_designs();  // "gpt2, ..." for messages

// Reads config.json: *layered is false for a GPT-2 configuration (no "architecture" entry), else `out` is filled.
int load_design_config(const std::string& path, bool* layered, LayeredConfig* out);

// Checks every tensor's presence and shape against the configuration and fills in the ranks.
int check_layered_tensors(const SafeTensorsFile& file, const std::string& path, LayeredConfig* cfg);
// A tensor's values as FP32 (BF16 or F32 in the file). The tensor must exist.
std::vector<float> tensor_f32(const SafeTensorsFile& file, const std::string& name);

}  // namespace pg
