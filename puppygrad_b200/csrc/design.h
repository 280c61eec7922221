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
  // which j <= i position i sees: chunk > 0: those in its own block of `chunk` positions; window > 0: the last `window`
  // ones (itself included) and the first `keep_first` of the sequence; neither: all
  int chunk = 0;
  int window = 0, keep_first = 0;
  bool bias = false;       // q, k and v have biases
  int rot_dims = 0;        // the first rot_dims entries of q and k are rotated: entry i with entry i + rot_dims / 2
  double rot_base = 0;     // ... by position * rot_base^(-2i / rot_dims)
  bool v_rot = false;      // values rotated by their position over all of vdim, outputs turned back by the query's
  bool head_mix = false;   // scores of the heads are mixed before the softmax (a [heads, heads] matrix)
  bool sink = false;       // a learned number per head joins the softmax denominator
  bool head_gate = false;  // each head's output is multiplied by a sigmoid of its own projection
  // > 0: latent attention. q = W_uq norm(W_dq h), and keys and values of every head come from one normed latent row of
  // kv_rank numbers per token, which is all that is cached (kv_heads is then 1)
  int q_rank = 0, kv_rank = 0;
};

// A recurrence over tokens whose state is one [dim, vdim] FP32 matrix per head.
//  RECUR_GLA    S = diag(alpha) S + k v^T, alpha = sigmoid(A2 (A1 h) + b)^(1/tau); out = S^T (q / sqrt(dim)); the
//               per-head RMS norm has a weight of size vdim shared by the heads, the gate is silu
//  RECUR_DELTA  S = diag(w) S - (a * u) (u^T S) + k v^T, w = exp(-e^-1/2 * sigmoid(W2 tanh(W1 h) + w0)),
//               a = sigmoid(W_a h + b), u = k / sqrt(|k|^2 + 1e-6); out = S^T r; the per-head RMS norm has no weight of
//               its own, the concatenation is multiplied by a weight of all heads' size and the gate is sigmoid
//  RECUR_CHANNEL  S = diag(g) S, then S = S + k u^T with u = beta (v - S^T k); out = S^T q (after the write). q, k and v pass
//               a short causal convolution and silu, q and k are unit vectors (q times dim^-1/2) shared by groups of heads;
//               g = exp(-e^A_log softplus(A2 (A1 h) + b)) per key channel, beta = sigmoid(W_b h) per head; the per-head RMS
//               norm has a weight of size vdim, the gate is sigmoid(G2 (G1 h))
enum RecurrenceKind { RECUR_GLA = 0, RECUR_DELTA = 1, RECUR_CHANNEL = 2 };
struct RecurrenceSpec {
  int kind = RECUR_GLA;
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;  // kv_heads: heads of q and k (the others: one per head)
  float tau = 1.f;
  int conv = 0;   // taps of the short convolution, the current token's included
  int rank = 0;   // inner size of the two-step decay projection, from the tensors' shapes
  int rank2 = 0;  // ... and of the two-step gate projection
};

// One branch of a layer's mixer; branches read the same input and their results are added, each times its scale.
struct BranchSpec {
  enum Kind { ATTENTION = 0, RECURRENCE = 1, LATENT = 2 } kind = ATTENTION;  // LATENT: attn with kv_rank > 0
  AttentionSpec attn;
  RecurrenceSpec rec;
  float scale = 1.f;
  std::string prefix;  // tensors of this branch: "<layer prefix>.<prefix>.<name>"
  int out_dim() const { return kind == RECURRENCE ? rec.heads * rec.vdim : attn.heads * attn.vdim; }
};

enum NormKind { NORM_LAYER = 0, NORM_RMS = 1 };  // LayerNorm with weight and bias; weight times x over its root mean square
enum Activation {
  ACT_NONE = 0,
  ACT_GELU_ERF = 1,
  ACT_XIELU = 2  // a z^2 + z / 2 above 0, b (e^z - 1 - z) + z / 2 below, a = softplus(p), b = 1/2 + softplus(q), p and q learned
};

struct LayerSpec {
  std::string type;
  std::vector<BranchSpec> branches;
  int ff = 0;  // 0: no feed-forward; else W_down act(W_up h)
};

struct LayeredConfig {
  std::string architecture;
  int vocab = 0, width = 0;
  float norm_eps = 1e-5f;  // every norm of the model
  int norm_kind = NORM_LAYER;
  int activation = ACT_GELU_ERF;
  bool post_norms = true;    // x += norm(sublayer(norm(x))); false: x += sublayer(norm(x))
  bool parallel_ff = false;  // mixer and feed-forward read the same normed input: x += mixer(norm(x)) + ff(norm(x))
  bool sinusoids = true;     // sinusoidal position vectors are added to the embedding
  float embed_scale = 1.f;
  bool tied_head = true;     // output projection = token embedding; false: tensor `head`
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
