// Launch wrappers of the kernels of the layered models. Pointers are device pointers; every wrapper returns the
// cudaError_t of its launch. "T" storage is FP32 or BF16, chosen per model by `bf16`: it is the type of the inputs of
// the matrix products and of cached keys and values. Row pitches are padded to a multiple of eight elements.
#pragma once
#include <cuda_runtime.h>

#include <cstdint>

#include "design.h"

namespace pg {

// ------------------------------------------------------------------ norms.cu
// One row per block: x = (scaled token embedding [+ sinusoidal position] | x_in) [+ y | + norm(y; post)], then h = norm(x; pre).
// All sums in FP32. `norm`: NormKind, or NORM_COPY for h = x.
constexpr int NORM_COPY = 2;
struct NormStepArgs {
  const int* ids;        // [rows] or nullptr: start from the embedding of ids at positions pos
  const int* pos;
  const void* embed;     // [vocab, ld_embed] in T
  int ld_embed;
  float embed_scale;
  const double* freq;    // [ceil(width / 2)] 10000^(-2i / width), or nullptr: no position vectors
  const int* row_index;  // optional: input row of x for every output row (gathered final norm)
  const float* x_in;     // [*, ld_in]
  int ld_in;
  float* x_out;          // [rows, ldx] or nullptr
  const float* y;        // [rows, ldx] sublayer output, or nullptr
  const float *post_g, *post_b;  // nullptr: y is added as it is
  const float *pre_g, *pre_b;    // pre_b: NORM_LAYER only
  void* h;               // [rows, ldh] in T ...
  float* h32;            // ... or in FP32 (when not nullptr); neither: only x_out
  int ldx, ldh, width;   // columns width..ldh of h are zero
  float eps;
  int norm;
};
cudaError_t launch_norm_step(const NormStepArgs& a, int rows, bool bf16, bool pdl, cudaStream_t s);
// The feed-forward's activation: `kind` is an Activation, a and b the learned numbers of ACT_XIELU.
struct ActArgs {
  int kind;
  float a, b;
};
// out[rows, ldo] = act(x[rows, ldx]) for `cols` columns of FP32 rows (the FP32 path's feed-forward; elsewhere it is fused into
// the product); x and out may be the same
cudaError_t launch_activation(const float* x, int ldx, float* out, int ldo, int rows, int cols, ActArgs act, bool pdl, cudaStream_t s);
// FP32 [rows, cols] -> BF16 [rows_padded, ld], zero outside rows x cols
cudaError_t launch_pack_bf16(const float* src, void* dst, int rows, int cols, int rows_padded, int ld, cudaStream_t s);
// BF16 [rows, ld] (ld % 64 == 0) -> tiles [ceil(rows / 128)][ld / 64][128][64], rows past the end zero: one 128 x 64 tile is
// one contiguous 16 KB run, which a decode step streams at full DRAM bandwidth (128 rows of 128 bytes each would not be)
size_t tiled_bf16_elems(int rows, int ld);
cudaError_t launch_tile_bf16(const void* src, void* dst, int rows, int ld, cudaStream_t s);

// ------------------------------------------------------------------ linear_bf16.cu
// out[m, n] = f(x)[m, k] . w[n, k]^T for at most 8 rows, BF16 weights, FP32 activations and sums. `norm` (optional)
// makes x itself (see NormStepArgs), computed by every block, x_out written by the first one (so x_in and x_out must differ).
// Output columns from `act_from` on pass the activation and go to out_act instead.
struct RowsLinearArgs {
  const void* w;   // [n, k] BF16, k % 8 == 0
  const float* x;  // [m, ldx] FP32 (norm_step == nullptr semantics: fuse_norm == 0)
  int ldx, kx;     // columns of x from kx on count as zero
  int fuse_norm;
  NormStepArgs norm;
  float* out;      // [m, ldo]
  int ldo;
  int m, n, k;
  int act_from;    // >= n: none
  ActArgs act;
  float* out_act;  // [m, ldo_act], column act_from first
  int ldo_act;
  float* part_val;  // optional row arg-max candidates per block: [m][grid]
  int* part_idx;
};
bool rows_linear_supported(int m, int k, bool fuse_norm, int width);
int rows_linear_grid(int m, int n, int k);
cudaError_t launch_rows_linear(const RowsLinearArgs& a, bool pdl, cudaStream_t s, int* grid_out);

// ------------------------------------------------------------------ gemm_bf16.cu
// out[m, n] = x[m, k] . w[n, k]^T, BF16 operands, FP32 accumulation (tcgen05 kind::f16), k % 8 == 0.
struct Bf16GemmArgs {
  const void* x;   // [m, k] BF16
  const void* w;   // [n, k] BF16
  const void* w_tiled;  // the same in 128 x 64 tiles (launch_tile_bf16): used for at most 64 rows
  float* out;      // [m, ldo] FP32, or nullptr
  void* out_h;     // [m, ldo] BF16, or nullptr
  int ldo;
  int* error_flag;
  int m, n, k;
  ActArgs act;      // applied to BF16 results
  // decode rows only: columns from act_from on pass the activation and go to out_act (BF16, column act_from first), the others
  // to `out` as they are
  int act_from;     // 0: off
  void* out_act;
  int ldo_act;
  // decode rows only: `heads` products side by side, head h over columns h * x_head.. of x with its own weights (tiled: n rounded up
  // to 128 rows per head) to columns h * out_head.. of out
  int heads, x_head, out_head, ldx;  // heads 0: one product; ldx: row pitch of x
};
// Whether a product of m rows takes the kernel that knows act_from.
bool gemm_bf16_rows_kernel(int m, int k);
cudaError_t launch_tc_gemm_bf16(const Bf16GemmArgs& a, bool pdl, cudaStream_t s);

// ------------------------------------------------------------------ recurrence.cu
// One recurrence branch of one layer (see RecurrenceSpec). Column offsets are into a row of the fused input projection.
struct RecurrenceLayer {
  int kind, heads, kv_heads, dim, vdim, dvp, rank;  // dvp: state row pitch, vdim rounded up to 4
  int off_q, off_k, off_v, off_g, off_a, off_t;  // q (or r), k, v, gate, removal-rate and low-rank columns
  const float* w2;     // [rank, heads * dim]
  const float* b2;     // [heads * dim]
  const float* a_bias; // [heads * dim] (delta)
  const float* norm;   // [vdim] (GLA, channel) or [heads * vdim] (delta)
  // channel delta rule: q, k, v are the `channels` columns from off_q on, off_b the write strengths; the second steps of decay
  // and gate come from a product of their own: columns [0, heads * dim) and [heads * dim, + heads * vdim) of z
  int off_b, taps, channels;
  const float* conv;   // [taps][channels], the current token's tap last
  const float* neg_a;  // [heads] -e^A_log
  float q_scale, inv_tau, eps;
  float out_scale;     // branch scale, applied to the mixer output before the output projection
};
// Floats of one slot's state matrices and of its convolution inputs.
size_t recurrence_state_floats(const RecurrenceLayer& l);
inline size_t recurrence_tap_floats(const RecurrenceLayer& l) { return (size_t)l.taps * l.channels; }
struct RecurrenceStepArgs {  // one new token for slots 0..batch-1
  RecurrenceLayer l;
  const float* p;   // [batch, ldp] input projection
  int ldp;
  const float* z;   // channel: [batch, ldz] second-step projections
  int ldz;
  float* state;     // [slot][head][dim][dvp]
  float* taps;      // channel: [slot][taps][channels], the input of position p at p % taps
  const int* pos;   // [batch]; position 0 starts from a zero state
  void* y;          // [batch, ldy]: this branch's columns of the mixer output, T
  int ldy;
  int batch;
};
cudaError_t launch_recurrence_step(const RecurrenceStepArgs& a, bool y_bf16, bool pdl, cudaStream_t s);
struct RecurrenceScanArgs {  // whole portions of `nseq` sequences
  RecurrenceLayer l;
  const float* p;        // [rows, ldp]
  int ldp, rows, nseq;
  const int* seq_start;  // [nseq + 1] row offsets
  const int* seq_slot;   // [nseq]
  const int* seq_pos;    // [nseq] position of the first row; 0 starts from a zero state
  const int* row_seq;    // [rows]
  const float* z;        // channel: as in RecurrenceStepArgs
  int ldz;
  float* taps;
  int max_len;           // longest portion
  // channel: scratch. Values after the convolution (unit and rate hold k and q, decay and unit_next what reads the state), writes
  // into the state, decay of four tokens and their numbers (see recurrence_scan.cu)
  float *vals, *writes;  // [rows, heads * vdim], [rows, heads * dim]
  float *quad_decay, *quads;  // [recurrence_quads()][heads * dim], [recurrence_quads()][heads][20]
  float* state;
  float *decay, *unit, *rate;  // [rows, heads * dim] scratch: decay; delta: unit key u, a * u ...
  float *unit_next;            // ... and the next token's u times this token's decay
  float *pair;                 // [rows, heads, 4] delta: next u . (a * u), next u . k
  int* error_flag;
  float* out_raw;              // [rows, heads * vdim] scratch: outputs before the head norm
  float* segments;             // scratch of the segmented scan (may be nullptr)
  int seg_tokens, max_segs;    // tokens per segment, segments of the longest sequence (0: one pass)
  void* y;
  int ldy;
};
// Whether a portion is cut into segments that run side by side (long sequences that alone would not fill the chip).
bool recurrence_use_segments(const RecurrenceLayer& l, int nseq, int max_len, int max_segs);
inline size_t recurrence_quads(int rows, int nseq) { return (size_t)rows / 4 + nseq + 1; }
size_t recurrence_segment_floats(const RecurrenceLayer& l, int nseq, int max_segs);
cudaError_t launch_recurrence_scan(const RecurrenceScanArgs& a, bool y_bf16, cudaStream_t s);

// ------------------------------------------------------------------ attn_chunked.cu
// Which cached positions a layer's tokens see, and where they lie. window == 0: position p sees its own block of `span`
// positions up to itself (span = the whole context: everything). window > 0: the last `window` positions and the first `keep`
// of the sequence. A sequence holds at most `span` positions: place() is the cache index of one.
// A portion that starts at position p0 is attended over a workspace: the context() cached positions that its first row
// sees, in order, then its own rows.
struct KeyLife {
  int span, window, keep;
  __host__ __device__ int place(int p) const { return window == 0 ? p % span : p < span ? p : keep + (p - keep) % (span - keep); }
  __host__ __device__ int kept(int p0) const { return window == 0 ? 0 : keep < p0 ? keep : p0; }
  __host__ __device__ int recent(int p0) const {  // first position of the moving part of the context
    if (window == 0) return p0 - p0 % span;
    const int k = kept(p0), lo = p0 - window + 1;
    return lo > k ? lo : k;
  }
  __host__ __device__ int context(int p0) const { return kept(p0) + p0 - recent(p0); }
  __host__ __device__ int context_position(int p0, int w) const { return w < kept(p0) ? w : recent(p0) + w - kept(p0); }
  __host__ __device__ int row(int p0, int p) const { return kept(p0) + p - recent(p0); }  // workspace row of a position >= recent(p0)
  // Row `pos` sees the workspace rows low()..row(), and those below `keep`.
  __host__ __device__ int low(int p0, int pos) const {
    const int lo = window == 0 ? pos / span * span : pos - window + 1, w = kept(p0) + lo - recent(p0);
    return w > 0 ? w : 0;
  }
  // Whether position p is seen by a token after position `end`, or lies in the last one's block.
  __host__ __device__ bool lives(int p, int end) const { return window == 0 ? p / span == end / span : p < keep || p > end - window; }
  bool operator==(const KeyLife& o) const { return span == o.span && window == o.window && keep == o.keep; }
};

// One attention branch (see AttentionSpec). Keys and values are kept ready for use (normed, rotated), in T, rows padded to
// dimp / vdimp; a latent row (vrow == 0) is key and value in one.
struct AttentionLayer {
  int heads, kv_heads, dim, vdim, dimp, vdimp, vrow;  // vrow: pitch of the cached value rows
  int wide;  // page layout: 1: a token's rows of all key heads side by side, 0: a key head's rows of all tokens
  KeyLife life;
  int off_q, off_k, off_v, off_gate;  // off_gate < 0: no gate per head
  const float *q_norm, *k_norm;  // [dim] or nullptr
  int v_norm;
  const float *q_bias, *k_bias, *v_bias;  // or nullptr
  int rot_dims, v_rot;
  const double *rot_freq, *v_freq;        // [rot_dims / 2], [vdim / 2]: radians per position
  const float *mix, *sink;                // [heads][heads], [heads] or nullptr
  float scale, eps, out_scale;
  int page_tokens, pages_per_seq;
};
// Elements of one page: keys [kv_heads][page_tokens][dimp] (wide: [page_tokens][kv_heads][dimp]), then the values alike.
size_t attention_page_elems(const AttentionLayer& l);
bool attention_supported(const AttentionLayer& l);
struct AttentionStepArgs {
  AttentionLayer l;
  const float* p;
  int ldp;
  const float* q;         // latent rows: [batch, heads * dimp] queries against them (FP32 path)
  const void* q16;        // launch_attention_heads_tc: [batch, heads * attention_q_width()] BF16 queries
  int num_pages;          // of the pool
  void* pool;
  const int* page_table;  // [slot][pages_per_seq]
  const int* pos;
  float* part;            // [batch * heads][splits][attention_part_floats()]
  unsigned* counters;     // [batch * max(kv_heads, heads)], zero between launches
  void* y;
  int ldy, ldyh, batch, splits;  // ldyh: columns between the outputs of two heads (the merge clears those past vdim)
  int* error_flag;
};
// A part of one head's result: maximum, sum, (padding), sums of values.
inline int attention_part_floats(const AttentionLayer& l) { return 4 + (l.vdim + 3) / 4 * 4; }
// One block per key head: no rotation, mixing, sink, window or latent rows.
cudaError_t launch_attention_step(const AttentionStepArgs& a, bool bf16, bool y_bf16, bool pdl, cudaStream_t s);
struct AttentionPortionArgs {
  AttentionLayer l;
  const float* p;
  int ldp, rows, nseq, max_len, krows;
  const int* seq_start;   // [nseq + 1] first row of each sequence
  const int* key_start;   // [nseq + 1] first row of each sequence in the key / value workspace
  const int* seq_slot;    // [nseq]
  const int* seq_pos;     // [nseq] position of the first row
  const int* row_seq;     // [rows] sequence of each row
  const float2 *rot, *v_rot;  // (cos, sin) of every row: [rows][rot_dims / 2], [rows][vdim / 2]
  const int* step_pos;    // one new token of slot `row` per row, at this position: keys and values go straight to the pages
  void* pool;
  const int* page_table;
  void *q, *k, *v;        // workspaces in T: [rows][heads * q_width()], [krows][ldk], [krows][ldv]
  int ldk, ldv;
  int* error_flag;
  void* y;
  int ldy;
};
// With mixed heads the mixing is moved to the queries: head h scores all key heads at once, against the whole row of keys.
__host__ __device__ inline int attention_q_width(const AttentionLayer& l) { return l.mix ? l.kv_heads * l.dimp : l.dimp; }
// Makes the rows' queries, keys and values ready in the workspaces, copies the cached keys and values that the first rows
// still see in front of them, attends, and stores what later tokens can still see into the pages.
cudaError_t launch_attention_portion(const AttentionPortionArgs& a, bool bf16, cudaStream_t s);
// Its parts: cached rows into the workspaces; attention over them; workspace rows into the pages.
cudaError_t launch_attention_context(const AttentionPortionArgs& a, bool bf16, cudaStream_t s);
cudaError_t launch_attention_core(const AttentionPortionArgs& a, bool bf16, cudaStream_t s);
cudaError_t launch_attention_store(const AttentionPortionArgs& a, bool bf16, cudaStream_t s);
cudaError_t launch_attention_tc(const AttentionPortionArgs& a, cudaStream_t s);  // the products of BF16 portions on the tensor cores

// ------------------------------------------------------------------ attn_heads.cu
// One token per sequence, all heads of it in a block: rotation, mixed heads, sink, window with kept first tokens, latent rows.
// Makes its queries, keys and values itself and appends the new token.
cudaError_t launch_attention_heads_step(const AttentionStepArgs& a, bool bf16, bool y_bf16, bool pdl, cudaStream_t s);
bool attention_heads_supported(const AttentionLayer& l);
// out[rows][half] = (cos, sin) of pos * freq
cudaError_t launch_angles(const int* pos, const double* freq, float2* out, int rows, int half, bool pdl, cudaStream_t s);
// The rows' rotated and mixed queries, rotated keys and values, into the workspaces (a step's keys and values into the pages).
cudaError_t launch_attention_rotate(const AttentionPortionArgs& a, bool bf16, cudaStream_t s, bool pdl = false);
// The rows' normed latents into the key workspace (a step's into the pages).
cudaError_t launch_attention_latent(const AttentionPortionArgs& a, bool bf16, cudaStream_t s, bool pdl = false);
// Turns FP32 outputs back by their rows' angles, in place.
cudaError_t launch_attention_turn_back(const AttentionPortionArgs& a, cudaStream_t s);
// Adds the parts of a step's heads: sink, turning back, gate, branch scale; y in FP32 or BF16.
cudaError_t launch_attention_merge(const AttentionStepArgs& a, const float2* v_rot, bool y_bf16, bool pdl, cudaStream_t s);

// ------------------------------------------------------------------ attn_heads_tc.cu
// One token per sequence on the tensor cores, for heads that share wide key rows (mixed heads, latent rows): BF16 queries a.q16
// against the cached rows, results as parts for launch_attention_merge. The new token's row must be in its page.
bool attention_heads_tc_supported(const AttentionLayer& l);
int attention_heads_tc_splits(const AttentionLayer& l, int batch, int tiles, int sms);  // parts for `tiles` tiles of 128 keys
cudaError_t launch_attention_heads_tc(const AttentionStepArgs& a, bool pdl, cudaStream_t s);

// ------------------------------------------------------------------ attn_heads.cu
// out[b, h * ldh + n] = sum_k x[b, h * ldxh + k] w[h][k][n], w in T with rows of np (a multiple of 8)
struct HeadProductArgs {
  const void* w;
  const float* x;
  int ldx, ldxh;
  void* out;
  int ldo, ldh;
  int batch, heads, k, n, np;
};
cudaError_t launch_head_product(const HeadProductArgs& a, bool bf16, bool out_bf16, bool pdl, cudaStream_t s);

}  // namespace pg
