// Launch wrappers of the kernels of the layered models. Pointers are device pointers; every wrapper returns the
// cudaError_t of its launch. "T" storage is FP32 or BF16, chosen per model by `bf16`: it is the type of the inputs of
// the matrix products and of cached keys and values. Row pitches are padded to a multiple of eight elements.
#pragma once
#include <cuda_runtime.h>

#include <cstdint>

namespace pg {

// ------------------------------------------------------------------ norms.cu
// One row per block: x = (token embedding + sinusoidal position | x_in) [+ LayerNorm(y; post)], then
// h = LayerNorm(x; pre). All sums in FP32.
struct NormStepArgs {
  const int* ids;        // [rows] or nullptr: start from the embedding of ids at positions pos
  const int* pos;
  const void* embed;     // [vocab, ld_embed] in T
  int ld_embed;
  const double* freq;    // [ceil(width / 2)] 10000^(-2i / width)
  const int* row_index;  // optional: input row of x for every output row (gathered final norm)
  const float* x_in;     // [*, ldx]
  float* x_out;          // [rows, ldx] or nullptr
  const float* y;        // [rows, ldx] sublayer output, or nullptr
  const float *post_g, *post_b;
  const float *pre_g, *pre_b;  // nullptr: no h
  void* h;               // [rows, ldh] in T ...
  float* h32;            // ... or in FP32 (when not nullptr)
  int ldx, ldh, width;
  float eps;
};
cudaError_t launch_norm_step(const NormStepArgs& a, int rows, bool bf16, bool pdl, cudaStream_t s);
// in-place exact gelu of an FP32 array (the FP32 path's feed-forward; elsewhere it is fused into the product)
cudaError_t launch_gelu_erf(float* x, size_t n, bool pdl, cudaStream_t s);
// FP32 [rows, cols] -> BF16 [rows_padded, ld], zero outside rows x cols
cudaError_t launch_pack_bf16(const float* src, void* dst, int rows, int cols, int rows_padded, int ld, cudaStream_t s);
// BF16 [rows, ld] (ld % 64 == 0) -> tiles [ceil(rows / 128)][ld / 64][128][64], rows past the end zero: one 128 x 64 tile is
// one contiguous 16 KB run, which a decode step streams at full DRAM bandwidth (128 rows of 128 bytes each would not be)
size_t tiled_bf16_elems(int rows, int ld);
cudaError_t launch_tile_bf16(const void* src, void* dst, int rows, int ld, cudaStream_t s);

// ------------------------------------------------------------------ linear_bf16.cu
// out[m, n] = f(x)[m, k] . w[n, k]^T for at most 8 rows, BF16 weights, FP32 activations and sums. `norm` (optional)
// makes x itself: x_out = x_in + LayerNorm(y; post), x = LayerNorm(x_out; pre), computed by every block, x_out written
// by the first one (so x_in and x_out must differ).
enum RowsEpilogue { ROWS_NONE = 0, ROWS_GELU_ERF = 1 };
struct RowsLinearArgs {
  const void* w;   // [n, k] BF16, k % 8 == 0
  const float* x;  // [m, ldx] FP32 (norm_step == nullptr semantics: fuse_norm == 0)
  int ldx;
  int fuse_norm;
  NormStepArgs norm;
  float* out;      // [m, ldo]
  int ldo;
  int m, n, k, epilogue;
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
  int gelu_erf;
};
cudaError_t launch_tc_gemm_bf16(const Bf16GemmArgs& a, bool pdl, cudaStream_t s);

// ------------------------------------------------------------------ recurrence.cu
// One recurrence branch of one layer (see RecurrenceSpec). Column offsets are into a row of the fused input projection.
struct RecurrenceLayer {
  int kind, heads, dim, vdim, dvp, rank;  // dvp: state row pitch, vdim rounded up to 4
  int off_q, off_k, off_v, off_g, off_a, off_t;  // q (or r), k, v, gate, removal-rate and low-rank columns
  const float* w2;     // [heads * dim, rank]
  const float* b2;     // [heads * dim]
  const float* a_bias; // [heads * dim] (delta)
  const float* norm;   // [vdim] (GLA) or [heads * vdim] (delta)
  float q_scale, inv_tau, eps;
  float out_scale;     // branch scale, applied to the mixer output before the output projection
};
// Floats of one slot's state.
size_t recurrence_state_floats(const RecurrenceLayer& l);
struct RecurrenceStepArgs {  // one new token for slots 0..batch-1
  RecurrenceLayer l;
  const float* p;   // [batch, ldp] input projection
  int ldp;
  float* state;     // [slot][head][dim][dvp]
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
size_t recurrence_segment_floats(const RecurrenceLayer& l, int nseq, int max_segs);
cudaError_t launch_recurrence_scan(const RecurrenceScanArgs& a, bool y_bf16, cudaStream_t s);

// ------------------------------------------------------------------ attn_chunked.cu
// One attention branch (see AttentionSpec). Keys and values are kept normed, in T, rows padded to dimp / vdimp.
struct AttentionLayer {
  int heads, kv_heads, dim, vdim, dimp, vdimp, span;  // span: keys of positions p and q share a block iff p / span == q / span
  int off_q, off_k, off_v;
  const float *q_norm, *k_norm;  // [dim] or nullptr
  int v_norm;
  float scale, eps, out_scale;
  int page_tokens, pages_per_seq;
};
size_t attention_page_elems(const AttentionLayer& l);  // elements of one page: [kv_heads][page_tokens][dimp] keys, then values
bool attention_supported(const AttentionLayer& l);
struct AttentionStepArgs {
  AttentionLayer l;
  const float* p;
  int ldp;
  void* pool;
  const int* page_table;  // [slot][pages_per_seq]
  const int* pos;
  float* part;            // [batch * heads][splits][vdim + 2]
  unsigned* counters;     // [batch * kv_heads], zero between launches
  void* y;
  int ldy, batch, splits;
};
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
  void* pool;
  const int* page_table;
  void *q, *k, *v;        // workspaces in T: [rows][heads * dimp], [krows][kv_heads * dimp], [krows][kv_heads * vdimp]
  int* error_flag;
  void* y;
  int ldy;
};
// Norms the rows' queries, keys and values into the workspaces, copies the cached keys and values that the first rows
// still see in front of them, attends, and stores what later tokens can still see into the pages.
cudaError_t launch_attention_tc(const AttentionPortionArgs& a, cudaStream_t s);  // the products of BF16 portions on the tensor cores
cudaError_t launch_attention_portion(const AttentionPortionArgs& a, bool bf16, cudaStream_t s);

}  // namespace pg
