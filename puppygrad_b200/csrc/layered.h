// Entry points of the layered models into the common runtime (model.cu): building, cache state, the decode step and
// the pass over portions of prompts.
#pragma once
#include <vector>

#include "design.h"
#include "runtime.h"

namespace pg {

int build_layered_model(const LayeredConfig& cfg, const SafeTensorsFile& file, const pg_backend_config* backend, pg_model** out);
const LayeredConfig& layered_config(const pg_model* m);
// Adds page tables, key / value pools, recurrent states and step buffers to a cache whose common part exists.
int layered_cache_init(pg_cache* c);
int layered_choose_splits(const pg_cache* c, int batch, int max_len);
// One token for slots 0..batch-1 (ids and positions on the device).
cudaError_t layered_enqueue_decode(pg_cache* c, int batch, int splits, cudaStream_t s, uint64_t* launches, StepProfiler* prof);
uint64_t layered_weight_bytes_per_step(const pg_model* m);
uint64_t layered_state_bytes_per_sequence(const pg_model* m);

// Portions of several sequences, rows concatenated. `out_rows` are the rows whose logits are written to `logits`
// [out_rows.size(), vocab] (device). Pages must exist; positions on the host are advanced by the caller.
struct PortionPlan {
  std::vector<int> ids, pos, row_seq;                   // [rows]
  std::vector<int> seq_start, slot, start_pos, out_rows;  // [n + 1], [n], [n]
  int max_len = 0;
  int n() const { return (int)slot.size(); }
  int rows() const { return (int)ids.size(); }
};
int layered_run_portions(pg_cache* c, const PortionPlan& plan, float* logits, StepProfiler* prof);
// Device buffer for the logits of `rows` rows (grow-only).
int layered_logits_buffer(pg_cache* c, size_t rows, float** out);

}  // namespace pg
