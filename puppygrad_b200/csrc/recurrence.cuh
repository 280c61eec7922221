// Arithmetic that the single-token step and the scan of the recurrent mixers share.
#pragma once
#include "device_util.cuh"
#include "layered_kernels.cuh"

namespace pg {
namespace {

enum { KIND_GLA = RECUR_GLA, KIND_DELTA = RECUR_DELTA, KIND_CHANNEL = RECUR_CHANNEL };
constexpr float DELTA_RATE = 0.60653065971263342f;  // e^-1/2: the strongest decay per token is exp(-DELTA_RATE)
constexpr float UNIT_EPS = 1e-6f;

__device__ __forceinline__ float decay_of(int kind, float z, float inv_tau) {
  return kind == KIND_GLA ? expf(log_sigmoid(z) * inv_tau) : expf(-DELTA_RATE * sigmoid_f(z));
}

__device__ __forceinline__ float softplus_f(float z) { return -log_sigmoid(-z); }

// Channel delta rule: decay of one key channel from the second-step projection.
__device__ __forceinline__ float channel_decay(const RecurrenceLayer& l, int head, int ch, float z) {
  return expf(l.neg_a[head] * softplus_f(z + l.b2[ch]));
}

// A convolution input `back` tokens before row r (position pos, portion from row `first` on): from the portion, from the
// cached inputs in front of it, or zero before the sequence's start.
__device__ __forceinline__ float conv_input(const RecurrenceLayer& l, const float* p, int ldp, const float* taps, int r, int first, int pos, int back, int ch) {
  if (r - back >= first) return p[(size_t)(r - back) * ldp + l.off_q + ch];
  return pos - back >= 0 ? taps[(size_t)((pos - back) % l.taps) * l.channels + ch] : 0.f;
}

}  // namespace
}  // namespace pg
