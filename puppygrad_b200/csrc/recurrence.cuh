// Arithmetic that the single-token step and the scan of the recurrent mixers share.
#pragma once
#include "device_util.cuh"
#include "layered_kernels.cuh"

namespace pg {
namespace {

enum { KIND_GLA = 0, KIND_DELTA = 1 };
constexpr float DELTA_RATE = 0.60653065971263342f;  // e^-1/2: the strongest decay per token is exp(-DELTA_RATE)
constexpr float UNIT_EPS = 1e-6f;

__device__ __forceinline__ float decay_of(int kind, float z, float inv_tau) {
  return kind == KIND_GLA ? expf(log_sigmoid(z) * inv_tau) : expf(-DELTA_RATE * sigmoid_f(z));
}

}  // namespace
}  // namespace pg
