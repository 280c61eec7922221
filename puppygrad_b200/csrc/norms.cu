// Row kernels of the layered models: embedding with sinusoidal positions, LayerNorm or RMS norm before and after a sublayer
// fused with the FP32 residual sum, activations, weight packing.
#include "device_util.cuh"
#include "layered_kernels.cuh"
#include "norm_step.cuh"

namespace pg {
namespace {

constexpr int NORM_THREADS = 256;

template <int V4, typename T>
__global__ void __launch_bounds__(NORM_THREADS) norm_step_kernel(NormStepArgs a) {
  __shared__ float red[33];
  grid_dep_launch();
  grid_dep_wait();
  const int row = blockIdx.x, tid = threadIdx.x;
  float4 x[V4];
#pragma unroll
  for (int j = 0; j < V4; ++j) {
    const int c = (tid + j * NORM_THREADS) * 4;
    x[j] = c < a.ldx ? norm_step_load_x<T>(a, row, c) : make_float4(0, 0, 0, 0);
  }
  const float inv_n = 1.f / (float)a.width;
  auto moments = [&](const float4 (&v)[V4], float* mean, float* rstd) {
    *mean = 0.f;
    if (a.norm == NORM_LAYER) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < V4; ++j) s += (v[j].x + v[j].y) + (v[j].z + v[j].w);  // columns past width are zero
      *mean = block_sum(s, red) * inv_n;
    }
    float q = 0.f;
#pragma unroll
    for (int j = 0; j < V4; ++j) q += norm_step_square(v[j], *mean, (tid + j * NORM_THREADS) * 4, a.width);
    *rstd = 1.f / sqrtf(block_sum(q, red) * inv_n + a.eps);
  };
  if (a.y) {
    float4 y[V4];
#pragma unroll
    for (int j = 0; j < V4; ++j) {
      const int c = (tid + j * NORM_THREADS) * 4;
      y[j] = c < a.ldx ? mask4(load4(a.y + (size_t)row * a.ldx + c), c, a.width) : make_float4(0, 0, 0, 0);
    }
    float mean = 0.f, rstd = 1.f;
    if (a.post_g) moments(y, &mean, &rstd);
#pragma unroll
    for (int j = 0; j < V4; ++j) {
      const int c = (tid + j * NORM_THREADS) * 4;
      if (c < a.width) {
        const float4 n = a.post_g ? norm_step_apply(y[j], mean, rstd, a.post_g, a.post_b, c, a.width) : y[j];
        x[j].x += n.x; x[j].y += n.y; x[j].z += n.z; x[j].w += n.w;
      }
    }
  }
  if (a.x_out) {
#pragma unroll
    for (int j = 0; j < V4; ++j) {
      const int c = (tid + j * NORM_THREADS) * 4;
      if (c < a.ldx) store4(a.x_out + (size_t)row * a.ldx + c, x[j]);
    }
  }
  if (a.h || a.h32) {
    float mean = 0.f, rstd = 1.f;
    if (a.norm != NORM_COPY) moments(x, &mean, &rstd);
#pragma unroll
    for (int j = 0; j < V4; ++j) {
      const int c = (tid + j * NORM_THREADS) * 4;
      if (c < a.ldh) {
        const float4 n = a.norm == NORM_COPY ? x[j] : norm_step_apply(x[j], mean, rstd, a.pre_g, a.pre_b, c, a.width);
        if (a.h32) store4(a.h32 + (size_t)row * a.ldh + c, n);
        else store4(static_cast<T*>(a.h) + (size_t)row * a.ldh + c, n);
      }
    }
  }
}

template <typename T>
cudaError_t launch_norm_step_t(const NormStepArgs& a, int rows, bool pdl, cudaStream_t s) {
  const int per = NORM_THREADS * 4;
  const dim3 g(rows), b(NORM_THREADS);
  if (a.ldx <= per) return launch_kernel(norm_step_kernel<1, T>, g, b, 0, s, pdl, a);
  if (a.ldx <= 2 * per) return launch_kernel(norm_step_kernel<2, T>, g, b, 0, s, pdl, a);
  if (a.ldx <= 4 * per) return launch_kernel(norm_step_kernel<4, T>, g, b, 0, s, pdl, a);
  if (a.ldx <= 8 * per) return launch_kernel(norm_step_kernel<8, T>, g, b, 0, s, pdl, a);
  if (a.ldx <= 16 * per) return launch_kernel(norm_step_kernel<16, T>, g, b, 0, s, pdl, a);
  return cudaErrorInvalidValue;
}

__global__ void __launch_bounds__(256) activation_kernel(const float* x, int ldx, float* out, int ldo, int rows, int cols, ActArgs act) {
  grid_dep_launch();
  grid_dep_wait();
  const size_t n = (size_t)rows * cols;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const size_t r = i / cols, c = i % cols;
    out[r * ldo + c] = activate(act, x[r * ldx + c]);
  }
}

__global__ void __launch_bounds__(256) pack_bf16_kernel(const float* __restrict__ src, __nv_bfloat16* dst, int rows, int cols,
                                                        int rows_padded, int ld) {
  const size_t n = (size_t)rows_padded * ld;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const int r = (int)(i / ld), c = (int)(i % ld);
    dst[i] = __float2bfloat16_rn(r < rows && c < cols ? src[(size_t)r * cols + c] : 0.f);
  }
}

__global__ void __launch_bounds__(256) tile_bf16_kernel(const uint4* __restrict__ src, uint4* __restrict__ dst, int rows, int ld) {
  const int nkb = ld / 64;
  const size_t n = (size_t)((rows + 127) / 128) * nkb * 128 * 8;  // 16-byte pieces
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
    const int piece = (int)(i & 7), r = (int)((i >> 3) & 127);
    const size_t tile = i >> 10;
    const int kb = (int)(tile % nkb);
    const size_t row = tile / nkb * 128 + r;
    dst[i] = row < (size_t)rows ? src[row * (ld / 8) + kb * 8 + piece] : make_uint4(0, 0, 0, 0);
  }
}

int grid_for(size_t n) { return (int)((n + 255) / 256 < 1184 ? (n + 255) / 256 : 1184); }

}  // namespace

cudaError_t launch_norm_step(const NormStepArgs& a, int rows, bool bf16, bool pdl, cudaStream_t s) {
  if (rows <= 0) return cudaSuccess;
  return bf16 ? launch_norm_step_t<__nv_bfloat16>(a, rows, pdl, s) : launch_norm_step_t<float>(a, rows, pdl, s);
}

cudaError_t launch_activation(const float* x, int ldx, float* out, int ldo, int rows, int cols, ActArgs act, bool pdl, cudaStream_t s) {
  if (rows <= 0 || cols <= 0) return cudaSuccess;
  return launch_kernel(activation_kernel, dim3(grid_for((size_t)rows * cols)), dim3(256), 0, s, pdl, x, ldx, out, ldo, rows, cols, act);
}

size_t tiled_bf16_elems(int rows, int ld) { return (size_t)((rows + 127) / 128) * 128 * ld; }

cudaError_t launch_tile_bf16(const void* src, void* dst, int rows, int ld, cudaStream_t s) {
  if (ld % 64 != 0) return cudaErrorInvalidValue;
  return launch_kernel(tile_bf16_kernel, dim3(1184), dim3(256), 0, s, false, static_cast<const uint4*>(src), static_cast<uint4*>(dst), rows, ld);
}

cudaError_t launch_pack_bf16(const float* src, void* dst, int rows, int cols, int rows_padded, int ld, cudaStream_t s) {
  return launch_kernel(pack_bf16_kernel, dim3(grid_for((size_t)rows_padded * ld)), dim3(256), 0, s, false, src,
                       static_cast<__nv_bfloat16*>(dst), rows, cols, rows_padded, ld);
}

}  // namespace pg
