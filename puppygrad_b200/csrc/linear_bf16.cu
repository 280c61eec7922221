// Decode-sized products over BF16 weights: at most eight rows of FP32 activations, weights streamed once with 16-byte
// loads, FP32 sums. The input rows can be made by the kernel itself from the residual stream (the LayerNorm after the
// previous sublayer, the residual sum, the LayerNorm before this one).
#include <algorithm>
#include <climits>

#include "device_util.cuh"
#include "layered_kernels.cuh"
#include "norm_step.cuh"

namespace pg {
namespace {

constexpr int RL_THREADS = 512, RL_WARPS = RL_THREADS / 32;
constexpr int RL_ROWS = 2;    // weight rows per warp and unit
constexpr int RL_CHUNK = 256; // columns a warp reads per step: 32 lanes x 8
constexpr int RL_PRE = 4;     // steps whose loads are in flight together
constexpr size_t RL_MAX_SMEM = 200 * 1024;

__device__ __forceinline__ uint4 ldg_weights(const uint4* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// Place of element k of an activation row in shared memory: inside every run of 256 the first halves of the lanes'
// eight values lie together, then the second halves, so that 16-byte reads of a warp do not collide.
__device__ __forceinline__ int act_slot(int k) { return (k & ~255) | ((k & 4) << 5) | ((k >> 1) & 124) | (k & 3); }

// Sum over the `wpr` neighbouring warps that share an activation row.
__device__ __forceinline__ float group_sum(float v, float* red, int warp, int lane, int wpr) {
  v = lane_sum(v);
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const int w0 = warp / wpr * wpr;
  float s = 0.f;
  for (int i = 0; i < wpr; ++i) s += red[w0 + i];
  __syncthreads();
  return s;
}

template <int MT>
__global__ void __launch_bounds__(RL_THREADS, 1) rows_linear_kernel(RowsLinearArgs a, int kp_shift, int kpad) {
  extern __shared__ __align__(16) float xs[];  // [MT][kpad] in act_slot order
  __shared__ float part[RL_WARPS][RL_ROWS * MT];
  __shared__ float red[RL_WARPS];
  __shared__ float best_v[RL_WARPS * RL_ROWS * MT];
  __shared__ int best_i[RL_WARPS * RL_ROWS * MT];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int kparts = 1 << kp_shift, upc = RL_WARPS >> kp_shift;  // parts of k per unit, units per block and round
  const int units = (a.n + RL_ROWS - 1) / RL_ROWS;
  const int steps = kpad / RL_CHUNK;                       // 256-column steps of a row
  const int kp = warp & (kparts - 1), wu = warp >> kp_shift;
  const int s0 = steps * kp / kparts, s1 = steps * (kp + 1) / kparts;
  const uint4* w = static_cast<const uint4*>(a.w);
  const int row16 = a.k / 8;  // 16-byte pieces of a weight row

  grid_dep_launch();
  uint4 pre[RL_PRE][RL_ROWS];
  auto request = [&](int unit, int st) {
#pragma unroll
    for (int j = 0; j < RL_PRE; ++j) {
      const int c = (st + j) * 32 + lane;
#pragma unroll
      for (int r = 0; r < RL_ROWS; ++r) {
        const int row = unit * RL_ROWS + r;
        pre[j][r] = (st + j < s1 && c < row16 && row < a.n) ? ldg_weights(w + (size_t)row * row16 + c) : make_uint4(0, 0, 0, 0);
      }
    }
  };
  // weights do not depend on the previous kernel: the first loads go out before the dependency wait
  // (unit u of round q of this block: units are dealt out over the blocks so that every SM streams its share)
  request(wu * gridDim.x + blockIdx.x, s0);
  if (a.fuse_norm) {  // the norms' vectors too, as far as L2
    const int c = (tid & 127) * 32;
    const float* v = (tid >> 7) == 0 ? a.norm.post_g : (tid >> 7) == 1 ? a.norm.post_b : (tid >> 7) == 2 ? a.norm.pre_g : a.norm.pre_b;
    if (v)
      for (int i = c; i < a.norm.ldx; i += 128 * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(v + i));
  }
  grid_dep_wait();

  if (!a.fuse_norm) {
    for (int i = tid; i < MT * (kpad / 4); i += RL_THREADS) {
      const int m = i / (kpad / 4), k = (i % (kpad / 4)) * 4;
      const float4 v = (m < a.m && k < a.kx) ? mask4(load4(a.x + (size_t)m * a.ldx + k), k, a.kx) : make_float4(0, 0, 0, 0);
      store4(xs + (size_t)m * kpad + act_slot(k), v);
    }
  } else {
    // wpr warps per row; the row stays in shared memory between the passes
    const NormStepArgs& n = a.norm;
    constexpr int WPR = RL_WARPS / MT;
    const int m = warp / WPR, t = (warp % WPR) * 32 + lane, nt = WPR * 32;
    const bool on = m < a.m;
    float* row = xs + (size_t)m * kpad;
    const float inv_n = 1.f / (float)n.width;
    for (int c = n.ldx + t * 4; c < kpad; c += nt * 4) store4(row + act_slot(c), make_float4(0, 0, 0, 0));
    float mean = 0.f, rstd = 0.f;
    if (n.y) {
      float s = 0.f;
      for (int c = t * 4; c < n.ldx; c += nt * 4) {
        const float4 v = on ? mask4(load4(n.y + (size_t)m * n.ldx + c), c, n.width) : make_float4(0, 0, 0, 0);
        store4(row + act_slot(c), v);
        s += (v.x + v.y) + (v.z + v.w);
      }
      if (n.post_g) {
        mean = n.norm == NORM_LAYER ? group_sum(s, red, warp, lane, WPR) * inv_n : 0.f;
        float q = 0.f;
        for (int c = t * 4; c < n.ldx; c += nt * 4) q += norm_step_square(load4(row + act_slot(c)), mean, c, n.width);
        rstd = 1.f / sqrtf(group_sum(q, red, warp, lane, WPR) * inv_n + n.eps);
      }
    }
    float s = 0.f;
    for (int c = t * 4; c < n.ldx; c += nt * 4) {
      float4 x = on ? norm_step_load_x<__nv_bfloat16>(n, m, c) : make_float4(0, 0, 0, 0);
      if (n.y && on) {
        float4 v = load4(row + act_slot(c));
        if (n.post_g) v = norm_step_apply(v, mean, rstd, n.post_g, n.post_b, c, n.width);
        x.x += v.x; x.y += v.y; x.z += v.z; x.w += v.w;
      }
      if (on && n.x_out && blockIdx.x == 0) store4(n.x_out + (size_t)m * n.ldx + c, x);
      store4(row + act_slot(c), x);
      s += (x.x + x.y) + (x.z + x.w);
    }
    mean = n.norm == NORM_LAYER ? group_sum(s, red, warp, lane, WPR) * inv_n : 0.f;
    float q = 0.f;
    for (int c = t * 4; c < n.ldx; c += nt * 4) q += norm_step_square(load4(row + act_slot(c)), mean, c, n.width);
    rstd = 1.f / sqrtf(group_sum(q, red, warp, lane, WPR) * inv_n + n.eps);
    for (int c = t * 4; c < n.ldx; c += nt * 4)
      store4(row + act_slot(c), norm_step_apply(load4(row + act_slot(c)), mean, rstd, n.pre_g, n.pre_b, c, n.width));
  }
  __syncthreads();

  float bv = -INFINITY;
  int bi = INT_MAX;
  for (int round = 0; round * upc * (int)gridDim.x + (int)blockIdx.x < units; ++round) {
    const int unit = (round * upc + wu) * gridDim.x + blockIdx.x;
    float acc[RL_ROWS * MT];
#pragma unroll
    for (int i = 0; i < RL_ROWS * MT; ++i) acc[i] = 0.f;
    for (int st = s0; st < s1; st += RL_PRE) {
      if (st != s0 || round > 0) request(unit, st);
#pragma unroll
      for (int j = 0; j < RL_PRE; ++j) {
        if (st + j < s1) {
          float wv[RL_ROWS][8];
#pragma unroll
          for (int r = 0; r < RL_ROWS; ++r) unpack8(pre[j][r], wv[r]);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            const float* x = xs + (size_t)m * kpad + (st + j) * RL_CHUNK + lane * 4;
            const float4 x0 = load4(x), x1 = load4(x + 128);
#pragma unroll
            for (int r = 0; r < RL_ROWS; ++r) {
              float& c = acc[r * MT + m];
              c = fmaf(wv[r][0], x0.x, c); c = fmaf(wv[r][1], x0.y, c); c = fmaf(wv[r][2], x0.z, c); c = fmaf(wv[r][3], x0.w, c);
              c = fmaf(wv[r][4], x1.x, c); c = fmaf(wv[r][5], x1.y, c); c = fmaf(wv[r][6], x1.z, c); c = fmaf(wv[r][7], x1.w, c);
            }
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < RL_ROWS * MT; ++i) {
      acc[i] = lane_sum(acc[i]);
      if (lane == 0) part[warp][i] = acc[i];
    }
    __syncthreads();
    for (int i = tid; i < upc * RL_ROWS * MT; i += RL_THREADS) {
      const int uu = i / (RL_ROWS * MT), e = i % (RL_ROWS * MT), r = e / MT, m = e % MT;
      float v = 0.f;
      for (int q = 0; q < kparts; ++q) v += part[uu * kparts + q][e];
      const int row = ((round * upc + uu) * (int)gridDim.x + (int)blockIdx.x) * RL_ROWS + r;
      if (row < a.n && m < a.m) {
        if (row >= a.act_from) a.out_act[(size_t)m * a.ldo_act + row - a.act_from] = activate(a.act, v);
        else if (a.out) a.out[(size_t)m * a.ldo + row] = v;
        if (v > bv) {  // a thread's rows only grow: strict > keeps the lowest index
          bv = v;
          bi = row;
        }
      }
    }
    __syncthreads();
  }
  if (!a.part_val) return;
  // i % MT is the activation row of thread i in every round (RL_THREADS is a multiple of MT)
  static_assert(RL_THREADS >= RL_WARPS * RL_ROWS * MT, "one candidate per thread");
  if (tid < upc * RL_ROWS * MT) {
    best_v[tid] = bv;
    best_i[tid] = bi;
  }
  __syncthreads();
  if (tid < a.m) {
    float v = -INFINITY;
    int x = INT_MAX;
    for (int i = tid; i < upc * RL_ROWS * MT; i += MT)
      if (best_v[i] > v || (best_v[i] == v && best_i[i] < x)) {
        v = best_v[i];
        x = best_i[i];
      }
    a.part_val[(size_t)tid * gridDim.x + blockIdx.x] = v;
    a.part_idx[(size_t)tid * gridDim.x + blockIdx.x] = x;
  }
}

int sm_count() {
  static const int n = [] {
    int dev = 0, v = 148;
    cudaGetDevice(&dev);
    if (cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) v = 148;
    return v;
  }();
  return n;
}
int row_tile(int m) { return m <= 1 ? 1 : m <= 2 ? 2 : m <= 4 ? 4 : 8; }
int padded_k(int k) { return (k + RL_CHUNK - 1) / RL_CHUNK * RL_CHUNK; }

// Parts of k: as many as keep every warp of the chip busy in one round, each at least one 256-column step.
int k_part_shift(int n, int k) {
  const int units = (n + RL_ROWS - 1) / RL_ROWS, steps = padded_k(k) / RL_CHUNK;
  int shift = 0;
  while (shift < 4 && ((long long)units << (shift + 1)) <= (long long)sm_count() * RL_WARPS && (steps >> (shift + 1)) >= 1) ++shift;
  return shift;
}

}  // namespace

bool rows_linear_supported(int m, int k, bool fuse_norm, int width) {
  (void)fuse_norm;
  (void)width;
  return m >= 1 && m <= 8 && k % 8 == 0 && (size_t)row_tile(m) * padded_k(k) * sizeof(float) <= RL_MAX_SMEM;
}

int rows_linear_grid(int m, int n, int k) {
  (void)m;
  (void)k;
  return std::max(1, std::min(sm_count(), (n + RL_ROWS - 1) / RL_ROWS));
}

cudaError_t launch_rows_linear(const RowsLinearArgs& a, bool pdl, cudaStream_t s, int* grid_out) {
  if (!rows_linear_supported(a.m, a.k, a.fuse_norm != 0, a.norm.width)) return cudaErrorInvalidValue;
  const int shift = k_part_shift(a.n, a.k), grid = rows_linear_grid(a.m, a.n, a.k), kpad = padded_k(a.k), mt = row_tile(a.m);
  const size_t smem = (size_t)mt * kpad * sizeof(float);
  if (grid_out) *grid_out = grid;
  const dim3 g(grid), b(RL_THREADS);
  cudaError_t e = cudaErrorInvalidValue;
#define PG_RL(MT_)                                                                                                     \
  e = cudaFuncSetAttribute(rows_linear_kernel<MT_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)RL_MAX_SMEM);    \
  return e != cudaSuccess ? e : launch_kernel(rows_linear_kernel<MT_>, g, b, smem, s, pdl, a, shift, kpad)
  if (mt == 1) { PG_RL(1); }
  if (mt == 2) { PG_RL(2); }
  if (mt == 4) { PG_RL(4); }
  PG_RL(8);
#undef PG_RL
}

}  // namespace pg
