// BF16 tensor-core products of the layered models (sm_100a): tcgen05.mma kind::f16, operands staged by TMA with
// 128-byte swizzle, FP32 accumulators in tensor memory, warp-specialised roles, bounded waits.
//
//   tc_gemm_bf16_kernel  out[m, n] = x[m, k] . w[n, k]^T for whole portions of prompts and for batches of decode rows.
//
// On an expired wait the kernel raises the error flag, stops issuing work, still frees its tensor memory and returns.
#include <algorithm>

#include "device_util.cuh"
#include "layered_kernels.cuh"
#include "tc_common.cuh"

namespace pg {
namespace {

constexpr int KB = 64;  // BF16 elements per k block: one 128-byte swizzle row

template <int BN>
struct BfSmem {
  static constexpr int STAGES = (BN == 256) ? 4 : 6;
  static constexpr int A_BYTES = TILE_M * KB * 2, B_BYTES = BN * KB * 2;
  static constexpr int EPI_BYTES = 4 * 32 * 33 * 4;  // one padded 32x32 transpose tile per epilogue warp
  static constexpr size_t BYTES = (size_t)STAGES * (A_BYTES + B_BYTES) + EPI_BYTES + 1024 /*align*/ + 256 /*barriers*/;
};

// Persistent over 128 x BN output tiles; two accumulators in tensor memory, so that the epilogue of a tile overlaps the
// products of the next. Warp 0 loads, warp 1 issues the MMAs and owns the tensor memory, warps 2..5 store.
template <int BN>
__global__ void __launch_bounds__(192, 1)
    tc_gemm_bf16_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, Bf16GemmArgs a) {
  using S = BfSmem<BN>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* smem_a = base;
  uint8_t* smem_b = base + (size_t)S::STAGES * S::A_BYTES;
  float* epi_tiles = reinterpret_cast<float*>(smem_b + (size_t)S::STAGES * S::B_BYTES);
  uint64_t* full = reinterpret_cast<uint64_t*>(reinterpret_cast<uint8_t*>(epi_tiles) + S::EPI_BYTES);
  uint64_t* empty = full + S::STAGES;
  uint64_t* d_full = empty + S::STAGES;  // [2]: accumulator holds a finished tile
  uint64_t* d_empty = d_full + 2;        // [2]: the epilogue warps have read it
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(d_empty + 2);
  volatile int* failed = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tiles_m = (a.m + TILE_M - 1) / TILE_M, tiles_n = (a.n + BN - 1) / BN, tiles = tiles_n * tiles_m;
  const int nkb = (a.k + KB - 1) / KB;

  if (threadIdx.x == 0) {
    for (int s = 0; s < S::STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&d_full[i], 1);
      mbar_init(&d_empty[i], 4);
    }
    *failed = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(tmem_slot, 2 * BN);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch();
  pdl_wait();

  if (warp == 0) {
    if (lane == 0) {
      uint32_t it = 0;  // stage counter over all tiles of this block
      bool ok = true;
      for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
        const int n0 = (tile % tiles_n) * BN, m0 = (tile / tiles_n) * TILE_M;
        for (int kb = 0; kb < nkb; ++kb, ++it) {
          const uint32_t s = it % S::STAGES;
          if (it >= S::STAGES) ok = mbar_wait(&empty[s], ((it / S::STAGES) - 1) & 1, failed, a.error_flag, 1);
          if (!ok) break;
          mbar_expect_tx(&full[s], S::A_BYTES + S::B_BYTES);
          tma_load_2d(smem_a + (size_t)s * S::A_BYTES, &map_x, kb * KB, m0, &full[s]);
          tma_load_2d(smem_b + (size_t)s * S::B_BYTES, &map_w, kb * KB, n0, &full[s]);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = umma_idesc_bf16(TILE_M, BN);
      uint32_t it = 0, ti = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++ti) {
        const uint32_t buf = ti & 1;
        if (ti >= 2) ok = mbar_wait(&d_empty[buf], ((ti >> 1) - 1) & 1, failed, a.error_flag, 4);
        if (!ok) break;
        tc_fence_after();
        const uint32_t tmem_d = tmem_base + buf * BN;
        for (int kb = 0; kb < nkb && ok; ++kb, ++it) {
          const uint32_t s = it % S::STAGES;
          ok = mbar_wait(&full[s], (it / S::STAGES) & 1, failed, a.error_flag, 2);
          if (!ok) break;
          tc_fence_after();
          const uint64_t da = umma_desc_sw128(smem_a + (size_t)s * S::A_BYTES);
          const uint64_t db = umma_desc_sw128(smem_b + (size_t)s * S::B_BYTES);
#pragma unroll
          for (int k = 0; k < KB / 16; ++k)
            umma_bf16_ss(tmem_d, da + (uint64_t)(k * 2), db + (uint64_t)(k * 2), idesc, (kb | k) != 0);
          umma_commit(&empty[s]);
        }
        if (ok) umma_commit(&d_full[buf]);
      }
    }
  } else {
    const int q = warp & 3;  // tensor-memory lane quarter of this warp
    float* tile_s = epi_tiles + (size_t)(warp - 2) * 32 * 33;
    uint32_t ti = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++ti) {
      const int n0 = (tile % tiles_n) * BN, m0 = (tile / tiles_n) * TILE_M;
      const uint32_t buf = ti & 1, tmem_d = tmem_base + buf * BN;
      ok = mbar_wait(&d_full[buf], (ti >> 1) & 1, failed, a.error_flag, 3);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
#pragma unroll 1
      for (int c0 = 0; c0 < BN; c0 += 32) {
        if (n0 + c0 >= a.n) break;  // whole block of columns outside
        float v[32];
        tmem_ld32(tmem_d + ((uint32_t)(q * 32) << 16) + (uint32_t)c0, v);
        if (a.gelu_erf) {
#pragma unroll
          for (int j = 0; j < 32; ++j) v[j] = gelu_erf(v[j]);
        }
#pragma unroll
        for (int j = 0; j < 32; ++j) tile_s[lane * 33 + j] = v[j];
        __syncwarp();
        const int col = n0 + c0 + lane;
        if (col < a.n) {
#pragma unroll
          for (int rr = 0; rr < 32; ++rr) {
            const int row = m0 + q * 32 + rr;
            if (row < a.m) {
              const float r = tile_s[rr * 33 + lane];
              if (a.out) a.out[(size_t)row * a.ldo + col] = r;
              if (a.out_h) static_cast<__nv_bfloat16*>(a.out_h)[(size_t)row * a.ldo + col] = __float2bfloat16_rn(r);
            }
          }
        }
        __syncwarp();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&d_empty[buf]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 2 * BN);
}

template <int BN>
cudaError_t launch_bn(const Bf16GemmArgs& a, bool pdl, cudaStream_t s) {
  CUtensorMap mx, mw;
  if (!make_map_bf16(&mx, a.x, a.m, a.k, TILE_M) || !make_map_bf16(&mw, a.w, a.n, a.k, BN)) return cudaErrorInvalidValue;
  const size_t smem = BfSmem<BN>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(tc_gemm_bf16_kernel<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  int dev = 0, sms = 148;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  const int tiles = ((a.m + TILE_M - 1) / TILE_M) * ((a.n + BN - 1) / BN);
  return launch_kernel(tc_gemm_bf16_kernel<BN>, dim3(std::min(tiles, sms)), dim3(192), smem, s, pdl, mx, mw, a);
}

}  // namespace

cudaError_t launch_tc_gemm_bf16(const Bf16GemmArgs& a, bool pdl, cudaStream_t s) {
  if (a.m <= 0 || a.n <= 0) return cudaSuccess;
  if (a.k <= 0 || a.k % 8 != 0) return cudaErrorInvalidValue;
  const long long m_tiles = (a.m + TILE_M - 1) / TILE_M;
  if (m_tiles * ((a.n + 255) / 256) >= 148) return launch_bn<256>(a, pdl, s);
  if (m_tiles * ((a.n + 127) / 128) >= 100) return launch_bn<128>(a, pdl, s);
  return launch_bn<64>(a, pdl, s);
}

}  // namespace pg
