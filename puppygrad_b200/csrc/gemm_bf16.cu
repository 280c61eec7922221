// BF16 tensor-core products of the layered models (sm_100a): tcgen05.mma kind::f16, operands staged by TMA with
// 128-byte swizzle, FP32 accumulators in tensor memory, warp-specialised roles, bounded waits.
//
//   tc_gemm_bf16_kernel       out[m, n] = x[m, k] . w[n, k]^T for whole portions of prompts: 128 x BN tiles of the
//                             output, persistent, results leave through shared memory by TMA stores
//   tc_gemm_bf16_rows_kernel  the same product for at most 64 rows (a decode step): 128 weight rows are the wide operand,
//                             read in 16 KB tiles, k is cut over a thread-block cluster whose blocks exchange partial sums through
//                             distributed shared memory, and the weight stream starts before the dependency wait
//
// On an expired wait a kernel raises the error flag, stops issuing work, still frees its tensor memory and returns.
#include <algorithm>

#include "device_util.cuh"
#include "layered_kernels.cuh"
#include "tc_common.cuh"

namespace pg {
namespace {

constexpr int KB = 64;  // BF16 elements per k block: one 128-byte swizzle row

// z * Phi(z) of two values for results that are rounded to BF16 next. Phi(z) - 1/2 = z P(2 z^2 / 4.5^2 - 1) on
// [-4.5, 4.5] with a degree-9 weighted least-squares fit of (Phi(z) - 1/2) / z on Chebyshev nodes; beyond that range Phi
// is taken at its end. Absolute error below 1e-5 inside and 5e-5 outside.
__device__ __forceinline__ void gelu_erf_pair(float& x, float& y) {
  constexpr float C[10] = {1.569053008e-01f, -7.718336822e-02f, 5.467184018e-02f, -4.029580498e-02f, 2.862407447e-02f,
                           -1.815922087e-02f, 1.014016557e-02f, -6.682699045e-03f, 4.655552699e-03f, -1.565833704e-03f};
  const float cx = fminf(fmaxf(x, -4.5f), 4.5f), cy = fminf(fmaxf(y, -4.5f), 4.5f);
  const unsigned long long c2 = pack2(cx, cy), zero = pack2(0.f, 0.f);
  const unsigned long long t = fma2(fma2(c2, c2, zero), pack2(2.f / 20.25f, 2.f / 20.25f), pack2(-1.f, -1.f));
  unsigned long long p = pack2(C[9], C[9]);
#pragma unroll
  for (int i = 8; i >= 0; --i) p = fma2(p, t, pack2(C[i], C[i]));
  p = fma2(p, c2, pack2(0.5f, 0.5f));
  float px, py;
  unpack2(p, px, py);
  x *= px;
  y *= py;
}

__device__ __forceinline__ float exp2_fast(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
// xIELU for results that are rounded to BF16 next: e^z - 1 - z is off by less than 1e-6 here, far below z / 2 wherever that
// rounds to a BF16 of its own.
__device__ __forceinline__ float xielu_fast(float z, float a, float b) {
  const float e = exp2_fast(fminf(z, 0.f) * 1.4426950408889634f) - 1.f - z;
  return fmaf(0.5f, z, z > 0.f ? a * z * z : b * e);
}
__device__ __forceinline__ void activate_pair(const ActArgs& act, float& x, float& y) {
  if (act.kind == ACT_GELU_ERF) {
    gelu_erf_pair(x, y);
  } else if (act.kind == ACT_XIELU) {
    x = xielu_fast(x, act.a, act.b);
    y = xielu_fast(y, act.a, act.b);
  }
}

__device__ __forceinline__ void tma_store_2d(const CUtensorMap* map, int x, int y, const void* smem_src) {
  asm volatile("cp.async.bulk.tensor.2d.global.shared::cta.bulk_group [%0, {%1, %2}], [%3];" ::"l"(map), "r"(x), "r"(y),
               "r"(smem_u32(smem_src))
               : "memory");
}
__device__ __forceinline__ void bulk_commit() { asm volatile("cp.async.bulk.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void bulk_wait_read() {
  asm volatile("cp.async.bulk.wait_group.read %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void bulk_wait_all() { asm volatile("cp.async.bulk.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ void fence_async_shared() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); }

template <int BN>
struct BfSmem {
  static constexpr int STAGES = (BN == 256) ? 4 : 6;
  static constexpr int A_BYTES = TILE_M * KB * 2, B_BYTES = BN * KB * 2;
  static constexpr int BOX_BYTES = 32 * 128;            // 32 rows of 128 bytes: one store box
  static constexpr int EPI_BYTES = 4 * 2 * BOX_BYTES;   // two boxes per epilogue warp
  static constexpr size_t BYTES = (size_t)STAGES * (A_BYTES + B_BYTES) + EPI_BYTES + 1024 /*align*/ + 256 /*barriers*/;
};

enum { OUT_F32 = 0, OUT_BF16 = 1, OUT_BF16_ACT = 2 };

// Persistent over 128 x BN output tiles; two accumulators in tensor memory, so that the epilogue of a tile overlaps the
// products of the next. Warp 0 loads, warp 1 issues the MMAs and owns the tensor memory, warps 2..5 store. `tma_out`:
// map_o can be used (16-byte aligned rows); else rows are stored element by element.
template <int BN>
__global__ void __launch_bounds__(192, 1)
    tc_gemm_bf16_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w,
                        const __grid_constant__ CUtensorMap map_o, Bf16GemmArgs a, int out_kind, int tma_out) {
  using S = BfSmem<BN>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* smem_a = base;
  uint8_t* smem_b = base + (size_t)S::STAGES * S::A_BYTES;
  uint8_t* epi = smem_b + (size_t)S::STAGES * S::B_BYTES;
  uint64_t* full = reinterpret_cast<uint64_t*>(epi + S::EPI_BYTES);
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
    uint8_t* boxes = epi + (size_t)(warp - 2) * 2 * S::BOX_BYTES;
    const int cols = out_kind == OUT_F32 ? 32 : 64;  // columns of one 128-byte box row
    uint32_t ti = 0, nbox = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++ti) {
      const int n0 = (tile % tiles_n) * BN, m0 = (tile / tiles_n) * TILE_M + q * 32;
      const uint32_t buf = ti & 1, tmem_d = tmem_base + buf * BN + ((uint32_t)(q * 32) << 16);
      ok = mbar_wait(&d_full[buf], (ti >> 1) & 1, failed, a.error_flag, 3);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
#pragma unroll 1
      for (int c0 = 0; c0 < BN && n0 + c0 < a.n; c0 += cols) {
        float v[32];
        tmem_ld32(tmem_d + (uint32_t)c0, v);
        uint8_t* box = boxes + (nbox & 1) * S::BOX_BYTES;
        uint4* row = reinterpret_cast<uint4*>(box + lane * 128);
        if (tma_out) {
          if (lane == 0) bulk_wait_read<1>();  // the box's previous store has read it
          __syncwarp();
        }
        if (out_kind == OUT_F32) {
          if (tma_out) {
#pragma unroll
            for (int j = 0; j < 8; ++j)
              row[j ^ (lane & 7)] = make_uint4(__float_as_uint(v[4 * j]), __float_as_uint(v[4 * j + 1]), __float_as_uint(v[4 * j + 2]),
                                               __float_as_uint(v[4 * j + 3]));
          } else if (m0 + lane < a.m) {
#pragma unroll
            for (int j = 0; j < 32; ++j)
              if (n0 + c0 + j < a.n) a.out[(size_t)(m0 + lane) * a.ldo + n0 + c0 + j] = v[j];
          }
        } else {
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            if (half) tmem_ld32(tmem_d + (uint32_t)(c0 + 32), v);
            if (out_kind == OUT_BF16_ACT) {
#pragma unroll
              for (int j = 0; j < 32; j += 2) activate_pair(a.act, v[j], v[j + 1]);
            }
            uint32_t p[16];
#pragma unroll
            for (int j = 0; j < 16; ++j) {
              const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
              p[j] = *reinterpret_cast<const uint32_t*>(&b);
            }
            if (tma_out) {
#pragma unroll
              for (int j = 0; j < 4; ++j)
                row[(half * 4 + j) ^ (lane & 7)] = make_uint4(p[4 * j], p[4 * j + 1], p[4 * j + 2], p[4 * j + 3]);
            } else if (m0 + lane < a.m) {
#pragma unroll
              for (int j = 0; j < 32; ++j)
                if (n0 + c0 + half * 32 + j < a.n)
                  static_cast<__nv_bfloat16*>(a.out_h)[(size_t)(m0 + lane) * a.ldo + n0 + c0 + half * 32 + j] = __float2bfloat16_rn(v[j]);
            }
          }
        }
        if (tma_out) {
          fence_async_shared();
          __syncwarp();
          if (lane == 0) {
            if (m0 < a.m) tma_store_2d(&map_o, n0 + c0, m0, box);
            bulk_commit();
          }
          ++nbox;
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&d_empty[buf]);
    }
    if (lane == 0) bulk_wait_all();
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 2 * BN);
}

// ------------------------------------------------------------------ decode rows
template <int BN, int SPLITS>
struct RowsSmem {
  static constexpr int STAGES = 6;
  static constexpr int A_BYTES = TILE_M * KB * 2, B_BYTES = BN * KB * 2;
  static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;  // both multiples of 1024
  static constexpr int RECV_BYTES = TILE_M * BN * 4;     // partial sums of this block's rows from every block of the cluster
  static constexpr size_t BYTES = (size_t)STAGES * STAGE_BYTES + RECV_BYTES + 1024 + 256;
};

__device__ __forceinline__ uint32_t cluster_addr(uint32_t addr, uint32_t rank) {
  uint32_t r;
  asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
  return r;
}
__device__ __forceinline__ void cluster_store(uint32_t addr, float v) {
  asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(addr), "f"(v) : "memory");
}
__device__ __forceinline__ void cluster_barrier() {
  asm volatile("barrier.cluster.arrive.release.aligned;\nbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <int BN, int SPLITS>
__global__ void __launch_bounds__(192, 1)
    tc_gemm_bf16_rows_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w, Bf16GemmArgs a,
                             int out_kind) {
  using S = RowsSmem<BN, SPLITS>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  float* recv = reinterpret_cast<float*>(base + (size_t)S::STAGES * S::STAGE_BYTES);  // [SPLITS][BN][TILE_M / SPLITS]
  uint64_t* full = reinterpret_cast<uint64_t*>(reinterpret_cast<uint8_t*>(recv) + S::RECV_BYTES);
  uint64_t* empty = full + S::STAGES;
  uint64_t* d_full = empty + S::STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(d_full + 1);
  volatile int* failed = reinterpret_cast<volatile int*>(tmem_slot + 1);
  constexpr uint32_t COLS = BN < 32 ? 32 : BN;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * TILE_M, split = blockIdx.y;
  const int nkb_all = (a.k + KB - 1) / KB, kb0 = nkb_all * split / SPLITS, nkb = nkb_all * (split + 1) / SPLITS - kb0;
  const int head = blockIdx.z, x0 = head * a.x_head;
  const int wrow = ((head * (int)gridDim.x + (int)blockIdx.x) * nkb_all + kb0) * TILE_M;  // first row of this block's run of weight tiles

  if (threadIdx.x == 0) {
    for (int s = 0; s < S::STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    mbar_init(d_full, 1);
    *failed = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(tmem_slot, COLS);
  tc_fence_before();
  __syncthreads();
  // nobody writes into a peer's receive buffer before every block of the cluster runs
  cluster_barrier();
  tc_fence_after();
  const uint32_t tmem_d = *tmem_slot;
  pdl_launch();

  if (warp == 0) {
    if (lane == 0) {
      const int ahead = min(nkb, S::STAGES);
      for (int i = 0; i < ahead; ++i) {  // weights do not depend on the previous kernel
        mbar_expect_tx(&full[i], S::STAGE_BYTES);
        tma_load_2d(base + (size_t)i * S::STAGE_BYTES, &map_w, 0, wrow + i * TILE_M, &full[i]);
      }
      pdl_wait();
      for (int i = 0; i < ahead; ++i)
        tma_load_2d(base + (size_t)i * S::STAGE_BYTES + S::A_BYTES, &map_x, x0 + (kb0 + i) * KB, 0, &full[i]);
      bool ok = true;
      for (int i = ahead; i < nkb; ++i) {
        const int s = i % S::STAGES;
        ok = mbar_wait(&empty[s], ((i / S::STAGES) - 1) & 1, failed, a.error_flag, 11);
        if (!ok) break;
        mbar_expect_tx(&full[s], S::STAGE_BYTES);
        tma_load_2d(base + (size_t)s * S::STAGE_BYTES, &map_w, 0, wrow + i * TILE_M, &full[s]);
        tma_load_2d(base + (size_t)s * S::STAGE_BYTES + S::A_BYTES, &map_x, x0 + (kb0 + i) * KB, 0, &full[s]);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = umma_idesc_bf16(TILE_M, BN);
      bool ok = true;
      for (int i = 0; i < nkb && ok; ++i) {
        const int s = i % S::STAGES;
        ok = mbar_wait(&full[s], (i / S::STAGES) & 1, failed, a.error_flag, 12);
        if (!ok) break;
        tc_fence_after();
        const uint64_t da = umma_desc_sw128(base + (size_t)s * S::STAGE_BYTES);
        const uint64_t db = umma_desc_sw128(base + (size_t)s * S::STAGE_BYTES + S::A_BYTES);
#pragma unroll
        for (int k = 0; k < KB / 16; ++k) umma_bf16_ss(tmem_d, da + (uint64_t)(k * 2), db + (uint64_t)(k * 2), idesc, (i | k) != 0);
        umma_commit(&empty[s]);
      }
      if (ok) umma_commit(d_full);
    }
  } else {
    // row r of the tile is finished by block r / RP of the cluster: this thread sends its partial sums there
    const int r = (warp & 3) * 32 + lane;
    constexpr int RP = TILE_M / SPLITS;
    bool ok = mbar_wait(d_full, 0, failed, a.error_flag, 13);
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tc_fence_after();
      const uint32_t dst = cluster_addr(smem_u32(recv), (uint32_t)(r / RP)) + (uint32_t)((split * BN) * RP + (r % RP)) * 4u;
#pragma unroll 1
      for (int c0 = 0; c0 < BN; c0 += 16) {
        float v[16];
        tmem_ld16(tmem_d + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)c0, v);
#pragma unroll
        for (int j = 0; j < 16; ++j) cluster_store(dst + (uint32_t)((c0 + j) * RP) * 4u, v[j]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  cluster_barrier();  // every partial sum has arrived; no peer touches this block's memory after it
  pdl_wait();         // nothing may be overwritten before the previous kernel has ended
  if (warp >= 2 && !*failed) {
    constexpr int RP = TILE_M / SPLITS;
    const int t = threadIdx.x - 64;
    for (int i = t; i < RP * BN; i += 128) {
      const int j = i / RP, rl = i % RP, feat = n0 + split * RP + rl;
      if (j < a.m && feat < a.n) {
        float s = 0.f;
#pragma unroll
        for (int sp = 0; sp < SPLITS; ++sp) s += recv[(size_t)(sp * BN + j) * RP + rl];  // in split order
        const bool split = a.act_from > 0 && feat >= a.act_from;
        if (out_kind == OUT_BF16_ACT || split) {
          float z = 0.f;
          activate_pair(a.act, s, z);
        }
        const size_t at = (size_t)j * a.ldo + (size_t)head * a.out_head + feat;
        if (split) static_cast<__nv_bfloat16*>(a.out_act)[(size_t)j * a.ldo_act + feat - a.act_from] = __float2bfloat16_rn(s);
        else if (out_kind == OUT_F32) a.out[at] = s;
        else static_cast<__nv_bfloat16*>(a.out_h)[at] = __float2bfloat16_rn(s);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_d, COLS);
}

// ------------------------------------------------------------------ host side
int sm_count() {
  static const int n = [] {
    int dev = 0, v = 148;
    cudaGetDevice(&dev);
    if (cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) v = 148;
    return v;
  }();
  return n;
}

// [rows, cols] with row pitch ld, FP32 or BF16, boxes of 32 rows x 128 bytes; false when the layout does not allow it
bool make_out_map(CUtensorMap* map, void* ptr, bool bf16, uint64_t rows, uint64_t cols, uint64_t ld) {
  EncodeTiledFn fn = encode_fn();
  const uint64_t elem = bf16 ? 2 : 4;
  if (!fn || (ld * elem) % 16 != 0 || (reinterpret_cast<uintptr_t>(ptr) & 15)) return false;
  cuuint64_t dims[2] = {cols, rows};
  cuuint64_t strides[1] = {ld * elem};
  cuuint32_t box[2] = {(cuuint32_t)(128 / elem), 32};
  cuuint32_t estr[2] = {1, 1};
  return fn(map, bf16 ? CU_TENSOR_MAP_DATA_TYPE_BFLOAT16 : CU_TENSOR_MAP_DATA_TYPE_FLOAT32, 2, ptr, dims, strides, box, estr,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

int out_kind_of(const Bf16GemmArgs& a) { return a.out ? OUT_F32 : a.act.kind != ACT_NONE ? OUT_BF16_ACT : OUT_BF16; }

template <int BN>
cudaError_t launch_bn(const Bf16GemmArgs& a, bool pdl, cudaStream_t s) {
  CUtensorMap mx, mw, mo{};
  if (!make_map_bf16(&mx, a.x, a.m, a.k, TILE_M) || !make_map_bf16(&mw, a.w, a.n, a.k, BN)) return cudaErrorInvalidValue;
  const int kind = out_kind_of(a);
  const int tma_out = make_out_map(&mo, kind == OUT_F32 ? (void*)a.out : a.out_h, kind != OUT_F32, a.m, a.n, a.ldo) ? 1 : 0;
  const size_t smem = BfSmem<BN>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(tc_gemm_bf16_kernel<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  const int tiles = ((a.m + TILE_M - 1) / TILE_M) * ((a.n + BN - 1) / BN);
  return launch_kernel(tc_gemm_bf16_kernel<BN>, dim3(std::min(tiles, sm_count())), dim3(192), smem, s, pdl, mx, mw, mo, a, kind, tma_out);
}

template <int BN, int SPLITS>
cudaError_t launch_rows(const Bf16GemmArgs& a, bool pdl, cudaStream_t s) {
  CUtensorMap mx, mw;
  const uint64_t heads = std::max(a.heads, 1), tiles = heads * ((a.n + TILE_M - 1) / TILE_M) * (a.k / KB);
  if (!make_map_bf16(&mx, a.x, a.m, a.heads ? a.ldx : a.k, BN) || !make_map_bf16(&mw, a.w_tiled, tiles * TILE_M, KB, TILE_M)) return cudaErrorInvalidValue;
  auto kernel = tc_gemm_bf16_rows_kernel<BN, SPLITS>;
  const size_t smem = RowsSmem<BN, SPLITS>::BYTES;
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((a.n + TILE_M - 1) / TILE_M, SPLITS, (unsigned)heads);
  cfg.blockDim = dim3(192);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = SPLITS;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 2 : 1;
  return cudaLaunchKernelEx(&cfg, kernel, mx, mw, a, out_kind_of(a));
}

template <int BN>
cudaError_t launch_rows_bn(const Bf16GemmArgs& a, bool pdl, cudaStream_t s) {
  // As many parts of k as fill the chip once, each at least two k blocks; clusters of eight only where a few of them are
  // needed: sixteen do not run at the same time (measured, 2048 output columns: 19 us in eight parts, 12 us in four).
  const int tiles = (a.n + TILE_M - 1) / TILE_M * std::max(a.heads, 1), nkb = (a.k + KB - 1) / KB;
  const int max_splits = tiles <= 8 ? 8 : 4;
  int splits = 1;
  while (splits < max_splits && tiles * splits * 2 <= sm_count() && splits * 4 <= nkb) splits *= 2;
  switch (splits) {
    case 1: return launch_rows<BN, 1>(a, pdl, s);
    case 2: return launch_rows<BN, 2>(a, pdl, s);
    case 4: return launch_rows<BN, 4>(a, pdl, s);
    default: return launch_rows<BN, 8>(a, pdl, s);
  }
}

}  // namespace

bool gemm_bf16_rows_kernel(int m, int k) { return m <= 64 && k % KB == 0; }

cudaError_t launch_tc_gemm_bf16(const Bf16GemmArgs& a, bool pdl, cudaStream_t s) {
  if (a.m <= 0 || a.n <= 0) return cudaSuccess;
  if (a.heads > 0 && (a.x_head % 8 != 0 || a.ldx % 8 != 0)) return cudaErrorInvalidValue;  // TMA boxes start on 16 bytes
  if ((a.act_from > 0 || a.heads > 0) && (!a.w_tiled || !gemm_bf16_rows_kernel(a.m, a.k))) return cudaErrorInvalidValue;
  if (a.k <= 0 || a.k % 8 != 0 || (!a.out && !a.out_h)) return cudaErrorInvalidValue;
  if (a.w_tiled && a.k % KB == 0) {
    if (a.m <= 16) return launch_rows_bn<16>(a, pdl, s);
    if (a.m <= 32) return launch_rows_bn<32>(a, pdl, s);
    if (a.m <= 64) return launch_rows_bn<64>(a, pdl, s);
  }
  const long long m_tiles = (a.m + TILE_M - 1) / TILE_M;
  if (m_tiles * ((a.n + 255) / 256) >= sm_count()) return launch_bn<256>(a, pdl, s);
  if (m_tiles * ((a.n + 127) / 128) >= 100) return launch_bn<128>(a, pdl, s);
  return launch_bn<64>(a, pdl, s);
}

}  // namespace pg
