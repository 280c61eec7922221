// Tensor-core attention of portions of prompts over the BF16 workspaces (see AttentionPortionArgs): tcgen05 products with
// S and P and O in tensor memory, FP32 scores and softmax, queries / keys / values by TMA.
//
// Block = 128 query rows of one head of one sequence. Warp 0 loads, warp 1 issues the MMAs, warps 2..5 do the softmax
// (thread = row). S(j + 1) = Q K^T is issued before O += P(j) V, so that the tensor cores work on the next scores while
// the softmax warps are busy; keys and values have rings of their own. A block walks only the key tiles that some row of
// it can see. Every wait is bounded: on expiry the error flag is set, work stops, tensor memory is freed.
#include <algorithm>

#include "device_util.cuh"
#include "layered_kernels.cuh"
#include "tc_common.cuh"

namespace pg {
namespace {

constexpr int QROWS = 128, KROWS = 128;
constexpr int PIECE = 128 * 128;  // bytes of one 128-row piece of 64 BF16 columns
constexpr uint32_t COL_S = 0, COL_P = 128, COL_O = 192;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float exp2_fast(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

// kstages / vstages: ring depths; dpieces / vpieces: 64-column pieces of a key / value row; vn: columns of O (multiple of 16)
struct TcShape {
  int dpieces, vpieces, ksteps, vn, kstages, vstages, tmem_cols;
};

__global__ void __launch_bounds__(192, 2)
    attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                        const __grid_constant__ CUtensorMap map_v, AttentionPortionArgs a, TcShape t) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t q_full, k_full[4], k_empty[4], v_full[4], v_empty[4], s_full, p_ready, pv_done;
  __shared__ uint32_t tmem_slot;
  __shared__ int failed_flag;
  const AttentionLayer& l = a.l;
  const int head = blockIdx.y, seq = blockIdx.z;
  const int first = a.seq_start[seq], n = a.seq_start[seq + 1] - first;
  // long tiles first: the last query rows see the most keys
  const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * QROWS;
  if (q0 >= n) return;
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* qs = base;
  uint8_t* ks = qs + (size_t)t.dpieces * PIECE;
  uint8_t* vs = ks + (size_t)t.kstages * t.dpieces * PIECE;
  volatile int* failed = &failed_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = head / (l.heads / l.kv_heads), p0 = a.seq_pos[seq];
  const int base_pos = p0 - p0 % l.span;  // position of the sequence's first workspace key
  const int pos_a = p0 + q0, pos_b = p0 + min(q0 + QROWS, n) - 1;
  const int lo = max(pos_a / l.span * l.span - base_pos, 0), hi = pos_b - base_pos;
  const int tiles = (hi - lo) / KROWS + 1;

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    for (int i = 0; i < 4; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    mbar_init(&s_full, 1);
    mbar_init(&p_ready, 4);
    mbar_init(&pv_done, 1);
    failed_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(&tmem_slot, (uint32_t)t.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      mbar_expect_tx(&q_full, t.dpieces * PIECE);
      for (int d = 0; d < t.dpieces; ++d) tma_load_3d(qs + (size_t)d * PIECE, &map_q, d * 64, head, first + q0, &q_full);
      for (int j = 0; j < tiles && ok; ++j) {
        const int krow = a.key_start[seq] + lo + j * KROWS;
        const int s = j % t.kstages, v = j % t.vstages;
        if (j >= t.kstages) ok = mbar_wait(&k_empty[s], ((j / t.kstages) - 1) & 1, failed, a.error_flag, 21);
        if (!ok) break;
        mbar_expect_tx(&k_full[s], t.dpieces * PIECE);
        for (int d = 0; d < t.dpieces; ++d) tma_load_3d(ks + (size_t)(s * t.dpieces + d) * PIECE, &map_k, d * 64, kvh, krow, &k_full[s]);
        if (j >= t.vstages) ok = mbar_wait(&v_empty[v], ((j / t.vstages) - 1) & 1, failed, a.error_flag, 22);
        if (!ok) break;
        mbar_expect_tx(&v_full[v], t.vpieces * PIECE);
        for (int d = 0; d < t.vpieces; ++d) tma_load_3d(vs + (size_t)(v * t.vpieces + d) * PIECE, &map_v, d * 64, kvh, krow, &v_full[v]);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16(QROWS, KROWS), idesc_o = umma_idesc_bf16(QROWS, t.vn, true);
      auto scores = [&](int j) -> bool {
        const int s = j % t.kstages;
        if (!mbar_wait(&k_full[s], (j / t.kstages) & 1, failed, a.error_flag, 23)) return false;
        tc_fence_after();
        for (int k = 0; k < t.ksteps; ++k) {
          const uint64_t dq = umma_desc_sw128(qs + (size_t)(k >> 2) * PIECE) + (uint64_t)((k & 3) * 2);
          const uint64_t dk = umma_desc_sw128(ks + (size_t)(s * t.dpieces + (k >> 2)) * PIECE) + (uint64_t)((k & 3) * 2);
          umma_bf16_ss(tmem + COL_S, dq, dk, idesc_s, k != 0);
        }
        umma_commit(&k_empty[s]);
        umma_commit(&s_full);
        return true;
      };
      bool ok = mbar_wait(&q_full, 0, failed, a.error_flag, 24) && scores(0);
      for (int j = 0; j < tiles && ok; ++j) {
        ok = mbar_wait(&p_ready, j & 1, failed, a.error_flag, 25);  // P(j) is written, S(j) has been read
        if (!ok) break;
        tc_fence_after();
        if (j + 1 < tiles) ok = scores(j + 1);
        const int v = j % t.vstages;
        ok = ok && mbar_wait(&v_full[v], (j / t.vstages) & 1, failed, a.error_flag, 26);
        if (!ok) break;
        tc_fence_after();
        for (int k = 0; k < KROWS / 16; ++k)
          umma_bf16_ts(tmem + COL_O, tmem + COL_P + (uint32_t)(k * 8),
                       umma_desc_mn_sw128(vs + (size_t)v * t.vpieces * PIECE + (size_t)k * 2048, PIECE), idesc_o, (j | k) != 0);
        umma_commit(&v_empty[v]);
        umma_commit(&pv_done);
      }
    }
  } else {
    const int q = warp & 3, r = q * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const int qrow = q0 + r, pos = p0 + min(qrow, n - 1);
    const int lo_row = max(pos / l.span * l.span - base_pos, 0), hi_row = pos - base_pos;
    const int lo_all = max(pos_b / l.span * l.span - base_pos, 0), hi_all = pos_a - base_pos;  // keys every row sees
    const float scale2 = l.scale * LOG2E;
    float m_ref = -1e30f, sum = 0.f;
    bool ok = true;
    for (int j = 0; j < tiles && ok; ++j) {
      ok = __all_sync(ALL_LANES, mbar_wait(&s_full, j & 1, failed, a.error_flag, 27));
      if (!ok) break;
      tc_fence_after();
      float s[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float v[32];
        tmem_ld32(tmem + COL_S + lane_addr + (uint32_t)(c * 32), v);
#pragma unroll
        for (int i = 0; i < 32; ++i) s[c * 32 + i] = v[i] * scale2;
      }
      const int k0 = lo + j * KROWS;
      if (k0 < lo_all || k0 + KROWS - 1 > hi_all) {
#pragma unroll
        for (int i = 0; i < 128; ++i)
          if (k0 + i < lo_row || k0 + i > hi_row) s[i] = -INFINITY;
      }
      float mx[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int i = 4; i < 128; ++i) mx[i & 3] = fmaxf(mx[i & 3], s[i]);
      const float m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
      // the reference maximum moves only when a row's scores outgrow it by 2^8
      const bool move = __any_sync(ALL_LANES, m_tile > m_ref + 8.f);
      float corr = 1.f;
      if (move) {
        const float m_new = fmaxf(m_ref, m_tile);
        corr = exp2_fast(m_ref - m_new);
        m_ref = m_new;
        sum *= corr;
      }
      float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < 128; ++i) {
        s[i] = exp2_fast(s[i] - m_ref);
        part[i & 3] += s[i];
      }
      sum += (part[0] + part[1]) + (part[2] + part[3]);
      if (j > 0) {  // P and O may be touched once O += P(j - 1) V is done
        ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (j - 1) & 1, failed, a.error_flag, 28));
        if (!ok) break;
        tc_fence_after();
        if (move) {
          for (int c = 0; c < t.vn; c += 16) {
            float o[16];
            tmem_ld16(tmem + COL_O + lane_addr + (uint32_t)c, o);
            uint32_t u[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) u[i] = __float_as_uint(o[i] * corr);
            tmem_st16(tmem + COL_O + lane_addr + (uint32_t)c, u);
          }
        }
      }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        uint32_t u[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const __nv_bfloat162 b = __floats2bfloat162_rn(s[h * 64 + 2 * i], s[h * 64 + 2 * i + 1]);
          u[i] = *reinterpret_cast<const uint32_t*>(&b);
        }
        tmem_st32(tmem + COL_P + lane_addr + (uint32_t)(h * 32), u);
      }
      tmem_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready);
    }
    if (ok) ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (tiles - 1) & 1, failed, a.error_flag, 29));
    if (ok) {
      tc_fence_after();
      const float inv = l.out_scale / sum;
      const size_t at = (size_t)(first + qrow) * a.ldy + head * l.vdim;
      __nv_bfloat16* y = static_cast<__nv_bfloat16*>(a.y) + at;
      const bool vec = l.vdim % 8 == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0;
      for (int c = 0; c < t.vn; c += 16) {
        float o[16];
        tmem_ld16(tmem + COL_O + lane_addr + (uint32_t)c, o);
        if (qrow >= n) {  // a row of the next sequence or none: nothing to store
        } else if (vec) {
#pragma unroll
          for (int h = 0; h < 2; ++h)
            if (c + h * 8 < l.vdim) {
              uint32_t u[4];
#pragma unroll
              for (int i = 0; i < 4; ++i) {
                const __nv_bfloat162 b = __floats2bfloat162_rn(o[h * 8 + 2 * i] * inv, o[h * 8 + 2 * i + 1] * inv);
                u[i] = *reinterpret_cast<const uint32_t*>(&b);
              }
              *reinterpret_cast<uint4*>(y + c + h * 8) = make_uint4(u[0], u[1], u[2], u[3]);
            }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (c + i < l.vdim) y[c + i] = __float2bfloat16_rn(o[i] * inv);
        }
        __syncwarp();
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, (uint32_t)t.tmem_cols);
}

// BF16 [rows][heads][dim] (dim % 8 == 0), box = 64 elements of one head of 128 rows, 128-byte swizzle; columns past dim and
// rows past the end read as zero.
bool make_head_map(CUtensorMap* map, const void* ptr, uint64_t rows, uint64_t heads, uint64_t dim) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return false;
  cuuint64_t dims[3] = {dim, heads, rows};
  cuuint64_t strides[2] = {dim * 2, heads * dim * 2};
  cuuint32_t box[3] = {64, 1, 128};
  cuuint32_t estr[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

constexpr size_t TC_MAX_SMEM = 225 * 1024;

}  // namespace

cudaError_t launch_attention_tc(const AttentionPortionArgs& a, cudaStream_t s) {
  const AttentionLayer& l = a.l;
  TcShape t;
  t.dpieces = (l.dimp + 63) / 64;
  t.vpieces = (l.vdimp + 63) / 64;
  t.ksteps = (l.dimp + 15) / 16;
  t.vn = (l.vdimp + 15) / 16 * 16;
  t.tmem_cols = (int)COL_O + t.vn <= 256 ? 256 : 512;
  auto bytes = [&](int stages) { return (size_t)(t.dpieces + stages * (t.dpieces + t.vpieces)) * PIECE + 1024; };
  const int stages = bytes(2) <= TC_MAX_SMEM ? 2 : 1;
  t.kstages = t.vstages = stages;
  if (bytes(stages) > TC_MAX_SMEM) return cudaErrorInvalidValue;
  CUtensorMap mq, mk, mv;
  if (!make_head_map(&mq, a.q, a.rows, l.heads, l.dimp) || !make_head_map(&mk, a.k, a.krows, l.kv_heads, l.dimp) ||
      !make_head_map(&mv, a.v, a.krows, l.kv_heads, l.vdimp))
    return cudaErrorInvalidValue;
  cudaError_t e = cudaFuncSetAttribute(attention_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TC_MAX_SMEM);
  if (e != cudaSuccess) return e;
  const dim3 grid((a.max_len + QROWS - 1) / QROWS, l.heads, a.nseq);
  return launch_kernel(attention_tc_kernel, grid, dim3(192), bytes(stages), s, false, mq, mk, mv, a, t);
}

}  // namespace pg
