// Tensor-core attention of portions of prompts over the BF16 workspaces (see AttentionPortionArgs): tcgen05 products with
// S and P and O in tensor memory, FP32 scores and softmax, queries / keys / values by TMA.
//
// Work item = 128 query rows of one head of one sequence; a persistent block takes items in turn, so that the loads and
// first scores of an item overlap the end of the one before. Warp 0 loads, warp 1 issues the MMAs, warps 2..5 do the
// softmax (thread = row). S(j + 1) = Q K^T is issued before O += P(j) V, so that the tensor cores work on the next scores
// while the softmax warps are busy; keys and values have rings of their own. An item walks only the key tiles that some
// row of it can see. Every wait is bounded: on expiry the error flag is set, work stops, tensor memory is freed.
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

struct TcItem {
  int head, seq, first, n, q0, kvh, p0, base_pos, pos_a, pos_b, lo, tiles;
  // false: no rows here
  __device__ __forceinline__ bool set(const AttentionPortionArgs& a, int index, int qtiles) {
    const AttentionLayer& l = a.l;
    const int per = l.heads * a.nseq;
    q0 = (qtiles - 1 - index / per) * QROWS;  // the last query rows see the most keys: they go first
    head = index % per % l.heads;
    seq = index % per / l.heads;
    first = a.seq_start[seq];
    n = a.seq_start[seq + 1] - first;
    if (q0 >= n) return false;
    kvh = head / (l.heads / l.kv_heads);
    p0 = a.seq_pos[seq];
    base_pos = p0 - p0 % l.span;  // position of the sequence's first workspace key
    pos_a = p0 + q0;
    pos_b = p0 + min(q0 + QROWS, n) - 1;
    lo = max(pos_a / l.span * l.span - base_pos, 0);
    tiles = (pos_b - base_pos - lo) / KROWS + 1;
    return true;
  }
};

__global__ void __launch_bounds__(192, 2)
    attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                        const __grid_constant__ CUtensorMap map_v, AttentionPortionArgs a, TcShape t, int items, int qtiles) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t q_full, q_empty, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full, p_ready, pv_done, o_free;
  __shared__ uint32_t tmem_slot;
  __shared__ int failed_flag;
  const AttentionLayer& l = a.l;
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* qs = base;
  uint8_t* ks = qs + (size_t)t.dpieces * PIECE;
  uint8_t* vs = ks + (size_t)t.kstages * t.dpieces * PIECE;
  volatile int* failed = &failed_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    mbar_init(&q_empty, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    mbar_init(&s_full, 1);
    mbar_init(&p_ready, 4);
    mbar_init(&pv_done, 1);
    mbar_init(&o_free, 4);
    failed_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(&tmem_slot, (uint32_t)t.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  TcItem w;
  uint32_t g = 0, done = 0;  // key tiles and items before the current ones: every role counts them alike
  bool ok = true;

  if (warp == 0) {
    if (lane == 0) {
      for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
        if (!w.set(a, it, qtiles)) continue;
        if (done > 0) ok = mbar_wait(&q_empty, (done - 1) & 1, failed, a.error_flag, 20);
        if (!ok) break;
        mbar_expect_tx(&q_full, t.dpieces * PIECE);
        for (int d = 0; d < t.dpieces; ++d) tma_load_3d(qs + (size_t)d * PIECE, &map_q, d * 64, w.head, w.first + w.q0, &q_full);
        for (int j = 0; j < w.tiles && ok; ++j) {
          const int krow = a.key_start[w.seq] + w.lo + j * KROWS;
          const uint32_t gt = g + j, s = gt % t.kstages, v = gt % t.vstages;
          if (gt >= (uint32_t)t.kstages) ok = mbar_wait(&k_empty[s], ((gt / t.kstages) - 1) & 1, failed, a.error_flag, 21);
          if (!ok) break;
          mbar_expect_tx(&k_full[s], t.dpieces * PIECE);
          for (int d = 0; d < t.dpieces; ++d) tma_load_3d(ks + (size_t)(s * t.dpieces + d) * PIECE, &map_k, d * 64, w.kvh, krow, &k_full[s]);
          if (gt >= (uint32_t)t.vstages) ok = mbar_wait(&v_empty[v], ((gt / t.vstages) - 1) & 1, failed, a.error_flag, 22);
          if (!ok) break;
          mbar_expect_tx(&v_full[v], t.vpieces * PIECE);
          for (int d = 0; d < t.vpieces; ++d) tma_load_3d(vs + (size_t)(v * t.vpieces + d) * PIECE, &map_v, d * 64, w.kvh, krow, &v_full[v]);
        }
        g += w.tiles;
        ++done;
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16(QROWS, KROWS), idesc_o = umma_idesc_bf16(QROWS, t.vn, true);
      auto scores = [&](uint32_t gt, bool last) -> bool {
        const uint32_t s = gt % t.kstages;
        if (!mbar_wait(&k_full[s], (gt / t.kstages) & 1, failed, a.error_flag, 23)) return false;
        tc_fence_after();
        for (int k = 0; k < t.ksteps; ++k) {
          const uint64_t dq = umma_desc_sw128(qs + (size_t)(k >> 2) * PIECE) + (uint64_t)((k & 3) * 2);
          const uint64_t dk = umma_desc_sw128(ks + (size_t)(s * t.dpieces + (k >> 2)) * PIECE) + (uint64_t)((k & 3) * 2);
          umma_bf16_ss(tmem + COL_S, dq, dk, idesc_s, k != 0);
        }
        umma_commit(&k_empty[s]);
        if (last) umma_commit(&q_empty);
        umma_commit(&s_full);
        return true;
      };
      // S(gt) may be overwritten once the softmax warps have read it, which they tell with p_ready(gt): every scores()
      // but the very first one follows such a wait.
      for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
        if (!w.set(a, it, qtiles)) continue;
        ok = mbar_wait(&q_full, done & 1, failed, a.error_flag, 24) && scores(g, w.tiles == 1);
        for (int j = 0; j < w.tiles && ok; ++j) {
          const uint32_t gt = g + j;
          ok = mbar_wait(&p_ready, gt & 1, failed, a.error_flag, 25);  // P is written, S has been read
          if (!ok) break;
          tc_fence_after();
          if (j + 1 < w.tiles) ok = scores(gt + 1, j + 2 == w.tiles);
          const uint32_t v = gt % t.vstages;
          ok = ok && mbar_wait(&v_full[v], (gt / t.vstages) & 1, failed, a.error_flag, 26);
          if (ok && j == 0 && done > 0) ok = mbar_wait(&o_free, (done - 1) & 1, failed, a.error_flag, 30);  // O of the item before has been read
          if (!ok) break;
          tc_fence_after();
          for (int k = 0; k < KROWS / 16; ++k)
            umma_bf16_ts(tmem + COL_O, tmem + COL_P + (uint32_t)(k * 8),
                         umma_desc_mn_sw128(vs + (size_t)v * t.vpieces * PIECE + (size_t)k * 2048, PIECE), idesc_o, (j | k) != 0);
          umma_commit(&v_empty[v]);
          umma_commit(&pv_done);
        }
        g += w.tiles;
        ++done;
      }
    }
  } else {
    const int q = warp & 3, r = q * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const float scale2 = l.scale == 0.f ? 1e-30f : l.scale * LOG2E;  // never 0: the mask is an infinite score
    for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
      if (!w.set(a, it, qtiles)) continue;
      const int qrow = w.q0 + r, pos = w.p0 + min(qrow, w.n - 1);
      const int lo_row = max(pos / l.span * l.span - w.base_pos, 0), hi_row = pos - w.base_pos;
      const int lo_all = max(w.pos_b / l.span * l.span - w.base_pos, 0), hi_all = w.pos_a - w.base_pos;  // keys every row sees
      float m_ref = -1e30f, sum = 0.f;
      for (int j = 0; j < w.tiles && ok; ++j) {
        const uint32_t gt = g + j;
        ok = __all_sync(ALL_LANES, mbar_wait(&s_full, gt & 1, failed, a.error_flag, 27));
        if (!ok) break;
        tc_fence_after();
        float s[128];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          float v[32];
          tmem_ld32(tmem + COL_S + lane_addr + (uint32_t)(c * 32), v);
#pragma unroll
          for (int i = 0; i < 32; ++i) s[c * 32 + i] = v[i];
        }
        const int k0 = w.lo + j * KROWS;
        if (k0 < lo_all || k0 + KROWS - 1 > hi_all) {
          const int lo_i = lo_row - k0, hi_i = hi_row - k0;
#pragma unroll
          for (int i = 0; i < 128; ++i)
            if (i < lo_i || i > hi_i) s[i] = scale2 < 0.f ? INFINITY : -INFINITY;
        }
        float mx[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) mx[i] = s[i] * scale2;
#pragma unroll
        for (int i = 4; i < 128; ++i) mx[i & 3] = fmaxf(mx[i & 3], s[i] * scale2);
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
          s[i] = exp2_fast(fmaf(s[i], scale2, -m_ref));
          part[i & 3] += s[i];
        }
        sum += (part[0] + part[1]) + (part[2] + part[3]);
        if (j > 0) {  // P and O may be touched once O += P(j - 1) V is done (for j = 0 the wait at the end of the item before)
          ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (gt - 1) & 1, failed, a.error_flag, 28));
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
      if (ok) ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (g + w.tiles - 1) & 1, failed, a.error_flag, 29));
      if (!ok) break;
      tc_fence_after();
      const float inv = l.out_scale / sum;
      __nv_bfloat16* y = static_cast<__nv_bfloat16*>(a.y) + (size_t)(w.first + qrow) * a.ldy + w.head * l.vdim;
      const bool vec = l.vdim % 8 == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0;
      for (int c = 0; c < t.vn; c += 16) {
        float o[16];
        tmem_ld16(tmem + COL_O + lane_addr + (uint32_t)c, o);
        if (c + 16 >= t.vn) {  // all of O is in registers or stored: the next item may overwrite it
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&o_free);
        }
        if (qrow >= w.n) {  // a row of the next sequence or none: nothing to store
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
      g += w.tiles;
      ++done;
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
  const int qtiles = (a.max_len + QROWS - 1) / QROWS, items = qtiles * l.heads * a.nseq;
  int dev = 0, sms = 148;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  const int per_sm = t.tmem_cols <= 256 && bytes(stages) <= 110 * 1024 ? 2 : 1;
  return launch_kernel(attention_tc_kernel, dim3(std::min(items, sms * per_sm)), dim3(192), bytes(stages), s, false, mq, mk, mv, a, t, items,
                       qtiles);
}

}  // namespace pg
