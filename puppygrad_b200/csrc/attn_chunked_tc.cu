// Tensor-core attention of portions of prompts over the BF16 workspaces (see AttentionPortionArgs): tcgen05 products with
// S and P and O in tensor memory, FP32 scores and softmax, queries / keys / values by TMA.
//
// Work item = 128 query rows of one head of one sequence; a persistent block takes items in turn, so that the loads and
// first scores of an item overlap the end of the one before. Warp 0 loads, warp 1 issues the MMAs, warps 2..9 do the
// softmax: two threads share a row, each with half of a tile's keys; they exchange maxima and sums through shared memory. S(j + 1) = Q K^T is issued as soon as the softmax warps hold S(j) in registers, so that the tensor cores
// work on the next scores while those warps are busy; keys and values have rings of their own. An item walks only the key tiles that some
// row of it can see: those of the moving range, and before them those of the sequence's kept first keys. Keys come in pieces of
// 64 columns through a ring; where the queries of an item do not fit beside it, their pieces come with the keys', again for
// every tile. Every wait is bounded: on expiry the error flag is set, work stops, tensor memory is freed.
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

constexpr int MAX_KSTAGES = 8, THREADS = 320, SOFTMAX_WARPS = 8;

__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* v) {
  uint32_t u[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 b = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    u[i] = *reinterpret_cast<const uint32_t*>(&b);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(u[0], u[1], u[2], u[3]);
}

// kstages / vstages: ring depths (pieces of keys, whole value tiles); dpieces / vpieces: 64-column pieces of a query or key / value
// row; vn: columns of O (multiple of 16); q_resident: an item's queries stay in shared memory
struct TcShape {
  int dpieces, vpieces, ksteps, vn, kstages, vstages, tmem_cols, q_resident;
};

struct TcItem {
  int head, seq, first, n, q0, kvh, p0, pos_a, pos_b, lo, kept, kept_tiles, tiles;
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
    pos_a = p0 + q0;
    pos_b = p0 + min(q0 + QROWS, n) - 1;
    lo = l.life.low(p0, pos_a);  // the moving range of the item's rows starts here
    kept = min(l.life.keep, lo);
    if (lo < KROWS) lo = kept = 0;
    kept_tiles = (kept + KROWS - 1) / KROWS;
    tiles = kept_tiles + (l.life.row(p0, pos_b) - lo) / KROWS + 1;
    return true;
  }
  // first workspace row of tile j, and the end of the rows that it stands for
  __device__ __forceinline__ int start(int j) const { return j < kept_tiles ? j * KROWS : lo + (j - kept_tiles) * KROWS; }
  __device__ __forceinline__ int end(int j) const { return j < kept_tiles ? kept : 1 << 30; }
};

__device__ __forceinline__ void pair_barrier(int quarter) { asm volatile("bar.sync %0, 64;" ::"r"(1 + quarter) : "memory"); }

template <int PER_SM>
__global__ void __launch_bounds__(THREADS, PER_SM)
    attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                        const __grid_constant__ CUtensorMap map_v, AttentionPortionArgs a, TcShape t, int items, int qtiles) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t q_full, q_empty, k_full[MAX_KSTAGES], k_empty[MAX_KSTAGES], v_full[2], v_empty[2], s_full, s_free, p_ready, pv_done, o_free;
  __shared__ uint32_t tmem_slot;
  __shared__ int failed_flag;
  __shared__ float row_max[2][2][QROWS], row_sum[2][2][QROWS];  // by parity of the tile (item) and side
  const AttentionLayer& l = a.l;
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* qs = base;
  uint8_t* ks = qs + (t.q_resident ? (size_t)t.dpieces * PIECE : 0);  // a stage: a piece of keys, and one of queries unless resident
  const uint32_t kstage_bytes = t.q_resident ? PIECE : 2 * PIECE;
  uint8_t* vs = ks + (size_t)t.kstages * kstage_bytes;
  volatile int* failed = &failed_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    mbar_init(&q_empty, 1);
    for (int i = 0; i < MAX_KSTAGES; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&v_full[i], 1);
      mbar_init(&v_empty[i], 1);
    }
    mbar_init(&s_full, 1);
    mbar_init(&s_free, SOFTMAX_WARPS);
    mbar_init(&p_ready, SOFTMAX_WARPS);
    mbar_init(&pv_done, 1);
    mbar_init(&o_free, SOFTMAX_WARPS);
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
      const int key_head = l.mix ? 0 : 1;  // mixed heads: all key heads are one wide row
      RingCursor kr, vr;
      for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
        if (!w.set(a, it, qtiles)) continue;
        if (t.q_resident) {
          ok = mbar_wait(&q_empty, (done & 1) ^ 1, failed, a.error_flag, 20);
          if (!ok) break;
          mbar_expect_tx(&q_full, t.dpieces * PIECE);
          for (int d = 0; d < t.dpieces; ++d) tma_load_3d(qs + (size_t)d * PIECE, &map_q, d * 64, w.head, w.first + w.q0, &q_full);
        }
        const int key0 = a.key_start[w.seq], kh = key_head * w.kvh;
        for (int j = 0; j < w.tiles && ok; ++j) {
          const int krow = key0 + w.start(j);
          for (int d = 0; d < t.dpieces; ++d, kr.next(t.kstages)) {
            ok = mbar_wait(&k_empty[kr.stage], kr.parity ^ 1, failed, a.error_flag, 21);
            if (!ok) break;
            uint8_t* dst = ks + kr.stage * kstage_bytes;
            mbar_expect_tx(&k_full[kr.stage], kstage_bytes);
            tma_load_3d(dst, &map_k, d * 64, kh, krow, &k_full[kr.stage]);
            if (!t.q_resident) tma_load_3d(dst + PIECE, &map_q, d * 64, w.head, w.first + w.q0, &k_full[kr.stage]);
          }
          if (ok) ok = mbar_wait(&v_empty[vr.stage], vr.parity ^ 1, failed, a.error_flag, 22);
          if (!ok) break;
          mbar_expect_tx(&v_full[vr.stage], t.vpieces * PIECE);
          for (int d = 0; d < t.vpieces; ++d) tma_load_3d(vs + (vr.stage * t.vpieces + d) * PIECE, &map_v, d * 64, w.kvh, krow, &v_full[vr.stage]);
          vr.next(t.vstages);
        }
        g += w.tiles;
        ++done;
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16(QROWS, KROWS), idesc_o = umma_idesc_bf16(QROWS, t.vn, true);
      RingCursor kr, vr;
      const uint64_t q_desc = umma_desc_sw128(qs), k_desc = umma_desc_sw128(ks), v_desc = umma_desc_mn_sw128(vs, PIECE);
      const uint32_t kstage16 = kstage_bytes >> 4, vstage16 = (uint32_t)t.vpieces * (PIECE >> 4);
      auto scores = [&](bool last) -> bool {
        for (int d = 0; d < t.dpieces; ++d, kr.next(t.kstages)) {
          if (!mbar_wait(&k_full[kr.stage], kr.parity, failed, a.error_flag, 23)) return false;
          tc_fence_after();
          const uint64_t dk = k_desc + kr.stage * kstage16, dq = t.q_resident ? q_desc + (uint32_t)d * (PIECE >> 4) : dk + (PIECE >> 4);
          const int steps = t.ksteps - d * 4;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (k < steps) umma_bf16_ss(tmem + COL_S, dq + (uint64_t)(k * 2), dk + (uint64_t)(k * 2), idesc_s, (d | k) != 0);
          umma_commit(&k_empty[kr.stage]);
        }
        if (last && t.q_resident) umma_commit(&q_empty);
        umma_commit(&s_full);
        return true;
      };
      // S(gt) may be overwritten once the softmax warps have read it, which they tell with s_free(gt): every scores() but the
      // very first one follows such a wait.
      for (int it = blockIdx.x; it < items && ok; it += gridDim.x) {
        if (!w.set(a, it, qtiles)) continue;
        ok = (!t.q_resident || mbar_wait(&q_full, done & 1, failed, a.error_flag, 24)) && scores(w.tiles == 1);
        for (int j = 0; j < w.tiles && ok; ++j) {
          const uint32_t gt = g + j;
          ok = mbar_wait(&s_free, gt & 1, failed, a.error_flag, 31);  // S has been read
          if (!ok) break;
          tc_fence_after();
          if (j + 1 < w.tiles) ok = scores(j + 2 == w.tiles);
          ok = ok && mbar_wait(&p_ready, gt & 1, failed, a.error_flag, 25);  // P is written
          if (!ok) break;
          tc_fence_after();
          ok = ok && mbar_wait(&v_full[vr.stage], vr.parity, failed, a.error_flag, 26);
          if (ok && j == 0 && done > 0) ok = mbar_wait(&o_free, (done - 1) & 1, failed, a.error_flag, 30);  // O of the item before has been read
          if (!ok) break;
          tc_fence_after();
          const uint64_t dv = v_desc + vr.stage * vstage16;
#pragma unroll
          for (int k = 0; k < KROWS / 16; ++k)
            umma_bf16_ts(tmem + COL_O, tmem + COL_P + (uint32_t)(k * 8), dv + (uint64_t)(k * (2048 >> 4)), idesc_o, (j | k) != 0);
          umma_commit(&v_empty[vr.stage]);
          vr.next(t.vstages);
          umma_commit(&pv_done);
        }
        g += w.tiles;
        ++done;
      }
    }
  } else {
    // on expiry these warps go on through their loops without work: the pairs' barriers need both sides
    const int q = warp & 3, side = (warp - 2) >> 2, r = q * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const float scale2 = l.scale == 0.f ? 1e-30f : l.scale * LOG2E;  // never 0: the mask is an infinite score
    for (int it = blockIdx.x; it < items; it += gridDim.x) {
      if (!w.set(a, it, qtiles)) continue;
      const int qrow = w.q0 + r, pos = w.p0 + min(qrow, w.n - 1);
      const int lo_row = l.life.low(w.p0, pos), hi_row = l.life.row(w.p0, pos), keep = l.life.keep;
      const int lo_all = l.life.low(w.p0, w.pos_b), hi_all = l.life.row(w.p0, w.pos_a);  // keys every row sees
      float m_ref = l.sink ? l.sink[w.head] * LOG2E : -1e30f, sum = l.sink && side == 0 ? 1.f : 0.f;
      for (int j = 0; j < w.tiles; ++j) {
        const uint32_t gt = g + j;
        if (ok) ok = __all_sync(ALL_LANES, mbar_wait(&s_full, gt & 1, failed, a.error_flag, 27));
        float s[64], m_tile = -INFINITY;
        if (ok) {
          tc_fence_after();
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            float v[32];
            tmem_ld32(tmem + COL_S + lane_addr + (uint32_t)(side * 64 + c * 32), v);
#pragma unroll
            for (int i = 0; i < 32; ++i) s[c * 32 + i] = v[i];
          }
          tc_fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(&s_free);
          const int k0 = w.start(j) + side * 64, k1 = w.end(j);
          if (j < w.kept_tiles ? k0 + 64 > k1 : k0 < lo_all || k0 + 63 > hi_all) {
            const int lo_i = lo_row - k0, hi_i = min(hi_row, k1 - 1) - k0, keep_i = keep - k0;
#pragma unroll
            for (int i = 0; i < 64; ++i)
              if ((i < lo_i && i >= keep_i) || i > hi_i) s[i] = scale2 < 0.f ? INFINITY : -INFINITY;
          }
          float mx[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) mx[i] = s[i] * scale2;
#pragma unroll
          for (int i = 4; i < 64; ++i) mx[i & 3] = fmaxf(mx[i & 3], s[i] * scale2);
          m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
        }
        row_max[gt & 1][side][r] = m_tile;
        pair_barrier(q);
        m_tile = fmaxf(m_tile, row_max[gt & 1][side ^ 1][r]);
        // the reference maximum moves only when a row's scores outgrow it by 2^8
        const bool move = __any_sync(ALL_LANES, m_tile > m_ref + 8.f);
        float corr = 1.f;
        if (move) {
          const float m_new = fmaxf(m_ref, m_tile);
          corr = exp2_fast(m_ref - m_new);
          m_ref = m_new;
          sum *= corr;
        }
        if (!ok) continue;
        float part[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          s[i] = exp2_fast(fmaf(s[i], scale2, -m_ref));
          part[i & 3] += s[i];
        }
        sum += (part[0] + part[1]) + (part[2] + part[3]);
        if (j > 0) {  // P and O may be touched once O += P(j - 1) V is done (for j = 0 the wait at the end of the item before)
          ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (gt - 1) & 1, failed, a.error_flag, 28));
          if (!ok) continue;
          tc_fence_after();
          if (move) {
            for (int c = side * 16; c < t.vn; c += 32) {
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
          uint32_t u[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(s[h * 32 + 2 * i], s[h * 32 + 2 * i + 1]);
            u[i] = *reinterpret_cast<const uint32_t*>(&b);
          }
          tmem_st16(tmem + COL_P + lane_addr + (uint32_t)(side * 32 + h * 16), u);
        }
        tmem_wait_st();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready);
      }
      row_sum[done & 1][side][r] = sum;
      pair_barrier(q);
      sum += row_sum[done & 1][side ^ 1][r];
      if (ok) ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (g + w.tiles - 1) & 1, failed, a.error_flag, 29));
      g += w.tiles;
      ++done;
      if (!ok) continue;
      tc_fence_after();
      float inv = l.out_scale / sum;
      if (l.off_gate >= 0 && qrow < w.n) inv *= sigmoid_f(a.p[(size_t)(w.first + qrow) * a.ldp + l.off_gate + w.head]);
      __nv_bfloat16* y = static_cast<__nv_bfloat16*>(a.y) + (size_t)(w.first + qrow) * a.ldy + w.head * l.vdim;
      const bool vec = l.vdim % 8 == 0 && (reinterpret_cast<uintptr_t>(y) & 15) == 0;
      if (l.v_rot) {  // pairs (c, c + half) are turned back by the row's angle
        const int half = l.vdim >> 1;
        const float2* cs = a.v_rot + (size_t)(w.first + min(qrow, w.n - 1)) * half;
        const bool vec2 = vec && half % 8 == 0;
        for (int c = side * 16; c < half; c += 32) {
          float u[16], v[16];
          tmem_ld16(tmem + COL_O + lane_addr + (uint32_t)c, u);
          tmem_ld16(tmem + COL_O + lane_addr + (uint32_t)(half + c), v);
          if (qrow < w.n) {
#pragma unroll
            for (int i = 0; i < 16; ++i)
              if (c + i < half) {
                const float2 r = cs[c + i];
                const float x = u[i] * inv, z = v[i] * inv;
                u[i] = x * r.x + z * r.y;
                v[i] = z * r.x - x * r.y;
              }
            if (vec2) {
#pragma unroll
              for (int h = 0; h < 2; ++h)
                if (c + h * 8 < half) {
                  store8(y + c + h * 8, u + h * 8);
                  store8(y + half + c + h * 8, v + h * 8);
                }
            } else {
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (c + i < half) {
                  y[c + i] = __float2bfloat16_rn(u[i]);
                  y[half + c + i] = __float2bfloat16_rn(v[i]);
                }
            }
          }
          __syncwarp();
        }
        tc_fence_before();  // this side's columns of O are in registers or stored: the next item may overwrite them
        __syncwarp();
        if (lane == 0) mbar_arrive(&o_free);
        continue;
      }
      for (int c = side * 16; c < t.vn; c += 32) {
        float o[16];
        tmem_ld16(tmem + COL_O + lane_addr + (uint32_t)c, o);
        if (qrow >= w.n) {  // a row of the next sequence or none: nothing to store
        } else if (vec) {
#pragma unroll
          for (int h = 0; h < 2; ++h)
            if (c + h * 8 < l.vdim) {
#pragma unroll
              for (int i = 0; i < 8; ++i) o[h * 8 + i] *= inv;
              store8(y + c + h * 8, o + h * 8);
            }
        } else {
#pragma unroll
          for (int i = 0; i < 16; ++i)
            if (c + i < l.vdim) y[c + i] = __float2bfloat16_rn(o[i] * inv);
        }
        __syncwarp();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&o_free);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, (uint32_t)t.tmem_cols);
}

// BF16 [rows][heads][dim] (dim % 8 == 0), rows `pitch` elements apart, box = 64 elements of one head of 128 rows, 128-byte swizzle; columns past dim and
// rows past the end read as zero.
bool make_head_map(CUtensorMap* map, const void* ptr, uint64_t rows, uint64_t heads, uint64_t dim, uint64_t pitch) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return false;
  cuuint64_t dims[3] = {dim, heads, rows};
  cuuint64_t strides[2] = {dim * 2, pitch * 2};
  cuuint32_t box[3] = {64, 1, 128};
  cuuint32_t estr[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(ptr), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

constexpr size_t TC_MAX_SMEM = 222 * 1024;  // beside the static arrays

}  // namespace

cudaError_t launch_attention_tc(const AttentionPortionArgs& a, cudaStream_t s) {
  const AttentionLayer& l = a.l;
  TcShape t;
  const int width = attention_q_width(l);
  t.dpieces = (width + 63) / 64;
  t.vpieces = (l.vdimp + 63) / 64;
  t.ksteps = (width + 15) / 16;
  t.vn = (l.vdimp + 15) / 16 * 16;
  t.tmem_cols = (int)COL_O + t.vn <= 256 ? 256 : 512;
  // queries stay resident while two value tiles and a few key pieces fit beside them
  auto bytes = [&] { return ((size_t)(t.q_resident ? t.dpieces + t.kstages : 2 * t.kstages) + (size_t)t.vstages * t.vpieces) * PIECE + 1024; };
  t.vstages = 2;
  t.q_resident = 1;
  t.kstages = std::min(t.dpieces == 1 ? 2 : 4, 2 * t.dpieces);
  if (bytes() > TC_MAX_SMEM) t.vstages = 1;
  if (bytes() > TC_MAX_SMEM) {
    t.q_resident = 0;
    t.vstages = 2;
    if (bytes() > TC_MAX_SMEM) t.vstages = 1;
  }
  if (bytes() > TC_MAX_SMEM) return cudaErrorInvalidValue;
  for (const int most = std::min(MAX_KSTAGES, 2 * t.dpieces); t.kstages < most && t.dpieces > 1;) {  // deeper rings where there is room
    ++t.kstages;
    if (bytes() > TC_MAX_SMEM) {
      --t.kstages;
      break;
    }
  }
  CUtensorMap mq, mk, mv;
  const int key_heads = l.mix ? 1 : l.kv_heads;
  if (!make_head_map(&mq, a.q, a.rows, l.heads, width, (uint64_t)l.heads * width) || !make_head_map(&mk, a.k, a.krows, key_heads, width, a.ldk) ||
      !make_head_map(&mv, a.v, a.krows, l.kv_heads, l.vdimp, a.ldv))
    return cudaErrorInvalidValue;
  const int qtiles = (a.max_len + QROWS - 1) / QROWS, items = qtiles * l.heads * a.nseq;
  int dev = 0, sms = 148;
  cudaGetDevice(&dev);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  auto run = [&](auto kernel, int per_sm) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TC_MAX_SMEM);
    return e != cudaSuccess ? e : launch_kernel(kernel, dim3(std::min(items, sms * per_sm)), dim3(THREADS), bytes(), s, false, mq, mk, mv, a, t, items, qtiles);
  };
  return t.tmem_cols <= 256 && bytes() <= 108 * 1024 ? run(attention_tc_kernel<2>, 2) : run(attention_tc_kernel<1>, 1);
}

}  // namespace pg
