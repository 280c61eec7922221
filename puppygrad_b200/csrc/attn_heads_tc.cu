// Decode attention on the tensor cores for heads that share wide key rows: heads whose scores are mixed (the mixing is in the
// queries, which then run against the rows of all key heads) and heads over one latent row per token. tcgen05, operands by TMA
// straight from the pages, FP32 scores and sums.
//
// The cached tokens are the wide side of both products: S^T[keys, heads] = K Q^T with 128 keys as rows, and
// O^T[value columns, heads] += V^T P^T with 128 value columns as rows (V as it lies, MN-major). Block = one part of the keys of
// one sequence, for `hn` heads. Warp 0 loads pages into a ring of stages (128 keys x 128 columns each), warp 1 issues the
// MMAs, warps 2..5 do the softmax: thread = key, its heads side by side; maxima and sums over the keys by lane exchanges and
// shared memory. Latent rows are key and value in one: a stage then serves both products. A window's ring of pages holds
// visible tokens only, so the order of the rows does not matter and only the end is masked. Every wait is bounded.
#include <algorithm>

#include "attn_pages.cuh"
#include "tc_common.cuh"

namespace pg {
namespace {

constexpr int ROWS = 128;                       // keys of a tile
constexpr uint32_t PIECE = ROWS * 128;          // bytes of 64 BF16 columns of a tile
constexpr uint32_t STAGE = 2 * PIECE;
constexpr int MAX_STAGES = 6;
constexpr float LOG2E = 1.4426950408889634f;
constexpr size_t TC_MAX_SMEM = 225 * 1024;

__device__ __forceinline__ float exp2_fast(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
__device__ __forceinline__ void softmax_barrier() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

struct HeadsTcShape {
  int hn, npad, groups;     // heads of a block, rounded up to 16, blocks over the heads
  int kpieces, kstages;     // 64-column pieces and stages of a tile's keys
  int vpieces, vstages;     // ... of its values (of the key heads that a block's heads read)
  int reuse;                // a tile's key stages are its value stages
  int stages, tmem_cols;
  size_t smem;
};

// Sum or maximum over the 32 lanes of 16 values: lane l ends with that of value l >> 1.
template <bool MAX>
__device__ __forceinline__ float across_lanes(float (&v)[16], int lane) {
#pragma unroll
  for (int o = 16, w = 8; o > 1; o >>= 1, w >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < w) {
        const float send = up ? v[i] : v[i + w], keep = up ? v[i + w] : v[i], got = __shfl_xor_sync(ALL_LANES, send, o);
        v[i] = MAX ? fmaxf(keep, got) : keep + got;
      }
  }
  const float got = __shfl_xor_sync(ALL_LANES, v[0], 1);
  return MAX ? fmaxf(v[0], got) : v[0] + got;
}

__global__ void __launch_bounds__(192, 1)
    attention_heads_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                              const __grid_constant__ CUtensorMap map_v, AttentionStepArgs a, HeadsTcShape t) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ uint64_t q_full, full[MAX_STAGES], empty[MAX_STAGES], s_full, p_ready, pv_done;
  __shared__ uint32_t tmem_slot;
  __shared__ int failed_flag;
  __shared__ float m_ref[256], corr[256], w_max[4][256], w_sum[4][256];
  __shared__ int moved[2], v_base[256];  // v_base: first value column of a head
  const AttentionLayer& l = a.l;
  uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  uint8_t* ps = ring + (size_t)t.stages * STAGE;               // two pieces of 64 keys: [npad][64]
  const uint32_t hpiece = (uint32_t)t.npad * 128;              // bytes of 64 columns of the heads' rows
  uint8_t* qs = ps + 2 * hpiece;                               // kpieces pieces [npad][64]
  volatile int* failed = &failed_flag;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int split = blockIdx.x, seq = blockIdx.y, h0 = (int)blockIdx.z * t.hn, nh = min(t.hn, l.heads - h0);

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    for (int i = 0; i < MAX_STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(&s_full, 1);
    mbar_init(&p_ready, 4);
    mbar_init(&pv_done, 1);
    failed_flag = 0;
    moved[0] = moved[1] = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(&tmem_slot, (uint32_t)t.tmem_cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot, tmem_o = tmem + (uint32_t)t.npad;
  pdl_launch();
  pdl_wait();
  const int pos = a.pos[seq], n = l.life.window > 0 ? min(pos + 1, l.life.span) : pos % l.life.span + 1;  // visible rows of the slot
  const int all = (n + ROWS - 1) / ROWS, t0 = all * split / a.splits, t1 = all * (split + 1) / a.splits;
  const int kv0 = l.mix ? h0 / (l.heads / l.kv_heads) : 0;  // first key head whose values are needed
  bool ok = true;
  RingCursor ring_at;

  if (warp == 0) {
    if (t0 < t1) {
      if (lane == 0) {
        mbar_expect_tx(&q_full, (uint32_t)t.kpieces * hpiece);
        for (int d = 0; d < t.kpieces; ++d) tma_load_2d(qs + (size_t)d * hpiece, &map_q, d * 64, seq * l.heads + h0, &q_full);
      }
      const int* table = a.page_table + (size_t)seq * l.pages_per_seq;
      const int ppt = ROWS / l.page_tokens, last = (n - 1) / l.page_tokens, piece = lane / ppt;  // lane = (column piece, page of the tile)
      for (int tile = t0; tile < t1 && ok; ++tile) {
        const int page = table[min(tile * ppt + lane % ppt, last)];  // rows past the end: the last page once more, masked
        for (int part = 0; part < (t.reuse ? 1 : 2) && ok; ++part) {
          const CUtensorMap* map = part == 0 ? &map_k : &map_v;
          const int pieces = part == 0 ? t.kpieces : t.vpieces, x0 = part == 0 ? 0 : kv0 * l.vdimp;
          for (int d = 0; d < pieces; d += 2, ring_at.next(t.stages)) {
            const uint32_t s = ring_at.stage;
            const int two = min(2, pieces - d);
            if (lane == 0) {
              ok = mbar_wait(&empty[s], ring_at.parity ^ 1, failed, a.error_flag, 61);
              if (ok) mbar_expect_tx(&full[s], (uint32_t)two * PIECE);
            }
            ok = __shfl_sync(ALL_LANES, ok ? 1 : 0, 0) != 0;
            if (!ok) break;
            if (piece < two)
              tma_load_3d(ring + (size_t)s * STAGE + piece * PIECE + (size_t)(lane % ppt) * l.page_tokens * 128, map, x0 + (d + piece) * 64, 0, page,
                          &full[s]);
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && t0 < t1) {
      const uint32_t idesc_s = umma_idesc_bf16(ROWS, t.npad), idesc_o = umma_idesc_bf16(ROWS, t.npad) | (1u << 15);  // A of O^T is MN-major
      const int ksteps = (attention_q_width(l) + 15) / 16;
      const uint64_t k_desc = umma_desc_sw128(ring), v_desc = umma_desc_mn_sw128(ring, PIECE), q_desc = umma_desc_sw128(qs), p_desc = umma_desc_sw128(ps);
      const uint32_t hpiece16 = hpiece >> 4;
      ok = mbar_wait(&q_full, 0, failed, a.error_flag, 62);
      for (int tile = t0; tile < t1 && ok; ++tile) {
        const uint32_t turn = (uint32_t)(tile - t0);
        RingCursor first = ring_at;
        for (int d = 0; d < t.kstages; ++d, ring_at.next(t.stages)) {
          ok = mbar_wait(&full[ring_at.stage], ring_at.parity, failed, a.error_flag, 63);
          if (!ok) break;
          tc_fence_after();
          const uint64_t dk = k_desc + ring_at.stage * (STAGE >> 4), dq = q_desc + (uint32_t)(2 * d) * hpiece16;
          const int steps = ksteps - d * 8;
#pragma unroll
          for (int k = 0; k < 8; ++k)
            if (k < steps)
              umma_bf16_ss(tmem, dk + (uint64_t)((k >> 2) * (PIECE >> 4) + (k & 3) * 2), dq + (uint64_t)((k >> 2) * hpiece16 + (k & 3) * 2), idesc_s, (d | k) != 0);
          if (!t.reuse) umma_commit(&empty[ring_at.stage]);
        }
        if (!ok) break;
        umma_commit(&s_full);
        ok = mbar_wait(&p_ready, turn & 1, failed, a.error_flag, 64);  // P is in shared memory, S has been read, O is rescaled
        if (!ok) break;
        tc_fence_after();
        RingCursor v = t.reuse ? first : ring_at;
        for (int d = 0; d < t.vstages; ++d, v.next(t.stages)) {
          if (!t.reuse) ok = mbar_wait(&full[v.stage], v.parity, failed, a.error_flag, 65);
          if (!ok) break;
          tc_fence_after();
          const uint64_t dv = v_desc + v.stage * (STAGE >> 4);
#pragma unroll
          for (int k = 0; k < ROWS / 16; ++k)
            umma_bf16_ss(tmem_o + (uint32_t)(d * t.npad), dv + (uint64_t)(k * (2048 >> 4)), p_desc + (uint64_t)((k >> 2) * hpiece16 + (k & 3) * 2), idesc_o,
                         turn != 0 || k != 0);
          umma_commit(&empty[v.stage]);
        }
        ring_at = v;
        if (ok) umma_commit(&pv_done);
      }
    }
  } else {
    const int q = warp & 3, r = q * 32 + lane, tid = (int)threadIdx.x - 64;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const float scale2 = l.scale * LOG2E;
    for (int i = tid; i < t.npad; i += 128) {
      m_ref[i] = -1e30f;
      v_base[i] = i >= nh ? 1 << 30 : l.mix ? ((h0 + i) / (l.heads / l.kv_heads) - kv0) * l.vdimp : 0;  // no columns past the last head
      for (int w = 0; w < 4; ++w) w_sum[w][i] = 0.f;
    }
    softmax_barrier();
    for (int tile = t0; tile < t1; ++tile) {  // on expiry too: the barriers need every softmax warp equally often
      const uint32_t turn = (uint32_t)(tile - t0);
      if (ok) ok = __all_sync(ALL_LANES, mbar_wait(&s_full, turn & 1, failed, a.error_flag, 66));
      const bool seen = tile * ROWS + r < n;
      if (ok) {
        tc_fence_after();
        for (int c = 0; c < t.npad; c += 16) {
          float v[16];
          tmem_ld16(tmem + lane_addr + (uint32_t)c, v);
#pragma unroll
          for (int i = 0; i < 16; ++i) v[i] = seen ? v[i] * scale2 : -INFINITY;
          const float m = across_lanes<true>(v, lane);
          if ((lane & 1) == 0) w_max[q][c + (lane >> 1)] = m;
        }
      }
      softmax_barrier();
      for (int h = tid; h < t.npad; h += 128) {  // a reference maximum moves only when it is outgrown by 2^8
        const float m = fmaxf(fmaxf(w_max[0][h], w_max[1][h]), fmaxf(w_max[2][h], w_max[3][h])), old = m_ref[h];
        const bool move = m > old + 8.f;
        corr[h] = move ? exp2_fast(old - m) : 1.f;
        if (move) {
          m_ref[h] = m;
          moved[turn & 1] = 1;
        }
      }
      softmax_barrier();
      if (tid == 0) moved[(turn + 1) & 1] = 0;
      if (turn > 0 && ok) {
        ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (turn - 1) & 1, failed, a.error_flag, 67));  // P and O may be touched
        if (ok && moved[turn & 1]) {
          tc_fence_after();
          for (int c = 0; c < t.vstages * t.npad; c += 16) {
            float o[16];
            tmem_ld16(tmem_o + lane_addr + (uint32_t)c, o);
            uint32_t u[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) u[i] = __float_as_uint(o[i] * corr[c % t.npad + i]);
            tmem_st16(tmem_o + lane_addr + (uint32_t)c, u);
          }
          tmem_wait_st();
        }
      }
      if (ok) {
        uint8_t* prow = ps + (size_t)(r >> 6) * hpiece;
        const uint32_t chunk = (uint32_t)(r & 63) >> 3, in = (uint32_t)(r & 7) * 2;
        for (int c = 0; c < t.npad; c += 16) {
          float v[16];
          tmem_ld16(tmem + lane_addr + (uint32_t)c, v);
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            v[i] = seen ? exp2_fast(fmaf(v[i], scale2, -m_ref[c + i])) : 0.f;
            const uint32_t h = (uint32_t)(c + i);
            *reinterpret_cast<__nv_bfloat16*>(prow + h * 128 + ((chunk ^ (h & 7)) << 4) + in) = __float2bfloat16_rn(v[i]);
          }
          const float sum = across_lanes<false>(v, lane);
          if ((lane & 1) == 0) {
            float& w = w_sum[q][c + (lane >> 1)];
            w = w * corr[c + (lane >> 1)] + sum;
          }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready);
      }
    }
    if (t0 < t1 && ok) ok = __all_sync(ALL_LANES, mbar_wait(&pv_done, (uint32_t)(t1 - t0 - 1) & 1, failed, a.error_flag, 68));
    softmax_barrier();  // every warp's sums are in
    const int pitch = 4 + ((l.vdim + 3) & ~3);
    auto part = [&](int h) { return a.part + (((size_t)seq * l.heads + h) * a.splits + split) * pitch; };
    for (int h = tid; h < nh; h += 128) {
      float* p = part(h0 + h);
      p[0] = m_ref[h];
      p[1] = t0 < t1 && ok ? (w_sum[0][h] + w_sum[1][h]) + (w_sum[2][h] + w_sum[3][h]) : 0.f;
    }
    if (t0 < t1 && ok) {
      tc_fence_after();
      for (int d = 0; d < t.vstages; ++d) {
        const int col = d * 128 + r;
        float* out = part(h0) + 4 + col;
        const size_t head_pitch = (size_t)a.splits * pitch;
        for (int c = 0; c < t.npad; c += 16) {
          float o[16];
          tmem_ld16(tmem_o + lane_addr + (uint32_t)(d * t.npad + c), o);
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const int at = col - v_base[c + i];  // this head's value column
            if (at >= 0 && at < l.vdim) out[(c + i) * head_pitch - v_base[c + i]] = o[i];
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, (uint32_t)t.tmem_cols);
}

bool shape_of(const AttentionLayer& l, HeadsTcShape* out) {
  if (!l.mix && l.vrow != 0) return false;           // one wide row for all heads
  if (l.mix && !l.wide) return false;
  if (ROWS % l.page_tokens != 0 || l.page_tokens % 8 != 0) return false;
  const int rep = l.heads / l.kv_heads, width = attention_q_width(l);
  for (int groups = 1; groups <= l.heads; ++groups) {
    HeadsTcShape t{};
    t.hn = (l.heads + groups - 1) / groups;
    if (l.mix && t.hn >= rep) t.hn = (t.hn + rep - 1) / rep * rep;  // whole key heads
    t.npad = (t.hn + 15) / 16 * 16;
    t.groups = (l.heads + t.hn - 1) / t.hn;
    if (t.npad > 256) continue;
    t.kpieces = (width + 63) / 64;
    t.kstages = (t.kpieces + 1) / 2;
    const int kvs = l.mix ? (t.hn >= rep ? t.hn / rep : (rep % t.hn == 0 ? 1 : 2)) : 1;
    t.vpieces = (kvs * l.vdimp + 63) / 64;
    t.vstages = (t.vpieces + 1) / 2;
    const int cols = t.npad * (1 + t.vstages);
    if (cols > 512) continue;
    t.tmem_cols = 32;
    while (t.tmem_cols < cols) t.tmem_cols *= 2;
    auto bytes = [&](int stages) { return (size_t)stages * STAGE + (size_t)(2 + t.kpieces) * t.npad * 128 + 1024; };
    t.stages = MAX_STAGES;
    while (t.stages > 0 && bytes(t.stages) > TC_MAX_SMEM - 12 * 1024) --t.stages;  // beside the static arrays
    t.reuse = l.vrow == 0 && t.stages >= t.kstages ? 1 : 0;
    if (t.stages < 2 && !(t.reuse && t.stages >= 1)) continue;
    // no more stages than two tiles need
    t.stages = std::min(t.stages, 2 * (t.kstages + (t.reuse ? 0 : t.vstages)));
    t.smem = bytes(t.stages);
    *out = t;
    return true;
  }
  return false;
}

// Cached rows [pages][page_tokens][width] (pages `pitch` elements apart), box = 64 columns of one page.
bool make_page_map(CUtensorMap* map, const __nv_bfloat16* ptr, uint64_t width, uint64_t tokens, uint64_t pages, uint64_t pitch) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return false;
  cuuint64_t dims[3] = {width, tokens, pages};
  cuuint64_t strides[2] = {width * 2, pitch * 2};
  cuuint32_t box[3] = {64, (cuuint32_t)tokens, 1};
  cuuint32_t estr[3] = {1, 1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<__nv_bfloat16*>(ptr), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace

bool attention_heads_tc_supported(const AttentionLayer& l) {
  HeadsTcShape t;
  return shape_of(l, &t);
}

int attention_heads_tc_splits(const AttentionLayer& l, int batch, int tiles, int sms) {
  HeadsTcShape t;
  if (!shape_of(l, &t)) return 1;
  // rounds of blocks, times tiles of a block and what a block costs beside them (about a tile and a half)
  int best = 1;
  double cost = 1e30;
  for (int s = 1; s <= 16 && s <= tiles; ++s) {
    const double c = (double)((batch * t.groups * s + sms - 1) / sms) * ((tiles + s - 1) / s + 1.5) + 0.02 * s;
    if (c < cost) {
      cost = c;
      best = s;
    }
  }
  return best;
}

cudaError_t launch_attention_heads_tc(const AttentionStepArgs& a, bool pdl, cudaStream_t s) {
  const AttentionLayer& l = a.l;
  HeadsTcShape t;
  if (!shape_of(l, &t)) return cudaErrorInvalidValue;
  const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(a.pool);
  const uint64_t pitch = attention_page_elems(l), kw = (uint64_t)l.kv_heads * l.dimp, vw = (uint64_t)l.kv_heads * l.vrow;
  CUtensorMap mq, mk, mv;
  if (!make_map_bf16(&mq, a.q16, (uint64_t)a.batch * l.heads, attention_q_width(l), t.npad) ||
      !make_page_map(&mk, pool, kw, l.page_tokens, a.num_pages, pitch))
    return cudaErrorInvalidValue;
  if (l.vrow == 0) mv = mk;
  else if (!make_page_map(&mv, pool + kw * l.page_tokens, vw, l.page_tokens, a.num_pages, pitch)) return cudaErrorInvalidValue;
  cudaError_t e = cudaFuncSetAttribute(attention_heads_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(TC_MAX_SMEM - 11 * 1024));
  if (e != cudaSuccess) return e;
  return launch_kernel(attention_heads_tc_kernel, dim3(a.splits, a.batch, t.groups), dim3(192), t.smem, s, pdl, mq, mk, mv, a, t);
}

}  // namespace pg
