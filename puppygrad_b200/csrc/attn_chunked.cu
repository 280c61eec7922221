// Attention of the layered models: grouped key / value heads, separate key and value sizes, optional per-head RMS norms
// of queries, keys and values. Which keys are visible, and where in the pages they lie, is KeyLife's matter; the single-token
// kernel here knows blocks of positions only, the portion kernels all of it.
#include <algorithm>
#include <cfloat>

#include "attn_pages.cuh"

namespace pg {
namespace {

// One warp: out[0..np) = norm(x[0..n)) * weight * mul, zero past n. `normed` false: only the copy.
template <typename T>
__device__ __forceinline__ void warp_norm_row(const float* x, int n, int np, const float* weight, bool normed, float eps,
                                              float mul, T* out, int lane) {
  float s = 0.f;
  if (normed)
    for (int c = lane; c < n; c += 32) s += x[c] * x[c];
  const float r = normed ? 1.f / sqrtf(lane_sum(s) / (float)n + eps) : 1.f;
  for (int c = lane; c < np; c += 32) {
    float v = 0.f;
    if (c < n) {
      v = x[c] * r;
      if (weight) v *= weight[c];
      v *= mul;
    }
    out[c] = from_f32<T>(v);
  }
}

// ------------------------------------------------------------------ one token per sequence
// Block = one kv head of one sequence and one part of its visible keys, for RB query heads of the group at a time.
// Eight lanes share a key (16-byte pieces of the row), the probabilities go through shared memory, and threads then own
// eight value columns each for a subset of the keys. Partial results of the parts are merged by the last block.
constexpr int STEP_THREADS = 256, STEP_KEYS = 256, RB = 4;

template <typename T>
__global__ void __launch_bounds__(STEP_THREADS) attention_step_kernel(AttentionStepArgs a, int y_bf16) {
  extern __shared__ __align__(16) float sm[];
  __shared__ int last_flag;
  const AttentionLayer& l = a.l;
  const int rep = l.heads / l.kv_heads;
  const int kvh = blockIdx.x, seq = blockIdx.y, split = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* qs = sm;                            // [rep][dimp]
  float* kn = qs + rep * l.dimp;             // [dimp] new key as stored
  float* vn = kn + l.dimp;                   // [vdimp] new value as stored
  float* sc = vn + l.vdimp;                  // [RB][STEP_KEYS]
  float* acc_s = sc + RB * STEP_KEYS;        // [groups][RB][vdimp] cross-thread sums
  __shared__ float red_m[RB], red_l[RB], corr_s[RB];

  grid_dep_launch();
  grid_dep_wait();
  const float* p = a.p + (size_t)seq * a.ldp;
  const int pos = a.pos[seq], last = pos % l.life.span;  // keys 0..last of this block of positions; `last` is the new one
  const int per = (last + 1 + a.splits - 1) / a.splits;
  const int k0 = split * per, k1 = min(last + 1, k0 + per);
  const int* table = a.page_table + (size_t)seq * l.pages_per_seq;
  T* pool = static_cast<T*>(a.pool);
  const bool owner = k0 <= last && last < k1;

  for (int i = warp; i < rep + 2; i += STEP_THREADS / 32) {
    if (i < rep)
      warp_norm_row<float>(p + l.off_q + (kvh * rep + i) * l.dim, l.dim, l.dimp, l.q_norm, l.q_norm != nullptr, l.eps, 1.f,
                           qs + i * l.dimp, lane);
    else if (i == rep)
      warp_norm_row<float>(p + l.off_k + kvh * l.dim, l.dim, l.dimp, l.k_norm, l.k_norm != nullptr, l.eps, 1.f, kn, lane);
    else
      warp_norm_row<float>(p + l.off_v + kvh * l.vdim, l.vdim, l.vdimp, nullptr, l.v_norm != 0, l.eps, 1.f, vn, lane);
  }
  __syncthreads();
  if (owner) {  // append; later reads of this row use the rounded copy in shared memory
    T* krow = page_row(l, pool, table, last, kvh, 0);
    T* vrow = page_row(l, pool, table, last, kvh, 1);
    for (int c = tid; c < l.dimp; c += STEP_THREADS) krow[c] = from_f32<T>(kn[c]);
    for (int c = tid; c < l.vdimp; c += STEP_THREADS) vrow[c] = from_f32<T>(vn[c]);
  }
  __syncthreads();
  for (int c = tid; c < l.dimp; c += STEP_THREADS) kn[c] = to_f32(from_f32<T>(kn[c]));
  for (int c = tid; c < l.vdimp; c += STEP_THREADS) vn[c] = to_f32(from_f32<T>(vn[c]));
  __syncthreads();

  const int nvec = l.vdimp / 8, groups = STEP_THREADS / nvec;  // value phase: thread = (8 columns, key subset)
  const int vc = tid % nvec, vg = tid / nvec;
  const int sub = lane >> 3, l8 = lane & 7;

  for (int r0 = 0; r0 < rep; r0 += RB) {
    const int nr = min(RB, rep - r0);
    float m_run[RB], l_run[RB], acc[RB][8];
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      m_run[r] = -FLT_MAX;
      l_run[r] = 0.f;
#pragma unroll
      for (int c = 0; c < 8; ++c) acc[r][c] = 0.f;
    }
    for (int kb = k0; kb < k1; kb += STEP_KEYS) {
      const int n = min(STEP_KEYS, k1 - kb);
      for (int j0 = warp * 4; j0 < n; j0 += STEP_THREADS / 32 * 4) {
        const int j = j0 + sub;
        float dot[RB];
#pragma unroll
        for (int r = 0; r < RB; ++r) dot[r] = 0.f;
        if (j < n) {
          const bool self = kb + j == last;
          const T* krow = self ? nullptr : page_row(l, pool, table, kb + j, kvh, 0);
          for (int c = l8 * 8; c < l.dimp; c += 64) {
            float kv[8];
            if (self) load8(kn + c, kv);
            else load8(krow + c, kv);
#pragma unroll
            for (int r = 0; r < RB; ++r) {
              if (r < nr) {
                float qv[8];
                load8(qs + (r0 + r) * l.dimp + c, qv);
#pragma unroll
                for (int e = 0; e < 8; ++e) dot[r] = fmaf(qv[e], kv[e], dot[r]);
              }
            }
          }
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1)
#pragma unroll
          for (int r = 0; r < RB; ++r) dot[r] += __shfl_xor_sync(ALL_LANES, dot[r], o);
        if (j < n && l8 == 0) {
#pragma unroll
          for (int r = 0; r < RB; ++r)
            if (r < nr) sc[r * STEP_KEYS + j] = dot[r] * l.scale;
        }
      }
      __syncthreads();
      if (warp < nr) {  // one warp per query head: running maximum, probabilities, sum
        float mx = -FLT_MAX;
        for (int j = lane; j < n; j += 32) mx = fmaxf(mx, sc[warp * STEP_KEYS + j]);
        mx = lane_max(mx);
        float m_old = -FLT_MAX;
#pragma unroll
        for (int r = 0; r < RB; ++r)
          if (r == warp) m_old = m_run[r];
        const float m_new = fmaxf(m_old, mx);
        float sum = 0.f;
        for (int j = lane; j < n; j += 32) {
          const float e = expf(sc[warp * STEP_KEYS + j] - m_new);
          sc[warp * STEP_KEYS + j] = e;
          sum += e;
        }
        sum = lane_sum(sum);
        if (lane == 0) {
          red_m[warp] = m_new;
          red_l[warp] = sum;
          corr_s[warp] = expf(m_old - m_new);
        }
      }
      __syncthreads();
#pragma unroll
      for (int r = 0; r < RB; ++r)
        if (r < nr) {
          m_run[r] = red_m[r];
          l_run[r] = l_run[r] * corr_s[r] + red_l[r];
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[r][c] *= corr_s[r];
        }
      if (vg < groups) {
        for (int j = vg; j < n; j += groups) {
          float vv[8];
          if (kb + j == last) load8(vn + vc * 8, vv);
          else load8(page_row(l, pool, table, kb + j, kvh, 1) + vc * 8, vv);
#pragma unroll
          for (int r = 0; r < RB; ++r)
            if (r < nr) {
              const float pr = sc[r * STEP_KEYS + j];
#pragma unroll
              for (int e = 0; e < 8; ++e) acc[r][e] = fmaf(pr, vv[e], acc[r][e]);
            }
        }
      }
      __syncthreads();
    }
    // sum over the key subsets
    if (vg < groups) {
#pragma unroll
      for (int r = 0; r < RB; ++r)
        if (r < nr)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc_s[((size_t)vg * RB + r) * l.vdimp + vc * 8 + e] = acc[r][e];
    }
    __syncthreads();
    for (int i = tid; i < nr * l.vdim; i += STEP_THREADS) {
      const int r = i / l.vdim, c = i % l.vdim;
      float s = 0.f;
      for (int g = 0; g < groups; ++g) s += acc_s[((size_t)g * RB + r) * l.vdimp + c];
      float lr = 0.f, mr = 0.f;
#pragma unroll
      for (int q = 0; q < RB; ++q)
        if (q == r) {
          lr = l_run[q];
          mr = m_run[q];
        }
      const int h = kvh * rep + r0 + r;
      if (a.splits == 1) {
        const float y = s / lr * l.out_scale;
        const size_t at = (size_t)seq * a.ldy + h * l.vdim + c;
        if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[at] = __float2bfloat16_rn(y);
        else static_cast<float*>(a.y)[at] = y;
      } else {
        float* pt = a.part + (((size_t)seq * l.heads + h) * a.splits + split) * (l.vdim + 2);
        pt[2 + c] = s;
        if (c == 0) {
          pt[0] = mr;
          pt[1] = lr;
        }
      }
    }
    __syncthreads();
  }
  if (a.splits == 1) return;
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    const unsigned n = atomicAdd(&a.counters[seq * l.kv_heads + kvh], 1u);
    last_flag = n == (unsigned)a.splits - 1;
    if (last_flag) a.counters[seq * l.kv_heads + kvh] = 0;
  }
  __syncthreads();
  if (!last_flag) return;
  __threadfence();
  for (int i = tid; i < rep * l.vdim; i += STEP_THREADS) {
    const int h = kvh * rep + i / l.vdim, c = i % l.vdim;
    const volatile float* pt = a.part + ((size_t)seq * l.heads + h) * a.splits * (l.vdim + 2);
    float m = -FLT_MAX;
    for (int s = 0; s < a.splits; ++s) m = fmaxf(m, pt[s * (l.vdim + 2)]);
    float num = 0.f, den = 0.f;
    for (int s = 0; s < a.splits; ++s) {
      const float w = expf(pt[s * (l.vdim + 2)] - m);
      num += w * pt[s * (l.vdim + 2) + 2 + c];
      den += w * pt[s * (l.vdim + 2) + 1];
    }
    const float y = num / den * l.out_scale;
    const size_t at = (size_t)seq * a.ldy + h * l.vdim + c;
    if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[at] = __float2bfloat16_rn(y);
    else static_cast<float*>(a.y)[at] = y;
  }
}

// ------------------------------------------------------------------ portions
// Norms of every row's queries, keys and values; a warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) attention_prep_kernel(AttentionPortionArgs a) {
  const AttentionLayer& l = a.l;
  const int per = l.heads + 2 * l.kv_heads, lane = threadIdx.x & 31;
  const long long total = (long long)a.rows * per;
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5; i < total;
       i += ((long long)gridDim.x * blockDim.x) >> 5) {
    const int row = (int)(i / per), j = (int)(i % per);
    const float* p = a.p + (size_t)row * a.ldp;
    const int seq = a.row_seq[row];
    const size_t krow = (size_t)a.key_start[seq] + l.life.context(a.seq_pos[seq]) + (row - a.seq_start[seq]);
    if (j < l.heads)
      warp_norm_row<T>(p + l.off_q + j * l.dim, l.dim, l.dimp, l.q_norm, l.q_norm != nullptr, l.eps, 1.f,
                       static_cast<T*>(a.q) + ((size_t)row * l.heads + j) * l.dimp, lane);
    else if (j < l.heads + l.kv_heads)
      warp_norm_row<T>(p + l.off_k + (j - l.heads) * l.dim, l.dim, l.dimp, l.k_norm, l.k_norm != nullptr, l.eps, 1.f,
                       static_cast<T*>(a.k) + krow * a.ldk + (j - l.heads) * l.dimp, lane);
    else
      warp_norm_row<T>(p + l.off_v + (j - l.heads - l.kv_heads) * l.vdim, l.vdim, l.vdimp, nullptr, l.v_norm != 0, l.eps, 1.f,
                       static_cast<T*>(a.v) + krow * a.ldv + (j - l.heads - l.kv_heads) * l.vdimp, lane);
  }
}

// The same when every size and offset is a multiple of four: eight lanes per (row, head), the row in registers.
template <typename T>
__global__ void __launch_bounds__(256) attention_prep_vec_kernel(AttentionPortionArgs a) {
  const AttentionLayer& l = a.l;
  const int per = l.heads + 2 * l.kv_heads, l8 = threadIdx.x & 7;
  const long long total = ((long long)a.rows * per + 3) / 4 * 4;  // whole warps stay together
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 3; i < total;
       i += ((long long)gridDim.x * blockDim.x) >> 3) {
    const bool on = i < (long long)a.rows * per;
    const int row = on ? (int)(i / per) : 0, j = on ? (int)(i % per) : 0;
    const int seq = a.row_seq[row];
    const size_t krow = (size_t)a.key_start[seq] + l.life.context(a.seq_pos[seq]) + (row - a.seq_start[seq]);
    const bool is_q = j < l.heads, is_k = !is_q && j < l.heads + l.kv_heads;
    const int h = is_q ? j : is_k ? j - l.heads : j - l.heads - l.kv_heads;
    const int n = is_q || is_k ? l.dim : l.vdim, np = is_q || is_k ? l.dimp : l.vdimp;
    const float* x = a.p + (size_t)row * a.ldp + (is_q ? l.off_q : is_k ? l.off_k : l.off_v) + h * n;
    const float* weight = is_q ? l.q_norm : is_k ? l.k_norm : nullptr;
    const bool normed = is_q ? l.q_norm != nullptr : is_k ? l.k_norm != nullptr : l.v_norm != 0;
    T* out = is_q   ? static_cast<T*>(a.q) + ((size_t)row * l.heads + h) * np
             : is_k ? static_cast<T*>(a.k) + krow * a.ldk + h * np
                    : static_cast<T*>(a.v) + krow * a.ldv + h * np;
    float4 v[8];
    float s = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      const int c = q * 32 + l8 * 4;
      v[q] = on && c < n ? load4(x + c) : make_float4(0, 0, 0, 0);
      s += (v[q].x * v[q].x + v[q].y * v[q].y) + (v[q].z * v[q].z + v[q].w * v[q].w);
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) s += __shfl_xor_sync(ALL_LANES, s, o);
    const float r = normed ? 1.f / sqrtf(s / (float)n + l.eps) : 1.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      const int c = q * 32 + l8 * 4;
      if (on && c < np) {
        float4 y = make_float4(v[q].x * r, v[q].y * r, v[q].z * r, v[q].w * r);
        if (weight && c < n) {
          y.x *= weight[c]; y.y *= weight[c + 1]; y.z *= weight[c + 2]; y.w *= weight[c + 3];
        }
        store4(out + c, y);
      }
    }
  }
}

// Eight elements between a workspace row (keys of all key heads, then their values) and a cached row.
template <typename T>
struct RowPiece {
  T *cached, *work;
  __device__ __forceinline__ RowPiece(const AttentionPortionArgs& a, const int* table, int place, size_t krow, int piece) {
    const AttentionLayer& l = a.l;
    const int e = piece * 8;
    const bool is_k = e < l.kv_heads * l.dimp;
    const int x = is_k ? e : e - l.kv_heads * l.dimp, w = is_k ? l.dimp : l.vrow;
    cached = page_row(l, static_cast<T*>(a.pool), table, place, x / w, is_k ? 0 : 1) + x % w;
    work = (is_k ? static_cast<T*>(a.k) + krow * a.ldk : static_cast<T*>(a.v) + krow * a.ldv) + x;
  }
  static __device__ __forceinline__ int count(const AttentionLayer& l) { return l.kv_heads * (l.dimp + l.vrow) / 8; }
  static __device__ __forceinline__ void copy(T* dst, const T* src) {
    reinterpret_cast<uint4*>(dst)[0] = reinterpret_cast<const uint4*>(src)[0];
    if (sizeof(T) == 4) reinterpret_cast<uint4*>(dst)[1] = reinterpret_cast<const uint4*>(src)[1];
  }
};

// Cached keys and values that the first row of each sequence still sees, copied in front of its own. Block = (key, seq).
template <typename T>
__global__ void __launch_bounds__(128) attention_context_kernel(AttentionPortionArgs a) {
  const AttentionLayer& l = a.l;
  const int seq = blockIdx.y, p0 = a.seq_pos[seq], ctx = l.life.context(p0);
  const int* table = a.page_table + (size_t)a.seq_slot[seq] * l.pages_per_seq;
  for (int c = blockIdx.x; c < ctx; c += gridDim.x)
    for (int i = threadIdx.x; i < RowPiece<T>::count(l); i += blockDim.x) {
      const RowPiece<T> r(a, table, l.life.place(l.life.context_position(p0, c)), (size_t)a.key_start[seq] + c, i);
      RowPiece<T>::copy(r.work, r.cached);
    }
}

// Stores the portion's keys and values that later tokens can still see.
template <typename T>
__global__ void __launch_bounds__(128) attention_store_kernel(AttentionPortionArgs a) {
  const AttentionLayer& l = a.l;
  const int row = blockIdx.x, seq = a.row_seq[row];
  const int first = a.seq_start[seq], n = a.seq_start[seq + 1] - first, p0 = a.seq_pos[seq], pos = p0 + (row - first);
  if (!l.life.lives(pos, p0 + n - 1)) return;
  const int* table = a.page_table + (size_t)a.seq_slot[seq] * l.pages_per_seq;
  for (int i = threadIdx.x; i < RowPiece<T>::count(l); i += blockDim.x) {
    const RowPiece<T> r(a, table, l.life.place(pos), (size_t)a.key_start[seq] + l.life.row(p0, pos), i);
    RowPiece<T>::copy(r.cached, r.work);
  }
}

// CUDA-core attention over the workspaces. Block = 32 query rows of one head of one sequence, 128 threads: four lanes
// per row, key tiles of 32, FP32 scores and sums, online softmax. Query and key rows are staged in pieces of DC columns, padded
// by one float.
constexpr int QT = 32, KT = 32, DC = 128;
template <typename T, int VR>
__global__ void __launch_bounds__(128) attention_rows_kernel(AttentionPortionArgs a) {
  extern __shared__ __align__(16) float sm[];
  const AttentionLayer& l = a.l;
  const int head = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
  const int first = a.seq_start[seq], n = a.seq_start[seq + 1] - first, q0 = blockIdx.x * QT;
  if (q0 >= n) return;
  const int rep = l.heads / l.kv_heads, kvh = head / rep, p0 = a.seq_pos[seq];
  const int width = l.mix ? l.kv_heads * l.dimp : l.dimp, koff = l.mix ? 0 : kvh * l.dimp, dc = min(width, DC);
  float* qs = sm;                       // [QT][dc + 1]
  float* ks = qs + QT * (dc + 1);       // [KT][dc + 1]
  float* vs = ks + KT * (dc + 1);       // [KT][vdimp]
  float* ps = vs + KT * l.vdimp;        // [QT][KT + 1]
  const int r = tid >> 2, sub = tid & 3;
  const int qrow = q0 + r;
  const bool live = qrow < n;
  auto stage = [&](float* dst, const T* src, size_t pitch, int rows, int c0) {  // rows past `rows` and columns past `width` as zero
    for (int i = tid; i < QT * dc; i += 128) {
      const int rr = i / dc, c = i % dc;
      dst[rr * (dc + 1) + c] = rr < rows && c0 + c < width ? to_f32(src[(size_t)rr * pitch + c0 + c]) : 0.f;
    }
  };
  const size_t qpitch = (size_t)l.heads * width;
  const T* qsrc = static_cast<const T*>(a.q) + (size_t)(first + q0) * qpitch + (size_t)head * width;
  if (width <= DC) stage(qs, qsrc, qpitch, n - q0, 0);
  // workspace keys [lo_row, hi_row] and those below `keep` are visible to this thread's row
  const int pos = p0 + min(qrow, n - 1);
  const int lo_row = l.life.low(p0, pos), hi_row = l.life.row(p0, pos), keep = l.life.keep;
  const int lo = l.life.low(p0, p0 + q0), hi = l.life.row(p0, p0 + min(q0 + QT, n) - 1);  // moving range of the block's rows
  const int kept = min(keep, lo);  // ... and the kept keys below it
  float m = l.sink ? l.sink[head] : -FLT_MAX, lsum = l.sink ? 1.f : 0.f, acc[VR];
#pragma unroll
  for (int c = 0; c < VR; ++c) acc[c] = 0.f;
  const int kept_tiles = (kept + KT - 1) / KT, tiles = kept_tiles + (hi - lo) / KT + 1;
  for (int tile = 0; tile < tiles; ++tile) {
    const int kt = tile < kept_tiles ? tile * KT : lo + (tile - kept_tiles) * KT;
    const int end = tile < kept_tiles ? min(kept, kt + KT) : min(hi + 1, kt + KT);
    __syncthreads();
    for (int i = tid; i < KT * l.vdimp; i += 128) {
      const int rr = i / l.vdimp, c = i % l.vdimp;
      vs[i] = kt + rr < end ? to_f32(static_cast<const T*>(a.v)[(size_t)(a.key_start[seq] + kt + rr) * a.ldv + kvh * l.vdimp + c]) : 0.f;
    }
    float s[KT / 4];
#pragma unroll
    for (int j = 0; j < KT / 4; ++j) s[j] = 0.f;
    for (int c0 = 0; c0 < width; c0 += dc) {
      if (c0 > 0) __syncthreads();
      stage(ks, static_cast<const T*>(a.k) + (size_t)(a.key_start[seq] + kt) * a.ldk + koff, a.ldk, end - kt, c0);
      if (width > DC) stage(qs, qsrc, qpitch, n - q0, c0);
      __syncthreads();
      for (int c = 0; c < dc; ++c) {
        const float q = qs[r * (dc + 1) + c];
#pragma unroll
        for (int j = 0; j < KT / 4; ++j) s[j] = fmaf(q, ks[(j * 4 + sub) * (dc + 1) + c], s[j]);
      }
    }
    float mx = -FLT_MAX;
#pragma unroll
    for (int j = 0; j < KT / 4; ++j) {
      const int key = kt + j * 4 + sub;
      s[j] = (live && key < end && key <= hi_row && (key >= lo_row || key < keep)) ? s[j] * l.scale : -FLT_MAX;
      mx = fmaxf(mx, s[j]);
    }
    mx = fmaxf(mx, __shfl_xor_sync(ALL_LANES, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(ALL_LANES, mx, 2));
    const float m_new = fmaxf(m, mx), corr = expf(m - m_new);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < KT / 4; ++j) {
      const float e = s[j] > -FLT_MAX ? expf(s[j] - m_new) : 0.f;
      ps[r * (KT + 1) + j * 4 + sub] = e;
      sum += e;
    }
    sum += __shfl_xor_sync(ALL_LANES, sum, 1);
    sum += __shfl_xor_sync(ALL_LANES, sum, 2);
    lsum = lsum * corr + sum;
    m = m_new;
    __syncwarp();  // the four lanes of a row exchange probabilities
#pragma unroll
    for (int c = 0; c < VR; ++c) acc[c] *= corr;
    for (int j = 0; j < KT; ++j) {
      const float pr = ps[r * (KT + 1) + j];
#pragma unroll
      for (int c = 0; c < VR; ++c) {
        const int col = c * 4 + sub;
        if (col < l.vdimp) acc[c] = fmaf(pr, vs[j * l.vdimp + col], acc[c]);
      }
    }
  }
  if (!live) return;
  float inv = l.out_scale / lsum;
  if (l.off_gate >= 0) inv *= sigmoid_f(a.p[(size_t)(first + qrow) * a.ldp + l.off_gate + head]);
#pragma unroll
  for (int c = 0; c < VR; ++c) {
    const int col = c * 4 + sub;
    if (col < l.vdim) static_cast<T*>(a.y)[(size_t)(first + qrow) * a.ldy + head * l.vdim + col] = from_f32<T>(acc[c] * inv);
  }
}

template <typename T>
cudaError_t ready_t(const AttentionPortionArgs& a, cudaStream_t s) {
  const AttentionLayer& l = a.l;
  if (l.rot_dims || l.v_rot || l.mix || l.q_bias) return launch_attention_rotate(a, sizeof(T) == 2, s);
  const long long warps = (long long)a.rows * (l.heads + 2 * l.kv_heads);
  const int pgrid = (int)std::min<long long>((warps + 7) / 8, 148 * 16);
  const bool vec = l.dim % 4 == 0 && l.vdim % 4 == 0 && l.off_q % 4 == 0 && l.off_k % 4 == 0 && l.off_v % 4 == 0 && a.ldp % 4 == 0;
  const int vgrid = (int)std::min<long long>((warps + 31) / 32, 148 * 16);
  return vec ? launch_kernel(attention_prep_vec_kernel<T>, dim3(vgrid), dim3(256), 0, s, false, a)
             : launch_kernel(attention_prep_kernel<T>, dim3(pgrid), dim3(256), 0, s, false, a);
}

cudaError_t rows_core(const AttentionPortionArgs& a, cudaStream_t s) {
  const AttentionLayer& l = a.l;
  const int dc = std::min(attention_q_width(l), DC);
  const dim3 grid((a.max_len + QT - 1) / QT, l.heads, a.nseq);
  const size_t smem = ((size_t)(QT + KT) * (dc + 1) + (size_t)KT * l.vdimp + (size_t)QT * (KT + 1)) * sizeof(float);
  cudaError_t e;
#define PG_ROWS(VR_)                                                                                                          \
  do {                                                                                                                        \
    e = cudaFuncSetAttribute(attention_rows_kernel<float, VR_>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);     \
    if (e == cudaSuccess) e = launch_kernel(attention_rows_kernel<float, VR_>, grid, dim3(128), smem, s, false, a);           \
  } while (0)
  if (l.vdimp <= 64) PG_ROWS(16);
  else if (l.vdimp <= 128) PG_ROWS(32);
  else PG_ROWS(64);
#undef PG_ROWS
  return e == cudaSuccess && l.v_rot ? launch_attention_turn_back(a, s) : e;
}

size_t step_smem(const AttentionLayer& l) {
  const int groups = STEP_THREADS / (l.vdimp / 8);
  return ((size_t)(l.heads / l.kv_heads) * l.dimp + l.dimp + l.vdimp + RB * STEP_KEYS + (size_t)groups * RB * l.vdimp) * sizeof(float);
}

}  // namespace

size_t attention_page_elems(const AttentionLayer& l) { return (size_t)l.kv_heads * l.page_tokens * (l.dimp + l.vrow); }

bool attention_supported(const AttentionLayer& l) { return step_smem(l) <= 200 * 1024; }

cudaError_t launch_attention_step(const AttentionStepArgs& a, bool bf16, bool y_bf16, bool pdl, cudaStream_t s) {
  const AttentionLayer& l = a.l;
  const size_t smem = step_smem(l);
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  const dim3 grid(l.kv_heads, a.batch, a.splits);
  const int yb = y_bf16 ? 1 : 0;
  cudaError_t e;
  if (bf16) {
    e = cudaFuncSetAttribute(attention_step_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    return e != cudaSuccess ? e : launch_kernel(attention_step_kernel<__nv_bfloat16>, grid, dim3(STEP_THREADS), smem, s, pdl, a, yb);
  }
  e = cudaFuncSetAttribute(attention_step_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  return e != cudaSuccess ? e : launch_kernel(attention_step_kernel<float>, grid, dim3(STEP_THREADS), smem, s, pdl, a, yb);
}

cudaError_t launch_attention_context(const AttentionPortionArgs& a, bool bf16, cudaStream_t s) {
  if (a.krows <= a.rows) return cudaSuccess;
  const dim3 grid(std::min(a.krows - a.rows, 1024), a.nseq);
  return bf16 ? launch_kernel(attention_context_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, false, a)
              : launch_kernel(attention_context_kernel<float>, grid, dim3(128), 0, s, false, a);
}

cudaError_t launch_attention_core(const AttentionPortionArgs& a, bool bf16, cudaStream_t s) {
  return bf16 ? launch_attention_tc(a, s) : rows_core(a, s);
}

cudaError_t launch_attention_store(const AttentionPortionArgs& a, bool bf16, cudaStream_t s) {
  return bf16 ? launch_kernel(attention_store_kernel<__nv_bfloat16>, dim3(a.rows), dim3(128), 0, s, false, a)
              : launch_kernel(attention_store_kernel<float>, dim3(a.rows), dim3(128), 0, s, false, a);
}

cudaError_t launch_attention_portion(const AttentionPortionArgs& a, bool bf16, cudaStream_t s) {
  if (a.rows <= 0) return cudaSuccess;
  cudaError_t e = bf16 ? ready_t<__nv_bfloat16>(a, s) : ready_t<float>(a, s);
  if (e == cudaSuccess) e = launch_attention_context(a, bf16, s);
  if (e == cudaSuccess) e = launch_attention_core(a, bf16, s);
  return e == cudaSuccess ? launch_attention_store(a, bf16, s) : e;
}

}  // namespace pg
