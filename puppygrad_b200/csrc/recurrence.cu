// Recurrent mixers with one [dim, vdim] FP32 state matrix per head (gated linear attention, generalized delta rule):
// the single-token step over the cached states, and the scan over whole portions of prompts.
//
// Both rules act on every column of the state on its own (S[:, c] needs only v[c] of the new token), so a column's
// `dim` entries are spread over a few lanes and the columns over groups of lanes, warps and blocks. Everything that
// enters the recurrence is FP32.
#include <algorithm>
#include <cstdlib>

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

// ------------------------------------------------------------------ one token per sequence
constexpr int STEP_THREADS = 256;

template <int NR>
__global__ void __launch_bounds__(STEP_THREADS) recurrence_step_kernel(RecurrenceStepArgs a, int y_bf16) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33];
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, dv = l.vdim, dvp = l.dvp, K = l.heads * dk;
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const bool delta = l.kind == KIND_DELTA;
  const int dka = (dk + 3) & ~3, rka = (l.rank + 3) & ~3;  // rows of shared memory start on 16-byte boundaries
  float* ks = sm;            // [dk] key
  float* ws = ks + dka;      // decay
  float* qs = ws + dka;      // query (r)
  float* us = qs + dka;      // unit key
  float* bs = us + dka;      // a * u
  float* ts = bs + dka;      // [rank]
  float* vs = ts + rka;      // [dvp]
  float* ds = vs + dvp;      // [dvp] u^T S
  float* os = ds + dvp;      // [dvp]
  float* part = os + dvp;    // [KG][dvp]
  const int dv4 = dvp / 4, KG = STEP_THREADS / dv4;
  const int c4 = tid % dv4, kg = tid / dv4;
  const bool active = kg < KG;

  grid_dep_launch();
  grid_dep_wait();
  const float* p = a.p + (size_t)seq * a.ldp;
  const bool fresh = a.pos[seq] == 0;
  float* S = a.state + ((size_t)seq * l.heads + head) * dk * dvp;
  constexpr int NRR = NR > 0 ? NR : 1;
  float4 st[NRR];
  if (NR > 0) {  // the state's loads overlap the gate arithmetic below
#pragma unroll
    for (int i = 0; i < NRR; ++i) {
      const int r = kg + i * KG;
      st[i] = (active && !fresh && r < dk) ? load4(S + (size_t)r * dvp + c4 * 4) : make_float4(0, 0, 0, 0);
    }
  }
  for (int r = tid; r < l.rank; r += STEP_THREADS) ts[r] = delta ? tanhf(p[l.off_t + r]) : p[l.off_t + r];
  float kk = 0.f;
  for (int c = tid; c < dk; c += STEP_THREADS) {
    ks[c] = p[l.off_k + head * dk + c];
    qs[c] = p[l.off_q + head * dk + c];
    kk += ks[c] * ks[c];
  }
  for (int c = tid; c < dvp; c += STEP_THREADS) vs[c] = c < dv ? p[l.off_v + head * dv + c] : 0.f;
  kk = block_sum(kk, red);  // also orders the shared-memory writes above
  const float inv_norm = 1.f / sqrtf(kk + UNIT_EPS);
  for (int c = tid; c < dk; c += STEP_THREADS) {
    const int ch = head * dk + c;
    float z = l.b2[ch];
    for (int r = 0; r < l.rank; ++r) z = fmaf(l.w2[(size_t)r * K + ch], ts[r], z);
    ws[c] = decay_of(l.kind, z, l.inv_tau);
    if (delta) {
      const float u = ks[c] * inv_norm;
      us[c] = u;
      bs[c] = sigmoid_f(p[l.off_a + ch] + l.a_bias[ch]) * u;
    }
  }
  __syncthreads();
  if (delta) {
    float4 d = make_float4(0, 0, 0, 0);
    if (active && !fresh) {
      for (int i = 0; i < (NR > 0 ? NRR : (dk + KG - 1) / KG); ++i) {
        const int r = kg + i * KG;
        if (r >= dk) break;
        const float4 s = NR > 0 ? st[NR > 0 ? i : 0] : load4(S + (size_t)r * dvp + c4 * 4);
        const float u = us[r];
        d.x = fmaf(u, s.x, d.x); d.y = fmaf(u, s.y, d.y); d.z = fmaf(u, s.z, d.z); d.w = fmaf(u, s.w, d.w);
      }
    }
    if (active) store4(part + (size_t)kg * dvp + c4 * 4, d);
    __syncthreads();
    for (int c = tid; c < dvp; c += STEP_THREADS) {
      float s = 0.f;
      for (int g = 0; g < KG; ++g) s += part[(size_t)g * dvp + c];
      ds[c] = s;
    }
    __syncthreads();
  }
  float4 o = make_float4(0, 0, 0, 0);
  if (active) {
    const float4 v = load4(vs + c4 * 4);
    const float4 d = delta ? load4(ds + c4 * 4) : make_float4(0, 0, 0, 0);
    for (int i = 0; i < (NR > 0 ? NRR : (dk + KG - 1) / KG); ++i) {
      const int r = kg + i * KG;
      if (r >= dk) break;
      float4 s = NR > 0 ? st[NR > 0 ? i : 0] : (fresh ? make_float4(0, 0, 0, 0) : load4(S + (size_t)r * dvp + c4 * 4));
      const float w = ws[r], k = ks[r], q = qs[r], b = delta ? bs[r] : 0.f;
      s.x = fmaf(w, s.x, fmaf(k, v.x, -b * d.x));
      s.y = fmaf(w, s.y, fmaf(k, v.y, -b * d.y));
      s.z = fmaf(w, s.z, fmaf(k, v.z, -b * d.z));
      s.w = fmaf(w, s.w, fmaf(k, v.w, -b * d.w));
      store4(S + (size_t)r * dvp + c4 * 4, s);
      o.x = fmaf(q, s.x, o.x); o.y = fmaf(q, s.y, o.y); o.z = fmaf(q, s.z, o.z); o.w = fmaf(q, s.w, o.w);
    }
    store4(part + (size_t)kg * dvp + c4 * 4, o);
  }
  __syncthreads();
  float sq = 0.f;
  for (int c = tid; c < dv; c += STEP_THREADS) {
    float s = 0.f;
    for (int g = 0; g < KG; ++g) s += part[(size_t)g * dvp + c];
    s *= l.q_scale;
    os[c] = s;
    sq += s * s;
  }
  sq = block_sum(sq, red);
  const float rinv = 1.f / sqrtf(sq / (float)dv + l.eps);
  for (int c = tid; c < dv; c += STEP_THREADS) {
    const float g = p[l.off_g + head * dv + c];
    const float gate = delta ? sigmoid_f(g) : silu_f(g);
    const float y = os[c] * rinv * l.norm[delta ? head * dv + c : c] * gate * l.out_scale;
    const size_t i = (size_t)seq * a.ldy + head * dv + c;
    if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[i] = __float2bfloat16_rn(y);
    else static_cast<float*>(a.y)[i] = y;
  }
}

// ------------------------------------------------------------------ gates of whole portions
constexpr int GATE_ROWS = 16;
// decay, and for the delta rule the unit keys u and the removal rates a * u, of GATE_ROWS rows per block
__global__ void __launch_bounds__(256) recurrence_gates_kernel(RecurrenceScanArgs a) {
  extern __shared__ __align__(16) float sm[];  // [rank][GATE_ROWS]
  const RecurrenceLayer& l = a.l;
  const int K = l.heads * l.dim, r0 = blockIdx.x * GATE_ROWS, tid = threadIdx.x;
  const int nr = min(GATE_ROWS, a.rows - r0);
  const bool delta = l.kind == KIND_DELTA;
  for (int i = tid; i < GATE_ROWS * l.rank; i += blockDim.x) {
    const int j = i / l.rank, r = i % l.rank;
    const float t = j < nr ? a.p[(size_t)(r0 + j) * a.ldp + l.off_t + r] : 0.f;
    sm[r * GATE_ROWS + j] = delta ? tanhf(t) : t;
  }
  __syncthreads();
  for (int c = tid; c < K; c += blockDim.x) {
    float z[GATE_ROWS];
#pragma unroll
    for (int j = 0; j < GATE_ROWS; ++j) z[j] = l.b2[c];
#pragma unroll 4
    for (int r = 0; r < l.rank; ++r) {
      const float w = l.w2[(size_t)r * K + c];
#pragma unroll
      for (int j = 0; j < GATE_ROWS; j += 4) {
        const float4 t = load4(sm + r * GATE_ROWS + j);
        z[j] = fmaf(w, t.x, z[j]);
        z[j + 1] = fmaf(w, t.y, z[j + 1]);
        z[j + 2] = fmaf(w, t.z, z[j + 2]);
        z[j + 3] = fmaf(w, t.w, z[j + 3]);
      }
    }
#pragma unroll
    for (int j = 0; j < GATE_ROWS; ++j)
      if (j < nr) a.decay[(size_t)(r0 + j) * K + c] = decay_of(l.kind, z[j], l.inv_tau);
  }
  if (!delta) return;
  const int warp = tid >> 5, lane = tid & 31;
  for (int i = warp; i < nr * l.heads; i += blockDim.x >> 5) {
    const int j = i / l.heads, head = i % l.heads;
    const float* row = a.p + (size_t)(r0 + j) * a.ldp;
    const float* k = row + l.off_k + head * l.dim;
    float s = 0.f;
    for (int c = lane; c < l.dim; c += 32) s += k[c] * k[c];
    const float inv = 1.f / sqrtf(lane_sum(s) + UNIT_EPS);
    for (int c = lane; c < l.dim; c += 32) {
      const int ch = head * l.dim + c;
      const float u = k[c] * inv;
      a.unit[(size_t)(r0 + j) * K + ch] = u;
      a.rate[(size_t)(r0 + j) * K + ch] = sigmoid_f(row[l.off_a + ch] + l.a_bias[ch]) * u;
    }
  }
}

// ------------------------------------------------------------------ scan
// Block = one head of one sequence (or of one segment of it). Eight lanes share a column of the state (lane l holds
// rows 32 j + 4 l + i in s[4 j + i]), a lane group has CPL columns, a warp four groups. Tokens are staged in shared
// memory TB at a time, two buffers, by asynchronous copies.
enum ScanMode {
  SCAN_FULL = 0,     // whole sequence: start from the cached state (or zero), outputs, final state to the cache
  SCAN_LOCAL = 1,    // one segment from a zero state, no outputs: its contribution to the state
  SCAN_TRANS = 2,    // one segment with identity columns and no values: its transition matrix (delta)
  SCAN_OUTPUT = 3    // one segment from its known start state: outputs
};
struct ScanArgs {
  RecurrenceScanArgs a;
  int mode, tb;
  float *seg_state, *seg_trans;  // [nseq][max_segs][heads][dim][dvp], [nseq][max_segs][heads][dim][dkp] (GLA: [..][dim] decays)
  int dkp;
  int col_blocks, block_cols;  // column blocks of a head, columns of each (the last may have fewer)
  int vec;      // 16-byte copies are possible
  int y_bf16;
};

__device__ __forceinline__ void copy_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Sum of CPL values over the eight lanes of a group. Afterwards every lane holds one column's total: the one
// owned_column() names.
template <int CPL>
__device__ __forceinline__ float group_reduce(const float (&v)[CPL], int lr) {
  float x;
  if (CPL == 4) {
    const bool up = lr & 4;
    const float a0 = up ? v[2 % CPL] : v[0], a1 = up ? v[3 % CPL] : v[1 % CPL];
    const float b0 = up ? v[0] : v[2 % CPL], b1 = up ? v[1 % CPL] : v[3 % CPL];
    const float c0 = a0 + __shfl_xor_sync(ALL_LANES, b0, 4), c1 = a1 + __shfl_xor_sync(ALL_LANES, b1, 4);
    const bool up2 = lr & 2;
    x = (up2 ? c1 : c0) + __shfl_xor_sync(ALL_LANES, up2 ? c0 : c1, 2);
  } else if (CPL == 2) {
    const bool up = lr & 4;
    x = (up ? v[1 % CPL] : v[0]) + __shfl_xor_sync(ALL_LANES, up ? v[0] : v[1 % CPL], 4);
    x += __shfl_xor_sync(ALL_LANES, x, 2);
  } else {
    x = v[0] + __shfl_xor_sync(ALL_LANES, v[0], 4);
    x += __shfl_xor_sync(ALL_LANES, x, 2);
  }
  return x + __shfl_xor_sync(ALL_LANES, x, 1);
}
template <int CPL>
__device__ __forceinline__ int owned_column(int lr) {
  return CPL == 4 ? ((lr & 4) >> 1) | ((lr & 2) >> 1) : CPL == 2 ? (lr & 4) >> 2 : 0;
}
// The totals of all columns in every lane.
template <int CPL>
__device__ __forceinline__ void group_all_reduce(float (&v)[CPL], int lr) {
  const float x = group_reduce<CPL>(v, lr);
  if (CPL == 4) {
    const float y = __shfl_xor_sync(ALL_LANES, x, 2);
    const float lo = lr & 2 ? y : x, hi = lr & 2 ? x : y;
    const float lo2 = __shfl_xor_sync(ALL_LANES, lo, 4), hi2 = __shfl_xor_sync(ALL_LANES, hi, 4);
    v[0] = lr & 4 ? lo2 : lo;
    v[1 % CPL] = lr & 4 ? hi2 : hi;
    v[2 % CPL] = lr & 4 ? lo : lo2;
    v[3 % CPL] = lr & 4 ? hi : hi2;
  } else if (CPL == 2) {
    const float y = __shfl_xor_sync(ALL_LANES, x, 4);
    v[0] = lr & 4 ? y : x;
    v[1 % CPL] = lr & 4 ? x : y;
  } else {
    v[0] = x;
  }
}

template <int KIND, int RPL, int CPL>
__global__ void __launch_bounds__(512, 1) recurrence_scan_kernel(ScanArgs sa) {
  extern __shared__ __align__(16) float sm[];
  constexpr int DKP = 8 * RPL, NA = KIND == KIND_DELTA ? 5 : 3;  // staged key-channel arrays
  const RecurrenceScanArgs& a = sa.a;
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, K = l.heads * dk, tid = threadIdx.x, nthreads = blockDim.x;
  const bool trans = sa.mode == SCAN_TRANS;
  // blockIdx.x = head * (column blocks) + column block; with several column blocks per head the outputs leave unnormed
  const int head = blockIdx.x / sa.col_blocks, cb = blockIdx.x % sa.col_blocks, seq = blockIdx.y, seg = blockIdx.z;
  const int all_cols = trans ? dk : l.vdim, cbase = cb * sa.block_cols;
  const int dv = min(sa.block_cols, all_cols - cbase);  // columns of this block
  const int W = nthreads >> 5, COLS = W * 4 * CPL, TB = sa.tb;
  const int stride = NA * DKP + 2 * COLS;  // floats of one staged token: k, decay, q, (u, rate), v, gate
  float* stage = sm;                       // [2][TB][stride]
  float* os = sm + (size_t)2 * TB * stride;  // [TB][COLS]
  const int lane = tid & 31, warp = tid >> 5, lr = lane & 7;
  const int col0 = (warp * 4 + (lane >> 3)) * CPL;
  const bool outputs = sa.mode == SCAN_FULL || sa.mode == SCAN_OUTPUT;

  int t0 = a.seq_start[seq], t1 = a.seq_start[seq + 1];
  if (sa.mode != SCAN_FULL) {
    t0 += seg * a.seg_tokens;
    t1 = min(t1, t0 + a.seg_tokens);
    if (t0 >= t1) return;
  }
  for (int i = tid; i < 2 * TB * stride; i += nthreads) stage[i] = 0.f;  // the padding stays zero
  __syncthreads();

  auto load_block = [&](int buf, int tb0) {
    const int n = min(TB, t1 - tb0);
    float* dst0 = stage + (size_t)buf * TB * stride;
    auto src_of = [&](int row, int arr) -> const float* {
      const float* p = a.p + (size_t)row * a.ldp;
      switch (arr) {
        case 0: return p + l.off_k + head * dk;
        case 1: return a.decay + (size_t)row * K + head * dk;
        case 2: return p + l.off_q + head * dk;
        case 3: return a.unit + (size_t)row * K + head * dk;
        default: return a.rate + (size_t)row * K + head * dk;
      }
    };
    const int vec = sa.vec, e = vec ? 4 : 1;
    const int nk = dk / e, nv = trans ? 0 : dv / e, ng = outputs && sa.col_blocks == 1 ? nv : 0;
    const int per = NA * nk + nv + ng;
    for (int i = tid; i < n * per; i += nthreads) {
      const int t = i / per, j = i - t * per, row = tb0 + t;
      float* d = dst0 + (size_t)t * stride;
      const float* s;
      if (j < NA * nk) {
        const int arr = j / nk, x = (j - arr * nk) * e;
        if (arr == 2 && !outputs) continue;
        d += arr * DKP + x;
        s = src_of(row, arr) + x;
      } else if (j < NA * nk + nv) {
        const int x = (j - NA * nk) * e;
        d += NA * DKP + x;
        s = a.p + (size_t)row * a.ldp + l.off_v + head * l.vdim + cbase + x;
      } else {
        const int x = (j - NA * nk - nv) * e;
        d += NA * DKP + COLS + x;
        s = a.p + (size_t)row * a.ldp + l.off_g + head * l.vdim + cbase + x;
      }
      if (vec) copy_async16(d, s);
      else copy_async4(d, s);
    }
  };

  // start state
  float s[RPL][CPL];
  const size_t seg_index = ((size_t)seq * a.max_segs + seg) * l.heads + head;
  const float* init = nullptr;
  if (sa.mode == SCAN_FULL && a.seq_pos[seq] > 0) init = a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp;
  if (sa.mode == SCAN_OUTPUT) init = sa.seg_state + seg_index * dk * l.dvp;
#pragma unroll
  for (int r = 0; r < RPL; ++r) {
    const int row = (r >> 2) * 32 + lr * 4 + (r & 3);
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      const int col = col0 + c;
      float v = 0.f;
      if (row < dk && col < dv) {
        if (init) v = init[(size_t)row * l.dvp + cbase + col];
        else if (trans) v = row == cbase + col ? 1.f : 0.f;
      }
      s[r][c] = v;
    }
  }
  load_block(0, t0);
  copy_commit();
  int buf = 0;
  for (int tb0 = t0; tb0 < t1; tb0 += TB, buf ^= 1) {
    copy_wait<0>();
    __syncthreads();  // this block of tokens is staged; everyone has left the other buffer and os
    if (tb0 + TB < t1) load_block(buf ^ 1, tb0 + TB);
    copy_commit();
    const int n = min(TB, t1 - tb0);
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      const float* x = stage + ((size_t)buf * TB + t) * stride;
      const float* xk = x + lr * 4;
      float v[CPL], o[CPL], d[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        v[c] = x[NA * DKP + col0 + c];
        o[c] = d[c] = 0.f;
      }
      if (KIND == KIND_DELTA) {
        float d2[CPL];
#pragma unroll
        for (int c = 0; c < CPL; ++c) d2[c] = 0.f;
#pragma unroll
        for (int j = 0; j < RPL / 4; ++j) {
          const float4 u = load4(xk + 3 * DKP + j * 32);
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            d[c] = fmaf(u.x, s[4 * j][c], d[c]);
            d2[c] = fmaf(u.y, s[4 * j + 1][c], d2[c]);
            d[c] = fmaf(u.z, s[4 * j + 2][c], d[c]);
            d2[c] = fmaf(u.w, s[4 * j + 3][c], d2[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < CPL; ++c) d[c] += d2[c];
        group_all_reduce<CPL>(d, lr);
      }
#pragma unroll
      for (int j = 0; j < RPL / 4; ++j) {
        const float4 k = load4(xk + j * 32), w = load4(xk + DKP + j * 32), q = load4(xk + 2 * DKP + j * 32);
        float4 b = make_float4(0, 0, 0, 0);
        if (KIND == KIND_DELTA) b = load4(xk + 4 * DKP + j * 32);
        const float kk[4] = {k.x, k.y, k.z, k.w}, ww[4] = {w.x, w.y, w.z, w.w}, qq[4] = {q.x, q.y, q.z, q.w};
        const float bb[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int r = 4 * j + i;
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            float add = kk[i] * v[c];
            if (KIND == KIND_DELTA) add = fmaf(-bb[i], d[c], add);
            s[r][c] = fmaf(ww[i], s[r][c], add);
            o[c] = fmaf(qq[i], s[r][c], o[c]);
          }
        }
      }
      if (outputs) {
        const float total = group_reduce<CPL>(o, lr);
        if (CPL == 4 ? (lr & 1) == 0 : CPL == 2 ? (lr & 3) == 0 : lr == 0)
          os[(size_t)t * COLS + col0 + owned_column<CPL>(lr)] = total * l.q_scale;
      }
    }
    if (outputs) {
      __syncthreads();
      if (sa.col_blocks > 1) {  // recurrence_output_kernel finishes the rows
        for (int i = tid; i < n * dv; i += nthreads)
          a.out_raw[(size_t)(tb0 + i / dv) * (l.heads * l.vdim) + head * l.vdim + cbase + i % dv] = os[(size_t)(i / dv) * COLS + i % dv];
        continue;
      }
      // head norm, gate and branch scale of the block's tokens, a warp per token
      for (int t = warp; t < n; t += W) {
        const float* o = os + (size_t)t * COLS;
        const float* g = stage + ((size_t)buf * TB + t) * stride + NA * DKP + COLS;
        float sq = 0.f;
        for (int c = lane; c < dv; c += 32) sq += o[c] * o[c];
        const float rinv = 1.f / sqrtf(lane_sum(sq) / (float)dv + l.eps);
        const size_t base = (size_t)(tb0 + t) * a.ldy + head * dv;
        for (int c = lane; c < dv; c += 32) {
          const float gate = KIND == KIND_DELTA ? sigmoid_f(g[c]) : silu_f(g[c]);
          const float y = o[c] * rinv * l.norm[KIND == KIND_DELTA ? head * dv + c : c] * gate * l.out_scale;
          if (sa.y_bf16) static_cast<__nv_bfloat16*>(a.y)[base + c] = __float2bfloat16_rn(y);
          else static_cast<float*>(a.y)[base + c] = y;
        }
      }
    }
  }
  copy_wait<0>();

  if (sa.mode == SCAN_OUTPUT) return;
  float* fin = sa.mode == SCAN_FULL ? a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp
               : trans              ? sa.seg_trans + seg_index * dk * sa.dkp
                                    : sa.seg_state + seg_index * dk * l.dvp;
  const int pitch = trans ? sa.dkp : l.dvp;
#pragma unroll
  for (int r = 0; r < RPL; ++r) {
    const int row = (r >> 2) * 32 + lr * 4 + (r & 3);
    if (row < dk) {
#pragma unroll
      for (int c = 0; c < CPL; ++c)
        if (col0 + c < dv) fin[(size_t)row * pitch + cbase + col0 + c] = s[r][c];
    }
  }
}

// Head norm, gate and branch scale of scan outputs that left in several column blocks; a warp per (row, head).
__global__ void __launch_bounds__(256) recurrence_output_kernel(RecurrenceScanArgs a, int y_bf16) {
  const RecurrenceLayer& l = a.l;
  const int lane = threadIdx.x & 31, dv = l.vdim;
  const long long total = (long long)a.rows * l.heads;
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5; i < total; i += ((long long)gridDim.x * blockDim.x) >> 5) {
    const int row = (int)(i / l.heads), head = (int)(i % l.heads);
    const float* o = a.out_raw + (size_t)row * (l.heads * dv) + head * dv;
    const float* g = a.p + (size_t)row * a.ldp + l.off_g + head * dv;
    float sq = 0.f;
    for (int c = lane; c < dv; c += 32) sq += o[c] * o[c];
    const float rinv = 1.f / sqrtf(lane_sum(sq) / (float)dv + l.eps);
    for (int c = lane; c < dv; c += 32) {
      const float gate = l.kind == KIND_DELTA ? sigmoid_f(g[c]) : silu_f(g[c]);
      const float y = o[c] * rinv * l.norm[l.kind == KIND_DELTA ? head * dv + c : c] * gate * l.out_scale;
      const size_t at = (size_t)row * a.ldy + head * dv + c;
      if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[at] = __float2bfloat16_rn(y);
      else static_cast<float*>(a.y)[at] = y;
    }
  }
}

// Product of the decays of every segment, per key channel (GLA).
__global__ void __launch_bounds__(256) segment_decay_kernel(ScanArgs sa) {
  const RecurrenceScanArgs& a = sa.a;
  const int K = a.l.heads * a.l.dim, seg = blockIdx.y, seq = blockIdx.z;
  const int t0 = a.seq_start[seq] + seg * a.seg_tokens, t1 = min(a.seq_start[seq + 1], t0 + a.seg_tokens);
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (t0 >= t1 || c >= K) return;
  float p = 1.f;
#pragma unroll 8
  for (int t = t0; t < t1; ++t) p *= a.decay[(size_t)t * K + c];
  sa.seg_trans[((size_t)seq * a.max_segs + seg) * K + c] = p;
}

// Turns the segments' own contributions into their start states, in order: start[0] = cached state (or zero),
// start[i + 1] = transition[i] start[i] + local[i]; the last one goes to the cache. Block = 16 columns of one head of
// one sequence; the running state stays in shared memory.
constexpr int COMBINE_COLS = 16, COMBINE_THREADS = 256;
template <int KIND>
__global__ void __launch_bounds__(COMBINE_THREADS) recurrence_combine_kernel(ScanArgs sa) {
  extern __shared__ __align__(16) float sm[];
  const RecurrenceScanArgs& a = sa.a;
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, head = blockIdx.x, seq = blockIdx.y, c0 = blockIdx.z * COMBINE_COLS, tid = threadIdx.x;
  const int nc = min(COMBINE_COLS, l.vdim - c0);
  const int len = a.seq_start[seq + 1] - a.seq_start[seq], segs = (len + a.seg_tokens - 1) / a.seg_tokens;
  float* cur = sm;                        // [dk][COMBINE_COLS]
  float* nxt = sm + dk * COMBINE_COLS;
  float* cached = a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp;
  const bool fresh = a.seq_pos[seq] == 0;
  for (int i = tid; i < dk * COMBINE_COLS; i += COMBINE_THREADS) {
    const int r = i / COMBINE_COLS, c = i % COMBINE_COLS;
    cur[i] = (!fresh && c < nc) ? cached[(size_t)r * l.dvp + c0 + c] : 0.f;
  }
  __syncthreads();
  for (int g = 0; g < segs; ++g) {
    const size_t si = ((size_t)seq * a.max_segs + g) * l.heads + head;
    float* loc = sa.seg_state + si * dk * l.dvp;
    for (int i = tid; i < dk * COMBINE_COLS; i += COMBINE_THREADS) {
      const int r = i / COMBINE_COLS, c = i % COMBINE_COLS;
      float v = c < nc ? loc[(size_t)r * l.dvp + c0 + c] : 0.f;
      if (KIND == KIND_GLA) {
        v = fmaf(sa.seg_trans[si * dk + r], cur[i], v);
      } else {
        const float* tr = sa.seg_trans + (si * dk + r) * sa.dkp;
        float acc = 0.f;
        for (int j = 0; j < dk; ++j) acc = fmaf(tr[j], cur[j * COMBINE_COLS + c], acc);
        v += acc;
      }
      if (c < nc) loc[(size_t)r * l.dvp + c0 + c] = cur[i];
      nxt[i] = v;
    }
    __syncthreads();
    float* t = cur;
    cur = nxt;
    nxt = t;
  }
  for (int i = tid; i < dk * COMBINE_COLS; i += COMBINE_THREADS) {
    const int r = i / COMBINE_COLS, c = i % COMBINE_COLS;
    if (c < nc) cached[(size_t)r * l.dvp + c0 + c] = cur[i];
  }
}

// ------------------------------------------------------------------ host side
constexpr size_t MAX_SMEM = 227 * 1024;

int sm_count() {
  static const int n = [] {
    int dev = 0, v = 148;
    cudaGetDevice(&dev);
    if (cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess) v = 148;
    return v;
  }();
  return n;
}

size_t scan_smem(int kind, int rpl, int cpl, int warps, int tb) {
  const size_t na = kind == KIND_DELTA ? 5 : 3, cols = (size_t)warps * 4 * cpl;
  return ((size_t)2 * tb * (na * 8 * rpl + 2 * cols) + (size_t)tb * cols) * sizeof(float);
}

template <int KIND, int RPL, int CPL>
cudaError_t launch_scan(ScanArgs sa, dim3 grid, int cols, cudaStream_t s) {
  const int warps = (cols + 4 * CPL - 1) / (4 * CPL);
  if (warps > 16) return cudaErrorInvalidValue;
  sa.tb = 16;
  while (sa.tb > 1 && scan_smem(KIND, RPL, CPL, warps, sa.tb) > MAX_SMEM) sa.tb /= 2;
  const size_t smem = scan_smem(KIND, RPL, CPL, warps, sa.tb);
  cudaError_t e = cudaFuncSetAttribute(recurrence_scan_kernel<KIND, RPL, CPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);
  if (e != cudaSuccess) return e;
  return launch_kernel(recurrence_scan_kernel<KIND, RPL, CPL>, grid, dim3(warps * 32), smem, s, false, sa);
}

template <int KIND, int RPL>
cudaError_t launch_scan_cols(const ScanArgs& sa, dim3 grid, int cols, int cpl, cudaStream_t s) {
  if (cpl == 4) return launch_scan<KIND, RPL, 4>(sa, grid, cols, s);
  if (cpl == 2) return launch_scan<KIND, RPL, 2>(sa, grid, cols, s);
  return launch_scan<KIND, RPL, 1>(sa, grid, cols, s);
}

int tune_int(const char* name, int otherwise) {
  const char* e = getenv(name);
  return e && *e ? atoi(e) : otherwise;
}

// `blocks` heads x sequences x segments are in flight. Few of them: the columns of a head are cut over several blocks
// (64 at least). Lanes take as many columns as leave every block at least four warps, so that a staged key, decay and
// query is read from shared memory for many products.
cudaError_t launch_scan_any(ScanArgs sa, dim3 grid, int cols, cudaStream_t s) {
  const int dk = sa.a.l.dim;
  const long long blocks = (long long)grid.x * grid.y * grid.z;
  int nb = (cols + 255) / 256;
  while (nb * 2 * blocks <= sm_count() && (cols + nb * 2 - 1) / (nb * 2) >= 48) nb *= 2;
  nb = std::max(nb, tune_int("PG_SCAN_BLOCKS", 0));
  sa.block_cols = ((cols + nb - 1) / nb + 3) / 4 * 4;
  sa.col_blocks = (cols + sa.block_cols - 1) / sa.block_cols;
  grid.x *= sa.col_blocks;
  const int bc = sa.block_cols;
  int cpl = bc > 32 ? 4 : bc > 16 ? 2 : 1;
  if (const int c = tune_int("PG_SCAN_CPL", 0)) cpl = std::max(c, (bc + 63) / 64);
  if (cpl == 3) cpl = 4;
#define PG_SCAN(KIND_)                                                                  \
  (dk <= 32    ? launch_scan_cols<KIND_, 4>(sa, grid, bc, cpl, s)                       \
   : dk <= 64  ? launch_scan_cols<KIND_, 8>(sa, grid, bc, cpl, s)                       \
   : dk <= 128 ? launch_scan_cols<KIND_, 16>(sa, grid, bc, cpl, s)                      \
   : dk <= 256 ? launch_scan_cols<KIND_, 32>(sa, grid, bc, cpl, s) : cudaErrorInvalidValue)
  cudaError_t e = sa.a.l.kind == KIND_DELTA ? PG_SCAN(KIND_DELTA) : PG_SCAN(KIND_GLA);
#undef PG_SCAN
  if (e == cudaSuccess && sa.col_blocks > 1 && (sa.mode == SCAN_FULL || sa.mode == SCAN_OUTPUT)) {
    const long long warps = (long long)sa.a.rows * sa.a.l.heads;
    e = launch_kernel(recurrence_output_kernel, dim3((unsigned)std::min<long long>((warps + 7) / 8, 148 * 16)), dim3(256), 0, s, false, sa.a,
                      sa.y_bf16);
  }
  return e;
}

}  // namespace

size_t recurrence_state_floats(const RecurrenceLayer& l) { return (size_t)l.heads * l.dim * l.dvp; }

bool recurrence_use_segments(const RecurrenceLayer& l, int nseq, int max_len, int max_segs) {
  return max_segs >= 4 && max_len >= 512 && (long long)nseq * l.heads < 48;
}

size_t recurrence_segment_floats(const RecurrenceLayer& l, int nseq, int max_segs) {
  return (size_t)nseq * max_segs * l.heads * l.dim * (l.dvp + (l.kind == KIND_DELTA ? (l.dim + 3) / 4 * 4 : 1));
}

cudaError_t launch_recurrence_step(const RecurrenceStepArgs& a, bool y_bf16, bool pdl, cudaStream_t s) {
  const RecurrenceLayer& l = a.l;
  const int dv4 = l.dvp / 4, kg = STEP_THREADS / dv4, nr = (l.dim + kg - 1) / kg;
  if (dv4 > STEP_THREADS) return cudaErrorInvalidValue;
  const size_t smem = ((size_t)5 * ((l.dim + 3) & ~3) + ((l.rank + 3) & ~3) + 3 * (size_t)l.dvp + (size_t)kg * l.dvp) * sizeof(float);
  const dim3 grid(l.heads, a.batch), block(STEP_THREADS);
  const int yb = y_bf16 ? 1 : 0;
  if (nr <= 4) return launch_kernel(recurrence_step_kernel<4>, grid, block, smem, s, pdl, a, yb);
  if (nr <= 8) return launch_kernel(recurrence_step_kernel<8>, grid, block, smem, s, pdl, a, yb);
  if (nr <= 16) return launch_kernel(recurrence_step_kernel<16>, grid, block, smem, s, pdl, a, yb);
  return launch_kernel(recurrence_step_kernel<0>, grid, block, smem, s, pdl, a, yb);
}

cudaError_t launch_recurrence_scan(const RecurrenceScanArgs& a, bool y_bf16, cudaStream_t s) {
  if (a.rows <= 0) return cudaSuccess;
  const RecurrenceLayer& l = a.l;
  cudaError_t e = launch_kernel(recurrence_gates_kernel, dim3((a.rows + GATE_ROWS - 1) / GATE_ROWS), dim3(256),
                                (size_t)GATE_ROWS * l.rank * sizeof(float), s, false, a);
  if (e != cudaSuccess) return e;
  ScanArgs sa{};
  sa.a = a;
  sa.y_bf16 = y_bf16 ? 1 : 0;
  const int K = l.heads * l.dim;
  auto m4 = [](int v) { return v % 4 == 0; };
  sa.vec = m4(l.dim) && m4(l.vdim) && m4(l.off_k) && m4(l.off_q) && m4(l.off_v) && m4(l.off_g) && m4(a.ldp) && m4(K);
  if (a.max_segs <= 1 || !a.segments) {
    sa.mode = SCAN_FULL;
    return launch_scan_any(sa, dim3(l.heads, a.nseq, 1), l.vdim, s);
  }
  const size_t units = (size_t)a.nseq * a.max_segs * l.heads;
  sa.dkp = (l.dim + 3) / 4 * 4;
  sa.seg_state = a.segments;
  sa.seg_trans = a.segments + units * l.dim * l.dvp;
  const dim3 grid(l.heads, a.nseq, a.max_segs);
  sa.mode = SCAN_LOCAL;
  if ((e = launch_scan_any(sa, grid, l.vdim, s)) != cudaSuccess) return e;
  if (l.kind == KIND_DELTA) {
    sa.mode = SCAN_TRANS;
    if ((e = launch_scan_any(sa, grid, l.dim, s)) != cudaSuccess) return e;
  } else {
    e = launch_kernel(segment_decay_kernel, dim3((K + 255) / 256, a.max_segs, a.nseq), dim3(256), 0, s, false, sa);
    if (e != cudaSuccess) return e;
  }
  const dim3 cgrid(l.heads, a.nseq, (l.vdim + COMBINE_COLS - 1) / COMBINE_COLS);
  const size_t csmem = (size_t)2 * l.dim * COMBINE_COLS * sizeof(float);
  e = l.kind == KIND_DELTA ? launch_kernel(recurrence_combine_kernel<KIND_DELTA>, cgrid, dim3(COMBINE_THREADS), csmem, s, false, sa)
                           : launch_kernel(recurrence_combine_kernel<KIND_GLA>, cgrid, dim3(COMBINE_THREADS), csmem, s, false, sa);
  if (e != cudaSuccess) return e;
  sa.mode = SCAN_OUTPUT;
  return launch_scan_any(sa, grid, l.vdim, s);
}

}  // namespace pg
