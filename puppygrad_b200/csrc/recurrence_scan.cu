// Recurrent mixers over whole portions of prompts: the gates of every row, the scan, and for long portions its
// segmented form. Everything that enters the recurrence is FP32.
//
// Both rules act on every column of a head's [dim, vdim] state on its own (S[:, c] needs only v[c] of the new token), so
// a column's `dim` entries are spread over eight lanes and the columns over groups of lanes, warps and blocks.
#include <algorithm>

#include "recurrence.cuh"
#include "tc_common.cuh"

namespace pg {
namespace {

// ------------------------------------------------------------------ gates
constexpr int GATE_ROWS = 16;
// decay of GATE_ROWS rows x 256 key channels per block
__global__ void __launch_bounds__(256) recurrence_decay_kernel(RecurrenceScanArgs a) {
  extern __shared__ __align__(16) float sm[];  // [rank][GATE_ROWS]
  const RecurrenceLayer& l = a.l;
  const int K = l.heads * l.dim, r0 = blockIdx.x * GATE_ROWS, tid = threadIdx.x, c = blockIdx.y * 256 + tid;
  const int nr = min(GATE_ROWS, a.rows - r0);
  for (int i = tid; i < GATE_ROWS * l.rank; i += 256) {
    const int j = i / l.rank, r = i - j * l.rank;
    const float t = j < nr ? a.p[(size_t)(r0 + j) * a.ldp + l.off_t + r] : 0.f;
    sm[r * GATE_ROWS + j] = l.kind == KIND_DELTA ? tanhf(t) : t;
  }
  __syncthreads();
  if (c >= K) return;
  float z[GATE_ROWS];
#pragma unroll
  for (int j = 0; j < GATE_ROWS; ++j) z[j] = l.b2[c];
  const float* __restrict__ w2 = l.w2 + c;
#pragma unroll 8
  for (int r = 0; r < l.rank; ++r) {
    const float w = w2[(size_t)r * K];
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

// Delta rule, after the decays; a warp per (row, head): the unit key u, the removal rate a * u, and what the scan needs
// to take two tokens at a time: the next token's u times this one's decay, next u . (a * u), next u . k.
__global__ void __launch_bounds__(256) delta_gates_kernel(RecurrenceScanArgs a) {
  const RecurrenceLayer& l = a.l;
  const int K = l.heads * l.dim, lane = threadIdx.x & 31;
  const long long total = (long long)a.rows * l.heads;
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5; i < total; i += ((long long)gridDim.x * blockDim.x) >> 5) {
    const int row = (int)(i / l.heads), head = (int)(i % l.heads);
    const float* pr = a.p + (size_t)row * a.ldp;
    const float* k = pr + l.off_k + head * l.dim;
    const float* kn = row + 1 < a.rows ? k + a.ldp : k;  // unused where the next row is another sequence's
    float s = 0.f, sn = 0.f;
    for (int c = lane; c < l.dim; c += 32) {
      s += k[c] * k[c];
      sn += kn[c] * kn[c];
    }
    const float inv = 1.f / sqrtf(lane_sum(s) + UNIT_EPS), invn = 1.f / sqrtf(lane_sum(sn) + UNIT_EPS);
    float ub = 0.f, uk = 0.f;
    for (int c = lane; c < l.dim; c += 32) {
      const int ch = head * l.dim + c;
      const size_t at = (size_t)row * K + ch;
      const float u = k[c] * inv, un = kn[c] * invn, b = sigmoid_f(pr[l.off_a + ch] + l.a_bias[ch]) * u;
      a.unit[at] = u;
      a.rate[at] = b;
      a.unit_next[at] = un * a.decay[at];
      ub += un * b;
      uk += un * k[c];
    }
    ub = lane_sum(ub);
    uk = lane_sum(uk);
    if (lane == 0) store4(a.pair + (size_t)i * 4, make_float4(ub, uk, 0.f, 0.f));
  }
}

// The same when every size and offset is a multiple of four: eight lanes per (row, head), four channels at a time.
__global__ void __launch_bounds__(256) delta_gates_vec_kernel(RecurrenceScanArgs a) {
  const RecurrenceLayer& l = a.l;
  const int K = l.heads * l.dim, l8 = threadIdx.x & 7;
  const long long total = (long long)a.rows * l.heads, rounded = (total + 3) / 4 * 4;  // whole warps stay together
  auto eight = [](float v) {
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) v += __shfl_xor_sync(ALL_LANES, v, o);
    return v;
  };
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 3; i < rounded; i += ((long long)gridDim.x * blockDim.x) >> 3) {
    const bool on = i < total;
    const int row = on ? (int)(i / l.heads) : 0, head = on ? (int)(i % l.heads) : 0;
    const float* pr = a.p + (size_t)row * a.ldp;
    const float* k = pr + l.off_k + head * l.dim;
    const float* kn = row + 1 < a.rows ? k + a.ldp : k;
    float4 kv[8], nv[8];
    float s = 0.f, sn = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      const int c = q * 32 + l8 * 4;
      const bool in = on && c < l.dim;
      kv[q] = in ? load4(k + c) : make_float4(0, 0, 0, 0);
      nv[q] = in ? load4(kn + c) : make_float4(0, 0, 0, 0);
      s += (kv[q].x * kv[q].x + kv[q].y * kv[q].y) + (kv[q].z * kv[q].z + kv[q].w * kv[q].w);
      sn += (nv[q].x * nv[q].x + nv[q].y * nv[q].y) + (nv[q].z * nv[q].z + nv[q].w * nv[q].w);
    }
    const float inv = 1.f / sqrtf(eight(s) + UNIT_EPS), invn = 1.f / sqrtf(eight(sn) + UNIT_EPS);
    float ub = 0.f, uk = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) {
      const int c = q * 32 + l8 * 4, ch = head * l.dim + c;
      if (on && c < l.dim) {
        const size_t at = (size_t)row * K + ch;
        const float4 al = load4(pr + l.off_a + ch), dec = load4(a.decay + at);
        const float* ab = l.a_bias + ch;
        float4 u, b, un;
        u.x = kv[q].x * inv; u.y = kv[q].y * inv; u.z = kv[q].z * inv; u.w = kv[q].w * inv;
        b.x = sigmoid_f(al.x + ab[0]) * u.x; b.y = sigmoid_f(al.y + ab[1]) * u.y;
        b.z = sigmoid_f(al.z + ab[2]) * u.z; b.w = sigmoid_f(al.w + ab[3]) * u.w;
        un.x = nv[q].x * invn; un.y = nv[q].y * invn; un.z = nv[q].z * invn; un.w = nv[q].w * invn;
        ub += (un.x * b.x + un.y * b.y) + (un.z * b.z + un.w * b.w);
        uk += (un.x * kv[q].x + un.y * kv[q].y) + (un.z * kv[q].z + un.w * kv[q].w);
        store4(a.unit + at, u);
        store4(a.rate + at, b);
        store4(a.unit_next + at, make_float4(un.x * dec.x, un.y * dec.y, un.z * dec.z, un.w * dec.w));
      }
    }
    ub = eight(ub);
    uk = eight(uk);
    if (on && l8 == 0) store4(a.pair + (size_t)i * 4, make_float4(ub, uk, 0.f, 0.f));
  }
}

// Channel delta rule: the convolutions of q, k and v with silu, unit vectors of q and k. A warp takes one head of q or k (2
// kv_heads units) or of v (heads units) over CONV_ROWS rows; the last inputs stay in registers (TAPS > 0) or are read again.
constexpr int CONV_ROWS = 16;
template <int TAPS, int NE>
__global__ void __launch_bounds__(256) channel_conv_kernel(RecurrenceScanArgs a) {
  const RecurrenceLayer& l = a.l;
  const int lane = threadIdx.x & 31, units = 2 * l.kv_heads + l.heads, ntaps = TAPS > 0 ? TAPS : l.taps;
  const int groups = (a.rows + CONV_ROWS - 1) / CONV_ROWS;
  const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (w >= (long long)groups * units) return;
  const int r0 = (int)(w / units) * CONV_ROWS, u = (int)(w % units), r1 = min(r0 + CONV_ROWS, a.rows);
  const bool is_q = u < l.kv_heads, is_k = !is_q && u < 2 * l.kv_heads;
  const int h = is_q ? u : is_k ? u - l.kv_heads : u - 2 * l.kv_heads, n = is_q || is_k ? l.dim : l.vdim;
  const int ch0 = (is_q ? l.off_q : is_k ? l.off_k : l.off_v) - l.off_q + h * n, pitch = (is_q || is_k ? l.kv_heads : l.heads) * n;
  float* dst = (is_q ? a.rate : is_k ? a.unit : a.vals) + h * n;
  constexpr int NT = TAPS > 0 ? TAPS : 1;
  float win[NT][NE], wt[NT][NE];  // inputs (the newest last) and weights
  if (TAPS > 0) {
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int i = 0; i < NE; ++i) wt[t][i] = lane + i * 32 < n ? l.conv[(size_t)t * l.channels + ch0 + lane + i * 32] : 0.f;
  }
  int seq = -1, first = 0;
  const float* taps = nullptr;
  for (int r = r0; r < r1; ++r) {
    const int s = a.row_seq[r];
    const bool enter = s != seq;
    if (enter) {
      seq = s;
      first = a.seq_start[s];
      taps = a.taps + (size_t)a.seq_slot[s] * l.taps * l.channels;
    }
    const int pos = a.seq_pos[seq] + r - first;
    float x[NE], sq = 0.f;
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      const int c = lane + i * 32;
      x[i] = 0.f;
      if (TAPS > 0) {
#pragma unroll
        for (int t = 0; t < NT; ++t) {
          if (t + 1 < NT && !enter) win[t][i] = win[t + 1 < NT ? t + 1 : t][i];
          else win[t][i] = c < n ? conv_input(l, a.p, a.ldp, taps, r, first, pos, NT - 1 - t, ch0 + c) : 0.f;
        }
#pragma unroll
        for (int t = 0; t < NT; ++t) x[i] = fmaf(wt[t][i], win[t][i], x[i]);
      } else if (c < n) {
        for (int back = ntaps - 1; back >= 0; --back)
          x[i] = fmaf(l.conv[(size_t)(ntaps - 1 - back) * l.channels + ch0 + c], conv_input(l, a.p, a.ldp, taps, r, first, pos, back, ch0 + c), x[i]);
      }
      x[i] = silu_f(x[i]);
      sq += x[i] * x[i];
    }
    const float inv = is_q || is_k ? 1.f / sqrtf(lane_sum(sq) + UNIT_EPS) : 1.f;
#pragma unroll
    for (int i = 0; i < NE; ++i)
      if (lane + i * 32 < n) dst[(size_t)r * pitch + lane + i * 32] = x[i] * inv;
  }
}

// The same when every size and offset is a multiple of four and heads have at most 128 channels: four channels per lane, the
// rows of a group requested four at a time.
template <int TAPS>
__global__ void __launch_bounds__(256) channel_conv_vec_kernel(RecurrenceScanArgs a) {
  const RecurrenceLayer& l = a.l;
  const int lane = threadIdx.x & 31, units = 2 * l.kv_heads + l.heads;
  const int groups = (a.rows + CONV_ROWS - 1) / CONV_ROWS;
  const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  if (w >= (long long)groups * units) return;
  const int r0 = (int)(w / units) * CONV_ROWS, u = (int)(w % units), r1 = min(r0 + CONV_ROWS, a.rows);
  const bool is_q = u < l.kv_heads, is_k = !is_q && u < 2 * l.kv_heads;
  const int h = is_q ? u : is_k ? u - l.kv_heads : u - 2 * l.kv_heads, n = is_q || is_k ? l.dim : l.vdim, c = lane * 4;
  const bool on = c < n;
  const int ch = (is_q ? l.off_q : is_k ? l.off_k : l.off_v) - l.off_q + h * n + (on ? c : 0), pitch = (is_q || is_k ? l.kv_heads : l.heads) * n;
  float* dst = (is_q ? a.rate : is_k ? a.unit : a.vals) + h * n + c;
  const float* src = a.p + l.off_q + ch;
  float4 win[TAPS], wt[TAPS];  // inputs (the newest last) and weights
#pragma unroll
  for (int t = 0; t < TAPS; ++t) wt[t] = load4(l.conv + (size_t)t * l.channels + ch);
  const bool one = a.row_seq[r0] == a.row_seq[r1 - 1];  // the whole group in one sequence
  int seq = -1;
  for (int rb = r0; rb < r1; rb += 4) {
    float4 x[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) x[j] = load4(src + (size_t)min(rb + j, r1 - 1) * a.ldp);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = rb + j;
      if (r >= r1) break;
      const int s = one && seq >= 0 ? seq : a.row_seq[r];
      if (s != seq) {  // entering a sequence: its cached inputs, or what the portion has before this group
        seq = s;
        const int first = a.seq_start[s], pos = a.seq_pos[s] + r - first;
        const float* taps = a.taps + (size_t)a.seq_slot[s] * l.taps * l.channels;
#pragma unroll
        for (int t = 0; t + 1 < TAPS; ++t) {
          const int back = TAPS - 1 - t;
          win[t + 1] = r - back >= first ? load4(src + (size_t)(r - back) * a.ldp)
                       : pos - back >= 0 ? load4(taps + (size_t)((pos - back) % TAPS) * l.channels + ch) : make_float4(0, 0, 0, 0);
        }
      }
#pragma unroll
      for (int t = 0; t + 1 < TAPS; ++t) win[t] = win[t + 1];
      win[TAPS - 1] = x[j];
      float4 y = make_float4(0, 0, 0, 0);
#pragma unroll
      for (int t = 0; t < TAPS; ++t) {
        y.x = fmaf(wt[t].x, win[t].x, y.x); y.y = fmaf(wt[t].y, win[t].y, y.y);
        y.z = fmaf(wt[t].z, win[t].z, y.z); y.w = fmaf(wt[t].w, win[t].w, y.w);
      }
      y.x = silu_f(y.x); y.y = silu_f(y.y); y.z = silu_f(y.z); y.w = silu_f(y.w);
      if (is_q || is_k) {
        const float sq = on ? (y.x * y.x + y.y * y.y) + (y.z * y.z + y.w * y.w) : 0.f, inv = 1.f / sqrtf(lane_sum(sq) + UNIT_EPS);
        y.x *= inv; y.y *= inv; y.z *= inv; y.w *= inv;
      }
      if (on) store4(dst + (size_t)r * pitch, y);
    }
  }
}

// Channel delta rule, after the convolutions. The scan takes QUAD tokens at a time from the state S before them. With D_ij the
// product of the decays of tokens j + 1..i of a quad and P_i that of tokens 0..i, token i reads S through A_i = P_i k_i and
// answers through Q_i = P_i q_i, and the four writes u_j become
//   u_i = beta_i (v_i - A_i^T S - sum_{j < i} c_ij u_j),  out_i = Q_i^T S + sum_{j <= i} r_ij u_j,  S = W S + sum_j B_j u_j^T
// with c_ij = k_i . D_ij k_j, r_ij = q_i . D_ij k_j, B_j = D_3j k_j, W = P_3. Quads are counted from a portion's first row; tokens
// past its end count as decay 1 and zeros. A warp makes the rows and numbers of one head of one quad.
constexpr int QUAD = 4, QUAD_NUMBERS = 20;  // c (6), r (10), beta (4)
__device__ __forceinline__ size_t first_quad(const RecurrenceScanArgs& a, int seq) { return (size_t)(a.seq_start[seq] / QUAD + seq); }
template <int NE>
__global__ void __launch_bounds__(256) channel_quads_kernel(RecurrenceScanArgs a) {
  const RecurrenceLayer& l = a.l;
  const int lane = threadIdx.x & 31, K = l.heads * l.dim, rep = l.heads / l.kv_heads, kv_pitch = l.kv_heads * l.dim;
  const int seq = blockIdx.y, first = a.seq_start[seq], len = a.seq_start[seq + 1] - first;
  const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int quad = (int)(w / l.heads), head = (int)(w % l.heads);
  if (quad * QUAD >= len) return;
  const int r0 = first + quad * QUAD, n = min(QUAD, len - quad * QUAD);
  const float beta = lane < n ? sigmoid_f(a.p[(size_t)(r0 + lane) * a.ldp + l.off_b + head]) : 0.f;
  float wd[QUAD][NE], k[QUAD][NE], q[QUAD][NE], sums[16];
#pragma unroll
  for (int t = 0; t < QUAD; ++t)
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      const int c = lane + i * 32;
      const bool on = t < n && c < l.dim;
      const size_t r = r0 + t;
      wd[t][i] = on ? a.z[r * a.ldz + head * l.dim + c] : 0.f;
      k[t][i] = on ? a.unit[r * kv_pitch + head / rep * l.dim + c] : 0.f;
      q[t][i] = on ? a.rate[r * kv_pitch + head / rep * l.dim + c] : 0.f;
    }
#pragma unroll
  for (int i = 0; i < 16; ++i) sums[i] = 0.f;
  const size_t quad_at = first_quad(a, seq) + quad;
#pragma unroll
  for (int i = 0; i < NE; ++i) {
    const int c = lane + i * 32;
    const bool in = c < l.dim;
    const float b = in ? l.b2[head * l.dim + c] : 0.f, na = l.neg_a[head];
#pragma unroll
    for (int t = 0; t < QUAD; ++t) wd[t][i] = in && t < n ? expf(na * softplus_f(wd[t][i] + b)) : 1.f;
    float p = 1.f, rest = 1.f;
#pragma unroll
    for (int t = 0; t < QUAD; ++t) {
      p *= wd[t][i];
      float d = 1.f;
#pragma unroll
      for (int j = t; j >= 0; --j) {
        const float dk = d * k[j][i];
        sums[6 + t * (t + 1) / 2 + j] = fmaf(q[t][i], dk, sums[6 + t * (t + 1) / 2 + j]);
        if (j < t) sums[t * (t - 1) / 2 + j] = fmaf(k[t][i], dk, sums[t * (t - 1) / 2 + j]);
        d *= wd[j][i];
      }
      if (in && t < n) {
        const size_t at = (size_t)(r0 + t) * K + head * l.dim + c;
        a.decay[at] = p * k[t][i];
        a.unit_next[at] = p * q[t][i];
      }
    }
    if (in) a.quad_decay[quad_at * K + head * l.dim + c] = p;
#pragma unroll
    for (int t = QUAD - 1; t >= 0; --t) {
      if (in && t < n) a.writes[(size_t)(r0 + t) * K + head * l.dim + c] = rest * k[t][i];
      rest *= wd[t][i];
    }
  }
  // sums over the lanes: lane l ends with that of number l >> 1
#pragma unroll
  for (int o = 16, m = 8; o > 1; o >>= 1, m >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < m) {
        const float send = up ? sums[i] : sums[i + m], keep = up ? sums[i + m] : sums[i];
        sums[i] = keep + __shfl_xor_sync(ALL_LANES, send, o);
      }
  }
  const float total = sums[0] + __shfl_xor_sync(ALL_LANES, sums[0], 1);
  float* out = a.quads + (quad_at * l.heads + head) * QUAD_NUMBERS;
  if ((lane & 1) == 0) out[lane >> 1] = total;
  if (lane < QUAD) out[16 + lane] = beta;
}

// The inputs that the next tokens' convolutions still need. Block = (sequence, one of its last taps - 1 rows, 256 channels).
__global__ void __launch_bounds__(256) channel_taps_kernel(RecurrenceScanArgs a) {
  const RecurrenceLayer& l = a.l;
  const int seq = blockIdx.x, first = a.seq_start[seq], r = a.seq_start[seq + 1] - 1 - (int)blockIdx.y;
  if (r < first) return;
  const int pos = a.seq_pos[seq] + r - first;
  float* dst = a.taps + ((size_t)a.seq_slot[seq] * l.taps + pos % l.taps) * l.channels;
  const int c = blockIdx.z * blockDim.x + threadIdx.x;
  if (c < l.channels) dst[c] = a.p[(size_t)r * a.ldp + l.off_q + c];
}

// ------------------------------------------------------------------ scan
// Block = one head of one sequence (or of one segment of it), or a part of its columns. The last warp stages the rows of
// TB tokens at a time in a ring of shared-memory stages (bulk copies where rows are 16-byte aligned); in the others
// eight lanes share a column (lane l holds rows 32 j + 4 l + i), a group of eight has CPL columns, a warp four groups.
// A lane's share of an output goes to shared memory; after TB tokens the shares are added and the head norm and output
// gate applied.
enum ScanMode {
  SCAN_FULL = 0,     // whole sequence: start from the cached state (or zero), outputs, final state to the cache
  SCAN_LOCAL = 1,    // one segment from a zero state, no outputs: its contribution to the state
  SCAN_TRANS = 2,    // one segment with identity columns and no values: its transition matrix (delta)
  SCAN_OUTPUT = 3    // one segment from its known start state: outputs
};
constexpr int SCAN_WARPS = 8;   // at most: 32 CPL columns
constexpr int SCAN_STAGES = 3;
struct ScanArgs {
  RecurrenceScanArgs a;
  int mode, tb;
  float *seg_state, *seg_trans;  // [nseq][max_segs][heads][dim][dvp], [nseq][max_segs][heads][dim][dkp] (GLA: [..][dim] decays)
  int dkp;
  const float *k, *q, *v, *g;  // rows of keys, queries, values and gates (heads side by side) and their pitches
  int ldk, ldq, ldv, ldg;
  int col_blocks, block_cols;  // column blocks of a head, columns of each (the last may have fewer)
  int vec;      // rows can be copied in 16-byte pieces
  int y_bf16;
};

__device__ __forceinline__ void bulk_row(float* dst, const float* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)), "l"(src),
               "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void named_barrier(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

// Sums of N values over the eight lanes of a group, in every lane: halves are exchanged on the way down, totals on the
// way back.
template <int N, int OFF>
struct GroupSum {
  static __device__ __forceinline__ void run(float* v, int lr) {
    const bool up = lr & OFF;
    if (N > 1) {
      constexpr int H = N > 1 ? N / 2 : 1;
#pragma unroll
      for (int i = 0; i < H; ++i) {
        const float send = up ? v[i] : v[i + H], keep = up ? v[i + H] : v[i];
        v[i] = keep + __shfl_xor_sync(ALL_LANES, send, OFF);
      }
      GroupSum<H, OFF / 2>::run(v, lr);
#pragma unroll
      for (int i = 0; i < H; ++i) {
        const float other = __shfl_xor_sync(ALL_LANES, v[i], OFF), own = v[i];
        v[i] = up ? other : own;
        v[i + H] = up ? own : other;
      }
    } else {
      v[0] += __shfl_xor_sync(ALL_LANES, v[0], OFF);
      GroupSum<1, OFF / 2>::run(v, lr);
    }
  }
};
template <int N>
struct GroupSum<N, 0> {
  static __device__ __forceinline__ void run(float*, int) {}
};

// The same sums, each in the lanes that share it only: lane l of the group ends with the values index(l).. (N / 8 of them, or one).
template <int N, int OFF>
struct GroupScatter {
  static __device__ __forceinline__ void run(float* v, int lr) {
    if (N > 1) {
      constexpr int H = N > 1 ? N / 2 : 1;
      const bool up = lr & OFF;
#pragma unroll
      for (int i = 0; i < H; ++i) {
        const float send = up ? v[i] : v[i + H], keep = up ? v[i + H] : v[i];
        v[i] = keep + __shfl_xor_sync(ALL_LANES, send, OFF);
      }
      GroupScatter<H, OFF / 2>::run(v, lr);
    } else {
      v[0] += __shfl_xor_sync(ALL_LANES, v[0], OFF);
      GroupScatter<1, OFF / 2>::run(v, lr);
    }
  }
  static __device__ __forceinline__ int index(int lr) { return (N > 1 && (lr & OFF) ? N / 2 : 0) + GroupScatter<(N > 1 ? N / 2 : 1), OFF / 2>::index(lr); }
};
template <int N>
struct GroupScatter<N, 0> {
  static __device__ __forceinline__ void run(float*, int) {}
  static __device__ __forceinline__ int index(int) { return 0; }
};

// The delta rule works on two tokens at a time: with e = (u' * w)^T S, where the dash marks the second token,
// u'^T S_t = e - (u' . b) d + (u' . k) v, so that both reads come from one reduction over the state before the pair.
template <int KIND, int RPL, int CPL>
__global__ void __launch_bounds__((SCAN_WARPS + 1) * 32, 1) recurrence_scan_kernel(ScanArgs sa) {
  extern __shared__ __align__(16) float sm[];
  __shared__ uint64_t full[SCAN_STAGES], empty[SCAN_STAGES];
  __shared__ int failed_flag;
  constexpr int DKP = 8 * RPL, NA = KIND == KIND_DELTA ? 6 : 3, J = RPL / 4;  // staged key-channel arrays
  constexpr bool PAIRS = KIND == KIND_DELTA;
  const RecurrenceScanArgs& a = sa.a;
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, K = l.heads * dk, tid = threadIdx.x;
  const bool trans = sa.mode == SCAN_TRANS;
  // blockIdx.x = head * (column blocks) + column block; with several column blocks per head the outputs leave unnormed
  const int head = blockIdx.x / sa.col_blocks, cb = blockIdx.x % sa.col_blocks, seq = blockIdx.y, seg = blockIdx.z;
  const int all_cols = trans ? dk : l.vdim, cbase = cb * sa.block_cols;
  const int dv = min(sa.block_cols, all_cols - cbase);  // columns of this block
  const int W = (blockDim.x >> 5) - 1, COLS = W * 4 * CPL, TB = sa.tb;
  // floats of one staged token: k, decay, q, (u, rate, next u * decay), v, gate, (next u . rate, next u . k)
  const int stride = NA * DKP + 2 * COLS + 4, OP = COLS + 4;
  float* stage = sm;                                   // [SCAN_STAGES][TB][stride]
  float* os0 = sm + (size_t)SCAN_STAGES * TB * stride;  // [2][TB][8 lanes of a group][OP]
  const int lane = tid & 31, warp = tid >> 5;
  const bool outputs = sa.mode == SCAN_FULL || sa.mode == SCAN_OUTPUT;
  const bool want_v = !trans, want_g = outputs && sa.col_blocks == 1;
  volatile int* failed = &failed_flag;

  int t0 = a.seq_start[seq], t1 = a.seq_start[seq + 1];
  if (sa.mode != SCAN_FULL) {
    t0 += seg * a.seg_tokens;
    t1 = min(t1, t0 + a.seg_tokens);
    if (t0 >= t1) return;
  }
  for (int i = tid; i < SCAN_STAGES * TB * stride; i += blockDim.x) stage[i] = 0.f;  // the padding stays zero
  if (tid == 0) {
    for (int i = 0; i < SCAN_STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], (uint32_t)W);
    }
    failed_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // the zeros come before the bulk copies
  __syncthreads();
  const int blocks = (t1 - t0 + TB - 1) / TB;

  if (warp == W) {  // ---- stages rows; lane = (token, array)
    const int arr = lane & 7;  // key-channel arrays, then values, then gates (GLA: lanes 5..7 idle; delta: all busy)
    const bool key = arr < NA, value = arr == NA && want_v, gate = arr == NA + 1 && want_g;
    const bool on = (key && !(arr == 2 && !outputs)) || value || gate;
    const float* src = nullptr;
    int pitch = a.ldp, off = 0;
    if (key) {
      off = arr * DKP;
      const float* gates[4] = {a.decay, a.unit, a.rate, a.unit_next};
      const int kv = head / (l.heads / l.kv_heads);
      if (arr == 0) {
        src = sa.k + kv * dk;
        pitch = sa.ldk;
      } else if (arr == 2) {
        src = sa.q + kv * dk;
        pitch = sa.ldq;
      } else {
        src = gates[arr == 1 ? 0 : arr - 2] + head * dk;
        pitch = K;
      }
    } else if (value || gate) {
      off = NA * DKP + (gate ? COLS : 0);
      src = (gate ? sa.g : sa.v) + head * l.vdim + cbase;
      pitch = gate ? sa.ldg : sa.ldv;
    }
    const int count = key ? dk : dv;
    const uint32_t token_bytes = 4u * (uint32_t)((NA - (outputs ? 0 : 1)) * dk + (want_v ? dv : 0) + (want_g ? dv : 0)) +
                                 (PAIRS ? 16u : 0u);
    for (int b = 0; b < blocks; ++b) {
      const int s = b % SCAN_STAGES, tb0 = t0 + b * TB, n = min(TB, t1 - tb0);
      if (b >= SCAN_STAGES && !mbar_wait(&empty[s], ((b / SCAN_STAGES) - 1) & 1, failed, a.error_flag, 41)) break;
      __syncwarp();
      float* dst = stage + (size_t)s * TB * stride;
      if (sa.vec) {
        if (lane == 0) mbar_expect_tx(&full[s], (uint32_t)n * token_bytes);
        __syncwarp();
        if (on)
          for (int t = lane >> 3; t < n; t += 4)
            bulk_row(dst + (size_t)t * stride + off, src + (size_t)(tb0 + t) * pitch, (uint32_t)(4 * count), &full[s]);
        if (PAIRS)
          for (int t = lane; t < n; t += 32)
            bulk_row(dst + (size_t)t * stride + NA * DKP + 2 * COLS, a.pair + ((size_t)(tb0 + t) * l.heads + head) * 4, 16, &full[s]);
      } else {
        if (on)
          for (int t = lane >> 3; t < n; t += 4)
            for (int i = 0; i < count; ++i) dst[(size_t)t * stride + off + i] = src[(size_t)(tb0 + t) * pitch + i];
        if (PAIRS)
          for (int t = lane; t < n; t += 32)
            store4(dst + (size_t)t * stride + NA * DKP + 2 * COLS, load4(a.pair + ((size_t)(tb0 + t) * l.heads + head) * 4));
        __syncwarp();
        if (lane == 0) mbar_arrive(&full[s]);
      }
    }
    return;
  }

  // ---- start state, two neighbouring rows per register pair
  const int lr = lane & 7, col0 = (warp * 4 + (lane >> 3)) * CPL;
  unsigned long long s[RPL / 2][CPL];
  const size_t seg_index = ((size_t)seq * a.max_segs + seg) * l.heads + head;
  const float* init = nullptr;
  if (sa.mode == SCAN_FULL && a.seq_pos[seq] > 0) init = a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp;
  if (sa.mode == SCAN_OUTPUT) init = sa.seg_state + seg_index * dk * l.dvp;
  auto row_of = [&](int r) { return (r >> 2) * 32 + lr * 4 + (r & 3); };
#pragma unroll
  for (int r = 0; r < RPL; r += 2) {
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      const int col = col0 + c;
      float v[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = row_of(r + e);
        v[e] = 0.f;
        if (row < dk && col < dv) {
          if (init) v[e] = init[(size_t)row * l.dvp + cbase + col];
          else if (trans) v[e] = row == cbase + col ? 1.f : 0.f;
        }
      }
      s[r / 2][c] = pack2(v[0], v[1]);
    }
  }

  using Row = ulonglong2;  // four entries of a key-channel row
  for (int b = 0; b < blocks; ++b) {
    const int sidx = b % SCAN_STAGES, tb0 = t0 + b * TB, n = min(TB, t1 - tb0);
    mbar_wait(&full[sidx], (b / SCAN_STAGES) & 1, failed, a.error_flag, 42);  // on expiry the numbers are void, the barriers below are kept
    __syncwarp();
    const float* x0 = stage + (size_t)sidx * TB * stride;
    float* os = os0 + (size_t)(b & 1) * TB * 8 * OP;

    auto values = [&](const float* x, float (&v)[CPL]) {
#pragma unroll
      for (int c = 0; c < CPL; ++c) v[c] = x[NA * DKP + col0 + c];
    };
    auto fetch = [&](const float* x, int arr, Row (&r)[J]) {
#pragma unroll
      for (int j = 0; j < J; ++j) r[j] = *reinterpret_cast<const Row*>(x + arr * DKP + j * 32 + lr * 4);
    };
    auto dot = [&](const Row (&u)[J], float* d) {
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        unsigned long long e = 0, f = 0;
#pragma unroll
        for (int j = 0; j < J; ++j) {
          e = fma2(u[j].x, s[2 * j][c], e);
          f = fma2(u[j].y, s[2 * j + 1][c], f);
        }
        float x, y, z, w;
        unpack2(e, x, y);
        unpack2(f, z, w);
        d[c] = (x + y) + (z + w);
      }
    };
    // one token: S = w S - b d + k v, and this lane's share of S^T q
    auto token = [&](int t, const Row (&k)[J], const Row (&w)[J], const Row (&q)[J], const Row (&bb)[J], const float (&v)[CPL], const float* d) {
      unsigned long long o[CPL], vv[CPL], dd[CPL];
#pragma unroll
      for (int c = 0; c < CPL; ++c) {
        o[c] = 0;
        vv[c] = pack2(v[c], v[c]);
        dd[c] = KIND == KIND_DELTA ? pack2(-d[c], -d[c]) : 0;
      }
#pragma unroll
      for (int j = 0; j < J; ++j) {
        const unsigned long long kk[2] = {k[j].x, k[j].y}, ww[2] = {w[j].x, w[j].y}, qq[2] = {q[j].x, q[j].y}, rr[2] = {bb[j].x, bb[j].y};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int r = 2 * j + i;
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            unsigned long long add = mul2(kk[i], vv[c]);
            if (KIND == KIND_DELTA) add = fma2(rr[i], dd[c], add);
            s[r][c] = fma2(ww[i], s[r][c], add);
            o[c] = fma2(qq[i], s[r][c], o[c]);
          }
        }
      }
      if (outputs) {
        float* po = os + (size_t)(t * 8 + lr) * OP + col0;
        float r[CPL];
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          float x, y;
          unpack2(o[c], x, y);
          r[c] = x + y;
        }
        if (CPL == 4) store4(po, make_float4(r[0], r[1 % CPL], r[2 % CPL], r[3 % CPL]));
        else if (CPL == 2) *reinterpret_cast<float2*>(po) = make_float2(r[0], r[1 % CPL]);
        else po[0] = r[0];
      }
    };
    if (KIND == KIND_GLA) {
#pragma unroll 2
      for (int t = 0; t < n; ++t) {
        const float* x = x0 + (size_t)t * stride;
        Row k[J], w[J], q[J];
        float v[CPL];
        fetch(x, 0, k);
        fetch(x, 1, w);
        fetch(x, 2, q);
        values(x, v);
        token(t, k, w, q, k, v, nullptr);
      }
    } else {
      int t = 0;
      for (; t + 1 < n; t += 2) {
        const float *xa = x0 + (size_t)t * stride, *xb = xa + stride;
        float d[2 * CPL], va[CPL], vb[CPL];
        Row k[J], w[J], q[J], r[J];
        fetch(xa, 3, k);
        fetch(xa, 5, w);
        dot(k, d);
        dot(w, d + CPL);
        fetch(xa, 0, k);
        fetch(xa, 1, w);
        fetch(xa, 2, q);
        fetch(xa, 4, r);
        values(xa, va);
        const float2 ab = *reinterpret_cast<const float2*>(xa + NA * DKP + 2 * COLS);
        GroupSum<2 * CPL, 4>::run(d, lr);
#pragma unroll
        for (int c = 0; c < CPL; ++c) d[CPL + c] = fmaf(ab.y, va[c], fmaf(-ab.x, d[c], d[CPL + c]));
        token(t, k, w, q, r, va, d);
        fetch(xb, 0, k);
        fetch(xb, 1, w);
        fetch(xb, 2, q);
        fetch(xb, 4, r);
        values(xb, vb);
        token(t + 1, k, w, q, r, vb, d + CPL);
      }
      if (t < n) {
        const float* xa = x0 + (size_t)t * stride;
        float d[CPL], va[CPL];
        Row k[J], w[J], q[J], r[J];
        fetch(xa, 3, k);
        dot(k, d);
        fetch(xa, 0, k);
        fetch(xa, 1, w);
        fetch(xa, 2, q);
        fetch(xa, 4, r);
        values(xa, va);
        GroupSum<CPL, 4>::run(d, lr);
        token(t, k, w, q, r, va, d);
      }
    }
    if (outputs) {
      // every warp's shares are in; this buffer is written again two blocks on, after the next barrier
      named_barrier(1, W * 32);
      for (int t = warp; t < n; t += W) {
        const float* po = os + (size_t)t * 8 * OP;
        const float* g = x0 + (size_t)t * stride + NA * DKP + COLS;
        float o[4], sq = 0.f;  // at most 128 columns
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int c = lane + i * 32;
          float x = 0.f;
          if (c < dv) {
#pragma unroll
            for (int e = 0; e < 8; ++e) x += po[e * OP + c];
          }
          o[i] = x * l.q_scale;
          sq += o[i] * o[i];
        }
        if (sa.col_blocks > 1) {  // recurrence_output_kernel finishes the rows
          float* out = a.out_raw + (size_t)(tb0 + t) * (l.heads * l.vdim) + head * l.vdim + cbase;
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (lane + i * 32 < dv) out[lane + i * 32] = o[i];
        } else {
          const float rinv = 1.f / sqrtf(lane_sum(sq) / (float)dv + l.eps);
          const size_t base = (size_t)(tb0 + t) * a.ldy + head * dv;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int c = lane + i * 32;
            if (c < dv) {
              const float gate = KIND == KIND_GLA ? silu_f(g[c]) : sigmoid_f(g[c]);
              const float y = o[i] * rinv * l.norm[KIND == KIND_DELTA ? head * dv + c : c] * gate * l.out_scale;
              if (sa.y_bf16) static_cast<__nv_bfloat16*>(a.y)[base + c] = __float2bfloat16_rn(y);
              else static_cast<float*>(a.y)[base + c] = y;
            }
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[sidx]);
  }

  if (sa.mode == SCAN_OUTPUT) return;
  float* fin = sa.mode == SCAN_FULL ? a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp
               : trans              ? sa.seg_trans + seg_index * dk * sa.dkp
                                    : sa.seg_state + seg_index * dk * l.dvp;
  const int pitch = trans ? sa.dkp : l.dvp;
#pragma unroll
  for (int r = 0; r < RPL; r += 2)
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      float v[2];
      unpack2(s[r / 2][c], v[0], v[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (row_of(r + e) < dk && col0 + c < dv) fin[(size_t)row_of(r + e) * pitch + cbase + col0 + c] = v[e];
    }
}

// The channel delta rule, four tokens at a time (see channel_quads_kernel); blocks, lanes, stages and modes as above.
template <int RPL, int CPL>
__global__ void __launch_bounds__((SCAN_WARPS + 1) * 32, 1) channel_scan_kernel(ScanArgs sa) {
  extern __shared__ __align__(16) float sm[];
  __shared__ uint64_t full[SCAN_STAGES], empty[SCAN_STAGES];
  __shared__ int failed_flag;
  constexpr int DKP = 8 * RPL, J = RPL / 4;
  const RecurrenceScanArgs& a = sa.a;
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, K = l.heads * dk, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const bool trans = sa.mode == SCAN_TRANS, outputs = sa.mode == SCAN_FULL || sa.mode == SCAN_OUTPUT;
  const int head = blockIdx.x / sa.col_blocks, cb = blockIdx.x % sa.col_blocks, seq = blockIdx.y, seg = blockIdx.z;
  const int all_cols = trans ? dk : l.vdim, cbase = cb * sa.block_cols;
  const int dv = min(sa.block_cols, all_cols - cbase);  // columns of this block
  const int W = (blockDim.x >> 5) - 1, COLS = W * 4 * CPL, TB = sa.tb;  // TB: tokens of a stage, a multiple of QUAD
  // a staged quad: per token A, B, Q, v, gate; then W and the numbers
  const int stride = 3 * DKP + 2 * COLS, qstride = QUAD * stride + DKP + QUAD_NUMBERS, OP = COLS + 4, quads = TB / QUAD;
  float* stage = sm;                                            // [SCAN_STAGES][quads][qstride]
  float* os0 = sm + (size_t)SCAN_STAGES * quads * qstride;      // [2][TB][OP] outputs
  const bool want_v = !trans, want_g = outputs && sa.col_blocks == 1;
  volatile int* failed = &failed_flag;

  const int first = a.seq_start[seq];
  int t0 = first, t1 = a.seq_start[seq + 1];
  if (sa.mode != SCAN_FULL) {
    t0 += seg * a.seg_tokens;
    t1 = min(t1, t0 + a.seg_tokens);
    if (t0 >= t1) return;
  }
  for (int i = tid; i < SCAN_STAGES * quads * qstride; i += blockDim.x) stage[i] = 0.f;  // the padding stays zero
  if (tid == 0) {
    for (int i = 0; i < SCAN_STAGES; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], (uint32_t)W);
    }
    failed_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // the zeros come before the bulk copies
  __syncthreads();
  const int blocks = (t1 - t0 + TB - 1) / TB;

  if (warp == W) {  // ---- stages rows; lane = (token, array) of a quad, then its W and its numbers
    const int tok = lane / 5, arr = lane % 5;
    const float* rows[5] = {a.decay + head * dk, a.writes + head * dk, a.unit_next + head * dk, sa.v + head * l.vdim + cbase, sa.g + head * l.vdim + cbase};
    const bool on = lane >= 20 ? lane < 22 : arr < 2 || (arr == 2 && outputs) || (arr == 3 && want_v) || (arr == 4 && want_g);
    const float* src = rows[arr];
    const int pitch = arr < 3 ? K : arr == 3 ? sa.ldv : sa.ldg, count = lane == 21 ? QUAD_NUMBERS : lane == 20 || arr < 3 ? dk : dv;
    const int off = lane == 21 ? QUAD * stride + DKP : lane == 20 ? QUAD * stride : tok * stride + (arr < 3 ? arr * DKP : 3 * DKP + (arr == 4 ? COLS : 0));
    const size_t quad0 = first_quad(a, seq) + (t0 - first) / QUAD;
    const uint32_t token_bytes = 4u * (uint32_t)((outputs ? 3 : 2) * dk + (want_v ? dv : 0) + (want_g ? dv : 0)), quad_bytes = 4u * (uint32_t)(dk + QUAD_NUMBERS);
    RingCursor r;
    for (int b = 0; b < blocks; ++b, r.next(SCAN_STAGES)) {
      const int tb0 = t0 + b * TB, n = min(TB, t1 - tb0), nq = (n + QUAD - 1) / QUAD;
      if (!mbar_wait(&empty[r.stage], r.parity ^ 1, failed, a.error_flag, 41)) break;
      __syncwarp();
      float* dst = stage + (size_t)r.stage * quads * qstride + off;
      if (sa.vec) {
        if (lane == 0) mbar_expect_tx(&full[r.stage], (uint32_t)n * token_bytes + (uint32_t)nq * quad_bytes);
        __syncwarp();
      }
      for (int g = 0; g < nq; ++g) {
        const size_t quad = quad0 + (size_t)b * quads + g;
        const bool have = on && (lane >= 20 || g * QUAD + tok < n);
        const float* from = lane == 21 ? a.quads + (quad * l.heads + head) * QUAD_NUMBERS
                            : lane == 20 ? a.quad_decay + quad * K + head * dk
                                         : src + (size_t)(tb0 + g * QUAD + tok) * pitch;
        if (have && sa.vec) bulk_row(dst + (size_t)g * qstride, from, (uint32_t)(4 * count), &full[r.stage]);
        else if (have)
          for (int i = 0; i < count; ++i) dst[(size_t)g * qstride + i] = from[i];
      }
      if (!sa.vec) {
        __syncwarp();
        if (lane == 0) mbar_arrive(&full[r.stage]);
      }
    }
    return;
  }

  // ---- start state, two neighbouring rows per register pair
  const int lr = lane & 7, col0 = (warp * 4 + (lane >> 3)) * CPL;
  unsigned long long s[RPL / 2][CPL];
  const size_t seg_index = ((size_t)seq * a.max_segs + seg) * l.heads + head;
  const float* init = nullptr;
  if (sa.mode == SCAN_FULL && a.seq_pos[seq] > 0) init = a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp;
  if (sa.mode == SCAN_OUTPUT) init = sa.seg_state + seg_index * dk * l.dvp;
  auto row_of = [&](int r) { return (r >> 2) * 32 + lr * 4 + (r & 3); };
#pragma unroll
  for (int r = 0; r < RPL; r += 2)
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      float v[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = row_of(r + e), col = col0 + c;
        v[e] = 0.f;
        if (row < dk && col < dv) {
          if (init) v[e] = init[(size_t)row * l.dvp + cbase + col];
          else if (trans) v[e] = row == cbase + col ? 1.f : 0.f;
        }
      }
      s[r / 2][c] = pack2(v[0], v[1]);
    }

  using Row = ulonglong2;  // four entries of a key-channel row
  auto row = [&](const float* x, int j) { return *reinterpret_cast<const Row*>(x + j * 32 + lr * 4); };
  RingCursor ring;
  for (int b = 0; b < blocks; ++b, ring.next(SCAN_STAGES)) {
    const int tb0 = t0 + b * TB, n = min(TB, t1 - tb0);
    mbar_wait(&full[ring.stage], ring.parity, failed, a.error_flag, 42);  // on expiry the numbers are void, the barriers below are kept
    __syncwarp();
    const float* x0 = stage + (size_t)ring.stage * quads * qstride;
    float* os = os0 + (size_t)(b & 1) * TB * OP;
    for (int g = 0; g * QUAD < n; ++g) {
      const float* x = x0 + (size_t)g * qstride;
      const float* num = x + QUAD * stride + DKP;
      const int have = n - g * QUAD;  // tokens of this quad, if below four
      float d[QUAD * CPL];
#pragma unroll
      for (int i = 0; i < QUAD; ++i) {
        unsigned long long e[CPL];
#pragma unroll
        for (int c = 0; c < CPL; ++c) e[c] = 0;
#pragma unroll
        for (int j = 0; j < J; ++j) {
          const Row k = row(x + i * stride, j);
#pragma unroll
          for (int c = 0; c < CPL; ++c) e[c] = fma2(k.y, s[2 * j + 1][c], fma2(k.x, s[2 * j][c], e[c]));
        }
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          float u, v;
          unpack2(e[c], u, v);
          d[i * CPL + c] = u + v;
        }
      }
      GroupSum<QUAD * CPL, 4>::run(d, lr);
      float nr[QUAD_NUMBERS];
#pragma unroll
      for (int i = 0; i < QUAD_NUMBERS; i += 4) {
        const float4 f = load4(num + i);
        nr[i] = f.x; nr[i + 1] = f.y; nr[i + 2] = f.z; nr[i + 3] = f.w;
      }
#pragma unroll
      for (int i = 0; i < QUAD; ++i)
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          float v = x[i * stride + 3 * DKP + col0 + c] - d[i * CPL + c];
#pragma unroll
          for (int j = 0; j < i; ++j) v = fmaf(-nr[i * (i - 1) / 2 + j], d[j * CPL + c], v);
          d[i * CPL + c] = i < have ? nr[16 + i] * v : 0.f;  // what token i writes
        }
      if (outputs) {
        float r[QUAD * CPL];
#pragma unroll
        for (int i = 0; i < QUAD; ++i) {
          unsigned long long e[CPL];
#pragma unroll
          for (int c = 0; c < CPL; ++c) e[c] = 0;
#pragma unroll
          for (int j = 0; j < J; ++j) {
            const Row q = row(x + i * stride + 2 * DKP, j);
#pragma unroll
            for (int c = 0; c < CPL; ++c) e[c] = fma2(q.y, s[2 * j + 1][c], fma2(q.x, s[2 * j][c], e[c]));
          }
#pragma unroll
          for (int c = 0; c < CPL; ++c) {
            float u, v;
            unpack2(e[c], u, v);
            r[i * CPL + c] = u + v;
            if (lr == 0) {
#pragma unroll
              for (int j = 0; j <= i; ++j) r[i * CPL + c] = fmaf(nr[6 + i * (i + 1) / 2 + j], d[j * CPL + c], r[i * CPL + c]);
            }
          }
        }
        using Scatter = GroupScatter<QUAD * CPL, 4>;
        Scatter::run(r, lr);
        const int at = Scatter::index(lr), i = at / CPL;
        float* po = os + (size_t)(g * QUAD + i) * OP + col0 + at % CPL;
        if (CPL == 4) *reinterpret_cast<float2*>(po) = make_float2(r[0], r[1]);
        else if (CPL == 2 || (lr & 1) == 0) po[0] = r[0];
      }
#pragma unroll
      for (int j = 0; j < J; ++j) {
        const Row w = row(x + QUAD * stride, j);
        Row k[QUAD];
#pragma unroll
        for (int i = 0; i < QUAD; ++i) k[i] = row(x + i * stride + DKP, j);
#pragma unroll
        for (int c = 0; c < CPL; ++c) {
          unsigned long long lo = mul2(w.x, s[2 * j][c]), hi = mul2(w.y, s[2 * j + 1][c]);
#pragma unroll
          for (int i = 0; i < QUAD; ++i) {
            const unsigned long long u = pack2(d[i * CPL + c], d[i * CPL + c]);
            lo = fma2(k[i].x, u, lo);
            hi = fma2(k[i].y, u, hi);
          }
          s[2 * j][c] = lo;
          s[2 * j + 1][c] = hi;
        }
      }
    }
    if (outputs) {
      // every warp's shares are in; this buffer is written again two blocks on, after the next barrier
      named_barrier(1, W * 32);
      for (int t = warp; t < n; t += W) {
        const float* po = os + (size_t)t * OP;
        const float* g = x0 + (size_t)(t / QUAD) * qstride + (t % QUAD) * stride + 3 * DKP + COLS;
        float o[4], sq = 0.f;  // at most 128 columns
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int c = lane + i * 32;
          o[i] = c < dv ? po[c] * l.q_scale : 0.f;
          sq += o[i] * o[i];
        }
        if (sa.col_blocks > 1) {  // recurrence_output_kernel finishes the rows
          float* out = a.out_raw + (size_t)(tb0 + t) * (l.heads * l.vdim) + head * l.vdim + cbase;
#pragma unroll
          for (int i = 0; i < 4; ++i)
            if (lane + i * 32 < dv) out[lane + i * 32] = o[i];
        } else {
          const float rinv = 1.f / sqrtf(lane_sum(sq) / (float)dv + l.eps);
          const size_t base = (size_t)(tb0 + t) * a.ldy + head * dv;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int c = lane + i * 32;
            if (c < dv) {
              const float y = o[i] * rinv * l.norm[c] * sigmoid_f(g[c]) * l.out_scale;
              if (sa.y_bf16) static_cast<__nv_bfloat16*>(a.y)[base + c] = __float2bfloat16_rn(y);
              else static_cast<float*>(a.y)[base + c] = y;
            }
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[ring.stage]);
  }

  if (sa.mode == SCAN_OUTPUT) return;
  float* fin = sa.mode == SCAN_FULL ? a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp
               : trans              ? sa.seg_trans + seg_index * dk * sa.dkp
                                    : sa.seg_state + seg_index * dk * l.dvp;
  const int pitch = trans ? sa.dkp : l.dvp;
#pragma unroll
  for (int r = 0; r < RPL; r += 2)
#pragma unroll
    for (int c = 0; c < CPL; ++c) {
      float v[2];
      unpack2(s[r / 2][c], v[0], v[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (row_of(r + e) < dk && col0 + c < dv) fin[(size_t)row_of(r + e) * pitch + cbase + col0 + c] = v[e];
    }
}

// Head norm, gate and branch scale of scan outputs that left in several column blocks; a warp per (row, head), at most
// 256 columns.
__global__ void __launch_bounds__(256) recurrence_output_kernel(ScanArgs sa) {
  const RecurrenceScanArgs& a = sa.a;
  const RecurrenceLayer& l = a.l;
  const int lane = threadIdx.x & 31, dv = l.vdim;
  const long long total = (long long)a.rows * l.heads;
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5; i < total; i += ((long long)gridDim.x * blockDim.x) >> 5) {
    const int row = (int)(i / l.heads), head = (int)(i % l.heads);
    const float* o = a.out_raw + (size_t)row * (l.heads * dv) + head * dv;
    const float* g = sa.g + (size_t)row * sa.ldg + head * dv;
    float ov[8], gv[8], sq = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = lane + j * 32;
      ov[j] = c < dv ? o[c] : 0.f;
      gv[j] = c < dv ? g[c] : 0.f;
      sq += ov[j] * ov[j];
    }
    const float rinv = 1.f / sqrtf(lane_sum(sq) / (float)dv + l.eps);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = lane + j * 32;
      if (c >= dv) break;
      const float gate = l.kind == KIND_GLA ? silu_f(gv[j]) : sigmoid_f(gv[j]);
      const float y = ov[j] * rinv * l.norm[l.kind == KIND_DELTA ? head * dv + c : c] * gate * l.out_scale;
      const size_t at = (size_t)row * a.ldy + head * dv + c;
      if (sa.y_bf16) static_cast<__nv_bfloat16*>(a.y)[at] = __float2bfloat16_rn(y);
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
// one sequence; the running state stays in shared memory, the next segment's numbers load one segment ahead.
constexpr int COMBINE_COLS = 16, COMBINE_THREADS = 256, ROW_STEP = COMBINE_THREADS / COMBINE_COLS;
template <int KIND, int PER>  // PER: rows of a thread, PER * ROW_STEP >= dim
__global__ void __launch_bounds__(COMBINE_THREADS) recurrence_combine_kernel(ScanArgs sa) {
  extern __shared__ __align__(16) float sm[];
  const RecurrenceScanArgs& a = sa.a;
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, head = blockIdx.x, seq = blockIdx.y, c0 = blockIdx.z * COMBINE_COLS, tid = threadIdx.x;
  const int nc = min(COMBINE_COLS, l.vdim - c0);
  const int len = a.seq_start[seq + 1] - a.seq_start[seq], segs = (len + a.seg_tokens - 1) / a.seg_tokens;
  const int tp = sa.dkp + 4;               // pitch of a transition row in shared memory
  float* cur = sm;                         // [dk][COMBINE_COLS]
  float* nxt = sm + dk * COMBINE_COLS;
  float* tr = sm + 2 * dk * COMBINE_COLS;  // delta: [2][dk][tp], the next one loading
  float* cached = a.state + ((size_t)a.seq_slot[seq] * l.heads + head) * dk * l.dvp;
  const bool fresh = a.seq_pos[seq] == 0;
  const int c = tid % COMBINE_COLS, row0 = tid / COMBINE_COLS;  // this thread: one column, rows row0 + q * ROW_STEP
  int at[PER];                                                  // where its rows of a transition matrix start
#pragma unroll
  for (int q = 0; q < PER; ++q) at[q] = min(row0 + q * ROW_STEP, dk - 1) * tp;
  auto seg_at = [&](int g) { return ((size_t)seq * a.max_segs + g) * l.heads + head; };
  auto load_trans = [&](int g, float* dst) {
    const float* src = sa.seg_trans + seg_at(g) * dk * sa.dkp;
    const int row4 = sa.dkp / 4;
    for (int i = tid; i < dk * row4; i += COMBINE_THREADS) {
      const int r = i / row4, x = i - r * row4;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + r * tp + x * 4)), "l"(src + (size_t)i * 4) : "memory");
    }
  };
  float loc[PER], dec[PER];
  auto load_next = [&](int g) {
    const float* p = sa.seg_state + seg_at(g) * dk * l.dvp;
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      const int r = row0 + q * ROW_STEP;
      if (r < dk) {
        loc[q] = c < nc ? p[(size_t)r * l.dvp + c0 + c] : 0.f;
        if (KIND == KIND_GLA) dec[q] = sa.seg_trans[seg_at(g) * dk + r];
      }
    }
  };
  for (int i = tid; i < dk * COMBINE_COLS; i += COMBINE_THREADS) {
    const int r = i / COMBINE_COLS, c = i % COMBINE_COLS;
    cur[i] = (!fresh && c < nc) ? cached[(size_t)r * l.dvp + c0 + c] : 0.f;
  }
  load_next(0);
  if (KIND == KIND_DELTA) load_trans(0, tr);
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int g = 0; g < segs; ++g) {
    float v[PER], w[PER];
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      v[q] = loc[q];
      w[q] = KIND == KIND_GLA ? dec[q] : 0.f;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (g + 1 < segs) {
      load_next(g + 1);
      if (KIND == KIND_DELTA) load_trans(g + 1, tr + (size_t)((g + 1) & 1) * dk * tp);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    float* start = sa.seg_state + seg_at(g) * dk * l.dvp;
    const float* m = tr + (size_t)(g & 1) * dk * tp;
    if (KIND == KIND_DELTA) {
      int j = 0;
      for (; j + 3 < dk; j += 4) {
        const float x0 = cur[j * COMBINE_COLS + c], x1 = cur[(j + 1) * COMBINE_COLS + c], x2 = cur[(j + 2) * COMBINE_COLS + c], x3 = cur[(j + 3) * COMBINE_COLS + c];
#pragma unroll
        for (int q = 0; q < PER; ++q) {
          const float4 t = load4(m + at[q] + j);
          v[q] = fmaf(t.x, x0, v[q]);
          v[q] = fmaf(t.y, x1, v[q]);
          v[q] = fmaf(t.z, x2, v[q]);
          v[q] = fmaf(t.w, x3, v[q]);
        }
      }
      for (; j < dk; ++j)
#pragma unroll
        for (int q = 0; q < PER; ++q)
          v[q] = fmaf(m[at[q] + j], cur[j * COMBINE_COLS + c], v[q]);
    }
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      const int r = row0 + q * ROW_STEP, i = r * COMBINE_COLS + c;
      if (r < dk) {
        const float old = cur[i];
        if (c < nc) start[(size_t)r * l.dvp + c0 + c] = old;
        nxt[i] = KIND == KIND_GLA ? fmaf(w[q], old, v[q]) : v[q];
      }
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
constexpr size_t MAX_SMEM = 225 * 1024;  // beside a little static shared memory

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
  if (kind == KIND_CHANNEL) {
    const size_t c = (size_t)warps * 4 * cpl, quad = QUAD * (3 * 8 * rpl + 2 * c) + 8 * rpl + QUAD_NUMBERS;
    return ((size_t)SCAN_STAGES * (tb / QUAD) * quad + (size_t)2 * tb * (c + 4)) * sizeof(float);
  }
  const size_t na = kind == KIND_DELTA ? 6 : 3, cols = (size_t)warps * 4 * cpl;
  return ((size_t)SCAN_STAGES * tb * (na * 8 * rpl + 2 * cols + 4) + (size_t)2 * tb * 8 * (cols + 4)) * sizeof(float);
}

template <int KIND, int RPL, int CPL>
auto scan_kernel() {
  if constexpr (KIND == KIND_CHANNEL) return channel_scan_kernel<RPL, CPL>;
  else return recurrence_scan_kernel<KIND, RPL, CPL>;
}

template <int KIND, int RPL, int CPL>
cudaError_t launch_scan(ScanArgs sa, dim3 grid, int cols, cudaStream_t s) {
  const int warps = (cols + 4 * CPL - 1) / (4 * CPL);
  if (warps > SCAN_WARPS) return cudaErrorInvalidValue;
  const int least = KIND == KIND_CHANNEL ? QUAD : 2;
  sa.tb = 16;
  while (sa.tb > least && scan_smem(KIND, RPL, CPL, warps, sa.tb) > MAX_SMEM) sa.tb /= 2;
  const size_t smem = scan_smem(KIND, RPL, CPL, warps, sa.tb);
  if (smem > MAX_SMEM) return cudaErrorInvalidValue;
  auto kernel = scan_kernel<KIND, RPL, CPL>();
  cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);
  if (e != cudaSuccess) return e;
  return launch_kernel(kernel, grid, dim3((warps + 1) * 32), smem, s, false, sa);
}

template <int KIND, int RPL>
cudaError_t launch_scan_cols(const ScanArgs& sa, dim3 grid, int cols, int cpl, cudaStream_t s) {
  if (cpl == 4) return launch_scan<KIND, RPL, 4>(sa, grid, cols, s);
  if (cpl == 2) return launch_scan<KIND, RPL, 2>(sa, grid, cols, s);
  return launch_scan<KIND, RPL, 1>(sa, grid, cols, s);
}

cudaError_t launch_scan_any(ScanArgs sa, dim3 grid, int cols, cudaStream_t s) {
  const int dk = sa.a.l.dim;
  const long long blocks = (long long)grid.x * grid.y * grid.z;
  // few blocks in flight: the columns of a head are cut over several of them
  int nb = (cols + 127) / 128;
  while (nb * 2 * blocks <= sm_count() && (cols + nb * 2 - 1) / (nb * 2) >= 48) nb *= 2;
  sa.block_cols = ((cols + nb - 1) / nb + 3) / 4 * 4;
  sa.col_blocks = (cols + sa.block_cols - 1) / sa.block_cols;
  grid.x *= sa.col_blocks;
  const int bc = sa.block_cols;
  int cpl = (bc + 31) / 32;
  if (cpl == 3) cpl = 4;
#define PG_SCAN(KIND_)                                                                  \
  (dk <= 32    ? launch_scan_cols<KIND_, 4>(sa, grid, bc, cpl, s)                       \
   : dk <= 64  ? launch_scan_cols<KIND_, 8>(sa, grid, bc, cpl, s)                       \
   : dk <= 128 ? launch_scan_cols<KIND_, 16>(sa, grid, bc, cpl, s)                      \
   : dk <= 256 ? launch_scan_cols<KIND_, 32>(sa, grid, bc, cpl, s) : cudaErrorInvalidValue)
  cudaError_t e = sa.a.l.kind == KIND_DELTA ? PG_SCAN(KIND_DELTA) : sa.a.l.kind == KIND_CHANNEL ? PG_SCAN(KIND_CHANNEL) : PG_SCAN(KIND_GLA);
#undef PG_SCAN
  if (e == cudaSuccess && sa.col_blocks > 1 && (sa.mode == SCAN_FULL || sa.mode == SCAN_OUTPUT)) {
    const long long warps = (long long)sa.a.rows * sa.a.l.heads;
    e = launch_kernel(recurrence_output_kernel, dim3((unsigned)std::min<long long>((warps + 7) / 8, 148 * 32)), dim3(256), 0, s, false, sa);
  }
  return e;
}

cudaError_t launch_channel_gates(const RecurrenceScanArgs& a, cudaStream_t s) {
  const RecurrenceLayer& l = a.l;
  const long long cw = (long long)((a.rows + CONV_ROWS - 1) / CONV_ROWS) * (2 * l.kv_heads + l.heads);
  const long long qw = (long long)((a.max_len + QUAD - 1) / QUAD) * l.heads;
  const dim3 cg((unsigned)((cw + 7) / 8)), qg((unsigned)((qw + 7) / 8), a.nseq), b(256);
  const int size = std::max(l.dim, l.vdim);
  const bool vec = l.dim % 4 == 0 && l.vdim % 4 == 0 && size <= 128 && l.taps >= 2 && l.taps <= 4 && a.ldp % 4 == 0 && l.off_q % 4 == 0 &&
                   l.off_k % 4 == 0 && l.off_v % 4 == 0 && l.channels % 4 == 0 && a.ldz % 4 == 0;
  cudaError_t e;
#define PG_CONV(TAPS_)                                                                                  \
  (vec           ? launch_kernel(channel_conv_vec_kernel<TAPS_>, cg, b, 0, s, false, a)                 \
   : size <= 64  ? launch_kernel(channel_conv_kernel<TAPS_, 2>, cg, b, 0, s, false, a)                  \
   : size <= 128 ? launch_kernel(channel_conv_kernel<TAPS_, 4>, cg, b, 0, s, false, a)                  \
                 : launch_kernel(channel_conv_kernel<TAPS_, 8>, cg, b, 0, s, false, a))
  if (l.taps == 2) e = PG_CONV(2);
  else if (l.taps == 3) e = PG_CONV(3);
  else if (l.taps == 4) e = PG_CONV(4);
  else
    e = size <= 64    ? launch_kernel(channel_conv_kernel<0, 2>, cg, b, 0, s, false, a)
        : size <= 128 ? launch_kernel(channel_conv_kernel<0, 4>, cg, b, 0, s, false, a)
                      : launch_kernel(channel_conv_kernel<0, 8>, cg, b, 0, s, false, a);
#undef PG_CONV
  if (e != cudaSuccess) return e;
  e = l.dim <= 64    ? launch_kernel(channel_quads_kernel<2>, qg, b, 0, s, false, a)
      : l.dim <= 128 ? launch_kernel(channel_quads_kernel<4>, qg, b, 0, s, false, a)
                     : launch_kernel(channel_quads_kernel<8>, qg, b, 0, s, false, a);
  if (e != cudaSuccess || l.taps == 1) return e;
  return launch_kernel(channel_taps_kernel, dim3(a.nseq, l.taps - 1, (l.channels + 255) / 256), b, 0, s, false, a);
}

}  // namespace

bool recurrence_use_segments(const RecurrenceLayer& l, int nseq, int max_len, int max_segs) {
  // the transition matrices of the delta rule must fit shared memory twice
  return max_segs >= 4 && max_len >= 512 && (long long)nseq * l.heads < 48 && (l.kind == KIND_GLA || l.dim <= 144);
}

size_t recurrence_segment_floats(const RecurrenceLayer& l, int nseq, int max_segs) {
  return (size_t)nseq * max_segs * l.heads * l.dim * (l.dvp + (l.kind != KIND_GLA ? (l.dim + 3) / 4 * 4 : 1));
}

cudaError_t launch_recurrence_scan(const RecurrenceScanArgs& a, bool y_bf16, cudaStream_t s) {
  if (a.rows <= 0) return cudaSuccess;
  const RecurrenceLayer& l = a.l;
  const int K = l.heads * l.dim;
  cudaError_t e = l.kind == KIND_CHANNEL ? launch_channel_gates(a, s) : launch_kernel(recurrence_decay_kernel, dim3((a.rows + GATE_ROWS - 1) / GATE_ROWS, (K + 255) / 256), dim3(256),
                                (size_t)GATE_ROWS * l.rank * sizeof(float), s, false, a);
  if (e != cudaSuccess) return e;
  if (l.kind == KIND_DELTA) {
    const long long warps = (long long)a.rows * l.heads;
    const bool vec = l.dim % 4 == 0 && l.off_k % 4 == 0 && l.off_a % 4 == 0 && a.ldp % 4 == 0;
    e = vec ? launch_kernel(delta_gates_vec_kernel, dim3((unsigned)std::min<long long>((warps + 31) / 32, 148 * 32)), dim3(256), 0, s, false, a)
            : launch_kernel(delta_gates_kernel, dim3((unsigned)std::min<long long>((warps + 7) / 8, 148 * 32)), dim3(256), 0, s, false, a);
    if (e != cudaSuccess) return e;
  }
  ScanArgs sa{};
  sa.a = a;
  sa.y_bf16 = y_bf16 ? 1 : 0;
  auto m4 = [](int v) { return v % 4 == 0; };
  if (l.kind == KIND_CHANNEL) {
    sa.v = a.vals; sa.g = a.z + K;
    sa.ldv = l.heads * l.vdim; sa.ldg = a.ldz;
  } else {
    sa.k = a.p + l.off_k; sa.q = a.p + l.off_q; sa.v = a.p + l.off_v; sa.g = a.p + l.off_g;
    sa.ldk = sa.ldq = sa.ldv = sa.ldg = a.ldp;
  }
  auto m16 = [](const float* v) { return (reinterpret_cast<uintptr_t>(v) & 15) == 0; };
  sa.vec = m4(l.dim) && m4(l.vdim) && m16(sa.k) && m16(sa.q) && m16(sa.v) && m16(sa.g) && m4(sa.ldk) && m4(sa.ldv) && m4(sa.ldg);
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
  if (l.kind != KIND_GLA) {
    sa.mode = SCAN_TRANS;
    e = launch_scan_any(sa, grid, l.dim, s);
  } else {
    e = launch_kernel(segment_decay_kernel, dim3((K + 255) / 256, a.max_segs, a.nseq), dim3(256), 0, s, false, sa);
  }
  if (e != cudaSuccess) return e;
  const dim3 cgrid(l.heads, a.nseq, (l.vdim + COMBINE_COLS - 1) / COMBINE_COLS);
  const size_t csmem = ((size_t)2 * l.dim * COMBINE_COLS + (l.kind != KIND_GLA ? (size_t)2 * l.dim * (sa.dkp + 4) : 0)) * sizeof(float);
  if (csmem > MAX_SMEM) return cudaErrorInvalidValue;
  auto combine = [&](auto kernel) {
    const cudaError_t r = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);
    return r != cudaSuccess ? r : launch_kernel(kernel, cgrid, dim3(COMBINE_THREADS), csmem, s, false, sa);
  };
#define PG_COMBINE(KIND_)                                                              \
  (l.dim <= 4 * ROW_STEP   ? combine(recurrence_combine_kernel<KIND_, 4>)              \
   : l.dim <= 8 * ROW_STEP ? combine(recurrence_combine_kernel<KIND_, 8>)              \
                           : combine(recurrence_combine_kernel<KIND_, 16>))
  e = l.kind != KIND_GLA ? PG_COMBINE(KIND_DELTA) : PG_COMBINE(KIND_GLA);
#undef PG_COMBINE
  if (e != cudaSuccess) return e;
  sa.mode = SCAN_OUTPUT;
  return launch_scan_any(sa, grid, l.vdim, s);
}

}  // namespace pg
