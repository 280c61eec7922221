// Attention steps whose heads belong together (mixed scores, shared latent rows), and the row work before and after the
// attention of portions: rotation, mixing, latents, products per head.
#include <algorithm>
#include <cfloat>

#include "attn_pages.cuh"

namespace pg {
namespace {

constexpr size_t MAX_SMEM = 200 * 1024;

// (cos, sin) of position * freq, the angle formed and reduced to one period in FP64.
__device__ __forceinline__ float2 angle(int pos, double freq) {
  const double ang = (double)pos * freq, two_pi = 6.283185307179586476925286766559;
  const float r = (float)(ang - two_pi * rint(ang * 0.15915494309189533576888376337251));
  float2 o;
  sincosf(r, &o.y, &o.x);
  return o;
}
// Entry c of a row of n values whose first `dims` entries are rotated in pairs (i, i + dims / 2).
template <typename F>
__device__ __forceinline__ float rotated(F x, int c, int dims, const float2* cs) {
  const int half = dims >> 1;
  if (c >= dims) return x(c);
  if (c < half) return x(c) * cs[c].x - x(c + half) * cs[c].y;
  return x(c) * cs[c - half].x + x(c - half) * cs[c - half].y;
}

__global__ void __launch_bounds__(256) angles_kernel(const int* pos, const double* freq, float2* out, int rows, int half) {
  grid_dep_launch();
  grid_dep_wait();
  const size_t n = (size_t)rows * half;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
    out[i] = angle(pos[i / half], freq[i % half]);
}

// ------------------------------------------------------------------ one token per sequence
// Block = one part of the visible keys of one sequence, for `hn` heads of it (all heads' scores where they are mixed).
// Scores: eight lanes share four keys at a time (16-byte pieces of the rows) for four heads that read the same key head; then
// the mixing, the running softmax, and threads that own eight value columns of up to NC heads. The last block of a sequence
// and head group merges the parts, adds the sink, turns the outputs back and applies the gate.
constexpr int THREADS = 256, WARPS = THREADS / 32, RB = 4, KB = 4;

struct StepShape {
  int hn, groups, raw, keys;  // heads of a block, blocks over the heads, heads whose scores a block makes, keys of a pass
  size_t smem;
};

template <typename T, int NC>
__global__ void __launch_bounds__(THREADS) attention_heads_step_kernel(AttentionStepArgs a, StepShape sh, int y_bf16) {
  extern __shared__ __align__(16) float sm[];
  __shared__ int last_flag;
  const AttentionLayer& l = a.l;
  const int split = blockIdx.x, seq = blockIdx.y, group = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = l.heads, G = l.kv_heads, rep = H / G, KC = sh.keys;
  const bool latent = l.vrow == 0;
  const int h0 = group * sh.hn, nh = min(sh.hn, H - h0), r0 = l.mix ? 0 : h0, nr = l.mix ? H : nh;  // output heads, scored heads
  float* qs = sm;                                   // [raw][dimp]
  float* kn = qs + (size_t)sh.raw * l.dimp;         // [G * dimp] the new keys as stored
  float* vn = latent ? kn : kn + G * l.dimp;        // [G * vdimp]
  float* raw = vn + G * l.vdimp;                    // [raw][KC] scores
  float* pr = l.mix ? raw + (size_t)sh.raw * KC : raw;  // [hn][KC] probabilities
  float* m_run = pr + (size_t)sh.hn * KC;           // [hn]
  float* l_run = m_run + sh.hn;
  float* corr = l_run + sh.hn;
  float2* kcs = reinterpret_cast<float2*>(corr + sh.hn + (sh.hn & 1));  // [rot_dims / 2]
  float2* vcs = kcs + (l.rot_dims >> 1);                               // [vdim / 2]
  size_t* kbase = reinterpret_cast<size_t*>(vcs + (l.v_rot ? l.vdim >> 1 : 0));  // [KC] page of a key, its row in it
  int* koff = reinterpret_cast<int*>(kbase + KC);
  float* os = reinterpret_cast<float*>(koff + KC);  // [max(hn * vdimp, 2048)] outputs
  float* red = os + max(sh.hn * l.vdimp, 8 * THREADS);  // [33]

  grid_dep_launch();
  grid_dep_wait();
  const float* p = a.p + (size_t)seq * a.ldp;
  const int pos = a.pos[seq];
  // visible: the kept first positions, then lo..pos
  const int lo = l.life.window > 0 ? max(pos - l.life.window + 1, 0) : pos / l.life.span * l.life.span;
  const int kept = l.life.window > 0 ? min(l.life.keep, lo) : 0, total = kept + pos - lo + 1;
  const int per = (total + a.splits - 1) / a.splits;
  const int k0 = split * per, k1 = min(total, k0 + per);
  const int* table = a.page_table + (size_t)seq * l.pages_per_seq;
  T* pool = static_cast<T*>(a.pool);
  const size_t page_elems = (size_t)G * l.page_tokens * (l.dimp + l.vrow), v_at = latent ? 0 : (size_t)G * l.page_tokens * l.dimp;
  const int vpitch = latent ? l.dimp : l.vrow;
  const int tok = l.wide ? G : 1, hd = l.wide ? 1 : l.page_tokens;  // rows between two tokens, two heads of a page

  for (int i = tid; i < (l.rot_dims >> 1); i += THREADS) kcs[i] = angle(pos, l.rot_freq[i]);
  if (l.v_rot)
    for (int i = tid; i < (l.vdim >> 1); i += THREADS) vcs[i] = angle(pos, l.v_freq[i]);
  for (int i = tid; i < nh; i += THREADS) {
    m_run[i] = -FLT_MAX;
    l_run[i] = 0.f;
  }
  __syncthreads();
  if (latent) {
    const float* q = a.q + ((size_t)seq * H + h0) * l.dimp;
    for (int i = tid; i < nh * l.dimp; i += THREADS) qs[i] = q[i];
    const float* x = p + l.off_k;
    float s = 0.f;
    for (int c = tid; c < l.dim; c += THREADS) s += x[c] * x[c];
    const float inv = 1.f / sqrtf(block_sum(s, red) / (float)l.dim + l.eps);
    for (int c = tid; c < l.dimp; c += THREADS) kn[c] = c < l.dim ? to_f32(from_f32<T>(x[c] * inv * l.k_norm[c])) : 0.f;
  } else {
    auto row = [&](const float* x, const float* bias, int n) { return [=](int c) { return x[c] + (bias ? bias[c] : 0.f); }; };
    for (int i = tid; i < nr * l.dimp; i += THREADS) {
      const int h = r0 + i / l.dimp, c = i % l.dimp;
      qs[i] = c < l.dim ? rotated(row(p + l.off_q + h * l.dim, l.q_bias ? l.q_bias + h * l.dim : nullptr, l.dim), c, l.rot_dims, kcs) : 0.f;
    }
    for (int i = tid; i < G * l.dimp; i += THREADS) {
      const int h = i / l.dimp, c = i % l.dimp;
      kn[i] = c < l.dim ? to_f32(from_f32<T>(rotated(row(p + l.off_k + h * l.dim, l.k_bias ? l.k_bias + h * l.dim : nullptr, l.dim), c, l.rot_dims, kcs))) : 0.f;
    }
    for (int i = tid; i < G * l.vdimp; i += THREADS) {
      const int h = i / l.vdimp, c = i % l.vdimp;
      vn[i] = c < l.vdim ? to_f32(from_f32<T>(rotated(row(p + l.off_v + h * l.vdim, l.v_bias ? l.v_bias + h * l.vdim : nullptr, l.vdim), c, l.v_rot ? l.vdim : 0, vcs))) : 0.f;
    }
  }
  __syncthreads();
  if (k0 <= total - 1 && total - 1 < k1 && group == 0) {  // append
    const int at = l.life.place(pos);
    for (int i = tid; i < G * l.dimp; i += THREADS) page_row(l, pool, table, at, i / l.dimp, 0)[i % l.dimp] = from_f32<T>(kn[i]);
    if (!latent)
      for (int i = tid; i < G * l.vdimp; i += THREADS) page_row(l, pool, table, at, i / l.vdimp, 1)[i % l.vdimp] = from_f32<T>(vn[i]);
  }

  // value phase: thread = (eight columns of a head, subset of the keys) where there are few, else NC such columns
  const int nvec = l.vdimp / 8, chunks = nh * nvec, KG = NC == 1 && chunks < THREADS ? THREADS / chunks : 1;
  const int kg = KG > 1 ? tid / chunks : 0;
  const bool one_v = G == 1 && NC > 1 && THREADS % nvec == 0;  // all of a thread's chunks are the same columns of the same row
  float acc[NC][8];
#pragma unroll
  for (int i = 0; i < NC; ++i)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[i][e] = 0.f;
  const int sub = lane >> 3, l8 = lane & 7;

  for (int kb = k0; kb < k1; kb += KC) {
    const int n = min(KC, k1 - kb);
    for (int j = tid; j < n; j += THREADS) {
      const int i = kb + j, at = l.life.place(i < kept ? i : lo + i - kept);
      kbase[j] = (size_t)table[at / l.page_tokens] * page_elems;
      koff[j] = i == total - 1 ? -1 : at % l.page_tokens;  // the new key is read from shared memory
    }
    __syncthreads();
    for (int j0 = warp * 16; j0 < n; j0 += WARPS * 16) {
      const int jt = j0 + sub * KB;
      for (int hb = 0; hb < nr;) {
        const int kvh = (r0 + hb) / rep, nb = min(min(RB, nr - hb), (kvh + 1) * rep - (r0 + hb));  // heads of one key head
        float dot[RB * KB];
#pragma unroll
        for (int i = 0; i < RB * KB; ++i) dot[i] = 0.f;
        for (int c = l8 * 8; c < l.dimp; c += 64) {
          float kv[KB][8];
#pragma unroll
          for (int k = 0; k < KB; ++k) {
            const int j = jt + k, off = j < n ? koff[j] : -2;
            if (off >= 0) load8(pool + kbase[j] + (size_t)(kvh * hd + off * tok) * l.dimp + c, kv[k]);
            else if (off == -1) load8(kn + kvh * l.dimp + c, kv[k]);
            else
#pragma unroll
              for (int e = 0; e < 8; ++e) kv[k][e] = 0.f;
          }
#pragma unroll
          for (int r = 0; r < RB; ++r) {
            if (r < nb) {
              float qv[8];
              load8(qs + (size_t)(hb + r) * l.dimp + c, qv);
#pragma unroll
              for (int k = 0; k < KB; ++k)
#pragma unroll
                for (int e = 0; e < 8; ++e) dot[r * KB + k] = fmaf(qv[e], kv[k][e], dot[r * KB + k]);
            }
          }
        }
        // sums over the eight lanes; every lane ends with two of them
#pragma unroll
        for (int o = 4, width = RB * KB / 2; o > 0; o >>= 1, width >>= 1) {
          const bool up = l8 & o;
#pragma unroll
          for (int i = 0; i < RB * KB / 2; ++i)
            if (i < width) {
              const float send = up ? dot[i] : dot[i + width], keep = up ? dot[i + width] : dot[i];
              dot[i] = keep + __shfl_xor_sync(ALL_LANES, send, o);
            }
        }
        const int r = l8 >> 1, k = (l8 & 1) * 2;
        if (r < nb) {
#pragma unroll
          for (int e = 0; e < 2; ++e)
            if (jt + k + e < n) raw[(size_t)(hb + r) * KC + jt + k + e] = dot[e] * l.scale;
        }
        hb += nb;
      }
    }
    __syncthreads();
    if (l.mix) {
      const int quads = (nh + 3) / 4;
      for (int i = tid; i < quads * n; i += THREADS) {
        const int j = i % n, h = i / n * 4;
        const float* t[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) t[r] = l.mix + (size_t)(h0 + min(h + r, nh - 1)) * H;
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        for (int g = 0; g < H; ++g) {
          const float x = raw[(size_t)g * KC + j];
#pragma unroll
          for (int r = 0; r < 4; ++r) s[r] = fmaf(__ldg(t[r] + g), x, s[r]);
        }
#pragma unroll
        for (int r = 0; r < 4; ++r)
          if (h + r < nh) pr[(size_t)(h + r) * KC + j] = s[r];
      }
      __syncthreads();
    }
    for (int h = warp; h < nh; h += WARPS) {  // running maximum, probabilities, sum
      float mx = -FLT_MAX;
      for (int j = lane; j < n; j += 32) mx = fmaxf(mx, pr[(size_t)h * KC + j]);
      const float m_old = m_run[h], m_new = fmaxf(m_old, lane_max(mx));
      float sum = 0.f;
      for (int j = lane; j < n; j += 32) {
        const float e = expf(pr[(size_t)h * KC + j] - m_new);
        pr[(size_t)h * KC + j] = e;
        sum += e;
      }
      sum = lane_sum(sum);
      __syncwarp();
      if (lane == 0) {
        const float c = expf(m_old - m_new);
        m_run[h] = m_new;
        l_run[h] = l_run[h] * c + sum;
        corr[h] = c;
      }
    }
    __syncthreads();
    auto value = [&](int j, int kvh, int vc, float (&v)[8]) {
      if (koff[j] < 0) load8(vn + kvh * l.vdimp + vc * 8, v);
      else load8(pool + kbase[j] + v_at + (size_t)(kvh * hd + koff[j] * tok) * vpitch + vc * 8, v);
    };
    if (one_v) {
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int c = tid + i * THREADS;
        const float f = c < chunks ? corr[c / nvec] : 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[i][e] *= f;
      }
      const int vc = tid % nvec, hs = tid / nvec, hstep = THREADS / nvec;
#pragma unroll 4
      for (int j = 0; j < n; ++j) {
        float v[8];
        value(j, 0, vc, v);
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const int h = hs + i * hstep;
          const float w = h < nh ? pr[(size_t)h * KC + j] : 0.f;
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[i][e] = fmaf(w, v[e], acc[i][e]);
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < NC; ++i) {
        const int c = KG > 1 ? tid % chunks : tid + i * THREADS;
        if (c >= chunks || kg >= KG) continue;
        const int h = c / nvec, vc = c % nvec, kvh = (h0 + h) / rep;
        const float f = corr[h];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[i][e] *= f;
#pragma unroll 4
        for (int j = kg; j < n; j += KG) {
          float v[8];
          value(j, kvh, vc, v);
          const float w = pr[(size_t)h * KC + j];
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[i][e] = fmaf(w, v[e], acc[i][e]);
        }
      }
    }
    __syncthreads();
  }
  // outputs of this part, the key subsets added
  if (KG > 1) {
    if (kg < KG)
#pragma unroll
      for (int e = 0; e < 8; ++e) os[(size_t)tid * 8 + e] = acc[0][e];  // [kg][chunk][8]
    __syncthreads();
    float v[8];
    if (tid < chunks) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = 0.f;
      for (int g = 0; g < KG; ++g)
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] += os[((size_t)g * chunks + tid) * 8 + e];
    }
    __syncthreads();
    if (tid < chunks)
#pragma unroll
      for (int e = 0; e < 8; ++e) os[(size_t)tid * 8 + e] = v[e];
  } else {
#pragma unroll
    for (int i = 0; i < NC; ++i) {
      const int c = tid + i * THREADS;
      if (c < chunks)
#pragma unroll
        for (int e = 0; e < 8; ++e) os[(size_t)c * 8 + e] = acc[i][e];
    }
  }
  __syncthreads();
  if (a.splits > 1) {
    const int vd2 = 4 + ((l.vdim + 3) & ~3);
    for (int i = tid; i < nh * l.vdim; i += THREADS) {
      const int h = i / l.vdim, c = i % l.vdim;
      float* pt = a.part + (((size_t)seq * H + h0 + h) * a.splits + split) * vd2;
      pt[4 + c] = os[(size_t)h * l.vdimp + c];
      if (c == 0) {
        pt[0] = m_run[h];
        pt[1] = l_run[h];
      }
    }
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      unsigned* counter = a.counters + (size_t)seq * gridDim.z + group;
      last_flag = atomicAdd(counter, 1u) == (unsigned)a.splits - 1;
      if (last_flag) *counter = 0;
    }
    __syncthreads();
    if (!last_flag) return;
    __threadfence();
    // weights of the parts: [nh][splits] in the space of the scores
    for (int h = tid; h < nh; h += THREADS) {
      const volatile float* pt = a.part + ((size_t)seq * H + h0 + h) * a.splits * vd2;
      float m = -FLT_MAX, den = 0.f;
      for (int s = 0; s < a.splits; ++s) m = fmaxf(m, pt[s * vd2]);
      for (int s = 0; s < a.splits; ++s) {
        const float w = expf(pt[s * vd2] - m);
        raw[h * a.splits + s] = w;
        den += w * pt[s * vd2 + 1];
      }
      m_run[h] = m;
      l_run[h] = den;
    }
    __syncthreads();
    for (int i = tid; i < nh * l.vdim; i += THREADS) {
      const int h = i / l.vdim, c = i % l.vdim;
      const volatile float* pt = a.part + ((size_t)seq * H + h0 + h) * a.splits * vd2 + 4 + c;
      float v = 0.f;
      for (int s = 0; s < a.splits; ++s) v = fmaf(raw[h * a.splits + s], pt[s * vd2], v);
      os[(size_t)h * l.vdimp + c] = v;
    }
    __syncthreads();
  }
  for (int h = tid; h < nh; h += THREADS) {
    float f = 1.f, den = l_run[h];
    if (l.sink) {  // the sink's share of the denominator; m may have to move up to it
      const float sink = l.sink[h0 + h], m = fmaxf(m_run[h], sink);
      f = expf(m_run[h] - m);
      den = den * f + expf(sink - m);
    }
    f *= l.out_scale / den;
    if (l.off_gate >= 0) f *= sigmoid_f(p[l.off_gate + h0 + h]);
    corr[h] = f;
  }
  __syncthreads();
  for (int i = tid; i < nh * l.vdim; i += THREADS) {
    const int h = i / l.vdim, c = i % l.vdim;
    const float* o = os + (size_t)h * l.vdimp;
    float y = o[c];
    if (l.v_rot) {
      const int half = l.vdim >> 1;
      y = c < half ? o[c] * vcs[c].x + o[c + half] * vcs[c].y : o[c] * vcs[c - half].x - o[c - half] * vcs[c - half].y;
    }
    y *= corr[h];
    const size_t at = (size_t)seq * a.ldy + (size_t)(h0 + h) * a.ldyh + c;
    if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[at] = __float2bfloat16_rn(y);
    else static_cast<float*>(a.y)[at] = y;
  }
}

// Shared memory of a block of hn heads with passes of `keys` keys.
size_t heads_smem(const AttentionLayer& l, int hn, int keys) {
  const size_t raw = l.mix ? l.heads : hn;
  size_t f = raw * l.dimp + (size_t)l.kv_heads * l.dimp + (l.vrow ? (size_t)l.kv_heads * l.vdimp : 0) + raw * std::max(keys, 16) +
             (l.mix ? (size_t)hn * keys : 0) + 3 * (size_t)hn + 1;
  f += l.rot_dims + (l.v_rot ? l.vdim : 0) + 3 * (size_t)keys;
  f += std::max(hn * l.vdimp, 8 * THREADS) + 33;
  return f * sizeof(float) + 16;
}
bool step_shape(const AttentionLayer& l, StepShape* sh) {
  const int nvec = l.vdimp / 8;
  // the fewest blocks over the heads that keep a block's outputs in registers
  for (int groups = 1; groups <= l.heads; ++groups) {
    const int hn = (l.heads + groups - 1) / groups;
    if (hn * nvec > 8 * THREADS) continue;
    for (int keys = 128; keys >= 16; keys /= 2) {
      const size_t smem = heads_smem(l, hn, keys);
      if (smem > MAX_SMEM) continue;
      *sh = StepShape{hn, (l.heads + hn - 1) / hn, l.mix ? l.heads : hn, keys, smem};
      return true;
    }
  }
  return false;
}

// ------------------------------------------------------------------ portions
// Where a row's key or value of one head goes: the workspace, or (a step) the page of its position.
template <typename T>
__device__ __forceinline__ T* key_target(const AttentionPortionArgs& a, int row, int head, int which) {
  const AttentionLayer& l = a.l;
  if (a.step_pos)
    return page_row(l, static_cast<T*>(a.pool), a.page_table + (size_t)row * l.pages_per_seq, l.life.place(a.step_pos[row]), head, which);
  const int seq = a.row_seq[row];
  const size_t krow = (size_t)a.key_start[seq] + l.life.context(a.seq_pos[seq]) + (row - a.seq_start[seq]);
  return which == 0 ? static_cast<T*>(a.k) + krow * a.ldk + head * l.dimp : static_cast<T*>(a.v) + krow * a.ldv + head * l.vdimp;
}

// Block = up to `rows` rows and one key head with the query heads that read it: biases, rotation. With mixed heads, piece c of
// head h's query (the part against key head c) = sum over the heads g that read key head c of mix[h][g] q_g. UNROLL rows are
// requested together; what depends on the column only is worked out once per block.
constexpr int ROT_THREADS = 256, ROT_MAX_ROWS = 32;
template <typename T, int UNROLL>
__global__ void __launch_bounds__(ROT_THREADS, 4) attention_rotate_kernel(AttentionPortionArgs a, int rows, int mix_staged) {
  extern __shared__ __align__(16) float sm[];  // [rows][rep][dimp] queries, [heads][rep] mixing
  __shared__ T* target[2 * ROT_MAX_ROWS];      // where the rows' key and value go
  const AttentionLayer& l = a.l;
  const int row0 = blockIdx.y * rows, c = blockIdx.x, nrows = min(rows, a.rows - row0), tid = threadIdx.x, H = l.heads, G = l.kv_heads, rep = H / G;
  const int qn = rep * l.dimp, per = qn + l.dimp + l.vdimp;
  float* qs = sm;
  const float* mix = mix_staged ? qs + (size_t)rows * qn : l.mix + c * rep;
  const int mix_row = mix_staged ? rep : H;
  grid_dep_launch();
  if (l.mix && mix_staged)
    for (int i = tid; i < H * rep; i += ROT_THREADS) qs[(size_t)rows * qn + i] = l.mix[(size_t)(i / rep) * H + c * rep + i % rep];
  grid_dep_wait();
  if (tid < 2 * nrows) target[tid] = key_target<T>(a, row0 + tid / 2, c, tid & 1);
  __syncthreads();
  for (int e = tid; e < per; e += ROT_THREADS) {  // a column of the block's rows
    const bool is_q = e < qn, is_k = !is_q && e < qn + l.dimp;
    const int x = is_q ? e : is_k ? e - qn : e - qn - l.dimp, np = is_q || is_k ? l.dimp : l.vdimp, n = is_q || is_k ? l.dim : l.vdim;
    const int head = is_q ? c * rep + x / np : c, col = x % np, dims = is_q || is_k ? l.rot_dims : l.v_rot ? l.vdim : 0;
    const float* bias = is_q ? l.q_bias : is_k ? l.k_bias : l.v_bias;
    // entry `col` = x cos + partner * (-sin or sin); past the rotated entries the factors are 1 and 0
    const int half = dims >> 1, turn = col < half ? col : col - half;
    const bool on = col < n, turned = on && col < dims;
    const int partner = turned ? (col < half ? col + half : col - half) : col;
    const float sign = !turned ? 0.f : col < half ? -1.f : 1.f;
    const float* src = a.p + (size_t)row0 * a.ldp + (is_q ? l.off_q : is_k ? l.off_k : l.off_v) + head * n;
    const float2* cs = turned ? (is_q || is_k ? a.rot : a.v_rot) + (size_t)row0 * half + turn : nullptr;
    const float b0 = bias && on ? bias[head * n + col] : 0.f, b1 = bias && on ? bias[head * n + partner] : 0.f;
    T* q16 = static_cast<T*>(a.q) + ((size_t)row0 * H + head) * l.dimp + col;
    for (int r0 = 0; r0 < nrows; r0 += UNROLL) {
      float u[UNROLL], v[UNROLL];
      float2 f[UNROLL];
#pragma unroll
      for (int i = 0; i < UNROLL; ++i) {
        const int r = min(r0 + i, nrows - 1);
        const float* p = src + (size_t)r * a.ldp;
        u[i] = on ? p[col] + b0 : 0.f;
        v[i] = on ? p[partner] + b1 : 0.f;
        f[i] = turned ? cs[(size_t)r * half] : make_float2(1.f, 0.f);
      }
#pragma unroll
      for (int i = 0; i < UNROLL; ++i) {
        const int r = r0 + i;
        if (r >= nrows) break;
        const float y = u[i] * f[i].x + sign * (v[i] * f[i].y);
        if (!is_q) target[2 * r + (is_k ? 0 : 1)][col] = from_f32<T>(y);
        else if (l.mix) qs[r * qn + x] = y;
        else q16[(size_t)r * H * l.dimp] = from_f32<T>(y);
      }
    }
  }
  if (!l.mix) return;
  __syncthreads();
  // thread = four columns of up to HPT heads at a time, whose mixing weights stay in registers over the rows
  constexpr int HPT = 2, MAX_REP = 8;
  const int nq = l.dimp / 4, lanes = nq < ROT_THREADS ? nq : ROT_THREADS, nhb = ROT_THREADS / lanes, hb = tid / lanes;
  if (hb >= nhb) return;
  for (int o = tid % lanes; o < nq; o += lanes)
    for (int h0 = hb; h0 < H; h0 += nhb * HPT) {
      float t[HPT][MAX_REP];
#pragma unroll
      for (int i = 0; i < HPT; ++i)
#pragma unroll
        for (int g = 0; g < MAX_REP; ++g) t[i][g] = g < rep && h0 + i * nhb < H ? mix[(size_t)(h0 + i * nhb) * mix_row + g] : 0.f;
      T* out = static_cast<T*>(a.q) + (((size_t)row0 * H + h0) * G + c) * l.dimp + o * 4;
      const size_t out_row = (size_t)H * G * l.dimp, out_head = (size_t)nhb * G * l.dimp;
      const float* q = qs + o * 4;
      for (int rr = 0; rr < nrows; ++rr, q += qn, out += out_row) {
        float4 acc[HPT];
#pragma unroll
        for (int i = 0; i < HPT; ++i) acc[i] = make_float4(0, 0, 0, 0);
        auto add = [&](float4& v, float f, const float4& x) {
          v.x = fmaf(f, x.x, v.x); v.y = fmaf(f, x.y, v.y); v.z = fmaf(f, x.z, v.z); v.w = fmaf(f, x.w, v.w);
        };
#pragma unroll
        for (int g = 0; g < MAX_REP; ++g)
          if (g < rep) {
            const float4 x = load4(q + g * l.dimp);
#pragma unroll
            for (int i = 0; i < HPT; ++i) add(acc[i], t[i][g], x);
          }
        for (int g = MAX_REP; g < rep; ++g) {
          const float4 x = load4(q + g * l.dimp);
#pragma unroll
          for (int i = 0; i < HPT; ++i)
            if (h0 + i * nhb < H) add(acc[i], mix[(size_t)(h0 + i * nhb) * mix_row + g], x);
        }
#pragma unroll
        for (int i = 0; i < HPT; ++i)
          if (h0 + i * nhb < H) store4(out + i * out_head, acc[i]);
      }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) attention_latent_kernel(AttentionPortionArgs a) {
  const AttentionLayer& l = a.l;
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  grid_dep_launch();
  grid_dep_wait();
  if (row >= a.rows) return;
  T* dst = key_target<T>(a, row, 0, 0);
  const float* p = a.p + (size_t)row * a.ldp + l.off_k;
  float4 x[8];  // at most 1024 columns; dimp and the weight are padded, the row is not
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = (i * 32 + lane) * 4;
    x[i] = make_float4(0, 0, 0, 0);
    if (c < l.dim) {
      x[i] = load4(p + c);
      if (c + 1 >= l.dim) x[i].y = 0.f;
      if (c + 2 >= l.dim) x[i].z = 0.f;
      if (c + 3 >= l.dim) x[i].w = 0.f;
    }
    s += (x[i].x * x[i].x + x[i].y * x[i].y) + (x[i].z * x[i].z + x[i].w * x[i].w);
  }
  const float inv = 1.f / sqrtf(lane_sum(s) / (float)l.dim + l.eps);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int c = (i * 32 + lane) * 4;
    if (c < l.dimp) {
      const float4 g = load4(l.k_norm + c);
      store4(dst + c, make_float4(x[i].x * inv * g.x, x[i].y * inv * g.y, x[i].z * inv * g.z, x[i].w * inv * g.w));
    }
  }
}

// Block = one head of one sequence. Parts hold maxima and sums in powers of two.
constexpr int MERGE_THREADS = 256;
__global__ void __launch_bounds__(MERGE_THREADS) attention_merge_kernel(AttentionStepArgs a, const float2* v_rot, int y_bf16) {
  __shared__ float w[64];
  const AttentionLayer& l = a.l;
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, pitch = 4 + ((l.vdim + 3) & ~3), half = l.vdim >> 1;
  constexpr float LOG2E = 1.4426950408889634f;
  grid_dep_launch();
  grid_dep_wait();
  const float* pt = a.part + ((size_t)seq * l.heads + h) * a.splits * pitch;
  if (tid < 32) {  // at most 32 parts
    const float sum = tid < a.splits ? pt[tid * pitch + 1] : 0.f, m = sum > 0.f ? pt[tid * pitch] : -1e30f;
    const float sink = l.sink ? l.sink[h] * LOG2E : -1e30f, top = fmaxf(lane_max(m), sink);
    const float f = sum > 0.f ? exp2f(m - top) : 0.f;
    const float den = lane_sum(f * sum) + (l.sink ? exp2f(sink - top) : 0.f);
    float scale = l.out_scale / den;
    if (l.off_gate >= 0) scale *= sigmoid_f(a.p[(size_t)seq * a.ldp + l.off_gate + h]);
    w[tid] = f * scale;
  }
  __syncthreads();
  auto sum = [&](int c) {
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < a.splits; ++s) {
      const float x = pt[s * pitch + 4 + c];  // an empty part holds no numbers
      v = w[s] != 0.f ? fmaf(w[s], x, v) : v;
    }
    return v;
  };
  auto put = [&](int c, float v) {
    const size_t at = (size_t)seq * a.ldy + (size_t)h * a.ldyh + c;
    if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[at] = __float2bfloat16_rn(v);
    else static_cast<float*>(a.y)[at] = v;
  };
  if (l.v_rot) {
    for (int c = tid; c < half; c += MERGE_THREADS) {
      const float2 r = v_rot[(size_t)seq * half + c];
      const float u = sum(c), v = sum(c + half);
      put(c, u * r.x + v * r.y);
      put(c + half, v * r.x - u * r.y);
    }
  } else {
    for (int c = tid; c < l.vdim; c += MERGE_THREADS) put(c, sum(c));
    for (int c = l.vdim + tid; c < a.ldyh; c += MERGE_THREADS) put(c, 0.f);
  }
}

__global__ void __launch_bounds__(256) attention_turn_back_kernel(AttentionPortionArgs a) {
  const AttentionLayer& l = a.l;
  const int half = l.vdim >> 1, row = blockIdx.x;
  const float2* cs = a.v_rot + (size_t)row * half;
  for (int i = threadIdx.x; i < l.heads * half; i += blockDim.x) {
    const int h = i / half, c = i % half;
    float* y = static_cast<float*>(a.y) + (size_t)row * a.ldy + h * l.vdim + c;
    const float u = y[0], v = y[half];
    y[0] = u * cs[c].x + v * cs[c].y;
    y[half] = v * cs[c].x - u * cs[c].y;
  }
}

// ------------------------------------------------------------------ products per head
// Block = 64 columns of one head for up to MB rows: lane = (eight columns, one of four subsets of k), warps take further
// subsets; the sums meet by shuffles and through shared memory. The first weights are requested before the dependency wait.
constexpr int HP_PRE = 4;
template <typename T>
struct Row8 {  // eight weights as they lie
  uint4 u[sizeof(T) / 2];
  __device__ __forceinline__ void load(const T* p) {
#pragma unroll
    for (int i = 0; i < (int)sizeof(T) / 2; ++i) u[i] = __ldg(reinterpret_cast<const uint4*>(p) + i);
  }
  __device__ __forceinline__ void get(float (&v)[8]) const { load8(reinterpret_cast<const T*>(u), v); }
};
template <typename T, int MB>
__global__ void __launch_bounds__(THREADS) head_product_kernel(HeadProductArgs a, int out_bf16) {
  extern __shared__ __align__(16) float sm[];  // [k][MB] inputs, then [WARPS][MB][64] sums
  const int n0 = blockIdx.x * 64, h = blockIdx.y, b0 = blockIdx.z * MB, nb = min(MB, a.batch - b0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int col = n0 + (lane & 7) * 8, ks = warp * 4 + (lane >> 3), kstep = 4 * WARPS;
  float* xs = sm;
  float* part = sm + (size_t)MB * a.k;
  const T* w = static_cast<const T*>(a.w) + (size_t)h * a.k * a.np + col;
  const bool on = col < a.np;
  grid_dep_launch();
  Row8<T> pre[HP_PRE];
#pragma unroll
  for (int i = 0; i < HP_PRE; ++i)
    if (on && ks + i * kstep < a.k) pre[i].load(w + (size_t)(ks + i * kstep) * a.np);
  grid_dep_wait();
  for (int i = tid; i < MB * a.k; i += THREADS) {
    const int b = i / a.k, k = i % a.k;
    xs[k * MB + b] = b < nb ? a.x[(size_t)(b0 + b) * a.ldx + (size_t)h * a.ldxh + k] : 0.f;
  }
  __syncthreads();
  float acc[MB][8];
#pragma unroll
  for (int b = 0; b < MB; ++b)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[b][e] = 0.f;
  if (on) {
    for (int k0 = ks; k0 < a.k; k0 += HP_PRE * kstep) {
      Row8<T> cur[HP_PRE];
#pragma unroll
      for (int i = 0; i < HP_PRE; ++i) {
        cur[i] = pre[i];
        const int next = k0 + (HP_PRE + i) * kstep;
        if (next < a.k) pre[i].load(w + (size_t)next * a.np);
      }
#pragma unroll
      for (int i = 0; i < HP_PRE; ++i) {
        const int k = k0 + i * kstep;
        if (k < a.k) {
          float v[8], x[MB];
          cur[i].get(v);
          if (MB % 4 == 0) {
#pragma unroll
            for (int b = 0; b < MB; b += 4) {
              const float4 f = load4(xs + k * MB + b);
              x[b] = f.x; x[(b + 1) % MB] = f.y; x[(b + 2) % MB] = f.z; x[(b + 3) % MB] = f.w;
            }
          } else {
#pragma unroll
            for (int b = 0; b < MB; ++b) x[b] = xs[k * MB + b];
          }
#pragma unroll
          for (int b = 0; b < MB; ++b)
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[b][e] = fmaf(x[b], v[e], acc[b][e]);
        }
      }
    }
  }
#pragma unroll
  for (int b = 0; b < MB; ++b)
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      acc[b][e] += __shfl_xor_sync(ALL_LANES, acc[b][e], 8);
      acc[b][e] += __shfl_xor_sync(ALL_LANES, acc[b][e], 16);
      if (lane < 8) part[((size_t)warp * MB + b) * 64 + lane * 8 + e] = acc[b][e];
    }
  __syncthreads();
  for (int i = tid; i < nb * 64; i += THREADS) {
    const int b = i / 64, c = i % 64;
    if (n0 + c >= a.n) continue;
    float v = 0.f;
    for (int q = 0; q < WARPS; ++q) v += part[((size_t)q * MB + b) * 64 + c];
    const size_t at = (size_t)(b0 + b) * a.ldo + (size_t)h * a.ldh + n0 + c;
    if (out_bf16) static_cast<__nv_bfloat16*>(a.out)[at] = __float2bfloat16_rn(v);
    else static_cast<float*>(a.out)[at] = v;
  }
}

template <typename T>
cudaError_t heads_step_t(const AttentionStepArgs& a, const StepShape& sh, int yb, bool pdl, cudaStream_t s) {
  const dim3 grid(a.splits, a.batch, sh.groups);
  const int nc = (sh.hn * (a.l.vdimp / 8) + THREADS - 1) / THREADS;
  cudaError_t e;
#define PG_STEP(NC_)                                                                                                                 \
  do {                                                                                                                               \
    e = cudaFuncSetAttribute(attention_heads_step_kernel<T, NC_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);       \
    return e != cudaSuccess ? e : launch_kernel(attention_heads_step_kernel<T, NC_>, grid, dim3(THREADS), sh.smem, s, pdl, a, sh, yb); \
  } while (0)
  if (nc <= 1) PG_STEP(1);
  if (nc <= 2) PG_STEP(2);
  if (nc <= 4) PG_STEP(4);
  PG_STEP(8);
#undef PG_STEP
}

}  // namespace

bool mix_staged(const AttentionLayer& l) { return l.mix && (size_t)l.heads * (l.heads / l.kv_heads) <= 16384; }
size_t rotate_smem(const AttentionLayer& l, int rows) {
  const int rep = l.heads / l.kv_heads;
  return l.mix ? ((size_t)rows * rep * l.dimp + (mix_staged(l) ? (size_t)l.heads * rep : 0)) * sizeof(float) : 0;
}

bool attention_heads_supported(const AttentionLayer& l) {
  StepShape sh;
  return step_shape(l, &sh) && rotate_smem(l, 1) <= MAX_SMEM;
}

cudaError_t launch_attention_heads_step(const AttentionStepArgs& a, bool bf16, bool y_bf16, bool pdl, cudaStream_t s) {
  StepShape sh;
  if (!step_shape(a.l, &sh)) return cudaErrorInvalidValue;
  return bf16 ? heads_step_t<__nv_bfloat16>(a, sh, y_bf16 ? 1 : 0, pdl, s) : heads_step_t<float>(a, sh, y_bf16 ? 1 : 0, pdl, s);
}

cudaError_t launch_angles(const int* pos, const double* freq, float2* out, int rows, int half, bool pdl, cudaStream_t s) {
  if (rows <= 0 || half <= 0) return cudaSuccess;
  const size_t blocks = ((size_t)rows * half + 255) / 256;
  return launch_kernel(angles_kernel, dim3((unsigned)std::min<size_t>(blocks, 148 * 16)), dim3(256), 0, s, pdl, pos, freq, out, rows, half);
}

cudaError_t launch_attention_rotate(const AttentionPortionArgs& a, bool bf16, cudaStream_t s, bool pdl) {
  int rows = a.step_pos ? 1 : ROT_MAX_ROWS;
  while (rows > 1 && rotate_smem(a.l, rows) > 48 * 1024) rows /= 2;
  const size_t smem = rotate_smem(a.l, rows);
  if (smem > MAX_SMEM) return cudaErrorInvalidValue;
  const dim3 grid(a.l.kv_heads, (a.rows + rows - 1) / rows);  // blocks of the same rows together: their queries are neighbours
  auto run = [&](auto kernel) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);
    return e != cudaSuccess ? e : launch_kernel(kernel, grid, dim3(ROT_THREADS), smem, s, pdl, a, rows, mix_staged(a.l) ? 1 : 0);
  };
  if (a.step_pos) return bf16 ? run(attention_rotate_kernel<__nv_bfloat16, 1>) : run(attention_rotate_kernel<float, 1>);
  return bf16 ? run(attention_rotate_kernel<__nv_bfloat16, 4>) : run(attention_rotate_kernel<float, 4>);
}

cudaError_t launch_attention_latent(const AttentionPortionArgs& a, bool bf16, cudaStream_t s, bool pdl) {
  const dim3 grid((a.rows + 7) / 8);
  return bf16 ? launch_kernel(attention_latent_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl, a)
              : launch_kernel(attention_latent_kernel<float>, grid, dim3(256), 0, s, pdl, a);
}

cudaError_t launch_attention_merge(const AttentionStepArgs& a, const float2* v_rot, bool y_bf16, bool pdl, cudaStream_t s) {
  if (a.splits > 32) return cudaErrorInvalidValue;
  return launch_kernel(attention_merge_kernel, dim3(a.l.heads, a.batch), dim3(MERGE_THREADS), 0, s, pdl, a, v_rot, y_bf16 ? 1 : 0);
}

cudaError_t launch_attention_turn_back(const AttentionPortionArgs& a, cudaStream_t s) {
  return launch_kernel(attention_turn_back_kernel, dim3(a.rows), dim3(256), 0, s, false, a);
}

template <typename T, int MB>
static cudaError_t head_product_mb(const HeadProductArgs& a, bool out_bf16, bool pdl, cudaStream_t s) {
  const size_t smem = ((size_t)MB * a.k + (size_t)WARPS * MB * 64) * sizeof(float);
  if (smem > MAX_SMEM || a.np % 8 != 0) return cudaErrorInvalidValue;
  const dim3 grid((a.n + 63) / 64, a.heads, (a.batch + MB - 1) / MB);
  cudaError_t e = cudaFuncSetAttribute(head_product_kernel<T, MB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);
  return e != cudaSuccess ? e : launch_kernel(head_product_kernel<T, MB>, grid, dim3(THREADS), smem, s, pdl, a, out_bf16 ? 1 : 0);
}

cudaError_t launch_head_product(const HeadProductArgs& a, bool bf16, bool out_bf16, bool pdl, cudaStream_t s) {
  if (bf16) {
    if (a.batch <= 1) return head_product_mb<__nv_bfloat16, 1>(a, out_bf16, pdl, s);
    if (a.batch <= 4) return head_product_mb<__nv_bfloat16, 4>(a, out_bf16, pdl, s);
    return head_product_mb<__nv_bfloat16, 8>(a, out_bf16, pdl, s);
  }
  return a.batch <= 1 ? head_product_mb<float, 1>(a, out_bf16, pdl, s) : head_product_mb<float, 8>(a, out_bf16, pdl, s);
}

}  // namespace pg
