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
            if (off >= 0) load8(pool + kbase[j] + (size_t)(kvh * l.page_tokens + off) * l.dimp + c, kv[k]);
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
      else load8(pool + kbase[j] + v_at + (size_t)(kvh * l.page_tokens + koff[j]) * vpitch + vc * 8, v);
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
    const int vd2 = l.vdim + 2;
    for (int i = tid; i < nh * l.vdim; i += THREADS) {
      const int h = i / l.vdim, c = i % l.vdim;
      float* pt = a.part + (((size_t)seq * H + h0 + h) * a.splits + split) * vd2;
      pt[2 + c] = os[(size_t)h * l.vdimp + c];
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
      const volatile float* pt = a.part + ((size_t)seq * H + h0 + h) * a.splits * vd2 + 2 + c;
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
    const size_t at = (size_t)seq * a.ldy + (size_t)(h0 + h) * l.vdim + c;
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
// Block = row. Queries with their bias, rotated; with mixed heads head h's query against the row of all key heads:
// piece c of it = sum over the heads g that read key head c of mix[h][g] q_g.
template <typename T>
__global__ void __launch_bounds__(256) attention_rotate_kernel(AttentionPortionArgs a, int mix_in_smem) {
  extern __shared__ __align__(16) float sm[];  // [heads][dimp] queries, [heads][heads] mixing
  const AttentionLayer& l = a.l;
  const int row = blockIdx.x, tid = threadIdx.x, H = l.heads, G = l.kv_heads, rep = H / G;
  const float* p = a.p + (size_t)row * a.ldp;
  const int seq = a.row_seq[row];
  const size_t krow = (size_t)a.key_start[seq] + l.life.context(a.seq_pos[seq]) + (row - a.seq_start[seq]);
  const float2* kcs = a.rot + (size_t)row * (l.rot_dims >> 1);
  const float2* vcs = a.v_rot + (size_t)row * (l.vdim >> 1);
  auto entry = [&](int off, const float* bias, int h, int n, int c, int dims, const float2* cs) {
    const float *x = p + off + h * n, *b = bias ? bias + h * n : nullptr;
    return c < n ? rotated([=](int e) { return x[e] + (b ? b[e] : 0.f); }, c, dims, cs) : 0.f;
  };
  for (int i = tid; i < G * l.dimp; i += 256)
    static_cast<T*>(a.k)[krow * a.ldk + i] = from_f32<T>(entry(l.off_k, l.k_bias, i / l.dimp, l.dim, i % l.dimp, l.rot_dims, kcs));
  for (int i = tid; i < G * l.vdimp; i += 256)
    static_cast<T*>(a.v)[krow * a.ldv + i] = from_f32<T>(entry(l.off_v, l.v_bias, i / l.vdimp, l.vdim, i % l.vdimp, l.v_rot ? l.vdim : 0, vcs));
  if (!l.mix) {
    for (int i = tid; i < H * l.dimp; i += 256)
      static_cast<T*>(a.q)[(size_t)row * H * l.dimp + i] = from_f32<T>(entry(l.off_q, l.q_bias, i / l.dimp, l.dim, i % l.dimp, l.rot_dims, kcs));
    return;
  }
  float* qs = sm;
  for (int i = tid; i < H * l.dimp; i += 256) qs[i] = entry(l.off_q, l.q_bias, i / l.dimp, l.dim, i % l.dimp, l.rot_dims, kcs);
  const float* mix = l.mix;
  if (mix_in_smem) {
    float* t = qs + (size_t)H * l.dimp;
    for (int i = tid; i < H * H; i += 256) t[i] = l.mix[i];
    mix = t;
  }
  __syncthreads();
  const int width = G * l.dimp;
  T* out = static_cast<T*>(a.q) + (size_t)row * H * width;
  for (int i = tid; i < width; i += 256) {
    const int c = i / l.dimp, e = i % l.dimp;
    const float* q = qs + (size_t)c * rep * l.dimp + e;
    const float* t = mix + c * rep;
    if (rep <= 8) {
      float x[8];
#pragma unroll
      for (int g = 0; g < 8; ++g) x[g] = g < rep ? q[g * l.dimp] : 0.f;
      for (int h = 0; h < H; ++h) {
        float s = 0.f;
#pragma unroll
        for (int g = 0; g < 8; ++g)
          if (g < rep) s = fmaf(t[h * H + g], x[g], s);
        out[(size_t)h * width + i] = from_f32<T>(s);
      }
    } else {
      for (int h = 0; h < H; ++h) {
        float s = 0.f;
        for (int g = 0; g < rep; ++g) s = fmaf(t[h * H + g], q[g * l.dimp], s);
        out[(size_t)h * width + i] = from_f32<T>(s);
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) attention_latent_kernel(AttentionPortionArgs a) {
  const AttentionLayer& l = a.l;
  const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= a.rows) return;
  const int seq = a.row_seq[row];
  const size_t krow = (size_t)a.key_start[seq] + l.life.context(a.seq_pos[seq]) + (row - a.seq_start[seq]);
  const float* x = a.p + (size_t)row * a.ldp + l.off_k;
  float s = 0.f;
  for (int c = lane; c < l.dim; c += 32) s += x[c] * x[c];
  const float inv = 1.f / sqrtf(lane_sum(s) / (float)l.dim + l.eps);
  for (int c = lane; c < l.dimp; c += 32)
    static_cast<T*>(a.k)[krow * a.ldk + c] = from_f32<T>(c < l.dim ? x[c] * inv * l.k_norm[c] : 0.f);
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
// subsets; the sums meet by shuffles and through shared memory.
constexpr int MB = 8;
template <typename T>
__global__ void __launch_bounds__(THREADS) head_product_kernel(HeadProductArgs a, int out_bf16) {
  extern __shared__ __align__(16) float sm[];  // [MB][k] inputs, then [WARPS][MB][64] sums
  const int n0 = blockIdx.x * 64, h = blockIdx.y, b0 = blockIdx.z * MB, nb = min(MB, a.batch - b0), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int col = n0 + (lane & 7) * 8, ks = warp * 4 + (lane >> 3);
  float* xs = sm;
  float* part = sm + (size_t)MB * a.k;
  grid_dep_launch();
  grid_dep_wait();
  for (int i = tid; i < MB * a.k; i += THREADS) {
    const int b = i / a.k, k = i % a.k;
    xs[i] = b < nb ? a.x[(size_t)(b0 + b) * a.ldx + (size_t)h * a.ldxh + k] : 0.f;
  }
  __syncthreads();
  float acc[MB][8];
#pragma unroll
  for (int b = 0; b < MB; ++b)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[b][e] = 0.f;
  if (col < a.np) {
    const T* w = static_cast<const T*>(a.w) + (size_t)h * a.k * a.np + col;
#pragma unroll 4
    for (int k = ks; k < a.k; k += 4 * WARPS) {
      float v[8];
      load8(w + (size_t)k * a.np, v);
#pragma unroll
      for (int b = 0; b < MB; ++b) {
        if (b < nb) {
          const float x = xs[b * a.k + k];
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[b][e] = fmaf(x, v[e], acc[b][e]);
        }
      }
    }
  }
#pragma unroll
  for (int b = 0; b < MB; ++b)
    if (b < nb) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        acc[b][e] += __shfl_xor_sync(ALL_LANES, acc[b][e], 8);
        acc[b][e] += __shfl_xor_sync(ALL_LANES, acc[b][e], 16);
        if (lane < 8) part[((size_t)warp * MB + b) * 64 + lane * 8 + e] = acc[b][e];
      }
    }
  __syncthreads();
  for (int i = tid; i < nb * 64; i += THREADS) {
    const int b = i / 64, c = i % 64;
    if (n0 + c >= a.n) continue;
    float v = 0.f;
    for (int w = 0; w < WARPS; ++w) v += part[((size_t)w * MB + b) * 64 + c];
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

bool attention_heads_supported(const AttentionLayer& l) {
  StepShape sh;
  return step_shape(l, &sh) && (!l.mix || (size_t)l.heads * l.dimp * sizeof(float) <= MAX_SMEM);
}

cudaError_t launch_attention_heads_step(const AttentionStepArgs& a, bool bf16, bool y_bf16, bool pdl, cudaStream_t s) {
  StepShape sh;
  if (!step_shape(a.l, &sh)) return cudaErrorInvalidValue;
  return bf16 ? heads_step_t<__nv_bfloat16>(a, sh, y_bf16 ? 1 : 0, pdl, s) : heads_step_t<float>(a, sh, y_bf16 ? 1 : 0, pdl, s);
}

cudaError_t launch_angles(const int* pos, const double* freq, float2* out, int rows, int half, cudaStream_t s) {
  if (rows <= 0 || half <= 0) return cudaSuccess;
  const size_t blocks = ((size_t)rows * half + 255) / 256;
  return launch_kernel(angles_kernel, dim3((unsigned)std::min<size_t>(blocks, 148 * 16)), dim3(256), 0, s, false, pos, freq, out, rows, half);
}

cudaError_t launch_attention_rotate(const AttentionPortionArgs& a, bool bf16, cudaStream_t s) {
  const AttentionLayer& l = a.l;
  size_t smem = l.mix ? (size_t)l.heads * l.dimp * sizeof(float) : 0;
  const size_t with = smem + (size_t)l.heads * l.heads * sizeof(float);
  const int in_smem = l.mix && with <= 96 * 1024 ? 1 : 0;
  if (in_smem) smem = with;
  if (smem > MAX_SMEM) return cudaErrorInvalidValue;
  auto run = [&](auto kernel) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);
    return e != cudaSuccess ? e : launch_kernel(kernel, dim3(a.rows), dim3(256), smem, s, false, a, in_smem);
  };
  return bf16 ? run(attention_rotate_kernel<__nv_bfloat16>) : run(attention_rotate_kernel<float>);
}

cudaError_t launch_attention_latent(const AttentionPortionArgs& a, bool bf16, cudaStream_t s) {
  const dim3 grid((a.rows + 7) / 8);
  return bf16 ? launch_kernel(attention_latent_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, false, a)
              : launch_kernel(attention_latent_kernel<float>, grid, dim3(256), 0, s, false, a);
}

cudaError_t launch_attention_turn_back(const AttentionPortionArgs& a, cudaStream_t s) {
  return launch_kernel(attention_turn_back_kernel, dim3(a.rows), dim3(256), 0, s, false, a);
}

cudaError_t launch_head_product(const HeadProductArgs& a, bool bf16, bool out_bf16, bool pdl, cudaStream_t s) {
  const size_t smem = ((size_t)MB * a.k + (size_t)WARPS * MB * 64) * sizeof(float);
  if (smem > MAX_SMEM || a.np % 8 != 0) return cudaErrorInvalidValue;
  const dim3 grid((a.n + 63) / 64, a.heads, (a.batch + MB - 1) / MB);
  auto run = [&](auto kernel) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SMEM);
    return e != cudaSuccess ? e : launch_kernel(kernel, grid, dim3(THREADS), smem, s, pdl, a, out_bf16 ? 1 : 0);
  };
  return bf16 ? run(head_product_kernel<__nv_bfloat16>) : run(head_product_kernel<float>);
}

}  // namespace pg
