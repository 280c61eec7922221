// One new token per sequence through a recurrent mixer (gated linear attention, delta rules): the cached
// [dim, vdim] FP32 state of every head is read, advanced and written back, with the gates before it and the head norm and
// output gate after it in the same kernel. Everything that enters the recurrence is FP32.
#include <algorithm>

#include "recurrence.cuh"

namespace pg {
namespace {

// ------------------------------------------------------------------ one token per sequence
constexpr int STEP_THREADS = 256;

template <int NR>
__global__ void __launch_bounds__(STEP_THREADS) recurrence_step_kernel(RecurrenceStepArgs a, int y_bf16) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33];
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, dv = l.vdim, dvp = l.dvp, K = l.heads * dk;
  const int head = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const bool delta = l.kind == KIND_DELTA, channel = l.kind == KIND_CHANNEL, reads = delta || channel;
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
  float* zs = os + dvp;      // [max(256, dk)] partial sums of the decay projection
  float* part = zs + (dk > STEP_THREADS ? dka : STEP_THREADS);  // [KG][dvp]
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
  float kk = 0.f, beta = 0.f;
  if (channel) {
    const int rep = l.heads / l.kv_heads, kv = head / rep, pos = a.pos[seq], slot = pos % l.taps;
    float* taps = a.taps + (size_t)seq * l.taps * l.channels;
    const float* z = a.z + (size_t)seq * a.ldz + head * dk;
    // a convolved input; the current one is cached where no token that still matters lies
    auto conv = [&](int col, bool keep) {
      const int ch = col - l.off_q;
      float x = 0.f;
      for (int back = l.taps - 1; back >= 0; --back)
        x = fmaf(l.conv[(size_t)(l.taps - 1 - back) * l.channels + ch], conv_input(l, p, 0, taps, 0, 0, pos, back, ch), x);
      if (keep) taps[(size_t)slot * l.channels + ch] = p[col];
      return silu_f(x);
    };
    const bool first = head % rep == 0;  // one block per group caches the shared q and k
    float qq = 0.f;
    for (int c = tid; c < dk; c += STEP_THREADS) {
      ks[c] = conv(l.off_k + kv * dk + c, first);
      qs[c] = conv(l.off_q + kv * dk + c, first);
      ws[c] = channel_decay(l, head, head * dk + c, z[c]);
      kk += ks[c] * ks[c];
      qq += qs[c] * qs[c];
    }
    for (int c = tid; c < dvp; c += STEP_THREADS) vs[c] = c < dv ? conv(l.off_v + head * dv + c, true) : 0.f;
    beta = sigmoid_f(p[l.off_b + head]);
    const float ki = 1.f / sqrtf(block_sum(kk, red) + UNIT_EPS), qi = 1.f / sqrtf(block_sum(qq, red) + UNIT_EPS);
    for (int c = tid; c < dk; c += STEP_THREADS) {
      ks[c] *= ki;
      qs[c] *= qi;
      us[c] = ws[c] * ks[c];  // what the key reads of the decayed state
      bs[c] = 0.f;
    }
  } else {
    for (int r = tid; r < l.rank; r += STEP_THREADS) ts[r] = delta ? tanhf(p[l.off_t + r]) : p[l.off_t + r];
    for (int c = tid; c < dk; c += STEP_THREADS) {
      ks[c] = p[l.off_k + head * dk + c];
      qs[c] = p[l.off_q + head * dk + c];
      kk += ks[c] * ks[c];
    }
    for (int c = tid; c < dvp; c += STEP_THREADS) vs[c] = c < dv ? p[l.off_v + head * dv + c] : 0.f;
    kk = block_sum(kk, red);  // also orders the shared-memory writes above
    const float inv_norm = 1.f / sqrtf(kk + UNIT_EPS);
    // second half of the decay projection: RG threads share a channel, so that its weights arrive in one round trip or two
    const int RG = dk >= STEP_THREADS ? 1 : STEP_THREADS / dk;
    for (int i = tid; i < RG * dk; i += STEP_THREADS) {
      const int c = i % dk, g = i / dk;
      const float* __restrict__ w2 = l.w2 + head * dk + c;
      float z = 0.f;
  #pragma unroll 16
      for (int r = g; r < l.rank; r += RG) z = fmaf(w2[(size_t)r * K], ts[r], z);
      zs[i] = z;
    }
    __syncthreads();
    for (int c = tid; c < dk; c += STEP_THREADS) {
      const int ch = head * dk + c;
      float z = l.b2[ch];
      for (int g = 0; g < RG; ++g) z += zs[g * dk + c];
      ws[c] = decay_of(l.kind, z, l.inv_tau);
      if (delta) {
        const float u = ks[c] * inv_norm;
        us[c] = u;
        bs[c] = sigmoid_f(p[l.off_a + ch] + l.a_bias[ch]) * u;
      }
    }
  }
  __syncthreads();
  if (reads) {
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
      if (channel) vs[c] = beta * (vs[c] - s);  // what is written; ds goes unused
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
    const float g = channel ? a.z[(size_t)seq * a.ldz + l.heads * dk + head * dv + c] : p[l.off_g + head * dv + c];
    const float gate = reads ? sigmoid_f(g) : silu_f(g);
    const float y = os[c] * rinv * l.norm[delta ? head * dv + c : c] * gate * l.out_scale;
    const size_t i = (size_t)seq * a.ldy + head * dv + c;
    if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[i] = __float2bfloat16_rn(y);
    else static_cast<float*>(a.y)[i] = y;
  }
}

}  // namespace

size_t recurrence_state_floats(const RecurrenceLayer& l) { return (size_t)l.heads * l.dim * l.dvp; }

cudaError_t launch_recurrence_step(const RecurrenceStepArgs& a, bool y_bf16, bool pdl, cudaStream_t s) {
  const RecurrenceLayer& l = a.l;
  const int dv4 = l.dvp / 4, kg = STEP_THREADS / dv4, nr = (l.dim + kg - 1) / kg;
  if (dv4 > STEP_THREADS) return cudaErrorInvalidValue;
  const size_t smem = ((size_t)5 * ((l.dim + 3) & ~3) + ((l.rank + 3) & ~3) + 3 * (size_t)l.dvp + std::max(STEP_THREADS, (l.dim + 3) & ~3) + (size_t)kg * l.dvp) * sizeof(float);
  const dim3 grid(l.heads, a.batch), block(STEP_THREADS);
  const int yb = y_bf16 ? 1 : 0;
  if (nr <= 4) return launch_kernel(recurrence_step_kernel<4>, grid, block, smem, s, pdl, a, yb);
  if (nr <= 8) return launch_kernel(recurrence_step_kernel<8>, grid, block, smem, s, pdl, a, yb);
  if (nr <= 16) return launch_kernel(recurrence_step_kernel<16>, grid, block, smem, s, pdl, a, yb);
  return launch_kernel(recurrence_step_kernel<0>, grid, block, smem, s, pdl, a, yb);
}

}  // namespace pg
