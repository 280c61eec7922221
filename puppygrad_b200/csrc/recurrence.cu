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

// ------------------------------------------------------------------ channel delta rule
// Block = one head of one sequence. A thread owns four columns of NR rows of the state (NR = 0: it is read twice instead). The
// unit lengths of k and q are factors of sums, so that the rows go on as they leave the convolutions.
constexpr int CH_THREADS = 512, CH_WARPS = CH_THREADS / 32;

template <int NR>
__global__ void __launch_bounds__(CH_THREADS, NR > 0 && NR <= 8 ? 2 : 1) channel_step_kernel(RecurrenceStepArgs a, int y_bf16) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[CH_WARPS], lengths[2];
  const RecurrenceLayer& l = a.l;
  const int dk = l.dim, dv = l.vdim, dvp = l.dvp, dka = (dk + 3) & ~3, rep = l.heads / l.kv_heads;
  const int head = blockIdx.x, seq = blockIdx.y, kv = head / rep, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* ks = sm;         // [dk] key
  float* qs = ks + dka;   // query
  float* ws = qs + dka;   // decay
  float* vs = ws + dka;   // [dvp] value, then what is written
  float* part = vs + dvp; // [KG][dvp]
  const int dv4 = dvp / 4, KG = CH_THREADS / dv4, c4 = tid % dv4, kg = tid / dv4;
  const bool active = kg < KG;
  float* S = a.state + ((size_t)seq * l.heads + head) * dk * dvp;

  grid_dep_launch();
  grid_dep_wait();
  constexpr int NRR = NR > 0 ? NR : 1;
  float4 st[NRR];
  if (NR > 0) {  // the state's loads overlap everything up to its first use
#pragma unroll
    for (int i = 0; i < NRR; ++i) {
      const int r = kg + i * KG;
      st[i] = active && r < dk ? load4(S + (size_t)r * dvp + c4 * 4) : make_float4(0, 0, 0, 0);
    }
  }
  const float* p = a.p + (size_t)seq * a.ldp;
  const float* z = a.z + (size_t)seq * a.ldz;
  const int pos = a.pos[seq], slot = pos % l.taps;
  const bool fresh = pos == 0;
  float* taps = a.taps + (size_t)seq * l.taps * l.channels;
  for (int i = tid; i < 3 * dk + dvp; i += CH_THREADS) {
    if (i < dk) {  // decay
      ws[i] = channel_decay(l, head, head * dk + i, z[head * dk + i]);
      continue;
    }
    const int j = i - dk;
    const bool is_k = j < dk, is_q = !is_k && j < 2 * dk;
    const int c = is_k ? j : is_q ? j - dk : j - 2 * dk;
    if (!is_k && !is_q && c >= dv) {
      vs[c] = 0.f;
      continue;
    }
    const int col = is_k ? l.off_k + kv * dk + c : is_q ? l.off_q + kv * dk + c : l.off_v + head * dv + c, ch = col - l.off_q;
    const float now = p[col];
    float x = 0.f;
    for (int back = l.taps - 1; back > 0; --back) {
      const int at = slot - back < 0 ? slot - back + l.taps : slot - back;
      const float past = taps[(size_t)at * l.channels + ch];
      if (pos >= back) x = fmaf(l.conv[(size_t)(l.taps - 1 - back) * l.channels + ch], past, x);
    }
    x = silu_f(fmaf(l.conv[(size_t)(l.taps - 1) * l.channels + ch], now, x));
    (is_k ? ks : is_q ? qs : vs)[c] = x;
    // the input is cached where no token that still matters lies; one block per group caches the shared q and k
    if (head % rep == 0 || (!is_k && !is_q)) taps[(size_t)slot * l.channels + ch] = now;
  }
  const float beta = sigmoid_f(p[l.off_b + head]);
  __syncthreads();
  if (warp >= CH_WARPS - 2) {  // squared lengths
    const float* x = warp == CH_WARPS - 1 ? qs : ks;
    float s = 0.f;
    for (int c = lane; c < dk; c += 32) s += x[c] * x[c];
    s = lane_sum(s);
    if (lane == 0) lengths[warp - (CH_WARPS - 2)] = 1.f / sqrtf(s + UNIT_EPS);
  }
  auto state = [&](int i, int r) { return fresh ? make_float4(0, 0, 0, 0) : NR > 0 ? st[i] : load4(S + (size_t)r * dvp + c4 * 4); };
  const int count = NR > 0 ? NRR : (dk + KG - 1) / KG;
  float4 d = make_float4(0, 0, 0, 0);
  if (active) {
#pragma unroll
    for (int i = 0; i < count; ++i) {
      const int r = kg + i * KG;
      if (r < dk) {
        const float4 s = state(NR > 0 ? i : 0, r);
        const float u = ws[r] * ks[r];
        d.x = fmaf(u, s.x, d.x); d.y = fmaf(u, s.y, d.y); d.z = fmaf(u, s.z, d.z); d.w = fmaf(u, s.w, d.w);
      }
    }
    store4(part + (size_t)kg * dvp + c4 * 4, d);
  }
  __syncthreads();
  const float ki = lengths[0], qi = lengths[1];
  for (int c = tid; c < dvp; c += CH_THREADS) {
    float s = 0.f;
    for (int g = 0; g < KG; ++g) s += part[(size_t)g * dvp + c];
    vs[c] = beta * ki * (vs[c] - ki * s);
  }
  __syncthreads();
  if (active) {
    const float4 v = load4(vs + c4 * 4);
    float4 o = make_float4(0, 0, 0, 0);
#pragma unroll
    for (int i = 0; i < count; ++i) {
      const int r = kg + i * KG;
      if (r < dk) {
        float4 s = state(NR > 0 ? i : 0, r);
        const float w = ws[r], k = ks[r], q = qs[r];
        s.x = fmaf(w, s.x, k * v.x); s.y = fmaf(w, s.y, k * v.y); s.z = fmaf(w, s.z, k * v.z); s.w = fmaf(w, s.w, k * v.w);
        store4(S + (size_t)r * dvp + c4 * 4, s);
        o.x = fmaf(q, s.x, o.x); o.y = fmaf(q, s.y, o.y); o.z = fmaf(q, s.z, o.z); o.w = fmaf(q, s.w, o.w);
      }
    }
    store4(part + (size_t)kg * dvp + c4 * 4, o);
  }
  __syncthreads();
  float out = 0.f;  // one column per thread: dv <= CH_THREADS
  if (tid < dv) {
    for (int g = 0; g < KG; ++g) out += part[(size_t)g * dvp + tid];
    out *= qi * l.q_scale;
  }
  const float sq = lane_sum(out * out);
  if (lane == 0) red[warp] = sq;
  __syncthreads();
  if (tid < dv) {
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < CH_WARPS; ++i) total += red[i];
    const float y = out / sqrtf(total / (float)dv + l.eps) * l.norm[tid] * sigmoid_f(z[l.heads * dk + head * dv + tid]) * l.out_scale;
    const size_t at = (size_t)seq * a.ldy + head * dv + tid;
    if (y_bf16) static_cast<__nv_bfloat16*>(a.y)[at] = __float2bfloat16_rn(y);
    else static_cast<float*>(a.y)[at] = y;
  }
}

cudaError_t launch_channel_step(const RecurrenceStepArgs& a, int yb, bool pdl, cudaStream_t s) {
  const RecurrenceLayer& l = a.l;
  const int kg = CH_THREADS / (l.dvp / 4), nr = (l.dim + kg - 1) / kg;
  if (l.dvp > CH_THREADS) return cudaErrorInvalidValue;
  const size_t smem = ((size_t)3 * ((l.dim + 3) & ~3) + l.dvp + (size_t)kg * l.dvp) * sizeof(float);
  const dim3 grid(l.heads, a.batch), block(CH_THREADS);
  if (nr <= 2) return launch_kernel(channel_step_kernel<2>, grid, block, smem, s, pdl, a, yb);
  if (nr <= 4) return launch_kernel(channel_step_kernel<4>, grid, block, smem, s, pdl, a, yb);
  if (nr <= 8) return launch_kernel(channel_step_kernel<8>, grid, block, smem, s, pdl, a, yb);
  if (nr <= 16) return launch_kernel(channel_step_kernel<16>, grid, block, smem, s, pdl, a, yb);
  return launch_kernel(channel_step_kernel<0>, grid, block, smem, s, pdl, a, yb);
}

}  // namespace

size_t recurrence_state_floats(const RecurrenceLayer& l) { return (size_t)l.heads * l.dim * l.dvp; }

cudaError_t launch_recurrence_step(const RecurrenceStepArgs& a, bool y_bf16, bool pdl, cudaStream_t s) {
  const RecurrenceLayer& l = a.l;
  if (l.kind == KIND_CHANNEL) return launch_channel_step(a, y_bf16 ? 1 : 0, pdl, s);
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
