// Element arithmetic of NormStepArgs, shared by the row kernel (norms.cu) and by the products that make their own
// input rows (linear_bf16.cu).
#pragma once
#include "device_util.cuh"
#include "layered_kernels.cuh"

namespace pg {
namespace {

// xIELU: expm1 keeps e^z - 1 - z accurate near 0.
__device__ __forceinline__ float xielu(float z, float a, float b) {
  return fmaf(0.5f, z, z > 0.f ? a * z * z : b * (expm1f(z) - z));
}
__device__ __forceinline__ float activate(const ActArgs& act, float z) {
  return act.kind == ACT_GELU_ERF ? gelu_erf(z) : act.kind == ACT_XIELU ? xielu(z, act.a, act.b) : z;
}

// Zeroes the elements of columns >= width.
__device__ __forceinline__ float4 mask4(float4 v, int c, int width) {
  if (c + 3 >= width) {
    if (c >= width) v.x = 0.f;
    if (c + 1 >= width) v.y = 0.f;
    if (c + 2 >= width) v.z = 0.f;
    v.w = c + 3 >= width ? 0.f : v.w;
  }
  return v;
}

// Entry c of the position vector: sin(p f) for even c, cos(p f) for odd c, f = freq[c / 2]. The angle is formed and
// reduced to one period in FP64 so that its error does not grow with the position.
__device__ __forceinline__ float2 sinusoid(int p, double f) {
  const double ang = (double)p * f, two_pi = 6.283185307179586476925286766559;
  const float r = (float)(ang - two_pi * rint(ang * 0.15915494309189533576888376337251));
  float2 o;
  sincosf(r, &o.x, &o.y);
  return o;
}

// Columns c..c+3 (c % 4 == 0, c < ldx) of a row of x before the sublayer is added.
template <typename T>
__device__ __forceinline__ float4 norm_step_load_x(const NormStepArgs& a, int row, int c) {
  float4 v;
  if (a.ids) {
    v = load4(static_cast<const T*>(a.embed) + (size_t)a.ids[row] * a.ld_embed + c);
    v.x *= a.embed_scale; v.y *= a.embed_scale; v.z *= a.embed_scale; v.w *= a.embed_scale;
    if (a.freq && c < a.width) {
      const float2 s = sinusoid(a.pos[row], a.freq[c >> 1]);
      v.x += s.x;
      v.y += s.y;
    }
    if (a.freq && c + 2 < a.width) {
      const float2 s = sinusoid(a.pos[row], a.freq[(c >> 1) + 1]);
      v.z += s.x;
      v.w += s.y;
    }
  } else {
    const int src = a.row_index ? a.row_index[row] : row;
    v = c < a.width ? load4(a.x_in + (size_t)src * a.ld_in + c) : make_float4(0, 0, 0, 0);
  }
  return mask4(v, c, a.width);
}

__device__ __forceinline__ float norm_step_square(float4 v, float mean, int c, int width) {
  const float dx = v.x - mean, dy = v.y - mean, dz = v.z - mean, dw = v.w - mean;
  float q = 0.f;
  if (c < width) q += dx * dx;
  if (c + 1 < width) q += dy * dy;
  if (c + 2 < width) q += dz * dz;
  if (c + 3 < width) q += dw * dw;
  return q;
}

// (v - mean) * rstd * g [+ b], zero past width (g and b are padded to the row pitch).
__device__ __forceinline__ float4 norm_step_apply(float4 v, float mean, float rstd, const float* g, const float* b, int c,
                                                  int width) {
  const float4 gg = load4(g + c), bb = b ? load4(b + c) : make_float4(0, 0, 0, 0);
  float4 o;
  o.x = (v.x - mean) * rstd * gg.x + bb.x;
  o.y = (v.y - mean) * rstd * gg.y + bb.y;
  o.z = (v.z - mean) * rstd * gg.z + bb.z;
  o.w = (v.w - mean) * rstd * gg.w + bb.w;
  return mask4(o, c, width);
}

}  // namespace
}  // namespace pg
