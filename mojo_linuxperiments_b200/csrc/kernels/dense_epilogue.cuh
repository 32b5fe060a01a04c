// What happens to a finished value of a dense (unquantised) linear before it leaves the kernel.
//
//   store     y[m][n] = v, optionally after an activation (square of relu) and times the sigmoid of a gate per (row, group);
//             grouped linears put group g at column g * y_group
//   residual  x[m][n] += mult * v (fp32, in place), optionally + add[m][n]; then, if y is given, the norm of the *next*
//             sub-layer is applied to the new residual and y[m][n] = norm(x) - possible here because the norm is
//             element-wise (dynamic tanh), so no second pass over the row is needed
//   glu       columns 2c / 2c+1 are gate / up of channel c (weight rows interleaved at load time):
//             y[m][c] = g sigmoid(1.702 g) (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit)
//
// Every buffer has a row pitch of at least N rounded up to four elements and 16-byte aligned rows, so a group of four
// columns is always handled as one vector; columns beyond N land in the padding.
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>
#include "api.h"

namespace b200 {

__device__ __forceinline__ float epi_sigmoid(float z, bool exact) {
  return exact ? 1.f / (1.f + expf(-z)) : __fdividef(1.f, 1.f + __expf(-z));
}
// tanh(z) = 1 - 2 / (e^2z + 1): absolute error of a few 1e-7, far below the bf16 rounding that follows; the 32-bit build
// of the model takes the library function.  z is bounded so that e^2z stays inside what __fdividef accepts.
__device__ __forceinline__ float epi_tanh(float z, bool exact) {
  if (exact) return tanhf(z);
  z = fminf(fmaxf(z, -15.f), 15.f);
  return 1.f - __fdividef(2.f, __expf(2.f * z) + 1.f);
}

__device__ __forceinline__ void store4_any(void* base, bool f32, long long off, float4 v) {
  if (f32) {
    *reinterpret_cast<float4*>(static_cast<float*>(base) + off) = v;
  } else {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&lo);
    raw.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(base) + off) = raw;
  }
}

// weight and shift of the element-wise norm for columns n .. n+3 (zeros when the epilogue has none)
struct EpiNorm { float4 w, b; };
__device__ __forceinline__ EpiNorm epi_norm_columns(const b200_dense_epilogue& e, int n) {
  EpiNorm k;
  k.w = k.b = make_float4(0.f, 0.f, 0.f, 0.f);
  if (e.y) {
    k.w = __ldg(reinterpret_cast<const float4*>(e.norm_w + n));
    k.b = __ldg(reinterpret_cast<const float4*>(e.norm_b + n));
  }
  return k;
}

__device__ __forceinline__ float4 epi_norm4(const b200_dense_epilogue& e, const EpiNorm& k, float4 x, bool exact) {
  float4 o;
  o.x = epi_tanh(e.norm_alpha * x.x, exact) * k.w.x + k.b.x;
  o.y = epi_tanh(e.norm_alpha * x.y, exact) * k.w.y + k.b.y;
  o.z = epi_tanh(e.norm_alpha * x.z, exact) * k.w.z + k.b.z;
  o.w = epi_tanh(e.norm_alpha * x.w, exact) * k.w.w + k.b.w;
  return o;
}

// residual form with the old residual values `x` of row m, columns n .. n+3, already loaded
__device__ __forceinline__ void epi_residual4(const b200_dense_epilogue& e, const EpiNorm& k, long long m, int n, float4 v, float4 x) {
  x.x += e.mult * v.x; x.y += e.mult * v.y; x.z += e.mult * v.z; x.w += e.mult * v.w;
  if (e.add) {
    const float4 a = *reinterpret_cast<const float4*>(e.add + m * e.ldx + n);
    x.x += a.x; x.y += a.y; x.z += a.z; x.w += a.w;
  }
  *reinterpret_cast<float4*>(e.x + m * e.ldx + n) = x;
  if (e.y) store4_any(e.y, e.out_f32 != 0, m * e.ldy + n, epi_norm4(e, k, x, e.exact != 0));
}

// columns n .. n+3 (n a multiple of four, n < N) of row m of group g
__device__ __forceinline__ void epi_apply4(const b200_dense_epilogue& e, long long m, int n, float4 v, int g = 0) {
  const bool f32 = e.out_f32 != 0;
  if (e.mode == B200_EPI_STORE) {
    if (e.act == B200_ACT_RELU2) {
      v.x = fmaxf(v.x, 0.f); v.y = fmaxf(v.y, 0.f); v.z = fmaxf(v.z, 0.f); v.w = fmaxf(v.w, 0.f);
      v.x *= v.x; v.y *= v.y; v.z *= v.z; v.w *= v.w;
    }
    if (e.gate) {
      const float s = epi_sigmoid(e.gate[m * e.ldg + g], e.exact != 0);
      v.x *= s; v.y *= s; v.z *= s; v.w *= s;
    }
    store4_any(e.y, f32, m * e.ldy + g * e.y_group + n, v);
  } else if (e.mode == B200_EPI_GLU) {
    const bool exact = e.exact != 0;
    const float g0 = fminf(v.x, e.limit), u0 = fminf(fmaxf(v.y, -e.limit), e.limit);
    const float g1 = fminf(v.z, e.limit), u1 = fminf(fmaxf(v.w, -e.limit), e.limit);
    const float o0 = g0 * epi_sigmoid(1.702f * g0, exact) * (u0 + 1.f);
    const float o1 = g1 * epi_sigmoid(1.702f * g1, exact) * (u1 + 1.f);
    const long long off = m * e.ldy + (n >> 1);
    if (f32) {
      *reinterpret_cast<float2*>(static_cast<float*>(e.y) + off) = make_float2(o0, o1);
    } else {
      *reinterpret_cast<__nv_bfloat162*>(static_cast<__nv_bfloat16*>(e.y) + off) = __floats2bfloat162_rn(o0, o1);
    }
  } else {
    epi_residual4(e, epi_norm_columns(e, n), m, n, v, *reinterpret_cast<const float4*>(e.x + m * e.ldx + n));
  }
}

}  // namespace b200
