// Routing for mixtures whose choice and weights differ, and the row gather in front of the grouped expert linears.
//
//   route_grouped     fp32 logits [M, E] -> s = softmax; choice = s + correction.  The E outputs form equal groups of
//                     neighbours; a group counts by its best choice score and only the members of the best `keep` groups
//                     are eligible; the `top` best eligible ones are chosen.  Weight: s * scale.  Ties: lowest index.
//   moe_gather_rows   rows of any element type into the slot order of a work list
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"

namespace b200 {

constexpr int RG_WARPS = 4;

// integers in the order of the floats they come from
__device__ __forceinline__ int rg_order(float v) { const int i = __float_as_int(v); return i ^ ((i >> 31) & 0x7fffffff); }
// index of the warp's largest value; the lowest index wins ties
__device__ __forceinline__ int rg_argmax(float v, int i) {
  const int key = rg_order(v), best = __reduce_max_sync(0xffffffffu, key);
  return static_cast<int>(__reduce_min_sync(0xffffffffu, key == best ? static_cast<unsigned>(i) : 0x7fffffffu));
}

// one warp per token; lane <-> outputs lane, lane + 32, ...
template <int EPL>
__global__ void __launch_bounds__(32 * RG_WARPS)
route_grouped_kernel(const float* logits, long long ld, const float* correction, int M, int E, int top, int groups, int keep,
                     float scale, int* ids, float* weights) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tok = blockIdx.x * RG_WARPS + warp;
  if (tok >= M) return;
  const float* x = logits + static_cast<size_t>(tok) * ld;
  float s[EPL], c[EPL];
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < E ? x[e] : -INFINITY;
    mx = fmaxf(mx, s[i]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    s[i] = lane + 32 * i < E ? expf(s[i] - mx) : 0.f;
    sum += s[i];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  const float inv = 1.f / sum;
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    const int e = lane + 32 * i;
    s[i] *= inv;
    c[i] = e < E ? s[i] + __ldg(correction + e) : -INFINITY;
  }
  if (keep < groups) {
    const int size = E / groups;
    int grp[EPL];
#pragma unroll
    for (int i = 0; i < EPL; ++i) grp[i] = lane + 32 * i < E ? (lane + 32 * i) / size : -1;
    // best group first: the group of the largest remaining choice score; its members are marked and leave the race
    unsigned in = 0;                       // bit i: output lane + 32 i is in a kept group
    for (int k = 0; k < keep; ++k) {
      float best = -INFINITY;
      int bi = 0x7fffffff;
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        const int e = lane + 32 * i;
        if (e < E && !(in >> i & 1u) && (c[i] > best || (c[i] == best && e < bi))) { best = c[i]; bi = e; }
      }
      bi = rg_argmax(best, bi);
      if (bi == 0x7fffffff) break;
      const int g = bi / size;
#pragma unroll
      for (int i = 0; i < EPL; ++i)
        if (grp[i] == g) in |= 1u << i;
    }
#pragma unroll
    for (int i = 0; i < EPL; ++i)
      if (!(in >> i & 1u)) c[i] = -INFINITY;
  }
  unsigned taken = 0;
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
      const int e = lane + 32 * i;
      if (e < E && !(taken >> i & 1u) && (c[i] > best || (c[i] == best && e < bi))) { best = c[i]; bi = e; }
    }
    bi = rg_argmax(best, bi);
    const size_t at = static_cast<size_t>(tok) * top + j;
#pragma unroll
    for (int i = 0; i < EPL; ++i)
      if (lane + 32 * i == bi) {                 // the winner's lane
        taken |= 1u << i;
        ids[at] = bi;
        weights[at] = s[i] * scale;
      }
    if (bi == 0x7fffffff && lane == 0) { ids[at] = E - 1; weights[at] = 0.f; }      // nothing eligible (no number among the scores)
  }
}

// grid = most slots; rows beyond meta[0] exit
__global__ void __launch_bounds__(128) moe_gather_rows_kernel(const uint8_t* x, long long row_bytes, const int* slot_token, const int* meta, uint8_t* out) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.x;
  if (s >= meta[0]) return;
  const uint4* src = reinterpret_cast<const uint4*>(x + slot_token[s] * row_bytes);
  uint4* dst = reinterpret_cast<uint4*>(out + s * row_bytes);
  for (int i = threadIdx.x; i < row_bytes / 16; i += blockDim.x) dst[i] = src[i];
}

}  // namespace b200

using namespace b200;

extern "C" int b200_route_grouped(const float* logits, long long ld, const float* correction, int M, int E, int top, int groups, int keep,
                                  float scale, int* ids, float* weights, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!logits || !correction || !ids || !weights || E <= 0 || E > 1024 || top <= 0 || groups <= 0 || E % groups || keep <= 0 || keep > groups || top > keep * (E / groups)) return -1;
  const dim3 grid((M + RG_WARPS - 1) / RG_WARPS), block(32 * RG_WARPS);
  // (3: a router of 64 experts and a few identity outputs)
  if (E <= 32) launch_ex(route_grouped_kernel<1>, grid, block, 0, stream, 0, logits, ld, correction, M, E, top, groups, keep, scale, ids, weights);
  else if (E <= 64) launch_ex(route_grouped_kernel<2>, grid, block, 0, stream, 0, logits, ld, correction, M, E, top, groups, keep, scale, ids, weights);
  else if (E <= 96) launch_ex(route_grouped_kernel<3>, grid, block, 0, stream, 0, logits, ld, correction, M, E, top, groups, keep, scale, ids, weights);
  else if (E <= 128) launch_ex(route_grouped_kernel<4>, grid, block, 0, stream, 0, logits, ld, correction, M, E, top, groups, keep, scale, ids, weights);
  else if (E <= 256) launch_ex(route_grouped_kernel<8>, grid, block, 0, stream, 0, logits, ld, correction, M, E, top, groups, keep, scale, ids, weights);
  else launch_ex(route_grouped_kernel<32>, grid, block, 0, stream, 0, logits, ld, correction, M, E, top, groups, keep, scale, ids, weights);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

extern "C" int b200_moe_gather_rows(const void* x, long long row_bytes, const int* slot_token, const int* meta, int max_slots, void* out,
                                    cudaStream_t stream) {
  if (max_slots <= 0) return 0;
  if (!x || !slot_token || !meta || !out || row_bytes <= 0 || row_bytes % 16 || (reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(out) & 15)) return -1;
  launch_ex(moe_gather_rows_kernel, dim3(max_slots), dim3(128), 0, stream, 0, static_cast<const uint8_t*>(x), row_bytes, slot_token, meta, static_cast<uint8_t*>(out));
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
