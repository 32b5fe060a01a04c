// fp32 linear on the CUDA cores (no reduced-precision matrix mode): v[m,n] = sum_k X[m,k] W[n,k] in fp32 fused
// multiply-adds along k, then the epilogue of dense_epilogue.cuh.  The 32-bit form of a model runs on it; 64 x 64 tiles,
// sixteen k at a time through shared memory, four by four outputs per thread.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "dense_epilogue.cuh"

namespace b200 {

int dense_epilogue_check(const b200_dense_epilogue* e, int N);

constexpr int FG_T = 64, FG_K = 16, FG_P = FG_T + 4;

__global__ void __launch_bounds__(256)
f32_gemm_kernel(const float* x, long long ldx, const float* w, long long ldw, int M, int N, int K,
                const __grid_constant__ b200_dense_epilogue epi, const __grid_constant__ b200_gemm_groups gr) {
  pdl_launch_dependents();
  pdl_wait();
  const int grp = blockIdx.z;
  int base = 0;                                      // first row of this group
  if (gr.groups > 0) {
    w += static_cast<long long>(grp) * N * ldw;
    if (gr.counts) { base = gr.offsets[grp]; M = min(M, gr.counts[grp]); x += base * ldx; }
    else x += grp * gr.x_group;
    if (static_cast<int>(blockIdx.y) * FG_T >= M) return;
  }
  __shared__ __align__(16) float xs[FG_K][FG_P], ws[FG_K][FG_P];
  const int m0 = blockIdx.y * FG_T, n0 = blockIdx.x * FG_T;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;      // loader: one row, four consecutive k
  const int tm = (threadIdx.x >> 4) * 4, tn = (threadIdx.x & 15) * 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += FG_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      xs[lk + i][lr] = (m0 + lr < M && k < K) ? x[static_cast<long long>(m0 + lr) * ldx + k] : 0.f;
      ws[lk + i][lr] = (n0 + lr < N && k < K) ? __ldg(w + static_cast<long long>(n0 + lr) * ldw + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < FG_K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][tm]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[k][tn]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (n0 + tn < N) {
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (m0 + tm + i < M) epi_apply4(epi, base + m0 + tm + i, n0 + tn, make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]), grp);
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_f32_gemm_grouped(const float* x, long long ldx, const float* w, long long ldw, int M, int N, int K,
                                     const b200_dense_epilogue* epi, const b200_gemm_groups* g, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (N <= 0 || K <= 0 || ldx < K || ldw < K || (M + FG_T - 1) / FG_T > 65535) return -1;
  b200_gemm_groups none = {};
  if (g && (g->groups <= 0 || g->groups > 65535 || (g->counts && !g->offsets) || !epi || epi->mode != B200_EPI_STORE)) return -1;
  if (int rc = dense_epilogue_check(epi, N)) return rc;
  launch_ex(f32_gemm_kernel, dim3((N + FG_T - 1) / FG_T, (M + FG_T - 1) / FG_T, g ? g->groups : 1), dim3(256), 0, stream, 0,
            x, ldx, w, ldw, M, N, K, *epi, g ? *g : none);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

extern "C" int b200_f32_gemm(const float* x, long long ldx, const float* w, long long ldw, int M, int N, int K,
                             const b200_dense_epilogue* epi, cudaStream_t stream) {
  return b200_f32_gemm_grouped(x, ldx, w, ldw, M, N, K, epi, nullptr, stream);
}
