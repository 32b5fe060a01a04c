// Gated linear recurrence whose gates read the current token only (minGRU), over portions of sequences:
//
//   z = sigmoid(z' + zb), c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0) with u = x' + xb
//   S_t = (1 - z) S_(t-1) + z c,   out = S_t * silu(g)
//
// S_t = a S_(t-1) + b is associative in (a, b), so a portion is cut into blocks of MG_BLOCK tokens: a first launch reduces
// every block to its (a, b), a second one starts each block from the composition of those before it (thread <-> channel).
// Entry 0 of the summaries is the state the portion starts from (zeros for a sequence's first token), so the second launch
// reads nothing of the state it writes.  One token per sequence (decoding) needs only the second launch.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"

namespace b200 {

constexpr int MG_BLOCK = 32;
constexpr int MG_THREADS = 128;

struct MingruParams {
  const float* in; long long ld;
  const float* zb; const float* xb;
  int width, M;
  float* state; long long state_ld; int num_seqs;
  const int* positions; const int* seq_ids; const int* active; const int* cu;
  float* scratch; int blocks;            // summaries [portion][blocks + 1][2][width]
  void* out; long long ldo; int f32;
};

__device__ __forceinline__ float mg_sigmoid(float v) { return 1.f / (1.f + expf(-v)); }

__device__ __forceinline__ void mg_gate(const float* row, int width, int c, float zb, float xb, float& a, float& b) {
  const float z = mg_sigmoid(row[c] + zb), u = row[width + c] + xb;
  a = 1.f - z;
  b = z * (u >= 0.f ? u + 0.5f : mg_sigmoid(u));
}

__device__ __forceinline__ float mg_start(const MingruParams& p, int row0, int seq, int c) {
  return p.positions[row0] > 0 && seq >= 0 && seq < p.num_seqs ? p.state[seq * p.state_ld + c] : 0.f;
}

__global__ void __launch_bounds__(MG_THREADS) mingru_reduce_kernel(const __grid_constant__ MingruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int portion = blockIdx.z, blk = blockIdx.y, c = blockIdx.x * MG_THREADS + threadIdx.x;
  const int row0 = p.cu[portion], len = p.cu[portion + 1] - row0;
  if (blk * MG_BLOCK >= len || c >= p.width) return;
  float* sum = p.scratch + static_cast<size_t>(portion) * (p.blocks + 1) * 2 * p.width + c;
  if (blk == 0) {
    sum[0] = 0.f;
    sum[p.width] = mg_start(p, row0, p.seq_ids ? p.seq_ids[row0] : portion, c);
  }
  const int n = min(MG_BLOCK, len - blk * MG_BLOCK);
  const float* row = p.in + static_cast<long long>(row0 + blk * MG_BLOCK) * p.ld;
  const float zb = __ldg(p.zb + c), xb = __ldg(p.xb + c);
  float A = 1.f, B = 0.f;
#pragma unroll 8
  for (int t = 0; t < n; ++t, row += p.ld) {
    float a, b;
    mg_gate(row, p.width, c, zb, xb, a, b);
    A *= a;
    B = a * B + b;
  }
  sum[static_cast<size_t>(blk + 1) * 2 * p.width] = A;
  sum[static_cast<size_t>(blk + 1) * 2 * p.width + p.width] = B;
}

template <typename T>
__global__ void __launch_bounds__(MG_THREADS) mingru_apply_kernel(const __grid_constant__ MingruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int portion = blockIdx.z, blk = blockIdx.y, c = blockIdx.x * MG_THREADS + threadIdx.x;
  const int row0 = p.cu ? p.cu[portion] : portion, len = p.cu ? p.cu[portion + 1] - row0 : 1;
  if (blk * MG_BLOCK >= len || c >= p.width) return;
  const int seq = p.seq_ids ? p.seq_ids[row0] : portion;
  float S;
  if (!p.cu) {
    S = mg_start(p, row0, seq, c);
  } else {
    const float* sum = p.scratch + static_cast<size_t>(portion) * (p.blocks + 1) * 2 * p.width + c;
    S = sum[p.width];
#pragma unroll 4
    for (int j = 1; j <= blk; ++j) S = sum[static_cast<size_t>(j) * 2 * p.width] * S + sum[static_cast<size_t>(j) * 2 * p.width + p.width];
  }
  const int n = min(MG_BLOCK, len - blk * MG_BLOCK);
  const long long m0 = row0 + blk * MG_BLOCK;
  const float* row = p.in + m0 * p.ld;
  T* out = static_cast<T*>(p.out) + m0 * p.ldo + c;
  const float zb = __ldg(p.zb + c), xb = __ldg(p.xb + c);
#pragma unroll 8
  for (int t = 0; t < n; ++t, row += p.ld, out += p.ldo) {
    float a, b;
    mg_gate(row, p.width, c, zb, xb, a, b);
    const float g = row[2 * p.width + c];
    S = a * S + b;
    *out = static_cast<T>(S * (g * mg_sigmoid(g)));
  }
  if (blk * MG_BLOCK + n == len && seq >= 0 && seq < p.num_seqs && (!p.active || p.active[seq] != 0)) p.state[seq * p.state_ld + c] = S;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_mingru_scratch_floats(int portions, int max_len, int width) {
  return portions * ((max_len + MG_BLOCK - 1) / MG_BLOCK + 1) * 2 * width;
}

extern "C" int b200_mingru(const float* zxg, long long ld, const float* zb, const float* xb, int M, int width, float* state, long long state_ld,
                           int num_seqs, const int* positions, const int* seq_ids, const int* active, const int* cu, int portions, int max_len,
                           float* scratch, void* out, long long ldo, int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!zxg || !zb || !xb || !state || !positions || !out || width <= 0 || ld < 3LL * width || state_ld < width || num_seqs <= 0 || ldo < width) return -1;
  if (cu && (portions <= 0 || max_len <= 0 || !scratch)) return -2;
  MingruParams p;
  p.in = zxg; p.ld = ld; p.zb = zb; p.xb = xb; p.width = width; p.M = M; p.state = state; p.state_ld = state_ld; p.num_seqs = num_seqs;
  p.positions = positions; p.seq_ids = seq_ids; p.active = active; p.cu = cu; p.scratch = scratch; p.out = out; p.ldo = ldo; p.f32 = f32;
  p.blocks = cu ? (max_len + MG_BLOCK - 1) / MG_BLOCK : 1;
  const int z = cu ? portions : M;
  if (z > 65535 || p.blocks > 65535) return -3;
  const dim3 grid((width + MG_THREADS - 1) / MG_THREADS, p.blocks, z), block(MG_THREADS);
  if (cu) launch_ex(mingru_reduce_kernel, grid, block, 0, stream, 0, p);
  if (f32) launch_ex(mingru_apply_kernel<float>, grid, block, 0, stream, 0, p);
  else launch_ex(mingru_apply_kernel<__nv_bfloat16>, grid, block, 0, stream, 0, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
