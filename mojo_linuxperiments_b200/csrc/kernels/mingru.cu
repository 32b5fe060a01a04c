// Gated linear recurrence whose gates read the current token only (minGRU), over portions of sequences:
//
//   z = sigmoid(z' + zb), c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0) with u = x' + xb
//   S_t = (1 - z) S_(t-1) + z c,   out = S_t * silu(g)
//
// S_t = a S_(t-1) + b is associative in (a, b), so a portion is cut into blocks: a first launch reduces every block to its
// (a, b), a second one starts each block from the composition of those before it (thread <-> four channels).  Blocks are 32
// tokens, more in long portions: the second launch walks the summaries before its block.  Entry 0 of the summaries is the state
// the portion starts from (zeros for a sequence's first token), so the second launch reads nothing of the state it writes.  One
// token per sequence (decoding) needs only the second launch.
//
// The 32-bit form takes the library's exponential and division, the bf16 form the hardware's (a few units in the last place of
// fp32, far below the rounding of what surrounds it); everything is fp32 in both.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "dense_epilogue.cuh"

namespace b200 {

constexpr int MG_THREADS = 128;

struct MingruParams {
  const float* in; long long ld;
  const float* zb; const float* xb;
  int width, M;
  float* state; long long state_ld; int num_seqs;
  const int* positions; const int* seq_ids; const int* active; const int* cu;
  float* scratch; int block, blocks;     // summaries [portion][blocks + 1][2][width]
  void* out; long long ldo;
};

template <bool EXACT>
__device__ __forceinline__ void mg_gate(float zr, float ur, float zb, float xb, float& a, float& b) {
  const float z = epi_sigmoid(zr + zb, EXACT), u = ur + xb;
  a = 1.f - z;
  b = z * (u >= 0.f ? u + 0.5f : epi_sigmoid(u, EXACT));
}
template <bool EXACT>
__device__ __forceinline__ void mg_gate4(const float* row, int width, float4 zb, float4 xb, float4& a, float4& b) {
  const float4 z = *reinterpret_cast<const float4*>(row), u = *reinterpret_cast<const float4*>(row + width);
  mg_gate<EXACT>(z.x, u.x, zb.x, xb.x, a.x, b.x);
  mg_gate<EXACT>(z.y, u.y, zb.y, xb.y, a.y, b.y);
  mg_gate<EXACT>(z.z, u.z, zb.z, xb.z, a.z, b.z);
  mg_gate<EXACT>(z.w, u.w, zb.w, xb.w, a.w, b.w);
}
__device__ __forceinline__ float4 mg_step(float4 a, float4 s, float4 b) {
  return make_float4(a.x * s.x + b.x, a.y * s.y + b.y, a.z * s.z + b.z, a.w * s.w + b.w);
}

__device__ __forceinline__ float4 mg_start(const MingruParams& p, int row0, int seq, int c) {
  return p.positions[row0] > 0 && seq >= 0 && seq < p.num_seqs ? *reinterpret_cast<const float4*>(p.state + seq * p.state_ld + c)
                                                               : make_float4(0.f, 0.f, 0.f, 0.f);
}

template <bool EXACT>
__global__ void __launch_bounds__(MG_THREADS) mingru_reduce_kernel(const __grid_constant__ MingruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int portion = blockIdx.z, blk = blockIdx.y, c = (blockIdx.x * MG_THREADS + threadIdx.x) * 4;
  const int row0 = p.cu[portion], len = p.cu[portion + 1] - row0;
  if (blk * p.block >= len || c >= p.width) return;
  float* sum = p.scratch + static_cast<size_t>(portion) * (p.blocks + 1) * 2 * p.width + c;
  if (blk == 0) {
    *reinterpret_cast<float4*>(sum) = make_float4(0.f, 0.f, 0.f, 0.f);
    *reinterpret_cast<float4*>(sum + p.width) = mg_start(p, row0, p.seq_ids ? p.seq_ids[row0] : portion, c);
  }
  const int n = min(p.block, len - blk * p.block);
  const float* row = p.in + static_cast<long long>(row0 + blk * p.block) * p.ld + c;
  const float4 zb = __ldg(reinterpret_cast<const float4*>(p.zb + c)), xb = __ldg(reinterpret_cast<const float4*>(p.xb + c));
  float4 A = make_float4(1.f, 1.f, 1.f, 1.f), B = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
  for (int t = 0; t < n; ++t, row += p.ld) {
    float4 a, b;
    mg_gate4<EXACT>(row, p.width, zb, xb, a, b);
    A = make_float4(A.x * a.x, A.y * a.y, A.z * a.z, A.w * a.w);
    B = mg_step(a, B, b);
  }
  *reinterpret_cast<float4*>(sum + static_cast<size_t>(blk + 1) * 2 * p.width) = A;
  *reinterpret_cast<float4*>(sum + static_cast<size_t>(blk + 1) * 2 * p.width + p.width) = B;
}

template <typename T>
__global__ void __launch_bounds__(MG_THREADS) mingru_apply_kernel(const __grid_constant__ MingruParams p) {
  constexpr bool EXACT = sizeof(T) == 4;
  pdl_launch_dependents();
  pdl_wait();
  const int portion = blockIdx.z, blk = blockIdx.y, c = (blockIdx.x * MG_THREADS + threadIdx.x) * 4;
  const int row0 = p.cu ? p.cu[portion] : portion, len = p.cu ? p.cu[portion + 1] - row0 : 1;
  if (blk * p.block >= len || c >= p.width) return;
  const int seq = p.seq_ids ? p.seq_ids[row0] : portion;
  float4 S;
  if (!p.cu) {
    S = mg_start(p, row0, seq, c);
  } else {
    const float* sum = p.scratch + static_cast<size_t>(portion) * (p.blocks + 1) * 2 * p.width + c;
    S = *reinterpret_cast<const float4*>(sum + p.width);
#pragma unroll 4
    for (int j = 1; j <= blk; ++j)
      S = mg_step(*reinterpret_cast<const float4*>(sum + static_cast<size_t>(j) * 2 * p.width), S,
                  *reinterpret_cast<const float4*>(sum + static_cast<size_t>(j) * 2 * p.width + p.width));
  }
  const int n = min(p.block, len - blk * p.block);
  const long long m0 = row0 + blk * p.block;
  const float* row = p.in + m0 * p.ld + c;
  const float4 zb = __ldg(reinterpret_cast<const float4*>(p.zb + c)), xb = __ldg(reinterpret_cast<const float4*>(p.xb + c));
#pragma unroll 4
  for (int t = 0; t < n; ++t, row += p.ld) {
    float4 a, b;
    mg_gate4<EXACT>(row, p.width, zb, xb, a, b);
    const float4 g = *reinterpret_cast<const float4*>(row + 2 * p.width);
    S = mg_step(a, S, b);
    store4_any(p.out, EXACT, (m0 + t) * p.ldo + c, make_float4(S.x * g.x * epi_sigmoid(g.x, EXACT), S.y * g.y * epi_sigmoid(g.y, EXACT),
                                                              S.z * g.z * epi_sigmoid(g.z, EXACT), S.w * g.w * epi_sigmoid(g.w, EXACT)));
  }
  if (blk * p.block + n == len && seq >= 0 && seq < p.num_seqs && (!p.active || p.active[seq] != 0))
    *reinterpret_cast<float4*>(p.state + seq * p.state_ld + c) = S;
}

static int mg_block(int max_len) { return max_len <= 1024 ? 32 : (max_len <= 8192 ? 64 : 256); }

}  // namespace b200

using namespace b200;

extern "C" int b200_mingru_scratch_floats(int portions, int max_len, int width) {
  const int block = mg_block(max_len);
  return portions * ((max_len + block - 1) / block + 1) * 2 * width;
}

extern "C" int b200_mingru(const float* zxg, long long ld, const float* zb, const float* xb, int M, int width, float* state, long long state_ld,
                           int num_seqs, const int* positions, const int* seq_ids, const int* active, const int* cu, int portions, int max_len,
                           float* scratch, void* out, long long ldo, int f32, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!zxg || !zb || !xb || !state || !positions || !out || width <= 0 || ld < 3LL * width || state_ld < width || num_seqs <= 0 || ldo < width) return -1;
  if (cu && (portions <= 0 || max_len <= 0 || !scratch)) return -2;
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (width % 4 || ld % 4 || state_ld % 4 || ldo % 8 || !al16(zxg) || !al16(zb) || !al16(xb) || !al16(state) || !al16(scratch) || !al16(out)) return -4;
  MingruParams p;
  p.in = zxg; p.ld = ld; p.zb = zb; p.xb = xb; p.width = width; p.M = M; p.state = state; p.state_ld = state_ld; p.num_seqs = num_seqs;
  p.positions = positions; p.seq_ids = seq_ids; p.active = active; p.cu = cu; p.scratch = scratch; p.out = out; p.ldo = ldo;
  p.block = cu ? mg_block(max_len) : 1;
  p.blocks = cu ? (max_len + p.block - 1) / p.block : 1;
  const int z = cu ? portions : M;
  if (z > 65535 || p.blocks > 65535) return -3;
  const dim3 grid((width / 4 + MG_THREADS - 1) / MG_THREADS, p.blocks, z), block(MG_THREADS);
  if (f32) {
    if (cu) launch_ex(mingru_reduce_kernel<true>, grid, block, 0, stream, 0, p);
    launch_ex(mingru_apply_kernel<float>, grid, block, 0, stream, 0, p);
  } else {
    if (cu) launch_ex(mingru_reduce_kernel<false>, grid, block, 0, stream, 0, p);
    launch_ex(mingru_apply_kernel<__nv_bfloat16>, grid, block, 0, stream, 0, p);
  }
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
