// bf16 linear for decode-sized calls (a few tokens) on sm_100a: the weight matrix is streamed from HBM exactly once.
//
//   v[m,n] = sum_k X[m,k] W[n,k], then the fused epilogue of dense_epilogue.cuh.
//
//   * The 128-row weight tile is the tcgen05 A operand (output channels fill the MMA M dimension), BN in {16,32,64} tokens
//     are B, so tokens are never padded to 128.  64 bf16 per k-block, 128-byte swizzled TMA tiles, STAGES-deep ring; the
//     weight tiles of the first ring-full are requested before the dependency wait (weights never change).
//   * K is split over a thread-block cluster of S CTAs.  Each CTA owns a slice of the tile's channels; partial sums travel
//     to the owner as fp32 through distributed shared memory ([sender][token][channel]), the owner adds them in rank
//     order (the result does not depend on timing) and runs the epilogue on four channels of a token at a time.
//   * More than BN tokens: blockIdx.z picks the token block; the weights come from L2 the second time.
//   * Grouped form: blockIdx.z also picks the group, whose weights are rows group * N .. of one stacked matrix (a tile that
//     reaches into the next group's rows is cut in the epilogue).  Heads take all rows at their own columns of x; experts
//     take their own rows, known only once the routing kernel has finished, so those CTAs wait first and leave if idle.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "gemm_common.cuh"
#include "dense_epilogue.cuh"

namespace b200 {

int dense_epilogue_check(const b200_dense_epilogue* e, int N);

struct BfDecodeParams {
  int M, N, kblocks, splits;
  int z_tiles, groups;                  // groups 0: one linear
  int x_group_bytes;
  const int* offsets; const int* counts;
  b200_dense_epilogue epi;
  int* status;
  unsigned long long limit_ns;
};

// first channel (of 128) that cluster rank r finishes: slices are multiples of four channels
__host__ __device__ __forceinline__ int bd_slice0(int r, int S) { return 4 * ((32 * r + S - 1) / S); }
// exchange rows: S senders x padded slice, at most 168 floats per token (S = 7: 24 x 7)
constexpr int BD_XROW = 168;

template <int BN, int STAGES>
constexpr int bd_smem_bytes() { return STAGES * (128 + BN) * 128 + BN * BD_XROW * 4 + 1024 + 256; }

template <int BN, int STAGES>
__global__ void __launch_bounds__(GEMM_THREADS, BN == 64 ? 1 : 2)
bf16_gemm_decode_kernel(const __grid_constant__ CUtensorMap tmap_w, const __grid_constant__ CUtensorMap tmap_x,
                        const __grid_constant__ BfDecodeParams p) {
  constexpr int A_BYTES = 128 * 128, B_BYTES = BN * 128, STAGE_BYTES = A_BYTES + B_BYTES;
  constexpr int TMEM_COLS = BN < 32 ? 32 : BN;
  constexpr uint32_t IDESC = umma_idesc_bf16(128, BN, 0, 0);
  constexpr int CH = BN >= 32 ? 32 : 16;

  pdl_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  float* ex = reinterpret_cast<float*>(smem + STAGES * STAGE_BYTES);                 // [S][BN][cw + 4]
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + STAGES * STAGE_BYTES + BN * BD_XROW * 4);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * STAGES + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t smem_base = smem_u32(smem), bar_base = smem_u32(bars);
  auto full_bar = [&](int s) { return bar_base + 8u * s; };
  auto empty_bar = [&](int s) { return bar_base + 8u * (STAGES + s); };
  const uint32_t tfull_bar = bar_base + 8u * (2 * STAGES);

  const int S = p.splits;
  const int rank = static_cast<int>(cluster_ctarank());
  const int grp = p.groups > 0 ? blockIdx.z / p.z_tiles : 0, zt = blockIdx.z - grp * p.z_tiles;
  const int n_tile = blockIdx.y;
  int m0 = zt * BN, rows = min(BN, p.M - m0);
  if (p.counts) {
    pdl_wait();
    rows = min(BN, p.counts[grp] - m0);
    if (rows <= 0) return;                      // the whole cluster
    m0 += p.offsets[grp];
  }
  const int w0 = grp * p.N + n_tile * 128, x0 = grp * p.x_group_bytes;
  const int kb0 = static_cast<int>(static_cast<long long>(p.kblocks) * rank / S);
  const int kb1 = static_cast<int>(static_cast<long long>(p.kblocks) * (rank + 1) / S);
  const uint64_t limit = p.limit_ns;

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) { mbar_init(full_bar(s), 1); mbar_init(empty_bar(s), 1); }
    mbar_init(tfull_bar, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(smem_u32(tmem_slot), TMEM_COLS); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  if (S > 1) cluster_arrive_relaxed();          // "this CTA runs": waited for just before the exchange

  if (warp == 0) {
    if (lane == 0) {
      const uint64_t pol_w = policy_evict_first();
      prefetch_tmap(&tmap_w);
      prefetch_tmap(&tmap_x);
      const int pre = min(STAGES, kb1 - kb0);
      for (int i = 0; i < pre; ++i) {
        mbar_expect_tx(full_bar(i), STAGE_BYTES);
        tma_load_2d_hint(smem_base + i * STAGE_BYTES, &tmap_w, full_bar(i), (kb0 + i) * 128, w0, pol_w);
      }
      pdl_wait();
      for (int i = 0; i < pre; ++i) tma_load_2d(smem_base + i * STAGE_BYTES + A_BYTES, &tmap_x, full_bar(i), x0 + (kb0 + i) * 128, m0);
      bool ok = true;
      int stage = pre == STAGES ? 0 : pre;
      uint32_t phase = pre == STAGES ? 1u : 0u;
      for (int kb = kb0 + pre; kb < kb1; ++kb) {
        if (!mbar_wait(empty_bar(stage), phase ^ 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_EMPTY | (10 << 8)), limit)) { ok = false; break; }
        mbar_expect_tx(full_bar(stage), STAGE_BYTES);
        const uint32_t a_dst = smem_base + stage * STAGE_BYTES;
        tma_load_2d_hint(a_dst, &tmap_w, full_bar(stage), kb * 128, w0, pol_w);
        tma_load_2d(a_dst + A_BYTES, &tmap_x, full_bar(stage), x0 + kb * 128, m0);
        if (++stage == STAGES) { stage = 0; phase ^= 1u; }
      }
      if (!ok) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 2000000ull) { } }   // copies in flight land
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      int stage = 0; uint32_t phase = 0;
      bool ok = true;
      for (int kb = kb0; kb < kb1; ++kb) {
        if (!mbar_wait(full_bar(stage), phase, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (10 << 8)), limit)) { ok = false; break; }
        tc_fence_after();
        const uint32_t a_src = smem_base + stage * STAGE_BYTES;
        const uint64_t a_desc = umma_desc_k_sw128(a_src), b_desc = umma_desc_k_sw128(a_src + A_BYTES);
#pragma unroll
        for (int k = 0; k < 4; ++k) umma_f16_ss(tmem_base, a_desc + 2ull * k, b_desc + 2ull * k, IDESC, (kb > kb0 || k > 0) ? 1u : 0u);
        umma_commit(empty_bar(stage));
        if (++stage == STAGES) { stage = 0; phase ^= 1u; }
      }
      if (ok) umma_commit(tfull_bar);
    }
    __syncwarp();
  }
  pdl_wait();                                   // the epilogue reads what earlier kernels wrote (residual rows)

  bool acc_ok = false;
  const int q = warp & 3, row = q * 32 + lane;  // channel inside the tile == TMEM lane
  if (warp >= 2) {
    acc_ok = kb1 > kb0 && mbar_wait(tfull_bar, 0, abort_flag, p.status, (ST_TIMEOUT_TMEM_FULL | (10 << 8)), limit);
    acc_ok = __all_sync(0xffffffffu, acc_ok);
    tc_fence_after();
  }
  if (S > 1) cluster_wait_acquire();            // every CTA of the cluster runs: its shared memory exists
  if (warp >= 2) {
    const int owner = (row >> 2) * S / 32;      // the rank whose slice holds this channel
    const int cwp = bd_slice0(owner + 1, S) - bd_slice0(owner, S) + 4;
    const uint32_t local = smem_u32(ex) + 4u * static_cast<uint32_t>(rank * BN * cwp + row - bd_slice0(owner, S));
    const uint32_t remote = mapa_shared(local, static_cast<uint32_t>(owner));
    const uint32_t t_addr = tmem_base + (static_cast<uint32_t>(q * 32) << 16);
#pragma unroll 1
    for (int c = 0; c < BN / CH; ++c) {
      if (c * CH >= rows) break;
      uint32_t r[CH];
      if (acc_ok) {
        if constexpr (CH == 32) tmem_ld_x32(t_addr + c * CH, r); else tmem_ld_x16(t_addr + c * CH, r);
        tmem_ld_wait();
      } else {
#pragma unroll
        for (int j = 0; j < CH; ++j) r[j] = 0u;             // empty K range (or aborted): contributes nothing
      }
#pragma unroll
      for (int j = 0; j < CH; ++j)
        if (c * CH + j < rows) st_shared_cluster_u32(remote + 4u * static_cast<uint32_t>((c * CH + j) * cwp), r[j]);
    }
  }
  tc_fence_before();
  if (S > 1) cluster_sync_all(); else __syncthreads();

  const int s0 = bd_slice0(rank, S), cw = bd_slice0(rank + 1, S) - s0, cwp = cw + 4, quads = cw >> 2;
  for (int i = threadIdx.x; i < rows * quads; i += GEMM_THREADS) {
    const int j = i / quads, c4 = (i - j * quads) * 4;
    const int n = n_tile * 128 + s0 + c4;
    if (n >= p.N) continue;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < S; ++s) {
      const float4 u = *reinterpret_cast<const float4*>(ex + (s * BN + j) * cwp + c4);
      v.x += u.x; v.y += u.y; v.z += u.z; v.w += u.w;
    }
    epi_apply4(p.epi, m0 + j, n, v, grp);
  }

  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, TMEM_COLS); }
}

template <int BN, int STAGES>
static int launch_bf16_decode(const CUtensorMap& tw, const CUtensorMap& tx, const BfDecodeParams& p, dim3 grid, cudaStream_t stream) {
  constexpr int SMEM = bd_smem_bytes<BN, STAGES>();
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(bf16_gemm_decode_kernel<BN, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return -1000 - static_cast<int>(e);
    cudaFuncSetAttribute(bf16_gemm_decode_kernel<BN, STAGES>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    configured = true;
  }
  launch_ex(bf16_gemm_decode_kernel<BN, STAGES>, grid, dim3(GEMM_THREADS), SMEM, stream, p.splits, tw, tx, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

// clusters of S CTAs that are resident at once with `per_sm` CTAs per SM (clusters are placed inside a GPC, hence less
// than per_sm x SMs / S for the larger sizes)
static int bd_resident(int S, int num_sms, int per_sm) {
  switch (S) {
    case 1: return per_sm * num_sms;
    case 2: return per_sm * (num_sms / 2);
    case 3: case 4: return per_sm * (num_sms * 33 / 148);
    default: return per_sm * (num_sms * 15 / 148);
  }
}

}  // namespace b200

using namespace b200;

// splits: 0 picks the K split, else 1..8 CTAs per cluster
static int bf16_decode_any(const void* x, long long ldx, const void* w, long long ldw, int M, int rows_total, int N, int K,
                           const b200_dense_epilogue* epi, const b200_gemm_groups* g, int* status, int num_sms, int splits, cudaStream_t stream) {
  if (M <= 0 || rows_total <= 0) return 0;
  if (N <= 0 || K <= 0 || ldx < K || ldw < K || (ldx % 8) || (ldw % 8) || splits < 0 || splits > 8) return -1;
  if ((reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(w) & 15)) return -2;
  if (int rc = dense_epilogue_check(epi, N)) return rc;
  if (g && (g->groups <= 0 || g->x_group % 8 || g->x_group < 0 || (g->counts && !g->offsets) || epi->mode != B200_EPI_STORE)) return -3;
  const bool lists = g && g->counts;
  if (g && !lists && (g->groups - 1) * g->x_group + K > ldx) return -3;
  const int bn = lists || M <= 16 ? 16 : (M <= 32 ? 32 : 64);
  BfDecodeParams p;
  p.M = M; p.N = N;
  p.kblocks = (K + 63) / 64;
  p.z_tiles = (M + bn - 1) / bn;
  p.groups = g ? g->groups : 0;
  p.x_group_bytes = g && !lists ? static_cast<int>(g->x_group * 2) : 0;
  p.offsets = lists ? g->offsets : nullptr;
  p.counts = lists ? g->counts : nullptr;
  p.epi = *epi;
  p.status = status;
  p.limit_ns = 2000000000ull;
  const int n_tiles = (N + 127) / 128, z = p.z_tiles * (g ? g->groups : 1);
  if (z > 65535) return -4;
  if (splits == 0) {
    double best = 0;
    const int busy = lists && g->expected > 0 && g->expected < g->groups ? g->expected : (lists ? g->groups : z);
    for (int s = 1; s <= 8 && s <= p.kblocks; ++s) {
      const int clusters = n_tiles * busy, res = bd_resident(s, num_sms, bn == 64 ? 1 : 2);
      const double cost = static_cast<double>((clusters + res - 1) / res) * ((p.kblocks + s - 1) / s + 6 + (s > 1 ? 1 : 0));
      if (splits == 0 || cost < best) { best = cost; splits = s; }
    }
  }
  if (splits > p.kblocks) splits = p.kblocks;
  p.splits = splits;
  const uint64_t x_cols = static_cast<uint64_t>(g && !lists ? (g->groups - 1) * g->x_group + K : K);
  CUtensorMap tw, tx;
  if (make_tmap_2d_u8(&tw, w, static_cast<uint64_t>(K) * 2, static_cast<uint64_t>(N) * (g ? g->groups : 1), static_cast<uint64_t>(ldw) * 2, 128)) return -11;
  if (make_tmap_2d_u8(&tx, x, x_cols * 2, rows_total, static_cast<uint64_t>(ldx) * 2, bn)) return -12;
  const dim3 grid(splits, n_tiles, z);
  switch (bn) {
    case 16: return launch_bf16_decode<16, 5>(tw, tx, p, grid, stream);
    case 32: return launch_bf16_decode<32, 4>(tw, tx, p, grid, stream);
    default: return launch_bf16_decode<64, 6>(tw, tx, p, grid, stream);
  }
}

// At most 128 tokens.
extern "C" int b200_bf16_gemm_decode(const void* x, long long ldx, const void* w, long long ldw, int M, int N, int K,
                                     const b200_dense_epilogue* epi, int* status, int num_sms, int splits, cudaStream_t stream) {
  if (M > 128) return -1;
  return bf16_decode_any(x, ldx, w, ldw, M, M, N, K, epi, nullptr, status, num_sms, splits, stream);
}

extern "C" int b200_bf16_gemm_decode_grouped(const void* x, long long ldx, const void* w, long long ldw, int M, int rows_total, int N,
                                             int K, const b200_dense_epilogue* epi, const b200_gemm_groups* g, int* status,
                                             int num_sms, int splits, cudaStream_t stream) {
  if (!g) return -3;
  return bf16_decode_any(x, ldx, w, ldw, M, rows_total, N, K, epi, g, status, num_sms, splits, stream);
}
