// bf16 linear for prefill-sized calls on sm_100a:  v[m,n] = sum_k X[m,k] W[n,k], then a fused epilogue (dense_epilogue.cuh).
//
//   X bf16 [M,K] (row pitch ldx), W bf16 [N,K] (row pitch ldw), fp32 accumulation in TMEM.
//
//   * 128 tokens are the rows of the tcgen05 A operand, BN (64..256) output channels the rows of B; both arrive by TMA
//     (128-byte swizzle, 64 bf16 per k-block) in a STAGES-deep ring.  K need not be a multiple of anything: the tensor
//     maps end at K and fill with zeros.
//   * Persistent grid over whole tiles; the accumulator is double buffered in TMEM, so the epilogue of one tile runs
//     under the main loop of the next.
//   * Warp 0 TMA producer, warp 1 MMA issuer, warps 2..5 epilogue.  An epilogue warp turns its 32 x 32 piece through
//     shared memory, so that eight lanes share one token row and every global access is a run of 128 bytes: the residual
//     form reads and writes fp32 rows.
//   * Grouped form (experts): a table of row tiles names each tile's rows and its group, whose weights are rows
//     group * N .. of one stacked matrix; a column tile that reaches into the next group's rows is cut in the epilogue.
//   * Every wait is bounded; a CTA that gives up records a status code, drains and exits.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "gemm_common.cuh"
#include "dense_epilogue.cuh"

namespace b200 {

constexpr int BG_BK = 64;              // bf16 per k-block: one 128-byte swizzle row
constexpr int BG_GROUP_M = 8;          // token tiles per rasterisation group
constexpr int BG_SP = 36;              // floats per row of an epilogue warp's staging piece (conflict-free 16-byte accesses)

struct BfGemmParams {
  int M, N, m_tiles, n_tiles, kblocks, num_tiles;
  b200_dense_epilogue epi;
  const int4* tiles; const int* tiles_used;      // row lists: {group, first row, rows, 0} per row tile, else NULL
  int* status;
  unsigned long long limit_ns;
};

struct BfTile { int m0, m_end, n_tile, group; };

__device__ __forceinline__ BfTile bg_tile_at(const BfGemmParams& p, int m_tiles, int tile) {
  const int per_group = BG_GROUP_M * p.n_tiles;
  const int g = tile / per_group;
  const int first_m = g * BG_GROUP_M;
  const int gsize = min(BG_GROUP_M, m_tiles - first_m);
  const int r = tile - g * per_group;
  const int m_tile = first_m + r % gsize;
  BfTile t;
  t.n_tile = r / gsize;
  if (p.tiles) {
    const int4 e = p.tiles[m_tile];
    t.group = e.x; t.m0 = e.y; t.m_end = e.y + e.z;
  } else {
    t.group = 0; t.m0 = m_tile * 128; t.m_end = p.M;
  }
  return t;
}

template <int BN, int STAGES>
constexpr int bg_smem_bytes() { return STAGES * (128 + BN) * 128 + 4 * 32 * BG_SP * 4 + 1024 + 256; }

template <int BN, int STAGES>
__global__ void __launch_bounds__(GEMM_THREADS, 1)
bf16_gemm_kernel(const __grid_constant__ CUtensorMap tmap_x, const __grid_constant__ CUtensorMap tmap_w,
                 const __grid_constant__ BfGemmParams p) {
  constexpr int A_BYTES = 128 * 128, B_BYTES = BN * 128, STAGE_BYTES = A_BYTES + B_BYTES;
  constexpr int TMEM_COLS = 2 * BN;
  constexpr uint32_t IDESC = umma_idesc_bf16(128, BN, 0, 0);

  pdl_launch_dependents();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  float* stage_f = reinterpret_cast<float*>(smem + STAGES * STAGE_BYTES);                  // [4 warps][32][BG_SP]
  uint64_t* bars = reinterpret_cast<uint64_t*>(stage_f + 4 * 32 * BG_SP);                  // full, empty, tfull[2], tempty[2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * STAGES + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t smem_base = smem_u32(smem), bar_base = smem_u32(bars);
  auto full_bar = [&](int s) { return bar_base + 8u * s; };
  auto empty_bar = [&](int s) { return bar_base + 8u * (STAGES + s); };
  auto tfull_bar = [&](int a) { return bar_base + 8u * (2 * STAGES + a); };
  auto tempty_bar = [&](int a) { return bar_base + 8u * (2 * STAGES + 2 + a); };

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) { mbar_init(full_bar(s), 1); mbar_init(empty_bar(s), 1); }
    for (int a = 0; a < 2; ++a) { mbar_init(tfull_bar(a), 1); mbar_init(tempty_bar(a), 4); }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(smem_u32(tmem_slot), TMEM_COLS); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint64_t limit = p.limit_ns;
  pdl_wait();                // everything before this kernel in the stream has completed
  const int m_tiles = p.tiles ? min(*p.tiles_used, p.m_tiles) : p.m_tiles;
  const int num_tiles = m_tiles * p.n_tiles;

  if (warp == 0) {
    if (lane == 0) {
      prefetch_tmap(&tmap_x);
      prefetch_tmap(&tmap_w);
      const uint64_t pol_w = p.m_tiles == 1 ? policy_evict_first() : policy_evict_last();
      int stage = 0; uint32_t phase = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x) {
        const BfTile t = bg_tile_at(p, m_tiles, tile);
        const int w0 = t.group * p.N + t.n_tile * BN;
        for (int kb = 0; kb < p.kblocks; ++kb) {
          if (!mbar_wait(empty_bar(stage), phase ^ 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_EMPTY | (9 << 8)), limit)) { ok = false; break; }
          mbar_expect_tx(full_bar(stage), STAGE_BYTES);
          const uint32_t a_dst = smem_base + stage * STAGE_BYTES;
          tma_load_2d(a_dst, &tmap_x, full_bar(stage), kb * 128, t.m0);
          tma_load_2d_hint(a_dst + A_BYTES, &tmap_w, full_bar(stage), kb * 128, w0, pol_w);
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
      }
      if (!ok) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 2000000ull) { } }   // copies in flight land
    }
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      int stage = 0; uint32_t phase = 0;
      int idx = 0;
      bool ok = true;
      for (int tile = blockIdx.x; tile < num_tiles && ok; tile += gridDim.x, ++idx) {
        const int a = idx & 1;
        if (!mbar_wait(tempty_bar(a), ((idx >> 1) & 1u) ^ 1u, abort_flag, p.status, (ST_TIMEOUT_TMEM_EMPTY | (9 << 8)), limit)) { ok = false; break; }
        tc_fence_after();
        const uint32_t d_tmem = tmem_base + a * BN;
        for (int kb = 0; kb < p.kblocks; ++kb) {
          if (!mbar_wait(full_bar(stage), phase, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (9 << 8)), limit)) { ok = false; break; }
          tc_fence_after();
          const uint32_t a_src = smem_base + stage * STAGE_BYTES;
          const uint64_t a_desc = umma_desc_k_sw128(a_src), b_desc = umma_desc_k_sw128(a_src + A_BYTES);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16_ss(d_tmem, a_desc + 2ull * k, b_desc + 2ull * k, IDESC, (kb > 0 || k > 0) ? 1u : 0u);
          umma_commit(empty_bar(stage));
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
        if (ok) umma_commit(tfull_bar(a));
      }
    }
    __syncwarp();
  } else {
    const int q = warp & 3;                 // TMEM lane quarter this warp may read
    float* piece = stage_f + (warp - 2) * 32 * BG_SP;
    int idx = 0;
    const bool residual = p.epi.mode == B200_EPI_RESIDUAL, plain = p.epi.mode == B200_EPI_STORE && !p.epi.gate;
    const bool plain16 = plain && !p.epi.out_f32, relu2 = p.epi.act == B200_ACT_RELU2;
    const int r8 = lane >> 2, c8 = (lane & 3) * 8;           // the same with eight columns per lane
    const int rr0 = lane >> 3, c4 = (lane & 7) * 4;          // row group and column quad of this lane in a 32 x 32 piece
    for (int tile = blockIdx.x; tile < num_tiles; tile += gridDim.x, ++idx) {
      const int a = idx & 1;
      const BfTile t = bg_tile_at(p, m_tiles, tile);
      const int m0 = t.m0 + q * 32, n0 = t.n_tile * BN;
      // The residual rows of a piece are requested one piece ahead (the first even before the accumulator is complete):
      // the epilogue is four warps, so what it needs is loads in flight.
      float4 xn[8];
      auto load_x = [&](int c) {
        const int n = n0 + c * 32 + c4;
#pragma unroll
        for (int it = 0; it < 8; ++it) {
          const int m = m0 + it * 4 + rr0;
          if (m < t.m_end && n < p.N) xn[it] = *reinterpret_cast<const float4*>(p.epi.x + static_cast<long long>(m) * p.epi.ldx + n);
        }
      };
      if (residual) load_x(0);
      // one verdict per warp: the lanes stay together at the TMEM loads
      const bool ok = __all_sync(0xffffffffu, mbar_wait(tfull_bar(a), (idx >> 1) & 1u, abort_flag, p.status, (ST_TIMEOUT_TMEM_FULL | (9 << 8)), limit));
      if (!ok) break;
      tc_fence_after();
      const uint32_t t_addr = tmem_base + (static_cast<uint32_t>(q * 32) << 16) + a * BN;
#pragma unroll 1
      for (int c = 0; c < BN / 32; ++c) {
        if (n0 + c * 32 >= p.N) break;
        uint32_t r[32];
        tmem_ld_x32(t_addr + c * 32, r);
        float4 xc[8];
        if (residual) {
#pragma unroll
          for (int it = 0; it < 8; ++it) xc[it] = xn[it];
          if (c + 1 < BN / 32) load_x(c + 1);
        }
        tmem_ld_wait();
        float* mine = piece + lane * BG_SP;
#pragma unroll
        for (int g = 0; g < 8; ++g)
          *reinterpret_cast<float4*>(mine + 4 * g) = make_float4(__uint_as_float(r[4 * g]), __uint_as_float(r[4 * g + 1]),
                                                                 __uint_as_float(r[4 * g + 2]), __uint_as_float(r[4 * g + 3]));
        __syncwarp();
        const int n = n0 + c * 32 + c4;
        if (plain16) {
          const int n8 = n0 + c * 32 + c8;
          if (n8 < p.N) {
            __nv_bfloat16* y = static_cast<__nv_bfloat16*>(p.epi.y) + static_cast<long long>(m0 + r8) * p.epi.ldy + n8;
#pragma unroll
            for (int it = 0; it < 4; ++it) {
              const float* src = piece + (it * 8 + r8) * BG_SP + c8;
              float v[8];
              *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(src);
              *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(src + 4);
              if (relu2) {
#pragma unroll
                for (int k = 0; k < 8; ++k) { v[k] = fmaxf(v[k], 0.f); v[k] *= v[k]; }
              }
              uint4 o;
              uint32_t* ow = reinterpret_cast<uint32_t*>(&o);
#pragma unroll
              for (int k = 0; k < 4; ++k) {
                const __nv_bfloat162 pb = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
                ow[k] = *reinterpret_cast<const uint32_t*>(&pb);
              }
              if (m0 + it * 8 + r8 < t.m_end) *reinterpret_cast<uint4*>(y + static_cast<long long>(it * 8) * p.epi.ldy) = o;
            }
          }
        } else if (plain) {
          if (n < p.N) {
            float* y = static_cast<float*>(p.epi.y) + static_cast<long long>(m0 + rr0) * p.epi.ldy + n;
#pragma unroll
            for (int it = 0; it < 8; ++it) {
              float4 v = *reinterpret_cast<const float4*>(piece + (it * 4 + rr0) * BG_SP + c4);
              if (relu2) {
                v.x = fmaxf(v.x, 0.f); v.y = fmaxf(v.y, 0.f); v.z = fmaxf(v.z, 0.f); v.w = fmaxf(v.w, 0.f);
                v.x *= v.x; v.y *= v.y; v.z *= v.z; v.w *= v.w;
              }
              if (m0 + it * 4 + rr0 < t.m_end) *reinterpret_cast<float4*>(y + static_cast<long long>(it * 4) * p.epi.ldy) = v;
            }
          }
        } else if (n < p.N) {
          if (residual) {
            const EpiNorm nw = epi_norm_columns(p.epi, n);
#pragma unroll
            for (int it = 0; it < 8; ++it) {
              const int rr = it * 4 + rr0, m = m0 + rr;
              if (m < t.m_end) epi_residual4(p.epi, nw, m, n, *reinterpret_cast<const float4*>(piece + rr * BG_SP + c4), xc[it]);
            }
          } else {
#pragma unroll
            for (int it = 0; it < 8; ++it) {
              const int rr = it * 4 + rr0, m = m0 + rr;
              if (m < t.m_end) epi_apply4(p.epi, m, n, *reinterpret_cast<const float4*>(piece + rr * BG_SP + c4), t.group);
            }
          }
        }
        __syncwarp();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(tempty_bar(a));
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, TMEM_COLS); }
}

template <int BN, int STAGES>
static int launch_bf16_gemm(const CUtensorMap& tx, const CUtensorMap& tw, const BfGemmParams& p, int grid, cudaStream_t stream) {
  constexpr int SMEM = bg_smem_bytes<BN, STAGES>();
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(bf16_gemm_kernel<BN, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return -1000 - static_cast<int>(e);
    configured = true;
  }
  launch_ex(bf16_gemm_kernel<BN, STAGES>, dim3(grid), dim3(GEMM_THREADS), SMEM, stream, 0, tx, tw, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

// shared with the decode form: everything epi_apply4 relies on
int dense_epilogue_check(const b200_dense_epilogue* e, int N) {
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const int n4 = (N + 3) & ~3;
  if (!e) return -3;
  if (e->mode == B200_EPI_STORE) return (e->y && al16(e->y) && e->ldy >= n4 && e->ldy % 8 == 0) ? 0 : -4;
  if (e->mode == B200_EPI_GLU) return (e->y && al16(e->y) && N % 2 == 0 && e->ldy >= n4 / 2 && e->ldy % 8 == 0) ? 0 : -5;
  if (e->mode != B200_EPI_RESIDUAL) return -6;
  if (!e->x || !al16(e->x) || e->ldx < n4 || e->ldx % 4 || !al16(e->add)) return -7;
  if (e->y && (!al16(e->y) || e->ldy < n4 || e->ldy % 8 || !e->norm_w || !e->norm_b || !al16(e->norm_w) || !al16(e->norm_b))) return -8;
  return 0;
}

}  // namespace b200

using namespace b200;

// g NULL: one linear over M rows; else row lists over M = rows of x
static int bf16_gemm_any(const void* x, long long ldx, const void* w, long long ldw, int M, int N, int K, const b200_dense_epilogue* epi,
                         const b200_gemm_groups* g, int* status, int num_sms, int force_bn, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (N <= 0 || K <= 0 || ldx < K || ldw < K || (ldx % 8) || (ldw % 8)) return -1;
  if ((reinterpret_cast<uintptr_t>(x) & 15) || (reinterpret_cast<uintptr_t>(w) & 15)) return -2;
  if (int rc = dense_epilogue_check(epi, N)) return rc;
  if (g && (g->groups <= 0 || !g->tiles || !g->num_tiles || g->max_tiles <= 0 || epi->mode != B200_EPI_STORE)) return -3;
  BfGemmParams p;
  p.M = M; p.N = N;
  p.m_tiles = g ? g->max_tiles : (M + 127) / 128;
  p.tiles = g ? static_cast<const int4*>(g->tiles) : nullptr;
  p.tiles_used = g ? g->num_tiles : nullptr;
  // row lists: a partly filled tile per group on top of the full ones is what to expect
  const int likely = g ? M / 128 + (g->expected > 0 ? g->expected : g->groups) : p.m_tiles;
  int bn = force_bn;
  if (bn != 64 && bn != 128 && bn != 256) {
    long long best_cost = -1;
    for (int cand : {256, 128, 64}) {
      const long long tiles = static_cast<long long>(likely) * ((N + cand - 1) / cand);
      const long long cost = (tiles + num_sms - 1) / num_sms * (cand + 64);
      if (best_cost < 0 || cost < best_cost) { best_cost = cost; bn = cand; }
    }
  }
  p.n_tiles = (N + bn - 1) / bn;
  p.kblocks = (K + BG_BK - 1) / BG_BK;
  p.num_tiles = p.m_tiles * p.n_tiles;
  p.epi = *epi;
  p.status = status;
  p.limit_ns = 2000000000ull;
  CUtensorMap tx, tw;
  if (make_tmap_2d_u8(&tx, x, static_cast<uint64_t>(K) * 2, M, static_cast<uint64_t>(ldx) * 2, 128)) return -11;
  if (make_tmap_2d_u8(&tw, w, static_cast<uint64_t>(K) * 2, static_cast<uint64_t>(N) * (g ? g->groups : 1), static_cast<uint64_t>(ldw) * 2, bn)) return -12;
  const int grid = p.num_tiles < num_sms ? p.num_tiles : num_sms;
  switch (bn) {
    case 64: return launch_bf16_gemm<64, 8>(tx, tw, p, grid, stream);
    case 128: return launch_bf16_gemm<128, 6>(tx, tw, p, grid, stream);
    default: return launch_bf16_gemm<256, 4>(tx, tw, p, grid, stream);
  }
}

extern "C" int b200_bf16_gemm(const void* x, long long ldx, const void* w, long long ldw, int M, int N, int K,
                              const b200_dense_epilogue* epi, int* status, int num_sms, int force_bn, cudaStream_t stream) {
  return bf16_gemm_any(x, ldx, w, ldw, M, N, K, epi, nullptr, status, num_sms, force_bn, stream);
}

extern "C" int b200_bf16_gemm_grouped(const void* x, long long ldx, const void* w, long long ldw, int rows_total, int N, int K,
                                      const b200_dense_epilogue* epi, const b200_gemm_groups* g, int* status, int num_sms,
                                      int force_bn, cudaStream_t stream) {
  if (!g) return -3;
  return bf16_gemm_any(x, ldx, w, ldw, rows_total, N, K, epi, g, status, num_sms, force_bn, stream);
}
