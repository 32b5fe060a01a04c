// Latent attention over the paged cache in the latent space (bf16, tcgen05): queries that were moved there against the cached
// latents and the shared rotated key part, for decoding and for short portions.  All heads read the same keys and a key's first
// `rank` dimensions are also its value, so a cached row is fetched once, by TMA, and serves both products from shared memory.
//
// Rows are (token, head) pairs of one portion in order, N = 16 or 32 of them per CTA.  So few rows would waste the MMA's 128, so
// the keys take that side:  S^T [keys, N] = C [keys, dk] . Q^T,   O^T [rank, N] = C^T [rank, keys] . P^T in blocks of 128 value
// dimensions - the same operand tile, once K-major and once MN-major.  Tiles are 128 keys (512 + 64 columns x 128 keys are
// 144 KB) where the queries leave room for one, else 64: the score MMA then still has 128 rows, and the upper half, whatever lies
// behind the operand, is never read back.
//   warps 0, 1  TMA producers, each for one of a slot's two 64-column chunks (a page is a box of its own and issuing one takes
//               some 50 cycles, so one warp alone cannot feed an SM): a tile is 8 or 4 pages, in slots of 128 latent columns and one of the rotated part, each
//               released as soon as its last product is done (rings).  In decoding the tiles of earlier tokens are requested before the dependency
//               wait: only the new token's row is written by a kernel that may still run.
//   warp 2      MMA issuer; the scores of the next tile go before the values of this one as far as its slots are there (entirely
//               where two tiles fit)
//   warps 3..10 softmax with keys on the lanes: a warp holds 32 keys of half the rows; maxima by warp reduction and through
//               shared memory, sums stay with their keys until the end.  They also turn the queries' second part, and keep the
//               accumulated values (128 dimensions x N per block) in registers.
// The splits of one row tile are a thread-block cluster that merges through distributed shared memory.  All waits are bounded.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "gemm_common.cuh"

namespace b200 {

constexpr int AL_THREADS = 352, AL_SOFTMAX = 256, AL_SOFTMAX0 = 96, AL_PS = 16;
constexpr int AL_MAX_SMEM = 232448, AL_MAX_SLOTS = 12, AL_MAX_ROT = 3;
constexpr float AL_LOG2E = 1.4426950408889634f;

struct AttnLatentParams {
  const __nv_bfloat16* q_rot; long long ldr; int head_ld_rot;
  __nv_bfloat16* out; long long ldo;
  b200_latent_dims d;
  float scale_log2;
  const int* cu; const int* positions; const int* seq_ids; const int* seq_lens;
  const float* cos_tab; const float* sin_tab;
  int max_pos, splits, slots, rot_slots, ahead;
  b200_paged_cache c;
  int* status;
  unsigned long long limit_ns;
};

__device__ __forceinline__ float al_ld_cluster(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ float4 al_ld_cluster4(uint32_t addr) {
  float4 v;
  asm volatile("ld.shared::cluster.v4.f32 {%0,%1,%2,%3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
  return v;
}
// integers in the order of the floats they come from
__device__ __forceinline__ int al_order(int i) { return i ^ ((i >> 31) & 0x7fffffff); }
__device__ __forceinline__ float al_warp_max(float v) {
  return __int_as_float(al_order(__reduce_max_sync(0xffffffffu, al_order(__float_as_int(v)))));
}
// element (row, key) of a K-major operand with 128-byte swizzle: rows of 64 elements, eight rows per 1024 bytes
__device__ __forceinline__ uint32_t al_swizzled(int row, int col) {
  return (row >> 3) * 1024 + (row & 7) * 128 + (((col >> 3) ^ (row & 7)) << 4) + (col & 7) * 2;
}

template <int N>
struct AlShared {      // behind the operands
  float red[2][4][N];  // maxima of the four key quarters, two turns
  float alpha[2][N];
  float m[N], l[N], lw[4][N];
  float f[8][N];       // factor of every split
  int pos[N];
  uint64_t bars[2 * AL_MAX_SLOTS + 2 * AL_MAX_ROT + 8];
  uint32_t tmem;
  int abort;
};

template <int N, int KEYS>
__global__ void __launch_bounds__(AL_THREADS, 1)
attn_latent_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_c,
                   const __grid_constant__ CUtensorMap tmap_r, const __grid_constant__ AttnLatentParams p) {
  constexpr int NC = N / 2;                              // columns of a softmax thread
  constexpr int AL_KEYS = KEYS, AL_CHUNK = KEYS * 128, AL_SLOT = 2 * AL_CHUNK, PAGES = KEYS / AL_PS;      // chunk: 64 bf16 of every key
  constexpr int PCHUNKS = KEYS / 64;                     // 64-key chunks of the softmax weights
  constexpr int QCHUNK = N * 128, TMEM_COLS = N == 32 ? 512 : 256, TMEM_O = 2 * N;
  pdl_launch_dependents();
  if (p.cu) pdl_wait();                                  // decoding: page table, positions and earlier rows are older than this step
  extern __shared__ __align__(1024) uint8_t al_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.d.heads, rank = p.d.rank, rot = p.d.rot;
  const int nd = (rank + 127) >> 7, kq = (rank + 63) >> 6, rc = (rot + 63) >> 6;      // slots per tile, chunks of each part
  const int b = blockIdx.z, S = p.splits, split = blockIdx.x, g0 = blockIdx.y * N;
  const int row0 = p.cu ? p.cu[b] : b, len = p.cu ? p.cu[b + 1] - row0 : 1;
  if (g0 >= len * H) return;                             // the same for all CTAs of the cluster, as below
  const int n_rows = min(N, len * H - g0);
  const int start = p.positions[row0], seq = p.seq_ids ? p.seq_ids[row0] : b;
  const int last_pos = start + (g0 + n_rows - 1) / H;
  const bool empty = p.seq_lens && p.seq_lens[b] <= 0;
  const bool bad = start < 0 || last_pos >= p.max_pos || seq < 0 || seq >= p.c.num_seqs || last_pos / AL_PS >= p.c.max_pages;
  if (empty || bad) {
    if (bad && tid == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (18 << 8));
    pdl_wait();
    if (split == 0)
      for (int i = tid; i < n_rows * rank; i += AL_THREADS) {
        const int g = g0 + i / rank, tok = g / H;
        p.out[static_cast<size_t>(row0 + tok) * p.ldo + static_cast<size_t>(g - tok * H) * rank + i % rank] = __float2bfloat16(0.f);
      }
    return;
  }
  const uint32_t sC = smem_u32(al_smem), sR = sC + p.slots * AL_SLOT, sQ = sR + p.rot_slots * rc * AL_CHUNK, sP = sQ + (kq + rc) * QCHUNK;
  uint8_t* pQr = al_smem + (sQ - sC) + kq * QCHUNK;
  uint8_t* pP = al_smem + (sP - sC);
  AlShared<N>& sh = *reinterpret_cast<AlShared<N>*>(pP + (p.ahead ? 2 : 1) * PCHUNKS * QCHUNK);
  const uint32_t bar0 = smem_u32(sh.bars);
  enum { B_Q = 0, B_QROT = 1, B_SFULL = 2, B_PFULL = 4, B_OFULL = 5, B_RFULL = 7, B_REMPTY = 7 + AL_MAX_ROT, B_CFULL = 7 + 2 * AL_MAX_ROT,
         B_CEMPTY = B_CFULL + AL_MAX_SLOTS, B_COUNT = B_CEMPTY + AL_MAX_SLOTS };
  auto bar = [&](int i) { return bar0 + 8u * i; };
  volatile int* abort_flag = &sh.abort;
  const uint64_t limit = p.limit_ns;

  const int n_tiles = last_pos / AL_KEYS + 1;
  const int ta = static_cast<int>(static_cast<long long>(n_tiles) * split / S), nt = static_cast<int>(static_cast<long long>(n_tiles) * (split + 1) / S) - ta;

  if (tid == 0) {
    for (int i = 0; i < B_COUNT; ++i) mbar_init(bar(i), i == B_PFULL || i == B_QROT ? AL_SOFTMAX / 32 : (i >= B_CFULL && i < B_CEMPTY) || (i >= B_RFULL && i < B_REMPTY) ? 2 : 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (tid < N) sh.pos[tid] = start + min(g0 + tid, len * H - 1) / H;
  if (warp == 2) { tmem_alloc(smem_u32(&sh.tmem), TMEM_COLS); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = sh.tmem;

  float o[2][N];                                         // softmax warps: value dimensions x rows, blocks half and half + 2
#pragma unroll
  for (int i = 0; i < N; ++i) o[0][i] = o[1][i] = 0.f;

  if (warp < 2) {
    const int* pt = p.c.page_table + static_cast<size_t>(seq) * p.c.max_pages;
    auto page_of = [&](int t) {                          // lane <-> page of tile t; past the last key: out of range, arrives as zeros
      const int tok = t * AL_KEYS + (lane % PAGES) * AL_PS;
      const int pg = tok <= last_pos ? pt[tok / AL_PS] : p.c.num_pages;
      return pg < 0 || pg > p.c.num_pages ? p.c.num_pages : pg;
    };
    if (lane == 0) { prefetch_tmap(&tmap_c); prefetch_tmap(&tmap_r); }
    bool waited = p.cu != nullptr, ok = true;
    int cs = 0, rs = 0;
    uint32_t cp = 0, rp = 0;
    int page = nt > 0 ? page_of(ta) : 0;
    // one chunk (if this warp has one of this slot) of the tile's pages
    auto fetch = [&](int full, int empty_bar, uint32_t phase, uint32_t dst, const CUtensorMap* map, int chunk, int chunks) -> bool {
      if (!__all_sync(0xffffffffu, mbar_wait(bar(empty_bar), phase ^ 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_EMPTY | (18 << 8)), limit))) return false;
      const bool has = chunk < chunks;
      if (lane == 0) { if (has) mbar_expect_tx(bar(full), AL_CHUNK); else mbar_arrive(bar(full)); }
      __syncwarp();
      if (has && lane < PAGES) tma_load_3d(dst + warp * AL_CHUNK + lane * 2048, map, bar(full), chunk * 64, 0, page);
      return true;
    };
    for (int j = 0; j < nt && ok; ++j) {
      if (!waited && (ta + j + 1) * AL_KEYS > last_pos) { pdl_wait(); waited = true; }      // holds the new token
      const int next = j + 1 < nt ? page_of(ta + j + 1) : 0;
      if (rc > 0) {
        ok = fetch(B_RFULL + rs, B_REMPTY + rs, rp, sR + rs * rc * AL_CHUNK, &tmap_r, warp, rc);
        if (++rs == p.rot_slots) { rs = 0; rp ^= 1u; }
      }
      for (int d = 0; d < nd && ok; ++d) {
        ok = fetch(B_CFULL + cs, B_CEMPTY + cs, cp, sC + cs * AL_SLOT, &tmap_c, 2 * d + warp, kq);
        if (++cs == p.slots) { cs = 0; cp ^= 1u; }
      }
      page = next;
    }
    if (!ok) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 2000000ull) { } }   // copies in flight land
    if (!waited) pdl_wait();
    __syncwarp();
  } else if (warp == 2) {
    pdl_wait();
    // The whole warp walks the loops, so that descriptors stay in uniform registers; one elected thread issues.
    if (nt > 0) {
      const bool one = elect_one();
      constexpr uint32_t IDESC_S = umma_idesc_bf16(128, N, 0, 0), IDESC_O = umma_idesc_bf16(128, N, 1, 0);      // C^T is MN-major
      if (one) mbar_expect_tx(bar(B_Q), kq * QCHUNK);
      for (int c = 0; c < kq; ++c) if (one) tma_load_3d(sQ + c * QCHUNK, &tmap_q, bar(B_Q), c * 64, row0 * H + g0, 0);
      const int c_steps = (rank + 15) >> 4, r_steps = (rot + 15) >> 4;
      int cs = 0, rs = 0, vs = 0;                        // slots: scores read cs, values vs
      uint32_t cp = 0, rp = 0;
      // One thread issues everything, so a descriptor must cost an addition: bases here, offsets known at compile time below
      // (the address field counts 16 bytes).
      const uint64_t c_desc = umma_desc_k_sw128(sC), ct_desc = umma_desc_mn_sw128(sC, AL_CHUNK, 1024), r_desc = umma_desc_k_sw128(sR),
                     q_desc = umma_desc_k_sw128(sQ), qr_desc = umma_desc_k_sw128(sQ + kq * QCHUNK), p_desc = umma_desc_k_sw128(sP);
      // Scores of tile j: (first:) the rotated part, and slots [d0, d1).  A tile's first slots are there before the values of the tile before
      // have freed the others, so their products go first.
      auto issue_s = [&](int j, bool first, int d0, int d1) -> bool {
        const uint32_t d_tmem = tmem_base + (j & 1) * N;
        if (first && rc > 0) {
          if (!mbar_wait(bar(B_RFULL + rs), rp, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (18 << 8)), limit)) return false;
          tc_fence_after();
          const uint64_t a = r_desc + static_cast<uint32_t>(rs * rc * (AL_CHUNK >> 4));
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            if (kk < r_steps && one)
              umma_f16_ss(d_tmem, a + ((kk >> 2) * (AL_CHUNK >> 4) + 2 * (kk & 3)), qr_desc + ((kk >> 2) * (QCHUNK >> 4) + 2 * (kk & 3)), IDESC_S, kk > 0 ? 1u : 0u);
          if (one) umma_commit(bar(B_REMPTY + rs));
          if (++rs == p.rot_slots) { rs = 0; rp ^= 1u; }
        }
        for (int d = d0; d < d1; ++d) {
          if (!mbar_wait(bar(B_CFULL + cs), cp, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (18 << 8)), limit)) return false;
          tc_fence_after();
          const int steps = c_steps - 8 * d;
          const uint64_t a = c_desc + static_cast<uint32_t>(cs * (AL_SLOT >> 4)), bq = q_desc + static_cast<uint32_t>(d * (2 * QCHUNK >> 4));
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            if (kk < steps && one)
              umma_f16_ss(d_tmem, a + ((kk >> 2) * (AL_CHUNK >> 4) + 2 * (kk & 3)), bq + ((kk >> 2) * (QCHUNK >> 4) + 2 * (kk & 3)), IDESC_S,
                          kk > 0 || rc > 0 || d > 0 ? 1u : 0u);
          if (++cs == p.slots) { cs = 0; cp ^= 1u; }
        }
        if (d1 == nd && one) umma_commit(bar(B_SFULL + (j & 1)));
        return true;
      };
      const int early = p.ahead ? nd : min(nd - 1, p.slots - nd);
      bool ok = mbar_wait(bar(B_Q), 0, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (18 << 8)), limit) &&
                mbar_wait(bar(B_QROT), 0, abort_flag, p.status, (ST_TIMEOUT_PEER_FLAG | (18 << 8)), limit);
      if (ok) { tc_fence_after(); ok = issue_s(0, true, 0, nd); }
      for (int j = 0; j < nt && ok; ++j) {
        if (j + 1 < nt && !issue_s(j + 1, true, 0, early)) { ok = false; break; }
        if (!mbar_wait(bar(B_PFULL), j & 1u, abort_flag, p.status, (ST_TIMEOUT_PEER_FLAG | (18 << 8)), limit)) { ok = false; break; }
        tc_fence_after();
        const uint64_t bp = p_desc + (p.ahead ? static_cast<uint32_t>((j & 1) * (PCHUNKS * QCHUNK >> 4)) : 0u);
        for (int d = 0; d < nd; ++d) {
          const uint32_t d_tmem = tmem_base + TMEM_O + ((j & 1) * 4 + d) * N;
          const uint64_t a = ct_desc + static_cast<uint32_t>(vs * (AL_SLOT >> 4));
#pragma unroll
          for (int kk = 0; kk < KEYS / 16; ++kk)
            if (one) umma_f16_ss(d_tmem, a + kk * (2048 >> 4), bp + ((kk >> 2) * (QCHUNK >> 4) + 2 * (kk & 3)), IDESC_O, kk > 0 ? 1u : 0u);
          if (one) umma_commit(bar(B_CEMPTY + vs));
          if (++vs == p.slots) vs = 0;
        }
        if (one) umma_commit(bar(B_OFULL + (j & 1)));
        if (early < nd && j + 1 < nt && !issue_s(j + 1, false, early, nd)) { ok = false; break; }
      }
    }
    __syncwarp();
  } else {
    pdl_wait();
    const int qd = warp & 3, half = (warp - 3) >> 2, c0 = half * NC;      // key quarter = TMEM lane quarter; first column
    const int st = tid - AL_SOFTMAX0;
    // the queries' rotated part; columns up to the end of its chunks and rows beyond the portion are zero
    const int np = p.d.true_rot / 2, wide = rc * 32;
    for (int i = st; i < N * wide; i += AL_SOFTMAX) {
      const int r = i / wide, j = i - r * wide, g = g0 + r, tok = g / H;
      float u = 0.f, v = 0.f;
      if (r < n_rows && j < np) {
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(p.q_rot + static_cast<size_t>(row0 + tok) * p.ldr + static_cast<size_t>(g - tok * H) * p.head_ld_rot + 2 * j);
        const float c = p.cos_tab[static_cast<size_t>(start + tok) * np + j], s = p.sin_tab[static_cast<size_t>(start + tok) * np + j];
        const float a = __low2float(x), e = __high2float(x);
        u = a * c - e * s;
        v = e * c + a * s;
      }
      *reinterpret_cast<__nv_bfloat162*>(pQr + (j >> 5) * QCHUNK + al_swizzled(r, (2 * j) & 63)) = __floats2bfloat162_rn(u, v);
    }
    fence_proxy_async_smem();
    __syncwarp();
    if (lane == 0) mbar_arrive(bar(B_QROT));

    const uint32_t t_lane = tmem_base + (static_cast<uint32_t>(qd * 32) << 16);
    float m_run[NC], l_run[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) { m_run[i] = -INFINITY; l_run[i] = 0.f; }
    bool ok = true;
    auto wait_all = [&](int i, uint32_t par) {           // one verdict per warp: the TMEM loads need all lanes
      return __all_sync(0xffffffffu, mbar_wait(bar(i), par, abort_flag, p.status, (ST_TIMEOUT_TMEM_FULL | (18 << 8)), limit)) != 0;
    };
    auto o_update = [&](int j) -> bool {
      if (!wait_all(B_OFULL + (j & 1), (j >> 1) & 1u)) return false;
      tc_fence_after();
      const float4* al = reinterpret_cast<const float4*>(sh.alpha[j & 1]);
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int d = half + 2 * k;
        if (d < nd) {
          uint32_t v[N];
          if constexpr (N == 32) tmem_ld_x32(t_lane + TMEM_O + ((j & 1) * 4 + d) * N, v);
          else tmem_ld_x16(t_lane + TMEM_O + ((j & 1) * 4 + d) * N, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < N / 4; ++i) {
            const float4 a = al[i];
            o[k][4 * i] = o[k][4 * i] * a.x + __uint_as_float(v[4 * i]);
            o[k][4 * i + 1] = o[k][4 * i + 1] * a.y + __uint_as_float(v[4 * i + 1]);
            o[k][4 * i + 2] = o[k][4 * i + 2] * a.z + __uint_as_float(v[4 * i + 2]);
            o[k][4 * i + 3] = o[k][4 * i + 3] * a.w + __uint_as_float(v[4 * i + 3]);
          }
        }
      }
      tc_fence_before();
      return true;
    };
    const int first_pos = start + g0 / H, key_in_chunk = (qd & 1) * 32 + lane;
    uint8_t* p_chunk = pP + (qd >> 1) * QCHUNK;
    // A warp whose wait fails still meets the others at the barriers: every turn has one, whatever happened before.
    for (int j = 0; j < nt; ++j) {
      const int turn = j & 1;
      ok = ok && wait_all(B_SFULL + turn, (j >> 1) & 1u);
      float v[NC];
      const int tile0 = (ta + j) * AL_KEYS, key = tile0 + qd * 32 + lane;
      if (ok) tc_fence_after();
      const bool mine_here = qd < KEYS / 32;             // the upper lanes of a 64-key tile hold nothing
      if (ok && mine_here) {
        uint32_t raw[NC];
        if constexpr (NC == 16) tmem_ld_x16(t_lane + turn * N + c0, raw); else tmem_ld_x8(t_lane + turn * N + c0, raw);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < NC; ++i) v[i] = __uint_as_float(raw[i]) * p.scale_log2;
        if (tile0 + AL_KEYS - 1 > first_pos) {
#pragma unroll
          for (int i = 0; i < NC; ++i) if (key > sh.pos[c0 + i]) v[i] = -INFINITY;
        }
        float mine = -INFINITY;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
          const float m = al_warp_max(v[i]);
          if (lane == i) mine = m;
        }
        if (lane < NC) sh.red[turn][qd][c0 + lane] = mine;
      }
      named_bar_sync(1, AL_SOFTMAX);
      if (!ok) continue;
      float a_mine = 0.f;
#pragma unroll
      for (int i = 0; i < NC; i += 4) {
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int q = 0; q < KEYS / 32; ++q) {
          const float4 x = *reinterpret_cast<const float4*>(&sh.red[turn][q][c0 + i]);
          mx[0] = fmaxf(mx[0], x.x); mx[1] = fmaxf(mx[1], x.y); mx[2] = fmaxf(mx[2], x.z); mx[3] = fmaxf(mx[3], x.w);
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int c = i + k;
          const float m_new = fmaxf(m_run[c], mx[k]), m_use = m_new == -INFINITY ? 0.f : m_new;
          const float alpha = m_run[c] == -INFINITY ? 0.f : exp2f(m_run[c] - m_use);
          m_run[c] = m_new;
          if (lane == c) a_mine = alpha;
          if (mine_here) {
            const __nv_bfloat16 e = __float2bfloat16(exp2f(v[c] - m_use));
            l_run[c] = l_run[c] * alpha + __bfloat162float(e);           // what the MMA will actually see
            *reinterpret_cast<__nv_bfloat16*>(p_chunk + (p.ahead ? turn * PCHUNKS * QCHUNK : 0) + al_swizzled(c0 + c, key_in_chunk)) = e;
          }
        }
      }
      if (qd == 0 && lane < NC) sh.alpha[turn][c0 + lane] = a_mine;
      tc_fence_before();
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(B_PFULL));          // one arrival per warp: they queue up at the barrier
      if (j > 0 && !o_update(j - 1)) ok = false;
    }
    named_bar_sync(1, AL_SOFTMAX);                       // the last turn's factors are written
    if (ok && nt > 0) ok = o_update(nt - 1);
#pragma unroll
    for (int i = 0; i < NC; ++i) {
#pragma unroll
      for (int w = 16; w > 0; w >>= 1) l_run[i] += __shfl_xor_sync(0xffffffffu, l_run[i], w);
      if (lane == i) {
        sh.lw[qd][c0 + i] = l_run[i];
        if (qd == 0) sh.m[c0 + i] = m_run[i];
      }
    }
  }
  tc_fence_before();
  __syncthreads();                                       // all products are done: the rings become the merge buffer
  float* obuf = reinterpret_cast<float*>(al_smem);
  const int OP = rank + 4;
  if (warp >= 3) {
    const int half = (warp - 3) >> 2, at = (warp & 3) * 32 + lane;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int dim = (half + 2 * k) * 128 + at;
      if (dim < rank) {
#pragma unroll
        for (int i = 0; i < N; ++i) obuf[i * OP + dim] = o[k][i];
      }
    }
    const int c = tid - AL_SOFTMAX0;
    if (c < N) sh.l[c] = sh.lw[0][c] + sh.lw[1][c] + sh.lw[2][c] + sh.lw[3][c];
  } else if (warp == 2) {
    tc_fence_after();
    tmem_dealloc(tmem_base, TMEM_COLS);
  }
  __syncwarp();
  if (S > 1) cluster_sync_all(); else __syncthreads();
  if (tid < n_rows) {                                    // the row's factor for every split
    const uint32_t ma = smem_u32(&sh.m[tid]), la = smem_u32(&sh.l[tid]);
    float ms[8], ls[8], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      ms[s] = s < S ? al_ld_cluster(mapa_shared(ma, s)) : -INFINITY;
      ls[s] = s < S ? al_ld_cluster(mapa_shared(la, s)) : 0.f;
    }
#pragma unroll
    for (int s = 0; s < 8; ++s) m = fmaxf(m, ms[s]);
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      ms[s] = ms[s] == -INFINITY ? 0.f : exp2f(ms[s] - m);
      l += ms[s] * ls[s];
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int s = 0; s < 8; ++s) if (s < S) sh.f[s][tid] = ms[s] * inv;
  }
  __syncthreads();
  const int quads = rank >> 2;
  for (int i = split * AL_THREADS + tid; i < n_rows * quads; i += S * AL_THREADS) {
    const int r = i / quads, d = (i - r * quads) * 4, g = g0 + r, tok = g / H;
    const uint32_t at = smem_u32(obuf + r * OP + d);
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < 8; ++s)
      if (s < S) {
        const float f = sh.f[s][r];
        const float4 x = al_ld_cluster4(mapa_shared(at, s));
        v.x += f * x.x; v.y += f * x.y; v.z += f * x.z; v.w += f * x.w;
      }
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p.out + static_cast<size_t>(row0 + tok) * p.ldo + static_cast<size_t>(g - tok * H) * rank + d) =
        make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  }
  if (S > 1) cluster_sync_all();                         // no CTA leaves while a peer may still read its partials
}

struct AlPlan { int keys, slots, rot_slots, ahead, smem; };

// tile and rings that fit; false: sizes beyond the kernel
static bool al_plan(int rank, int rot, int n, AlPlan& plan) {
  if (rank <= 0 || rank > 512 || rot < 0 || rot > 128 || rank % 8 || rot % 8) return false;
  const int nd = (rank + 127) / 128, kq = (rank + 63) / 64, rc = (rot + 63) / 64;
  const int tail = n == 16 ? static_cast<int>(sizeof(AlShared<16>)) : static_cast<int>(sizeof(AlShared<32>));
  for (int keys = 128; keys >= 64; keys /= 2)
    for (int ahead = 1; ahead >= 0; --ahead) {
      auto bytes = [&](int slots, int rs) { return slots * keys * 256 + rs * rc * keys * 128 + (kq + rc) * n * 128 + (ahead ? 2 : 1) * (keys / 64) * n * 128 + tail; };
      int slots = ahead ? 2 * nd : nd, rs = 1;
      if (bytes(slots, rs) > AL_MAX_SMEM) continue;
      // a spare slot first, then a second tile of the rotated part; a third one only beside a third tile of latents
      while (true) {
        if (rs < 2 && slots > nd && bytes(slots, rs + 1) <= AL_MAX_SMEM) ++rs;
        else if (slots < AL_MAX_SLOTS && bytes(slots + 1, rs) <= AL_MAX_SMEM) ++slots;
        else if (rs < AL_MAX_ROT && slots >= 3 * nd && bytes(slots, rs + 1) <= AL_MAX_SMEM) ++rs;
        else break;
      }
      plan = {keys, slots, rs, ahead, bytes(slots, rs)};
      return n * (rank + 4) * 4 <= slots * keys * 256;
    }
  return false;
}

template <int N, int KEYS>
static int launch_attn_latent(const CUtensorMap& tq, const CUtensorMap& tc, const CUtensorMap& tr, const AttnLatentParams& p, dim3 grid, int smem, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_latent_kernel<N, KEYS>, cudaFuncAttributeMaxDynamicSharedMemorySize, AL_MAX_SMEM);
    if (e != cudaSuccess) return -1000 - static_cast<int>(e);
    configured = true;
  }
  launch_ex(attn_latent_kernel<N, KEYS>, grid, dim3(AL_THREADS), smem, stream, p.splits, tq, tc, tr, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

bool latent_cache_ok(const b200_paged_cache* c, const b200_latent_dims* d);      // latent.cu

}  // namespace b200

using namespace b200;

extern "C" int b200_attn_latent_fits(int rank, int rot) {
  AlPlan plan;
  return al_plan(rank, rot, 16, plan) && al_plan(rank, rot, 32, plan) ? 1 : 0;
}

extern "C" int b200_attn_latent(const void* q, long long ldq, const void* q_rot, long long ldr, int head_ld_rot, void* out, long long ldo,
                                int M, const b200_latent_dims* d, float scale, const int* cu, int portions, int max_len, const int* positions,
                                const int* seq_ids, const int* seq_lens, const float* cos_tab, const float* sin_tab, int max_pos,
                                const b200_paged_cache* cache, int splits, int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!q || !q_rot || !out || !positions || !latent_cache_ok(cache, d) || cache->f32 || cache->page_size != AL_PS) return -1;
  if (ldq != static_cast<long long>(d->heads) * d->rank || ldo % 4 || ldr % 2 || head_ld_rot % 2 || (reinterpret_cast<uintptr_t>(q) & 15) ||
      (reinterpret_cast<uintptr_t>(out) & 7) || (reinterpret_cast<uintptr_t>(q_rot) & 3)) return -2;
  if (splits < 1 || splits > 8 || max_pos <= 0 || (d->true_rot > 0 && (!cos_tab || !sin_tab)) || (cu && (portions <= 0 || max_len <= 0))) return -3;
  const int longest = cu ? max_len : 1, batch = cu ? portions : M;
  const int n = static_cast<long long>(longest) * d->heads > 16 ? 32 : 16;
  AlPlan plan;
  if (!al_plan(d->rank, d->rot, n, plan)) return -4;
  const long long tiles = (static_cast<long long>(longest) * d->heads + n - 1) / n;
  if (tiles > 65535 || batch > 65535) return -5;
  const int dk = d->rank + d->rot;
  const uint64_t rows = static_cast<uint64_t>(M) * d->heads, pitch = static_cast<uint64_t>(dk) * 2;
  CUtensorMap tq, tc, tr;
  if (make_tmap_3d_bf16(&tq, q, d->rank, rows, 1, static_cast<uint64_t>(d->rank) * 2, rows * d->rank * 2, n, 1)) return -11;
  if (make_tmap_3d_bf16(&tc, cache->data, d->rank, AL_PS, cache->num_pages, pitch, pitch * AL_PS, AL_PS, 1)) return -12;
  tr = tc;
  if (d->rot > 0 && make_tmap_3d_bf16(&tr, static_cast<const uint8_t*>(cache->data) + static_cast<size_t>(d->rank) * 2, d->rot, AL_PS, cache->num_pages, pitch, pitch * AL_PS, AL_PS, 1)) return -13;
  AttnLatentParams p;
  p.q_rot = static_cast<const __nv_bfloat16*>(q_rot); p.ldr = ldr; p.head_ld_rot = head_ld_rot;
  p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.d = *d; p.scale_log2 = scale * AL_LOG2E; p.cu = cu; p.positions = positions;
  p.seq_ids = seq_ids; p.seq_lens = seq_lens; p.cos_tab = cos_tab; p.sin_tab = sin_tab; p.max_pos = max_pos; p.splits = splits;
  p.slots = plan.slots; p.rot_slots = plan.rot_slots; p.ahead = plan.ahead; p.c = *cache; p.status = status; p.limit_ns = 2000000000ull;
  const dim3 grid(splits, static_cast<unsigned>(tiles), batch);
  if (plan.keys == 128) return n == 16 ? launch_attn_latent<16, 128>(tq, tc, tr, p, grid, plan.smem, stream) : launch_attn_latent<32, 128>(tq, tc, tr, p, grid, plan.smem, stream);
  return n == 16 ? launch_attn_latent<16, 64>(tq, tc, tr, p, grid, plan.smem, stream) : launch_attn_latent<32, 64>(tq, tc, tr, p, grid, plan.smem, stream);
}
