// Flash attention for prefill portions over the paged cache on sm_100a tensor cores (bf16 in, fp32 accumulate), with an
// optional chunk mask, a softmax sink per head and a sigmoid gate per (token, head) on the output.
//
// One CTA = 128 consecutive query rows of one head of one portion.  The portion's own keys are in the cache already, so a
// portion that continues a sequence and a whole prompt are the same case: keys run from the start of the first row's
// chunk (rounded down to a page) to the last row's position, in tiles of 128 tokens = 8 pages.
//   warp 0      TMA producer: Q once, then K and V pages (16 x 64-column boxes straight into the swizzled operand layout)
//               into two-stage rings; lane <-> page.  Pages past the last key are requested at an out-of-range
//               coordinate, which fills with zeros.
//   warp 1      MMA issuer: S = Q.K^T and PV = P.V, both tcgen05.mma.kind::f16, S and PV double buffered in TMEM
//   warps 2..5  softmax: thread <-> query row, as in attn_prefill.cu; the sink joins the denominator and the gate the
//               scale of the final store
// Head sizes are free up to 128: the tensor maps end at dk / dv and fill with zeros, the MMAs take ceil(dk / 16) steps and
// dv rounded up to 16 columns.  All waits are bounded.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "gemm_common.cuh"

namespace b200 {

constexpr int PP_THREADS = 192;
constexpr int PP_BM = 128, PP_BN = 128, PP_PS = 16;
constexpr int PP_CHUNK_BYTES = 128 * 128;            // 128 rows x 64 bf16
constexpr int PP_TILE_BYTES = 2 * PP_CHUNK_BYTES;    // up to 128 columns
constexpr float PP_LOG2E = 1.4426950408889634f;

struct PrefillPagedParams {
  const int* cu_seqlens; const int* positions; const int* seq_ids;
  const int* page_table; int num_seqs, max_pages, num_pages;
  __nv_bfloat16* out; long long ldo;
  int hq, hkv, dk, dv, chunk;
  float scale_log2;
  const float* sink;
  const __nv_bfloat16* gate; long long ldg;
  int* status;
  unsigned long long limit_ns;
};

__global__ void __launch_bounds__(PP_THREADS, 1)
attn_prefill_paged_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                          const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ PrefillPagedParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  // [Q][K0][K1][V0][V1][P][barriers]
  const uint32_t sQ = smem_u32(smem), sK = sQ + PP_TILE_BYTES, sV = sK + 2 * PP_TILE_BYTES, sP = sV + 2 * PP_TILE_BYTES;
  uint8_t* pP = smem + 5 * PP_TILE_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + 6 * PP_TILE_BYTES);
  const uint32_t bar0 = smem_u32(bars);
  enum { B_QFULL = 0, B_KFULL = 1, B_VFULL = 3, B_KEMPTY = 5, B_VEMPTY = 7, B_SFULL = 9, B_PFULL = 11, B_OFULL = 12, B_COUNT = 14 };
  auto bar = [&](int i) { return bar0 + 8u * i; };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + B_COUNT);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qt = gridDim.x - 1 - blockIdx.x;        // heavy (late) query tiles first
  const int head = blockIdx.y, b = blockIdx.z;
  const int row0 = p.cu_seqlens[b];
  const int len = p.cu_seqlens[b + 1] - row0;
  const int q0 = qt * PP_BM;
  if (q0 >= len) return;                            // uniform across the CTA, before any barrier / TMEM use
  const int start = p.positions[row0];              // position of the portion's first token
  const int seq = p.seq_ids ? p.seq_ids[row0] : b;
  const int last_pos = start + min(q0 + PP_BM, len) - 1;
  if (start < 0 || seq < 0 || seq >= p.num_seqs || last_pos / PP_PS >= p.max_pages) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (11 << 8));
    return;
  }
  int kv_start = p.chunk > 0 ? (start + q0) - (start + q0) % p.chunk : 0;
  kv_start -= kv_start % PP_PS;
  const int n_tiles = (last_pos - kv_start) / PP_BN + 1;
  const int kvh = head / (p.hq / p.hkv);
  const int kchunks = (p.dk + 63) >> 6, vchunks = (p.dv + 63) >> 6, ksteps = (p.dk + 15) >> 4, dv16 = (p.dv + 15) & ~15;
  const uint64_t limit = p.limit_ns;

  if (threadIdx.x == 0) {
    for (int i = 0; i < B_COUNT; ++i) mbar_init(bar(i), (i == B_PFULL) ? 128 : 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(smem_u32(tmem_slot), 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      prefetch_tmap(&tmap_q); prefetch_tmap(&tmap_k); prefetch_tmap(&tmap_v);
      mbar_expect_tx(bar(B_QFULL), kchunks * PP_CHUNK_BYTES);
      for (int c = 0; c < kchunks; ++c) tma_load_3d(sQ + c * PP_CHUNK_BYTES, &tmap_q, bar(B_QFULL), c * 64, head, row0 + q0);
    }
    const int* pt = p.page_table + static_cast<size_t>(seq) * p.max_pages;
    auto page_of = [&](int j) {
      const int tok = kv_start + j * PP_BN + (lane & 7) * PP_PS;
      const int pg = tok <= last_pos ? pt[tok / PP_PS] : p.num_pages;
      return (pg < 0 || pg > p.num_pages) ? p.num_pages : pg;
    };
    int page = page_of(0);
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      const int st = j & 1;
      const uint32_t ph = (j >> 1) & 1u;
      const int next_page = j + 1 < n_tiles ? page_of(j + 1) : 0;
      ok = __all_sync(0xffffffffu, mbar_wait(bar(B_KEMPTY + st), ph ^ 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_EMPTY | (11 << 8)), limit));
      if (!ok) break;
      if (lane == 0) mbar_expect_tx(bar(B_KFULL + st), kchunks * PP_CHUNK_BYTES);
      __syncwarp();
      if (lane < 8)
        for (int c = 0; c < kchunks; ++c)
          tma_load_3d(sK + st * PP_TILE_BYTES + c * PP_CHUNK_BYTES + lane * 2048, &tmap_k, bar(B_KFULL + st), c * 64, kvh * PP_PS, page);
      ok = __all_sync(0xffffffffu, mbar_wait(bar(B_VEMPTY + st), ph ^ 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_EMPTY | (11 << 8)), limit));
      if (!ok) break;
      if (lane == 0) mbar_expect_tx(bar(B_VFULL + st), vchunks * PP_CHUNK_BYTES);
      __syncwarp();
      if (lane < 8)
        for (int c = 0; c < vchunks; ++c)
          tma_load_3d(sV + st * PP_TILE_BYTES + c * PP_CHUNK_BYTES + lane * 2048, &tmap_v, bar(B_VFULL + st), c * 64, kvh * PP_PS, page);
      page = next_page;
    }
    if (!ok) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 2000000ull) { } }   // copies in flight land
    __syncwarp();
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t IDESC_S = umma_idesc_bf16(128, 128, 0, 0);
      const uint32_t idesc_pv = umma_idesc_bf16(128, dv16, 0, 1);        // B (= V) is MN-major
      auto issue_s = [&](int j) {
        const int st = j & 1;
        const uint32_t d = tmem_base + (j & 1) * 128;
        for (int kk = 0; kk < ksteps; ++kk) {
          const uint32_t off = (kk >> 2) * PP_CHUNK_BYTES;
          const uint64_t a = umma_desc_k_sw128(sQ + off) + 2ull * (kk & 3);
          const uint64_t bd = umma_desc_k_sw128(sK + st * PP_TILE_BYTES + off) + 2ull * (kk & 3);
          umma_f16_ss(d, a, bd, IDESC_S, kk > 0 ? 1u : 0u);
        }
        umma_commit(bar(B_KEMPTY + st));
        umma_commit(bar(B_SFULL + (j & 1)));
      };
      bool ok = mbar_wait(bar(B_QFULL), 0, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (11 << 8)), limit) &&
                mbar_wait(bar(B_KFULL + 0), 0, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (11 << 8)), limit);
      if (ok) { tc_fence_after(); issue_s(0); }
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int st = j & 1;
        const uint32_t ph = (j >> 1) & 1u;
        if (j + 1 < n_tiles) {
          if (!mbar_wait(bar(B_KFULL + ((j + 1) & 1)), ((j + 1) >> 1) & 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (11 << 8)), limit)) { ok = false; break; }
          tc_fence_after();
          issue_s(j + 1);
        }
        if (!mbar_wait(bar(B_PFULL), j & 1u, abort_flag, p.status, (ST_TIMEOUT_PEER_FLAG | (11 << 8)), limit)) { ok = false; break; }
        if (!mbar_wait(bar(B_VFULL + st), ph, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (11 << 8)), limit)) { ok = false; break; }
        tc_fence_after();
        const uint32_t d = tmem_base + 256 + (j & 1) * 128;
#pragma unroll
        for (int kk = 0; kk < 8; ++kk) {
          const uint64_t a = umma_desc_k_sw128(sP + (kk >> 2) * PP_CHUNK_BYTES) + 2ull * (kk & 3);
          const uint64_t bd = umma_desc_mn_sw128(sV + st * PP_TILE_BYTES + kk * 2048, PP_CHUNK_BYTES, 1024);
          umma_f16_ss(d, a, bd, idesc_pv, kk > 0 ? 1u : 0u);
        }
        umma_commit(bar(B_VEMPTY + st));
        umma_commit(bar(B_OFULL + (j & 1)));
      }
    }
    __syncwarp();
  } else {
    const int qd = warp & 3;
    const int r = qd * 32 + lane;                    // row inside the tile == TMEM lane
    const int pos = start + q0 + r;
    const int lo = p.chunk > 0 ? pos - pos % p.chunk : 0;
    const uint32_t t_lane = tmem_base + (static_cast<uint32_t>(qd * 32) << 16);
    float o[128];
#pragma unroll
    for (int i = 0; i < 128; ++i) o[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f, alpha_prev = 1.f;
    bool ok = true;
    uint8_t* p_row = pP + (r >> 3) * 1024 + (r & 7) * 128;
    const int sw = r & 7;
    auto wait_all = [&](int i, uint32_t par) {       // one verdict per warp: the TMEM loads need all lanes
      return __all_sync(0xffffffffu, mbar_wait(bar(i), par, abort_flag, p.status, (ST_TIMEOUT_TMEM_FULL | (11 << 8)), limit)) != 0;
    };
    auto o_update = [&](int j, float alpha) -> bool {
      if (!wait_all(B_OFULL + (j & 1), (j >> 1) & 1u)) return false;
      tc_fence_after();
      const uint32_t t_pv = t_lane + 256 + (j & 1) * 128;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        if (c * 32 < dv16) {
          uint32_t v[32];
          tmem_ld_x32(t_pv + c * 32, v);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) o[c * 32 + i] = o[c * 32 + i] * alpha + __uint_as_float(v[i]);
        }
      }
      tc_fence_before();
      return true;
    };

    for (int j = 0; j < n_tiles; ++j) {
      if (!wait_all(B_SFULL + (j & 1), (j >> 1) & 1u)) { ok = false; break; }
      tc_fence_after();
      const uint32_t t_s = t_lane + (j & 1) * 128;
      const int kv0 = kv_start + j * PP_BN;
      // whole warp takes the masked form when any of its rows needs it
      const bool need_mask = __any_sync(0xffffffffu, kv0 + PP_BN - 1 > pos || kv0 < lo);
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t v[32];
        tmem_ld_x32(t_s + c * 32, v);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          float s = __uint_as_float(v[i]);
          if (need_mask) { const int kv = kv0 + c * 32 + i; if (kv > pos || kv < lo) s = -INFINITY; }
          mx = fmaxf(mx, s);
        }
      }
      const float m_new = fmaxf(m_run, mx * p.scale_log2);
      const float alpha = (m_run == -INFINITY) ? 0.f : exp2f(m_run - m_new);
      const float m_use = (m_new == -INFINITY) ? 0.f : m_new;
      // the P buffer is free once the PV MMA of the previous tile has completed
      if (j > 0) {
        if (!wait_all(B_OFULL + ((j - 1) & 1), ((j - 1) >> 1) & 1u)) { ok = false; break; }
      }
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t v[32];
        tmem_ld_x32(t_s + c * 32, v);
        tmem_ld_wait();
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float s0 = __uint_as_float(v[i]), s1 = __uint_as_float(v[i + 1]);
          if (need_mask) {
            const int kv = kv0 + c * 32 + i;
            if (kv > pos || kv < lo) s0 = -INFINITY;
            if (kv + 1 > pos || kv + 1 < lo) s1 = -INFINITY;
          }
          const float e0 = exp2f(s0 * p.scale_log2 - m_use), e1 = exp2f(s1 * p.scale_log2 - m_use);
          const __nv_bfloat162 pb = __floats2bfloat162_rn(e0, e1);
          sum += __low2float(pb) + __high2float(pb);          // what the MMA will actually see
          pk[i >> 1] = *reinterpret_cast<const uint32_t*>(&pb);
        }
        uint8_t* chunk = p_row + (c >> 1) * PP_CHUNK_BYTES;
#pragma unroll
        for (int u4 = 0; u4 < 4; ++u4) {
          const int u = (c & 1) * 4 + u4;
          *reinterpret_cast<uint4*>(chunk + ((u ^ sw) << 4)) = make_uint4(pk[4 * u4], pk[4 * u4 + 1], pk[4 * u4 + 2], pk[4 * u4 + 3]);
        }
      }
      l_run = l_run * alpha + sum;
      m_run = m_new;
      tc_fence_before();
      fence_proxy_async_smem();
      mbar_arrive(bar(B_PFULL));
      if (j > 0) { if (!o_update(j - 1, alpha_prev)) { ok = false; break; } }
      alpha_prev = alpha;
    }
    if (ok) ok = o_update(n_tiles - 1, alpha_prev);
    if (ok && q0 + r < len) {
      const size_t tok = static_cast<size_t>(row0) + q0 + r;
      float f = l_run > 0.f ? 1.f / l_run : 0.f;
      if (p.sink) {
        const float s2 = p.sink[head] * PP_LOG2E, m = fmaxf(m_run, s2), a = exp2f(m_run - m);
        f = a / (l_run * a + exp2f(s2 - m));
      }
      if (p.gate) f *= 1.f / (1.f + __expf(-__bfloat162float(p.gate[tok * p.ldg + head])));
      uint4* dst = reinterpret_cast<uint4*>(p.out + tok * p.ldo + static_cast<size_t>(head) * p.dv);
#pragma unroll
      for (int u = 0; u < 16; ++u) {
        if (u * 8 < p.dv) {
          uint32_t w[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const __nv_bfloat162 pb = __floats2bfloat162_rn(o[u * 8 + 2 * k] * f, o[u * 8 + 2 * k + 1] * f);
            w[k] = *reinterpret_cast<const uint32_t*>(&pb);
          }
          dst[u] = make_uint4(w[0], w[1], w[2], w[3]);
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, 512); }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_attn_prefill_paged(const void* q, long long ldq, void* out, long long ldo, int hq, int M, int B, int max_len,
                                       const int* cu_seqlens, const int* positions, const int* seq_ids,
                                       const b200_paged_cache* c, const b200_attn_spec* s, int* status, cudaStream_t stream) {
  if (M <= 0 || B <= 0 || max_len <= 0) return 0;
  if (!q || !out || !cu_seqlens || !positions || !c || !c->data || !c->page_table || !s) return -1;
  if (c->f32 || c->page_size != PP_PS || c->dk <= 0 || c->dv <= 0 || c->dk > 128 || c->dv > 128 || c->dk % 8 || c->dv % 8) return -2;
  if (hq <= 0 || c->kv_heads <= 0 || hq % c->kv_heads || ldq % 8 || ldo % 8 || ldq < static_cast<long long>(hq) * c->dk || c->num_pages <= 0) return -3;
  if ((reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(out) & 15) || (reinterpret_cast<uintptr_t>(c->data) & 15)) return -4;
  const uint64_t rec = static_cast<uint64_t>(c->kv_heads) * PP_PS * (c->dk + c->dv) * 2, kbytes = static_cast<uint64_t>(c->kv_heads) * PP_PS * c->dk * 2;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d_bf16(&tq, q, c->dk, hq, M, static_cast<uint64_t>(c->dk) * 2, static_cast<uint64_t>(ldq) * 2, 1, 128)) return -11;
  if (make_tmap_3d_bf16(&tk, c->data, c->dk, static_cast<uint64_t>(c->kv_heads) * PP_PS, c->num_pages, static_cast<uint64_t>(c->dk) * 2, rec, PP_PS, 1)) return -12;
  if (make_tmap_3d_bf16(&tv, static_cast<const uint8_t*>(c->data) + kbytes, c->dv, static_cast<uint64_t>(c->kv_heads) * PP_PS, c->num_pages, static_cast<uint64_t>(c->dv) * 2, rec, PP_PS, 1)) return -13;
  PrefillPagedParams p;
  p.cu_seqlens = cu_seqlens; p.positions = positions; p.seq_ids = seq_ids; p.page_table = c->page_table;
  p.num_seqs = c->num_seqs; p.max_pages = c->max_pages; p.num_pages = c->num_pages;
  p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.hq = hq; p.hkv = c->kv_heads; p.dk = c->dk; p.dv = c->dv; p.chunk = s->chunk;
  p.scale_log2 = s->scale * PP_LOG2E; p.sink = s->sink; p.gate = static_cast<const __nv_bfloat16*>(s->gate); p.ldg = s->ldg;
  p.status = status; p.limit_ns = 2000000000ull;
  constexpr int SMEM = 6 * PP_TILE_BYTES + 1024 + 256;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_prefill_paged_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return -1000 - static_cast<int>(e);
    configured = true;
  }
  launch_ex(attn_prefill_paged_kernel, dim3((max_len + PP_BM - 1) / PP_BM, hq, B), dim3(PP_THREADS), SMEM, stream, 0, tq, tk, tv, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
