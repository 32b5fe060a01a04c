// Flash attention for long portions of latent attention on sm_100a tensor cores (bf16 in, fp32 accumulate): keys and values have
// been expanded from the latents into consecutive rows; a head's key is its own part next to one rotated part that all heads
// share, and the two are fetched side by side into one operand.
//
// One CTA = 128 consecutive query rows of one head of one portion, keys in tiles of 128 rows.
//   warp 0      TMA producer: Q once, then key tiles (own part, shared part) and value tiles into rings of one or two stages
//               (what fits); rows beyond the buffers arrive as zeros
//   warp 1      MMA issuer: S = Q.K^T and PV = P.V, tcgen05.mma.kind::f16, S and PV double buffered in TMEM
//   warps 2..9  softmax: two threads per query row, each half of the tile's keys (kept in registers between maximum and
//               exponential; the halves exchange their maxima through shared memory) and half of the value columns
// The output gate is the scale of the final store.  Every head part is a whole number of 64-column chunks in shared memory, the
// tensor maps end at its true size and fill with zeros; the MMAs take ceil(size / 16) steps of each part.  All waits are bounded.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "gemm_common.cuh"

namespace b200 {

constexpr int PL_THREADS = 320, PL_SOFTMAX = 256;
constexpr int PL_BM = 128, PL_BN = 128;
constexpr int PL_CHUNK = 128 * 128;                   // 128 rows x 64 bf16
constexpr int PL_MAX_SMEM = 232448;
constexpr int PL_TAIL = 2 * 2 * 128 * 4 + 256;        // maxima of the halves, two turns; barriers
constexpr float PL_LOG2E = 1.4426950408889634f;

struct PrefillLatentParams {
  const int* cu; const int* ctx; const int* positions;
  __nv_bfloat16* out; long long ldo;
  int dn, dr, dv;
  int k_stages, v_stages, p_stages;
  float scale_log2;
  const float* gate; long long ldg;
  int* status;
  unsigned long long limit_ns;
};

__global__ void __launch_bounds__(PL_THREADS, 1)
attn_prefill_latent_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_qr,
                           const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_kr,
                           const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ PrefillLatentParams p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(1024) uint8_t pl_smem[];
  const int nc = (p.dn + 63) >> 6, kc = nc + ((p.dr + 63) >> 6), vc = (p.dv + 63) >> 6;      // 64-column chunks
  const int k_bytes = kc * PL_CHUNK, v_bytes = vc * PL_CHUNK;
  const uint32_t sQ = smem_u32(pl_smem), sK = sQ + k_bytes, sV = sK + p.k_stages * k_bytes, sP = sV + p.v_stages * v_bytes;
  uint8_t* pP = pl_smem + (sP - sQ);
  float* mx_buf = reinterpret_cast<float*>(pP + p.p_stages * 2 * PL_CHUNK);                  // [turn][half][row]
  uint64_t* bars = reinterpret_cast<uint64_t*>(mx_buf + 2 * 2 * 128);
  const uint32_t bar0 = smem_u32(bars);
  enum { B_QFULL = 0, B_KFULL = 1, B_VFULL = 3, B_KEMPTY = 5, B_VEMPTY = 7, B_SFULL = 9, B_PFULL = 11, B_OFULL = 12, B_COUNT = 14 };
  auto bar = [&](int i) { return bar0 + 8u * i; };
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + B_COUNT);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qt = gridDim.x - 1 - blockIdx.x;            // heavy (late) query tiles first
  const int head = blockIdx.y, b = blockIdx.z;
  const int row0 = p.cu[b], len = p.cu[b + 1] - row0, q0 = qt * PL_BM;
  if (q0 >= len) return;                                // uniform across the CTA, before any barrier / TMEM use
  const int start = p.positions[row0], key0 = p.ctx[b], keys = p.ctx[b + 1] - key0;
  const int last_pos = start + min(q0 + PL_BM, len) - 1;
  if (start < 0 || last_pos >= keys) {                  // the rows of this sequence must hold every key up to the last query
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (19 << 8));
    return;
  }
  const int n_tiles = last_pos / PL_BN + 1;
  const int dv16 = (p.dv + 15) & ~15;
  const uint64_t limit = p.limit_ns;

  if (threadIdx.x == 0) {
    for (int i = 0; i < B_COUNT; ++i) mbar_init(bar(i), i == B_PFULL ? PL_SOFTMAX / 32 : 1);
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
      prefetch_tmap(&tmap_q); prefetch_tmap(&tmap_qr); prefetch_tmap(&tmap_k); prefetch_tmap(&tmap_kr); prefetch_tmap(&tmap_v);
      mbar_expect_tx(bar(B_QFULL), k_bytes);
      for (int c = 0; c < nc; ++c) tma_load_3d(sQ + c * PL_CHUNK, &tmap_q, bar(B_QFULL), c * 64, head, row0 + q0);
      for (int c = nc; c < kc; ++c) tma_load_3d(sQ + c * PL_CHUNK, &tmap_qr, bar(B_QFULL), (c - nc) * 64, head, row0 + q0);
      bool ok = true;
      int ks = 0, vs = 0;
      uint32_t kp = 0, vp = 0;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int row = key0 + j * PL_BN;
        ok = mbar_wait(bar(B_KEMPTY + ks), kp ^ 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_EMPTY | (19 << 8)), limit);
        if (!ok) break;
        mbar_expect_tx(bar(B_KFULL + ks), k_bytes);
        const uint32_t kd = sK + ks * k_bytes;
        for (int c = 0; c < nc; ++c) tma_load_3d(kd + c * PL_CHUNK, &tmap_k, bar(B_KFULL + ks), c * 64, head, row);
        for (int c = nc; c < kc; ++c) tma_load_3d(kd + c * PL_CHUNK, &tmap_kr, bar(B_KFULL + ks), (c - nc) * 64, 0, row);
        if (++ks == p.k_stages) { ks = 0; kp ^= 1u; }
        ok = mbar_wait(bar(B_VEMPTY + vs), vp ^ 1u, abort_flag, p.status, (ST_TIMEOUT_SMEM_EMPTY | (19 << 8)), limit);
        if (!ok) break;
        mbar_expect_tx(bar(B_VFULL + vs), v_bytes);
        for (int c = 0; c < vc; ++c) tma_load_3d(sV + vs * v_bytes + c * PL_CHUNK, &tmap_v, bar(B_VFULL + vs), c * 64, head, row);
        if (++vs == p.v_stages) { vs = 0; vp ^= 1u; }
      }
      if (!ok) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 2000000ull) { } }   // copies in flight land
    }
    __syncwarp();
  } else if (warp == 1) {
    // The whole warp walks the loops, so that descriptors stay in uniform registers; one elected thread issues.
    {
      const bool one = elect_one();
      constexpr uint32_t IDESC_S = umma_idesc_bf16(128, 128, 0, 0);
      const uint32_t idesc_pv = umma_idesc_bf16(128, dv16, 0, 1);        // B (= V) is MN-major
      const int n_steps = (p.dn + 15) >> 4, r_steps = (p.dr + 15) >> 4;
      int ks = 0, vs = 0;
      uint32_t kp = 0, vp = 0;
      // a descriptor costs an addition (the address field counts 16 bytes)
      const uint64_t q_desc = umma_desc_k_sw128(sQ), k_desc = umma_desc_k_sw128(sK), p_desc = umma_desc_k_sw128(sP), v_desc = umma_desc_mn_sw128(sV, PL_CHUNK, 1024);
      auto issue_s = [&](int j) {                                        // the K stage has been waited for
        const uint32_t d = tmem_base + (j & 1) * 128;
        const uint64_t kd = k_desc + static_cast<uint32_t>(ks * (k_bytes >> 4));
        for (int c = 0; c < kc; ++c) {
          const int steps = c < nc ? n_steps - 4 * c : r_steps - 4 * (c - nc);
          const uint32_t off = c * (PL_CHUNK >> 4);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk)
            if (kk < steps && one) umma_f16_ss(d, q_desc + (off + 2 * kk), kd + (off + 2 * kk), IDESC_S, kk > 0 ? 1u : (c > 0 ? 1u : 0u));
        }
        if (one) { umma_commit(bar(B_KEMPTY + ks)); umma_commit(bar(B_SFULL + (j & 1))); }
        if (++ks == p.k_stages) { ks = 0; kp ^= 1u; }
      };
      bool ok = mbar_wait(bar(B_QFULL), 0, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (19 << 8)), limit) &&
                mbar_wait(bar(B_KFULL), 0, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (19 << 8)), limit);
      if (ok) { tc_fence_after(); issue_s(0); }
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles) {
          if (!mbar_wait(bar(B_KFULL + ks), kp, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (19 << 8)), limit)) { ok = false; break; }
          tc_fence_after();
          issue_s(j + 1);
        }
        if (!mbar_wait(bar(B_PFULL), j & 1u, abort_flag, p.status, (ST_TIMEOUT_PEER_FLAG | (19 << 8)), limit)) { ok = false; break; }
        if (!mbar_wait(bar(B_VFULL + vs), vp, abort_flag, p.status, (ST_TIMEOUT_SMEM_FULL | (19 << 8)), limit)) { ok = false; break; }
        tc_fence_after();
        const uint32_t d = tmem_base + 256 + (j & 1) * 128;
        const uint64_t a = p_desc + (p.p_stages == 2 ? static_cast<uint32_t>((j & 1) * (2 * PL_CHUNK >> 4)) : 0u), bv = v_desc + static_cast<uint32_t>(vs * (v_bytes >> 4));
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          if (one) umma_f16_ss(d, a + ((kk >> 2) * (PL_CHUNK >> 4) + 2 * (kk & 3)), bv + kk * (2048 >> 4), idesc_pv, kk > 0 ? 1u : 0u);
        if (one) { umma_commit(bar(B_VEMPTY + vs)); umma_commit(bar(B_OFULL + (j & 1))); }
        if (++vs == p.v_stages) { vs = 0; vp ^= 1u; }
      }
    }
    __syncwarp();
  } else {
    const int qd = warp & 3, half = (warp - 2) >> 2;    // TMEM lane quarter this warp may read; which half of the columns
    const int r = qd * 32 + lane, pos = start + q0 + r;
    const uint32_t t_lane = tmem_base + (static_cast<uint32_t>(qd * 32) << 16);
    const int ov = ((dv16 / 2 + 31) / 32) * 32, o0 = half * ov;          // value columns o0 .. o0 + ov of this thread (up to dv)
    float o[64];
#pragma unroll
    for (int i = 0; i < 64; ++i) o[i] = 0.f;
    float m_run = -INFINITY, l_run = 0.f, alpha_prev = 1.f;
    bool ok = true;
    const int sw = r & 7;
    auto wait_all = [&](int i, uint32_t par) {          // one verdict per warp: the TMEM loads need all lanes
      return __all_sync(0xffffffffu, mbar_wait(bar(i), par, abort_flag, p.status, (ST_TIMEOUT_TMEM_FULL | (19 << 8)), limit)) != 0;
    };
    auto o_update = [&](int j, float alpha) -> bool {
      if (!wait_all(B_OFULL + (j & 1), (j >> 1) & 1u)) return false;
      tc_fence_after();
      const uint32_t t_pv = t_lane + 256 + (j & 1) * 128 + o0;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        if (c * 32 < ov && o0 + c * 32 < dv16) {
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

    // A warp whose wait fails still meets the others at the barriers below: every step is taken by all or, once the flag is
    // up, fails for all within the same bounded time.
    for (int j = 0; j < n_tiles; ++j) {
      ok = ok && wait_all(B_SFULL + (j & 1), (j >> 1) & 1u);
      const int kv0 = j * PL_BN + half * 64;
      float s[64];
      float mx = -INFINITY;
      if (ok) {
        tc_fence_after();
        const uint32_t t_s = t_lane + (j & 1) * 128 + half * 64;
        uint32_t v[32], u[32];
        tmem_ld_x32(t_s, v);
        tmem_ld_x32(t_s + 32, u);
        tmem_ld_wait();
        const bool need_mask = __any_sync(0xffffffffu, kv0 + 63 > pos);
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          s[i] = __uint_as_float(v[i]);
          s[32 + i] = __uint_as_float(u[i]);
        }
        if (need_mask) {
#pragma unroll
          for (int i = 0; i < 64; ++i) if (kv0 + i > pos) s[i] = -INFINITY;
        }
#pragma unroll
        for (int i = 0; i < 64; ++i) mx = fmaxf(mx, s[i]);
      }
      mx_buf[((j & 1) * 2 + half) * 128 + r] = mx;
      named_bar_sync(1, PL_SOFTMAX);
      mx = fmaxf(mx, mx_buf[((j & 1) * 2 + (half ^ 1)) * 128 + r]);
      if (!ok) continue;
      const float m_new = fmaxf(m_run, mx * p.scale_log2);
      const float alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - m_new);
      const float m_use = m_new == -INFINITY ? 0.f : m_new;
      // with one weight buffer it is free once the PV MMA of the previous tile has completed; with two, once that of the tile
      // before has, which o_update waited for
      if (j > 0 && p.p_stages == 1 && !wait_all(B_OFULL + ((j - 1) & 1), ((j - 1) >> 1) & 1u)) { ok = false; continue; }
      uint8_t* chunk = pP + (p.p_stages == 2 ? (j & 1) * 2 * PL_CHUNK : 0) + half * PL_CHUNK + (r >> 3) * 1024 + sw * 128;
      float sum = 0.f;
#pragma unroll
      for (int g = 0; g < 8; ++g) {
        uint32_t pk[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const __nv_bfloat162 e = __floats2bfloat162_rn(exp2f(s[g * 8 + 2 * i] * p.scale_log2 - m_use), exp2f(s[g * 8 + 2 * i + 1] * p.scale_log2 - m_use));
          sum += __low2float(e) + __high2float(e);      // what the MMA will actually see
          pk[i] = *reinterpret_cast<const uint32_t*>(&e);
        }
        *reinterpret_cast<uint4*>(chunk + ((g ^ sw) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
      }
      l_run = l_run * alpha + sum;
      m_run = m_new;
      tc_fence_before();
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar(B_PFULL));         // one arrival per warp: they queue up at the barrier
      if (j > 0 && !o_update(j - 1, alpha_prev)) { ok = false; continue; }
      alpha_prev = alpha;
    }
    if (ok) ok = o_update(n_tiles - 1, alpha_prev);
    // the halves' sums belong to the same maximum
    named_bar_sync(1, PL_SOFTMAX);
    mx_buf[half * 128 + r] = l_run;
    named_bar_sync(1, PL_SOFTMAX);
    const float l = l_run + mx_buf[(half ^ 1) * 128 + r];
    if (ok && q0 + r < len) {
      const size_t tok = static_cast<size_t>(row0) + q0 + r;
      float f = l > 0.f ? 1.f / l : 0.f;
      if (p.gate) f *= 1.f / (1.f + __expf(-p.gate[tok * p.ldg + head]));
      uint4* dst = reinterpret_cast<uint4*>(p.out + tok * p.ldo + static_cast<size_t>(head) * p.dv + o0);
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (u * 8 < ov && o0 + u * 8 < p.dv) {
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

// stages of keys, values and softmax weights that fit; false: sizes beyond the kernel
static bool pl_stages(int dn, int dr, int dv, int& k, int& v, int& w, int& smem) {
  if (dn <= 0 || dr < 0 || dv <= 0 || dv > 128 || dn % 8 || dr % 8 || dv % 8) return false;
  const int kc = (dn + 63) / 64 + (dr + 63) / 64, vc = (dv + 63) / 64;
  const int plans[5][3] = {{2, 2, 2}, {1, 2, 2}, {1, 2, 1}, {2, 1, 1}, {1, 1, 1}};
  for (const auto& s : plans) {
    const int need = (kc + s[0] * kc + s[1] * vc + s[2] * 2) * PL_CHUNK + PL_TAIL;
    if (need <= PL_MAX_SMEM) { k = s[0]; v = s[1]; w = s[2]; smem = need; return true; }
  }
  return false;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_attn_prefill_latent_fits(int dn, int dr, int dv) {
  int k, v, w, smem;
  return pl_stages(dn, dr, dv, k, v, w, smem) ? 1 : 0;
}

extern "C" int b200_attn_prefill_latent(const void* q, long long ldq, int heads, int dn, int dr, int dv, const void* kv, long long ldkv,
                                        const void* k_rot, long long ldkr, int rows_kv, void* out, long long ldo, int M, int B, int max_len,
                                        float scale, const int* cu, const int* ctx, const int* positions, const float* gate, long long ldg,
                                        int* status, cudaStream_t stream) {
  if (M <= 0 || B <= 0 || max_len <= 0) return 0;
  if (!q || !kv || !k_rot || !out || !cu || !ctx || !positions || heads <= 0 || rows_kv <= 0 || heads > 65535 || B > 65535) return -1;
  auto al16 = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) == 0; };
  if (ldq % 8 || ldkv % 8 || ldkr % 8 || ldo % 8 || ldq < static_cast<long long>(heads) * (dn + dr) || ldkv < static_cast<long long>(heads) * (dn + dv) ||
      ldo < static_cast<long long>(heads) * dv || ldkr < dr || !al16(q) || !al16(kv) || !al16(k_rot) || !al16(out)) return -2;
  PrefillLatentParams p;
  int smem = 0;
  if (!pl_stages(dn, dr, dv, p.k_stages, p.v_stages, p.p_stages, smem)) return -3;
  const uint64_t head_pitch = static_cast<uint64_t>(dn + dr) * 2, q_pitch = static_cast<uint64_t>(ldq) * 2, kv_pitch = static_cast<uint64_t>(ldkv) * 2;
  CUtensorMap tq, tqr, tk, tkr, tv;
  if (make_tmap_3d_bf16(&tq, q, dn, heads, M, head_pitch, q_pitch, 1, PL_BM)) return -11;
  if (make_tmap_3d_bf16(&tk, kv, dn, heads, rows_kv, static_cast<uint64_t>(dn) * 2, kv_pitch, 1, PL_BN)) return -12;
  if (make_tmap_3d_bf16(&tv, static_cast<const uint8_t*>(kv) + static_cast<size_t>(heads) * dn * 2, dv, heads, rows_kv, static_cast<uint64_t>(dv) * 2, kv_pitch, 1, PL_BN)) return -13;
  if (dr > 0) {
    if (make_tmap_3d_bf16(&tqr, static_cast<const uint8_t*>(q) + static_cast<size_t>(dn) * 2, dr, heads, M, head_pitch, q_pitch, 1, PL_BM)) return -14;
    if (make_tmap_3d_bf16(&tkr, k_rot, dr, 1, rows_kv, static_cast<uint64_t>(ldkr) * 2, static_cast<uint64_t>(ldkr) * 2, 1, PL_BN)) return -15;
  } else {
    tqr = tq; tkr = tk;
  }
  p.cu = cu; p.ctx = ctx; p.positions = positions; p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.dn = dn; p.dr = dr; p.dv = dv;
  p.scale_log2 = scale * PL_LOG2E; p.gate = gate; p.ldg = ldg; p.status = status; p.limit_ns = 2000000000ull;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_prefill_latent_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, PL_MAX_SMEM);
    if (e != cudaSuccess) return -1000 - static_cast<int>(e);
    configured = true;
  }
  launch_ex(attn_prefill_latent_kernel, dim3((max_len + PL_BM - 1) / PL_BM, heads, B), dim3(PL_THREADS), smem, stream, 0, tq, tqr, tk, tkr, tv, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
