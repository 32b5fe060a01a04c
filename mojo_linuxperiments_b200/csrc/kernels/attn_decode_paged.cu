// Decode attention over the paged cache in one launch: rotary embedding of the new token's q and k, cache append, attention
// over the visible keys (all earlier ones, or the token's own chunk), softmax sink, sigmoid output gate.
//
// Grid (split, kv head x group of up to 16 query heads, sequence); the splits of one (kv head, sequence) are a thread-block
// cluster that merges through distributed shared memory.  The op is bound by the K/V bytes, so the design is about
// keeping loads in flight: each of the four warps walks its own 16-token pages with its own cp.async ring (no barrier
// between warps inside the loop) and its own online softmax; up to 16 query heads are the rows of m16n8k16 MMAs, so a page
// is read once for the whole group.  Cached pages do not depend on the preceding kernel and are requested before the
// dependency wait; the new token never goes through the cache: it is scored from the projection row by the last split.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"

namespace b200 {

constexpr int DP_THREADS = 128, DP_WARPS = 4, DP_PS = 16;
constexpr float DP_LOG2E = 1.4426950408889634f;

struct DecodePagedParams {
  const __nv_bfloat16* qkv; long long ld;
  __nv_bfloat16* out; long long ldo;
  int hq, hgroups;
  const int* positions; const int* seq_lens;
  const float* cos_tab; const float* sin_tab;
  int pairs, interleaved, max_pos;
  b200_paged_cache c;
  int chunk;
  float scale_log2;
  const float* sink;
  const __nv_bfloat16* gate; long long ldg;
  int splits;
  int* status;
};

__device__ __forceinline__ void dp_cp16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;      // 0 source bytes: the destination is filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void dp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void dp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void dp_ldm(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dp_ldm_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dp_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float dp_ld_cluster(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ uint32_t dp_pack(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}

template <int DK, int DV, int STG>
struct DpShape {
  static constexpr int KP = DK + 8, VP = DV + 8;                       // row pitches: 16-byte skew, ldmatrix without conflicts
  static constexpr int STAGE = 16 * (KP + VP) * 2;
  static constexpr int RING = DP_WARPS * STG * STAGE;
  static constexpr int QBYTES = 16 * KP * 2;
  static constexpr int OP = DV + 4;                                    // floats per row of the merge buffers
  static constexpr int MERGE = (DP_WARPS + 1) * (16 * OP + 32) * 4;    // four warps' partials + the CTA's own
  static constexpr int SMEM = (RING > MERGE ? RING : MERGE) + QBYTES + 128;
};

// FULL: dk == DK and dv == DV, so the MMA steps and the copies unroll without conditions
template <int DK, int DV, int STG, bool FULL>
__global__ void __launch_bounds__(DP_THREADS)
attn_decode_paged_kernel(const __grid_constant__ DecodePagedParams p) {
  using Sh = DpShape<DK, DV, STG>;
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t dp_smem[];
  uint8_t* smem = dp_smem;
  constexpr int QOFF = Sh::SMEM - 128 - Sh::QBYTES;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem + QOFF);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rank = blockIdx.x, S = p.splits, b = blockIdx.z;
  const int kvh = blockIdx.y / p.hgroups, hg = blockIdx.y - kvh * p.hgroups;
  const int group = p.hq / p.c.kv_heads, g0 = hg * 16, G = min(16, group - g0), h0 = kvh * group + g0;
  const int dk = FULL ? DK : p.c.dk, dv = FULL ? DV : p.c.dv, ksteps = (dk + 15) >> 4, vsteps = (dv + 15) >> 4;
  const int pos = p.positions[b];
  const bool empty = p.seq_lens[b] <= 0;
  const bool bad = pos < 0 || pos >= p.max_pos || pos / DP_PS >= p.c.max_pages;
  if (empty || bad) {                            // the same for all CTAs of the cluster
    if (bad && tid == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (13 << 8));
    pdl_wait();
    if (rank == 0)
      for (int i = tid; i < G * dv; i += DP_THREADS) p.out[static_cast<size_t>(b) * p.ldo + static_cast<size_t>(h0) * dv + i] = __float2bfloat16(0.f);
    return;
  }
  const int first = p.chunk > 0 ? pos - pos % p.chunk : 0;
  const int t_first = first / DP_PS, n_tiles = pos / DP_PS - t_first + 1;
  const int ta = t_first + static_cast<int>(static_cast<long long>(n_tiles) * rank / S);
  const int tb = t_first + static_cast<int>(static_cast<long long>(n_tiles) * (rank + 1) / S);
  const int mine = tb - ta > warp ? (tb - ta - warp + DP_WARPS - 1) / DP_WARPS : 0;      // pages of this warp
  const int* pt = p.c.page_table + static_cast<size_t>(b) * p.c.max_pages;
  const size_t rec = static_cast<size_t>(p.c.kv_heads) * DP_PS * (dk + dv);
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.c.data);
  const size_t k_off = static_cast<size_t>(kvh) * DP_PS * dk, v_off = static_cast<size_t>(p.c.kv_heads) * DP_PS * dk + static_cast<size_t>(kvh) * DP_PS * dv;
  uint8_t* ring = smem + warp * STG * Sh::STAGE;

  // columns dk .. 16 * ksteps of the key rows are never loaded: zero once
  if (dk & 15)
    for (int i = lane; i < STG * 16; i += 32)
      *reinterpret_cast<uint4*>(ring + (i >> 4) * Sh::STAGE + ((i & 15) * Sh::KP + dk) * 2) = make_uint4(0u, 0u, 0u, 0u);
  // Page ids of this warp's next 32 pages sit in its lanes, so that a request never waits for a table look-up; the
  // (row, 16-byte column) of a lane's first copy and its step to the next one avoid divisions.
  const int kc = dk >> 3, vc = dv >> 3;
  const int kr0 = lane / kc, kc0 = lane - kr0 * kc, krs = 32 / kc, kcs = 32 - krs * kc;
  const int vr0 = lane / vc, vc0 = lane - vr0 * vc, vrs = 32 / vc, vcs = 32 - vrs * vc;
  int ids = 0, ids_from = -32;
  auto issue = [&](int i) {
    if (i < mine) {
      if (i >= ids_from + 32) {
        ids_from = i;
        ids = i + lane < mine ? pt[ta + warp + (i + lane) * DP_WARPS] : 0;
      }
      const int t = ta + warp + i * DP_WARPS;
      const int page = __shfl_sync(0xffffffffu, ids, i - ids_from);
      const bool page_ok = page >= 0 && page < p.c.num_pages;
      const __nv_bfloat16* src = cache + (page_ok ? static_cast<size_t>(page) * rec : 0);
      const uint32_t kd = smem_u32(ring + (i % STG) * Sh::STAGE), vd = kd + 16 * Sh::KP * 2;
      const int left = page_ok ? pos - t * DP_PS : 0;           // rows of this page before the new token
      const __nv_bfloat16* ks = src + k_off + lane * 8;
      const __nv_bfloat16* vs = src + v_off + lane * 8;
      if constexpr (FULL) {
#pragma unroll
        for (int u = 0; u < DK / 16; ++u) {
          const int r = kr0 + u * (256 / DK);
          dp_cp16(kd + (r * Sh::KP + kc0 * 8) * 2, ks + u * 256, r < left);
        }
#pragma unroll
        for (int u = 0; u < DV / 16; ++u) {
          const int r = vr0 + u * (256 / DV);
          dp_cp16(vd + (r * Sh::VP + vc0 * 8) * 2, vs + u * 256, r < left);
        }
      } else {
        for (int r = kr0, c = kc0; r < 16; ks += 256) {
          dp_cp16(kd + (r * Sh::KP + c * 8) * 2, ks, r < left);
          r += krs; c += kcs;
          if (c >= kc) { c -= kc; ++r; }
        }
        for (int r = vr0, c = vc0; r < 16; vs += 256) {
          dp_cp16(vd + (r * Sh::VP + c * 8) * 2, vs, r < left);
          r += vrs; c += vcs;
          if (c >= vc) { c -= vc; ++r; }
        }
      }
    }
    dp_commit();
  };
#pragma unroll
  for (int i = 0; i < STG - 1; ++i) issue(i);

  for (int i = tid; i < Sh::QBYTES / 16; i += DP_THREADS) reinterpret_cast<uint4*>(qs)[i] = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();
  pdl_wait();                                    // the projections are the previous kernel's output

  const __nv_bfloat16* row = p.qkv + static_cast<size_t>(b) * p.ld;
  const float* ct = p.cos_tab + static_cast<size_t>(pos) * p.pairs;
  const float* st = p.sin_tab + static_cast<size_t>(pos) * p.pairs;
  const int np = p.pairs, su = p.interleaved ? 2 : 1, ov = p.interleaved ? 1 : np;
  // rotated head `h` of the projection row: dimensions j and its partner (j < np), or d itself beyond the rotated ones
  auto rotate = [&](const __nv_bfloat16* x, int j, float& ru, float& rv) {
    const float u = __bfloat162float(x[j * su]), v = __bfloat162float(x[j * su + ov]), c = ct[j], s = st[j];
    ru = u * c - v * s;
    rv = v * c + u * s;
  };
  for (int i = tid; i < G * np; i += DP_THREADS) {
    const int g = i / np, j = i - g * np;
    float ru, rv;
    rotate(row + static_cast<size_t>(h0 + g) * dk, j, ru, rv);
    qs[g * Sh::KP + j * su] = __float2bfloat16(ru);
    qs[g * Sh::KP + j * su + ov] = __float2bfloat16(rv);
  }
  for (int i = tid; i < G * (dk - 2 * np); i += DP_THREADS) {
    const int g = i / (dk - 2 * np), d = 2 * np + i - g * (dk - 2 * np);
    qs[g * Sh::KP + d] = row[static_cast<size_t>(h0 + g) * dk + d];
  }
  __syncthreads();
  uint32_t qa[DK / 16][4];
  const uint32_t qaddr = smem_u32(qs) + (((lane & 7) + ((lane >> 3) & 1) * 8) * Sh::KP + (lane >> 4) * 8) * 2;
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk)
    if (FULL || kk < ksteps) dp_ldm(qaddr + kk * 32, qa[kk]);

  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int k = 0; k < 4; ++k) o[i][k] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;      // rows lane / 4 and lane / 4 + 8
  // keys [lo, hi) of the 16 in the tile take part
  auto compute = [&](uint32_t kd, int lo, int hi) {
    const uint32_t vd = kd + 16 * Sh::KP * 2;
    float s[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int k = 0; k < 4; ++k) s[n][k] = 0.f;
    const uint32_t ka = kd + (((lane & 7) + (lane >> 4) * 8) * Sh::KP + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk)
      if (FULL || kk < ksteps) {
        uint32_t kb[4];
        dp_ldm(ka + kk * 32, kb);
        dp_mma(s[0], qa[kk], kb[0], kb[1]);
        dp_mma(s[1], qa[kk], kb[2], kb[3]);
      }
    float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = n * 8 + (lane & 3) * 2 + e;
        const bool on = key >= lo && key < hi;
        s[n][e] = on ? s[n][e] * p.scale_log2 : -INFINITY;
        s[n][2 + e] = on ? s[n][2 + e] * p.scale_log2 : -INFINITY;
        x0 = fmaxf(x0, s[n][e]);
        x1 = fmaxf(x1, s[n][2 + e]);
      }
    x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
    x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
    const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);          // finite: every tile has at least one visible key
    const float a0 = exp2f(m0 - n0), a1 = exp2f(m1 - n1);
    m0 = n0; m1 = n1;
    uint32_t pa[4];
    float t0 = 0.f, t1 = 0.f;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const __nv_bfloat162 lo2 = __floats2bfloat162_rn(exp2f(s[n][0] - n0), exp2f(s[n][1] - n0));
      const __nv_bfloat162 hi2 = __floats2bfloat162_rn(exp2f(s[n][2] - n1), exp2f(s[n][3] - n1));
      t0 += __low2float(lo2) + __high2float(lo2);
      t1 += __low2float(hi2) + __high2float(hi2);
      pa[2 * n] = *reinterpret_cast<const uint32_t*>(&lo2);
      pa[2 * n + 1] = *reinterpret_cast<const uint32_t*>(&hi2);
    }
    l0 = l0 * a0 + t0;
    l1 = l1 * a1 + t1;
    if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) { o[i][0] *= a0; o[i][1] *= a0; o[i][2] *= a1; o[i][3] *= a1; }
    }
    const uint32_t va = vd + (((lane & 7) + ((lane >> 3) & 1) * 8) * Sh::VP + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int n = 0; n < DV / 16; ++n)
      if (FULL || n < vsteps) {
        uint32_t vb[4];
        dp_ldm_t(va + n * 32, vb);
        dp_mma(o[2 * n], pa, vb[0], vb[1]);
        dp_mma(o[2 * n + 1], pa, vb[2], vb[3]);
      }
  };

  for (int i = 0; i < mine; ++i) {
    dp_wait<STG - 2>();
    __syncwarp();                                // everyone's copies of page i are in, everyone is done with page i - 1
    issue(i + STG - 1);
    const int t = ta + warp + i * DP_WARPS;
    const int lo = max(0, first - t * DP_PS), hi = min(DP_PS, pos - t * DP_PS);
    if (lo < hi) compute(smem_u32(ring + (i % STG) * Sh::STAGE), lo, hi);
  }
  dp_wait<0>();
  __syncwarp();
  if (rank == S - 1 && warp == 0) {
    // the new token: row 0 of a tile of its own (in this warp's first stage), and its place in the cache
    __nv_bfloat16* kt = reinterpret_cast<__nv_bfloat16*>(ring);
    __nv_bfloat16* vt = kt + 16 * Sh::KP;
    const int page = pt[pos / DP_PS];
    const bool keep = hg == 0 && page >= 0 && page < p.c.num_pages;
    if (hg == 0 && !keep && lane == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (13 << 8));
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.c.data) + (keep ? static_cast<size_t>(page) * rec : 0);
    __nv_bfloat16* kdst = dst + k_off + static_cast<size_t>(pos % DP_PS) * dk;
    __nv_bfloat16* vdst = dst + v_off + static_cast<size_t>(pos % DP_PS) * dv;
    const __nv_bfloat16* kr = row + static_cast<size_t>(p.hq + kvh) * dk;
    const __nv_bfloat16* vr = row + static_cast<size_t>(p.hq + p.c.kv_heads) * dk + static_cast<size_t>(kvh) * dv;
    for (int i = lane; i < 15 * Sh::VP; i += 32) vt[Sh::VP + i] = __float2bfloat16(0.f);      // weight 0 must not meet a NaN
    for (int j = lane; j < np; j += 32) {
      float ru, rv;
      rotate(kr, j, ru, rv);
      const __nv_bfloat16 bu = __float2bfloat16(ru), bv = __float2bfloat16(rv);
      kt[j * su] = bu; kt[j * su + ov] = bv;
      if (keep) { kdst[j * su] = bu; kdst[j * su + ov] = bv; }
    }
    for (int d = 2 * np + lane; d < dk; d += 32) { kt[d] = kr[d]; if (keep) kdst[d] = kr[d]; }
    for (int d = lane; d < dv; d += 32) { vt[d] = vr[d]; if (keep) vdst[d] = vr[d]; }
    __syncwarp();
    compute(smem_u32(ring), 0, 1);
  }
  // row sums live in four lanes
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  __syncthreads();                               // the rings become the merge buffers

  float* wbuf = reinterpret_cast<float*>(smem) + warp * (16 * Sh::OP + 32);
  const int r0 = lane >> 2, r1 = r0 + 8;
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
    if (i * 8 < dv) {
      const int d = i * 8 + (lane & 3) * 2;
      if (r0 < G) *reinterpret_cast<float2*>(wbuf + r0 * Sh::OP + d) = make_float2(o[i][0], o[i][1]);
      if (r1 < G) *reinterpret_cast<float2*>(wbuf + r1 * Sh::OP + d) = make_float2(o[i][2], o[i][3]);
    }
  if ((lane & 3) == 0) {
    wbuf[16 * Sh::OP + r0] = m0; wbuf[16 * Sh::OP + 16 + r0] = l0;
    wbuf[16 * Sh::OP + r1] = m1; wbuf[16 * Sh::OP + 16 + r1] = l1;
  }
  __syncthreads();
  float* all = reinterpret_cast<float*>(smem);
  float* cbuf = all + DP_WARPS * (16 * Sh::OP + 32);
  for (int i = tid; i < G * dv; i += DP_THREADS) {
    const int g = i / dv, d = i - g * dv;
    float m = -INFINITY, v = 0.f, l = 0.f;
#pragma unroll
    for (int w = 0; w < DP_WARPS; ++w) m = fmaxf(m, all[w * (16 * Sh::OP + 32) + 16 * Sh::OP + g]);
#pragma unroll
    for (int w = 0; w < DP_WARPS; ++w) {
      const float* wb = all + w * (16 * Sh::OP + 32);
      const float mw = wb[16 * Sh::OP + g], f = mw == -INFINITY ? 0.f : exp2f(mw - m);
      if (f > 0.f) { v += f * wb[g * Sh::OP + d]; l += f * wb[16 * Sh::OP + 16 + g]; }
    }
    cbuf[g * Sh::OP + d] = v;
    if (d == 0) { cbuf[16 * Sh::OP + g] = m; cbuf[16 * Sh::OP + 16 + g] = l; }
  }
  if (S > 1) cluster_sync_all(); else __syncthreads();
  const uint32_t c_addr = smem_u32(cbuf);
  for (int i = rank * DP_THREADS + tid; i < G * dv; i += S * DP_THREADS) {
    const int g = i / dv, d = i - g * dv;
    float m = p.sink ? p.sink[h0 + g] * DP_LOG2E : -INFINITY;
    float l = p.sink ? 1.f : 0.f, v = 0.f;
    for (int s = 0; s < S; ++s) {
      const uint32_t base = S > 1 ? mapa_shared(c_addr, s) : c_addr;
      const float ms = dp_ld_cluster(base + 4u * (16 * Sh::OP + g));
      if (ms == -INFINITY) continue;
      const float mn = fmaxf(m, ms), fo = m == -INFINITY ? 0.f : exp2f(m - mn), fn = exp2f(ms - mn);
      l = l * fo + fn * dp_ld_cluster(base + 4u * (16 * Sh::OP + 16 + g));
      v = v * fo + fn * dp_ld_cluster(base + 4u * (g * Sh::OP + d));
      m = mn;
    }
    float f = l > 0.f ? 1.f / l : 0.f;
    if (p.gate) f *= 1.f / (1.f + __expf(-__bfloat162float(p.gate[static_cast<size_t>(b) * p.ldg + h0 + g])));
    p.out[static_cast<size_t>(b) * p.ldo + static_cast<size_t>(h0 + g) * dv + d] = __float2bfloat16(v * f);
  }
  if (S > 1) cluster_sync_all();                 // no CTA leaves while a peer may still read its partials
}

template <int DK, int DV, int STG, bool FULL>
static int launch_decode_paged(const DecodePagedParams& p, dim3 grid, cudaStream_t stream) {
  constexpr int SMEM = DpShape<DK, DV, STG>::SMEM;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_decode_paged_kernel<DK, DV, STG, FULL>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return -1000 - static_cast<int>(e);
    cudaFuncSetAttribute(attn_decode_paged_kernel<DK, DV, STG, FULL>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    configured = true;
  }
  launch_ex(attn_decode_paged_kernel<DK, DV, STG, FULL>, grid, dim3(DP_THREADS), SMEM, stream, p.splits, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_attn_decode_paged(const void* qkv, long long ld, void* out, long long ldo, int hq, int B, const int* positions,
                                      const int* seq_lens, const float* cos_tab, const float* sin_tab, int pairs, int interleaved,
                                      int max_pos, const b200_paged_cache* c, const b200_attn_spec* s, int splits, int* status,
                                      cudaStream_t stream) {
  if (B <= 0) return 0;
  if (!qkv || !out || !positions || !seq_lens || !c || !c->data || !c->page_table || !s || splits < 1 || splits > 8) return -1;
  if (c->f32 || c->page_size != DP_PS || c->dk <= 0 || c->dv <= 0 || c->dk > 256 || c->dv > 256 || c->dk % 8 || c->dv % 8) return -2;
  if (hq <= 0 || c->kv_heads <= 0 || hq % c->kv_heads || pairs < 0 || 2 * pairs > c->dk || max_pos <= 0 || B > c->num_seqs || B > 65535) return -3;
  if ((pairs > 0 && (!cos_tab || !sin_tab)) || (reinterpret_cast<uintptr_t>(c->data) & 15)) return -4;
  DecodePagedParams p;
  p.qkv = static_cast<const __nv_bfloat16*>(qkv); p.ld = ld; p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.hq = hq;
  p.hgroups = (hq / c->kv_heads + 15) / 16; p.positions = positions; p.seq_lens = seq_lens; p.cos_tab = cos_tab; p.sin_tab = sin_tab;
  p.pairs = pairs; p.interleaved = interleaved; p.max_pos = max_pos; p.c = *c; p.chunk = s->chunk; p.scale_log2 = s->scale * DP_LOG2E;
  p.sink = s->sink; p.gate = static_cast<const __nv_bfloat16*>(s->gate); p.ldg = s->ldg; p.splits = splits; p.status = status;
  const dim3 grid(splits, c->kv_heads * p.hgroups, B);
  const int d = c->dk > c->dv ? c->dk : c->dv;
  if (c->dk == 64 && c->dv == 64) return launch_decode_paged<64, 64, 6, true>(p, grid, stream);
  if (c->dk == 128 && c->dv == 128) return launch_decode_paged<128, 128, 3, true>(p, grid, stream);
  if (d <= 64) return launch_decode_paged<64, 64, 6, false>(p, grid, stream);
  if (d <= 128) return launch_decode_paged<128, 128, 3, false>(p, grid, stream);
  return launch_decode_paged<256, 256, 3, false>(p, grid, stream);
}
