// Latent attention over the paged cache in the latent space (bf16): queries that were moved there against the cached latents
// and the shared rotated key part, for decoding and for short portions.  All heads read the same keys, and a key's first
// `rank` dimensions are also its value, so a cached row is fetched once for scores and values.
//
// Rows are (token, head) pairs of one portion in order; a CTA takes 16 or 32 of them against 64 keys at a time.  The op is
// bound by the cached bytes for a few heads, so a tile of 64 rows (up to 80 KB) is in flight while the one before is
// computed.  The eight warps share a tile: scores by keys (8 each, m16n8k16 MMAs over the whole row), softmax by rows through
// shared memory, values by columns (16-column units), so no warp holds more than its part of the accumulators.  The splits of
// one row tile are a thread-block cluster that merges through distributed shared memory.  The rotary embedding of the query's
// second part happens while it is loaded.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"

namespace b200 {

constexpr int AL_THREADS = 256, AL_KEYS = 64, AL_PS = 16, AL_PP = AL_KEYS + 8, AL_SP = AL_KEYS + 4;
constexpr float AL_LOG2E = 1.4426950408889634f;
constexpr int AL_MAX_SMEM = 232448;

struct AttnLatentParams {
  const __nv_bfloat16* q; long long ldq;
  const __nv_bfloat16* q_rot; long long ldr; int head_ld_rot;
  __nv_bfloat16* out; long long ldo;
  b200_latent_dims d;
  float scale_log2;
  const int* cu; const int* positions; const int* seq_ids; const int* seq_lens;
  const float* cos_tab; const float* sin_tab;
  int max_pos, splits;
  b200_paged_cache c;
  int* status;
};

__device__ __forceinline__ void al_cp16(uint32_t dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;      // 0 source bytes: the destination is filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void al_ldm(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void al_ldm_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void al_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float al_ld_cluster(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}

// shared memory: two tiles of keys, the queries, softmax weights, scores, per-row numbers; the key tiles become the merge buffer
__host__ __device__ inline int al_kp(int dk) { return ((dk + 15) / 16) * 16 + 8; }      // row pitch: 16-byte skew, ldmatrix without conflicts
__host__ __device__ inline int al_smem(int dk, int mt) {
  const int kp = al_kp(dk);
  return 2 * AL_KEYS * kp * 2 + 16 * mt * (kp * 2 + AL_PP * 2 + AL_SP * 4) + 16 * mt * 4 * (3 + 8);
}

template <int MT, int NU>
__global__ void __launch_bounds__(AL_THREADS, NU == 4 ? 1 : 2)
attn_latent_kernel(const __grid_constant__ AttnLatentParams p) {
  constexpr int ROWS = 16 * MT, TPR = AL_THREADS / ROWS, KPT = AL_KEYS / TPR;      // softmax: threads per row, keys per thread
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(128) uint8_t al_smem_raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.d.heads, rank = p.d.rank, rot = p.d.rot, dk = rank + rot, ks = (dk + 15) >> 4, KP = al_kp(dk);
  const int b = blockIdx.z, S = p.splits, split = blockIdx.x, g0 = blockIdx.y * ROWS;
  const int row0 = p.cu ? p.cu[b] : b, len = p.cu ? p.cu[b + 1] - row0 : 1;
  if (g0 >= len * H) return;                             // the same for all CTAs of the cluster, as below
  const int n_rows = min(ROWS, len * H - g0);
  const int start = p.positions[row0], seq = p.seq_ids ? p.seq_ids[row0] : b;
  const int last_pos = start + (g0 + n_rows - 1) / H;
  const bool empty = p.seq_lens && p.seq_lens[b] <= 0;
  const bool bad = start < 0 || last_pos >= p.max_pos || seq < 0 || seq >= p.c.num_seqs || last_pos / AL_PS >= p.c.max_pages;
  if (empty || bad) {
    if (bad && tid == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (18 << 8));
    if (split == 0)
      for (int i = tid; i < n_rows * rank; i += AL_THREADS) {
        const int g = g0 + i / rank, tok = g / H;
        p.out[static_cast<size_t>(row0 + tok) * p.ldo + static_cast<size_t>(g - tok * H) * rank + i % rank] = __float2bfloat16(0.f);
      }
    return;
  }
  const int stage_bytes = AL_KEYS * KP * 2;
  uint8_t* s_q = al_smem_raw + 2 * stage_bytes;
  __nv_bfloat16* s_p = reinterpret_cast<__nv_bfloat16*>(s_q + ROWS * KP * 2);
  float* s_s = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(s_p) + ROWS * AL_PP * 2);
  float* s_alpha = s_s + ROWS * AL_SP;                   // [ROWS], then the row's maximum and sum, then a factor per split
  float* s_m = s_alpha + ROWS;
  float* s_l = s_m + ROWS;
  float* s_f = s_l + ROWS;
  const uint32_t ring = smem_u32(al_smem_raw);

  const int n_tiles = last_pos / AL_KEYS + 1;
  const int ta = static_cast<int>(static_cast<long long>(n_tiles) * split / S), tb = static_cast<int>(static_cast<long long>(n_tiles) * (split + 1) / S);
  const int* pt = p.c.page_table + static_cast<size_t>(seq) * p.c.max_pages;
  const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.c.data);
  const int kc = dk >> 3, r_first = lane / kc, c_first = lane - r_first * kc, r_step = 32 / kc, c_step = 32 - r_step * kc;
  // a warp fetches eight consecutive rows, half a page: one contiguous run
  auto issue = [&](int t, int st) {
    const int key0 = t * AL_KEYS + warp * 8, left = last_pos + 1 - key0;
    const int page = left > 0 ? pt[key0 / AL_PS] : -1;
    const bool ok = page >= 0 && page < p.c.num_pages;
    const __nv_bfloat16* src = cache + (ok ? (static_cast<size_t>(page) * AL_PS + key0 % AL_PS) * dk : 0) + lane * 8;
    const uint32_t dst = ring + st * stage_bytes + warp * 8 * KP * 2;
    for (int r = r_first, c = c_first; r < 8; src += 256) {
      al_cp16(dst + (r * KP + c * 8) * 2, ok ? src : cache, ok && r < left);
      r += r_step; c += c_step;
      if (c >= kc) { c -= kc; ++r; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (ta < tb) issue(ta, 0);

  // columns dk .. of the key rows are never fetched: zero once
  if (dk & 15)
    for (int i = tid; i < 2 * AL_KEYS; i += AL_THREADS) *reinterpret_cast<uint4*>(al_smem_raw + (i * KP + dk) * 2) = make_uint4(0u, 0u, 0u, 0u);
  for (int i = tid; i < ROWS * ks * 2; i += AL_THREADS) {
    const int r = i / (ks * 2), c = (i - r * ks * 2) * 8, g = g0 + r, tok = g / H;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < n_rows && c < rank) v = *reinterpret_cast<const uint4*>(p.q + static_cast<size_t>(row0 + tok) * p.ldq + static_cast<size_t>(g - tok * H) * rank + c);
    if (c < rank || c >= dk) *reinterpret_cast<uint4*>(s_q + (r * KP + c) * 2) = v;
  }
  const int np = p.d.true_rot / 2;
  for (int i = tid; i < ROWS * (rot / 2); i += AL_THREADS) {
    const int r = i / (rot / 2), j = i - r * (rot / 2), g = g0 + r, tok = g / H;
    float u = 0.f, v = 0.f;
    if (r < n_rows && j < np) {
      const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(p.q_rot + static_cast<size_t>(row0 + tok) * p.ldr + static_cast<size_t>(g - tok * H) * p.head_ld_rot + 2 * j);
      const float c = p.cos_tab[static_cast<size_t>(start + tok) * np + j], s = p.sin_tab[static_cast<size_t>(start + tok) * np + j];
      const float a = __low2float(x), d = __high2float(x);
      u = a * c - d * s;
      v = d * c + a * s;
    }
    *reinterpret_cast<__nv_bfloat162*>(s_q + (r * KP + rank + 2 * j) * 2) = __floats2bfloat162_rn(u, v);
  }

  float o[MT][2 * NU][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2 * NU; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) o[mt][i][k] = 0.f;
  // this thread's share of the softmax
  const int my_row = tid / TPR, my_key = (tid % TPR) * KPT;
  const int my_pos = start + min(g0 + my_row, len * H - 1) / H;
  float m_run = -INFINITY, l_run = 0.f;
  const uint32_t a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;      // ldmatrix rows / columns of an A operand

  for (int t = ta; t < tb; ++t) {
    const uint32_t kt = ring + ((t - ta) & 1) * stage_bytes;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                     // tile t is in for everyone; everyone is done with tile t - 1
    if (t + 1 < tb) issue(t + 1, (t + 1 - ta) & 1);
    float s[MT][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) s[mt][i][k] = 0.f;
    const uint32_t ka = kt + ((warp * 8 + (lane & 7)) * KP + (lane >> 3) * 8) * 2;
    const uint32_t qa0 = smem_u32(s_q) + (a_row * KP + a_col) * 2;
#pragma unroll 4
    for (int kk = 0; kk < ks; kk += 2) {
      uint32_t kb[4];
      al_ldm(ka + kk * 32, kb);                          // keys x 32 dimensions (the last 16 unused when ks is odd)
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t qa[4];
        al_ldm(qa0 + mt * 16 * KP * 2 + kk * 32, qa);
        al_mma(s[mt][0], qa, kb[0], kb[1]);
        if (kk + 1 < ks) {
          al_ldm(qa0 + mt * 16 * KP * 2 + kk * 32 + 32, qa);
          al_mma(s[mt][1], qa, kb[2], kb[3]);
        }
      }
    }
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      float* at = s_s + (mt * 16 + (lane >> 2)) * AL_SP + warp * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(at) = make_float2(s[mt][0][0] + s[mt][1][0], s[mt][0][1] + s[mt][1][1]);
      *reinterpret_cast<float2*>(at + 8 * AL_SP) = make_float2(s[mt][0][2] + s[mt][1][2], s[mt][0][3] + s[mt][1][3]);
    }
    __syncthreads();
    {
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT; i += 4) {
        const float4 x = *reinterpret_cast<const float4*>(s_s + my_row * AL_SP + my_key + i);
        v[i] = x.x; v[i + 1] = x.y; v[i + 2] = x.z; v[i + 3] = x.w;
      }
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        v[i] = t * AL_KEYS + my_key + i <= my_pos ? v[i] * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int w = TPR / 2; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float m_new = fmaxf(m_run, mx), m_use = m_new == -INFINITY ? 0.f : m_new;
      const float alpha = m_run == -INFINITY ? 0.f : exp2f(m_run - m_use);
      m_run = m_new;
      float sum = 0.f;
      uint32_t pk[KPT / 2];
#pragma unroll
      for (int i = 0; i < KPT; i += 2) {
        const __nv_bfloat162 e = __floats2bfloat162_rn(exp2f(v[i] - m_use), exp2f(v[i + 1] - m_use));
        sum += __low2float(e) + __high2float(e);         // what the MMA will actually see
        pk[i / 2] = *reinterpret_cast<const uint32_t*>(&e);
      }
#pragma unroll
      for (int i = 0; i < KPT / 2; i += 2) *reinterpret_cast<uint2*>(s_p + my_row * AL_PP + my_key + 2 * i) = make_uint2(pk[i], pk[i + 1]);
      l_run = l_run * alpha + sum;
      if (my_key == 0) s_alpha[my_row] = alpha;
    }
    __syncthreads();
    uint32_t pa[MT][4][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float f0 = s_alpha[mt * 16 + (lane >> 2)], f1 = s_alpha[mt * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int k = 0; k < 4; ++k) al_ldm(smem_u32(s_p) + ((mt * 16 + a_row) * AL_PP + k * 16 + a_col) * 2, pa[mt][k]);
      if (__any_sync(0xffffffffu, f0 != 1.f || f1 != 1.f)) {
#pragma unroll
        for (int i = 0; i < 2 * NU; ++i) { o[mt][i][0] *= f0; o[mt][i][1] *= f0; o[mt][i][2] *= f1; o[mt][i][3] *= f1; }
      }
    }
#pragma unroll
    for (int u = 0; u < NU; ++u) {
      const int col = (warp + 8 * u) * 16;
      if (col < rank) {
        const uint32_t va = kt + (a_row * KP + col + a_col) * 2;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          uint32_t vb[4];
          al_ldm_t(va + k * 16 * KP * 2, vb);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            al_mma(o[mt][2 * u], pa[mt][k], vb[0], vb[1]);
            al_mma(o[mt][2 * u + 1], pa[mt][k], vb[2], vb[3]);
          }
        }
      }
    }
  }

#pragma unroll
  for (int w = TPR / 2; w > 0; w >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, w);
  __syncthreads();                                       // the key tiles become the merge buffer
  float* obuf = reinterpret_cast<float*>(al_smem_raw);
  const int OP = rank + 4;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < 2 * NU; ++i) {
      const int d = (warp + 8 * (i >> 1)) * 16 + (i & 1) * 8 + (lane & 3) * 2, r = mt * 16 + (lane >> 2);
      if (d < rank) {
        *reinterpret_cast<float2*>(obuf + r * OP + d) = make_float2(o[mt][i][0], o[mt][i][1]);
        *reinterpret_cast<float2*>(obuf + (r + 8) * OP + d) = make_float2(o[mt][i][2], o[mt][i][3]);
      }
    }
  if (my_key == 0) { s_m[my_row] = m_run; s_l[my_row] = l_run; }
  if (S > 1) cluster_sync_all(); else __syncthreads();
  if (tid < n_rows) {                                    // the row's factor for every split
    const uint32_t ma = smem_u32(s_m + tid), la = smem_u32(s_l + tid);
    float m = -INFINITY, l = 0.f;
    for (int s = 0; s < S; ++s) m = fmaxf(m, al_ld_cluster(mapa_shared(ma, s)));
    for (int s = 0; s < S; ++s) {
      const float ms = al_ld_cluster(mapa_shared(ma, s)), f = ms == -INFINITY ? 0.f : exp2f(ms - m);
      s_f[s * ROWS + tid] = f;
      l += f * al_ld_cluster(mapa_shared(la, s));
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    for (int s = 0; s < S; ++s) s_f[s * ROWS + tid] *= inv;
  }
  __syncthreads();
  const int half = rank >> 1;
  for (int i = split * AL_THREADS + tid; i < n_rows * half; i += S * AL_THREADS) {
    const int r = i / half, d = (i - r * half) * 2, g = g0 + r, tok = g / H;
    const uint32_t at = smem_u32(obuf + r * OP + d);
    float v0 = 0.f, v1 = 0.f;
    for (int s = 0; s < S; ++s) {
      const uint32_t a = mapa_shared(at, s);
      const float f = s_f[s * ROWS + r];
      v0 += f * al_ld_cluster(a);
      v1 += f * al_ld_cluster(a + 4);
    }
    *reinterpret_cast<__nv_bfloat162*>(p.out + static_cast<size_t>(row0 + tok) * p.ldo + static_cast<size_t>(g - tok * H) * rank + d) = __floats2bfloat162_rn(v0, v1);
  }
  if (S > 1) cluster_sync_all();                         // no CTA leaves while a peer may still read its partials
}

template <int MT, int NU>
static int launch_attn_latent(const AttnLatentParams& p, dim3 grid, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_latent_kernel<MT, NU>, cudaFuncAttributeMaxDynamicSharedMemorySize, AL_MAX_SMEM);
    if (e != cudaSuccess) return -1000 - static_cast<int>(e);
    cudaFuncSetAttribute(attn_latent_kernel<MT, NU>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    configured = true;
  }
  launch_ex(attn_latent_kernel<MT, NU>, grid, dim3(AL_THREADS), al_smem(p.d.rank + p.d.rot, MT), stream, p.splits, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

bool latent_cache_ok(const b200_paged_cache* c, const b200_latent_dims* d);      // latent.cu

}  // namespace b200

using namespace b200;

// CTAs per SM the kernel reaches with these sizes (16 or 32 rows per CTA); 0: sizes beyond it
extern "C" int b200_attn_latent_ctas_per_sm(int rank, int rot, int rows) {
  if (rank <= 0 || rank > 512 || rot < 0 || rank % 8 || rot % 8) return 0;
  const int smem = al_smem(rank + rot, rows > 16 ? 2 : 1) + 1024, merge = 16 * (rows > 16 ? 2 : 1) * (rank + 4) * 4;
  if (smem > AL_MAX_SMEM || merge > 2 * AL_KEYS * al_kp(rank + rot) * 2) return 0;
  return rank <= 256 && 2 * smem <= AL_MAX_SMEM ? 2 : 1;
}

extern "C" int b200_attn_latent(const void* q, long long ldq, const void* q_rot, long long ldr, int head_ld_rot, void* out, long long ldo,
                                int M, const b200_latent_dims* d, float scale, const int* cu, int portions, int max_len, const int* positions,
                                const int* seq_ids, const int* seq_lens, const float* cos_tab, const float* sin_tab, int max_pos,
                                const b200_paged_cache* cache, int splits, int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!q || !q_rot || !out || !positions || !latent_cache_ok(cache, d) || cache->f32 || cache->page_size != AL_PS) return -1;
  if (ldq % 8 || ldo % 2 || ldr % 2 || head_ld_rot % 2 || (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(q_rot) & 3)) return -2;
  if (splits < 1 || splits > 8 || max_pos <= 0 || (d->true_rot > 0 && (!cos_tab || !sin_tab)) || (cu && (portions <= 0 || max_len <= 0))) return -3;
  const int longest = cu ? max_len : 1, batch = cu ? portions : M;
  const int mt = static_cast<long long>(longest) * d->heads > 16 ? 2 : 1;
  if (b200_attn_latent_ctas_per_sm(d->rank, d->rot, 16 * mt) == 0) return -4;
  AttnLatentParams p;
  p.q = static_cast<const __nv_bfloat16*>(q); p.ldq = ldq; p.q_rot = static_cast<const __nv_bfloat16*>(q_rot); p.ldr = ldr; p.head_ld_rot = head_ld_rot;
  p.out = static_cast<__nv_bfloat16*>(out); p.ldo = ldo; p.d = *d; p.scale_log2 = scale * AL_LOG2E; p.cu = cu; p.positions = positions;
  p.seq_ids = seq_ids; p.seq_lens = seq_lens; p.cos_tab = cos_tab; p.sin_tab = sin_tab; p.max_pos = max_pos; p.splits = splits; p.c = *cache; p.status = status;
  const long long tiles = (static_cast<long long>(longest) * d->heads + 16 * mt - 1) / (16 * mt);
  if (tiles > 65535 || batch > 65535) return -5;
  const dim3 grid(splits, static_cast<unsigned>(tiles), batch);
  const int nu = d->rank <= 128 ? 1 : (d->rank <= 256 ? 2 : 4);
  if (mt == 1) return nu == 1 ? launch_attn_latent<1, 1>(p, grid, stream) : (nu == 2 ? launch_attn_latent<1, 2>(p, grid, stream) : launch_attn_latent<1, 4>(p, grid, stream));
  return nu == 1 ? launch_attn_latent<2, 1>(p, grid, stream) : (nu == 2 ? launch_attn_latent<2, 2>(p, grid, stream) : launch_attn_latent<2, 4>(p, grid, stream));
}
