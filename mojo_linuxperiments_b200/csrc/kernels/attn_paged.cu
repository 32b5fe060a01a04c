// General attention over a paged cache, bf16 or fp32, any head size: one warp per (query token, query head).
//
// The 32-bit form of a model and head sizes beyond the tensor-core kernels run here.  Keys are taken 32 at a time (lane <->
// key, exact dot product in fp32), online softmax per block of 32, then the lanes share out the value dimensions (512 at a
// time; blockIdx.z picks the part).  The latent form reads the query in two parts and takes the first dimensions of a
// cached key as its value.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"

namespace b200 {

template <typename T> __device__ __forceinline__ float ap_f(T v);
template <> __device__ __forceinline__ float ap_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float ap_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

constexpr int APG_WARPS = 4;
constexpr int APG_MAX_DV = 512;

struct AttnPagedParams {
  const void* q; long long ldq;
  const void* q2; long long ldq2;        // latent form: the query's last dk - q_len dimensions, q2_head apart per head
  int q_len, q_head, q2_head;            // q_len = dk otherwise
  int dv, latent;                        // latent: values are the first dv dimensions of the keys
  void* out; long long ldo;
  int hq, M;
  const int* positions; const int* seq_ids; const int* seq_lens;
  b200_paged_cache c;
  b200_attn_spec s;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(32 * APG_WARPS) attn_paged_kernel(const __grid_constant__ AttnPagedParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * APG_WARPS + warp, tok = blockIdx.x;
  if (h >= p.hq) return;
  const int dk = p.c.dk, dv = p.dv, ps = p.c.page_size, d0 = blockIdx.z * APG_MAX_DV;
  const int seq = p.seq_ids ? p.seq_ids[tok] : tok;
  T* o = static_cast<T*>(p.out) + static_cast<size_t>(tok) * p.ldo + static_cast<size_t>(h) * dv;
  const int pos = p.positions[tok];
  const bool empty = p.seq_lens && p.seq_lens[tok] <= 0;            // decode over a slot without a sequence
  const bool bad = pos < 0 || seq < 0 || seq >= p.c.num_seqs || pos / ps >= p.c.max_pages;
  if (bad || empty) {
    if (bad && lane == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (14 << 8));
    for (int d = d0 + lane; d < min(dv, d0 + APG_MAX_DV); d += 32) o[d] = T(0.f);
    return;
  }
  const int kvh = h / (p.hq / p.c.kv_heads);
  const T* q = static_cast<const T*>(p.q) + static_cast<size_t>(tok) * p.ldq + static_cast<size_t>(h) * p.q_head;
  const T* q2 = static_cast<const T*>(p.q2) + static_cast<size_t>(tok) * p.ldq2 + static_cast<size_t>(h) * p.q2_head;
  const int* pt = p.c.page_table + static_cast<size_t>(seq) * p.c.max_pages;
  const size_t rec = static_cast<size_t>(p.c.kv_heads) * ps * (dk + (p.latent ? 0 : dv));
  const int vp = p.latent ? dk : dv;                                 // pitch of the value rows
  const T* cache = static_cast<const T*>(p.c.data);
  const int first = p.s.chunk > 0 ? pos - pos % p.s.chunk : 0;
  // the sink opens the softmax: a term of the denominator without a value
  float m = p.s.sink ? p.s.sink[h] : -INFINITY, l = p.s.sink ? 1.f : 0.f;
  float acc[APG_MAX_DV / 32];
#pragma unroll
  for (int i = 0; i < APG_MAX_DV / 32; ++i) acc[i] = 0.f;
  for (int k0 = first; k0 <= pos; k0 += 32) {
    const int key = k0 + lane;
    float s = -INFINITY;
    if (key <= pos) {
      const int page = pt[key / ps];
      if (page >= 0 && page < p.c.num_pages) {
        const T* kr = cache + static_cast<size_t>(page) * rec + (static_cast<size_t>(kvh) * ps + key % ps) * dk;
        float d = 0.f;
        for (int i = 0; i < p.q_len; ++i) d = fmaf(ap_f(q[i]), ap_f(kr[i]), d);
        for (int i = p.q_len; i < dk; ++i) d = fmaf(ap_f(q2[i - p.q_len]), ap_f(kr[i]), d);
        s = d * p.s.scale;
      }
    }
    float mx = s;
#pragma unroll
    for (int t = 16; t > 0; t >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, t));
    const float m_new = fmaxf(m, mx);
    if (m_new == -INFINITY) continue;
    const float a = m == -INFINITY ? 0.f : expf(m - m_new);
    const float e = s == -INFINITY ? 0.f : expf(s - m_new);
    float sum = e;
#pragma unroll
    for (int t = 16; t > 0; t >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, t);
    l = l * a + sum;
    m = m_new;
#pragma unroll
    for (int i = 0; i < APG_MAX_DV / 32; ++i) acc[i] *= a;
    const int n = min(32, pos - k0 + 1);
    for (int j = 0; j < n; ++j) {
      const float w = __shfl_sync(0xffffffffu, e, j);
      const int kj = k0 + j, page = pt[kj / ps];
      if (page < 0 || page >= p.c.num_pages) continue;
      const T* vr = cache + static_cast<size_t>(page) * rec + (p.latent ? 0 : static_cast<size_t>(p.c.kv_heads) * ps * dk) +
                    (static_cast<size_t>(kvh) * ps + kj % ps) * vp + d0;
#pragma unroll
      for (int i = 0; i < APG_MAX_DV / 32; ++i)
        if (d0 + i * 32 + lane < dv) acc[i] = fmaf(w, ap_f(vr[i * 32 + lane]), acc[i]);
    }
  }
  float f = l > 0.f ? 1.f / l : 0.f;
  if (p.s.gate) f *= 1.f / (1.f + expf(-ap_f(static_cast<const T*>(p.s.gate)[static_cast<size_t>(tok) * p.s.ldg + h])));
#pragma unroll
  for (int i = 0; i < APG_MAX_DV / 32; ++i)
    if (d0 + i * 32 + lane < dv) o[d0 + i * 32 + lane] = T(acc[i] * f);
}

}  // namespace b200

using namespace b200;

static int launch_attn_paged(const AttnPagedParams& p, cudaStream_t stream) {
  const dim3 grid(p.M, (p.hq + APG_WARPS - 1) / APG_WARPS, (p.dv + APG_MAX_DV - 1) / APG_MAX_DV);
  if (p.c.f32) launch_ex(attn_paged_kernel<float>, grid, dim3(32 * APG_WARPS), 0, stream, 0, p);
  else launch_ex(attn_paged_kernel<__nv_bfloat16>, grid, dim3(32 * APG_WARPS), 0, stream, 0, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

extern "C" int b200_attn_paged(const void* q, long long ldq, void* out, long long ldo, int hq, int M, const int* positions,
                               const int* seq_ids, const int* seq_lens, const b200_paged_cache* cache, const b200_attn_spec* spec,
                               int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!q || !out || !positions || !cache || !cache->data || !cache->page_table || !spec) return -1;
  if (hq <= 0 || cache->kv_heads <= 0 || hq % cache->kv_heads || cache->page_size <= 0 || cache->dk <= 0 || cache->dv <= 0) return -2;
  AttnPagedParams p = {};
  p.q = p.q2 = q; p.ldq = ldq; p.q_len = p.q_head = cache->dk; p.dv = cache->dv; p.out = out; p.ldo = ldo; p.hq = hq; p.M = M;
  p.positions = positions; p.seq_ids = seq_ids; p.seq_lens = seq_lens; p.c = *cache; p.s = *spec; p.status = status;
  return launch_attn_paged(p, stream);
}

namespace b200 { bool latent_cache_ok(const b200_paged_cache* c, const b200_latent_dims* d); }      // latent.cu

extern "C" int b200_attn_latent_any(const void* q, long long ldq, const void* q_rot, long long ldr, int head_ld_rot, void* out, long long ldo,
                                    int M, const b200_latent_dims* d, float scale, const int* positions, const int* seq_ids,
                                    const int* seq_lens, const b200_paged_cache* cache, int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!q || !q_rot || !out || !positions || !latent_cache_ok(cache, d)) return -1;
  AttnPagedParams p = {};
  p.q = q; p.ldq = ldq; p.q2 = q_rot; p.ldq2 = ldr; p.q_len = p.q_head = d->rank; p.q2_head = head_ld_rot; p.dv = d->rank; p.latent = 1;
  p.out = out; p.ldo = ldo; p.hq = d->heads; p.M = M; p.positions = positions; p.seq_ids = seq_ids; p.seq_lens = seq_lens; p.c = *cache;
  p.s.scale = scale; p.status = status;
  return launch_attn_paged(p, stream);
}
