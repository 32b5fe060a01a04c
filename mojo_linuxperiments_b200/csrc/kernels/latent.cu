// Token-wise pieces around latent attention: the paged cache keeps one normalised latent and one rotated key part per token.
//
//   latent_append   norms of the query latent and of the key/value latent, rotation of the shared key part, cache append
//   rotary_heads    rotation of one part of every query head, in place
//   latent_gather   cached latents of whole sequences into consecutive rows (a portion that continues a sequence and
//                   expands its keys needs those of earlier portions too)
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "dense_epilogue.cuh"

namespace b200 {

template <typename T> __device__ __forceinline__ float la_f(T v);
template <> __device__ __forceinline__ float la_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float la_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

struct LatentAppendParams {
  const float* in; long long ld;
  int q_rank, true_q_rank;
  const float* q_gain; const float* c_gain;
  float eps;
  b200_latent_dims d;
  const int* positions; const int* seq_ids; const int* seq_lens;
  const float* cos_tab; const float* sin_tab;
  int max_pos;
  b200_paged_cache c;
  void* cq; long long ldq;
  void* lat;
  int* status;
};

// one CTA per token, four columns at a time
template <typename T, int THREADS>
__global__ void __launch_bounds__(THREADS) latent_append_kernel(const __grid_constant__ LatentAppendParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int tok = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = p.positions[tok], seq = p.seq_ids ? p.seq_ids[tok] : tok, ps = p.c.page_size;
  const bool empty = p.seq_lens && p.seq_lens[tok] <= 0;            // decode over a slot without a sequence
  // a position outside the tables or the sequence's pages must not become a stray write: skipped and reported
  bool bad = pos < 0 || pos >= p.max_pos || seq < 0 || seq >= p.c.num_seqs || pos / ps >= p.c.max_pages;
  int page = 0;
  if (!bad && !empty) page = p.c.page_table[static_cast<size_t>(seq) * p.c.max_pages + pos / ps];
  const float* row = p.in + static_cast<size_t>(tok) * p.ld;
  const float* lat_in = row + p.q_rank;
  const float* rot_in = lat_in + p.d.rank;
  auto squares = [](float4 v, int left) {               // of the first `left` of four
    return (left > 0 ? v.x * v.x : 0.f) + (left > 1 ? v.y * v.y : 0.f) + (left > 2 ? v.z * v.z : 0.f) + (left > 3 ? v.w * v.w : 0.f);
  };
  float sq = 0.f, sc = 0.f;
#pragma unroll 4
  for (int i = threadIdx.x * 4; i < p.q_rank; i += THREADS * 4) sq += squares(*reinterpret_cast<const float4*>(row + i), p.true_q_rank - i);
#pragma unroll 2
  for (int i = threadIdx.x * 4; i < p.d.rank; i += THREADS * 4) sc += squares(*reinterpret_cast<const float4*>(lat_in + i), p.d.true_rank - i);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) { sq += __shfl_xor_sync(0xffffffffu, sq, o); sc += __shfl_xor_sync(0xffffffffu, sc, o); }
  __shared__ float red[2][THREADS / 32];
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sc; }
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int w = 0; w < THREADS / 32; ++w) { sq += red[0][w]; sc += red[1][w]; }
  const float fq = 1.f / sqrtf(sq / static_cast<float>(p.true_q_rank) + p.eps), fc = 1.f / sqrtf(sc / static_cast<float>(p.d.true_rank) + p.eps);
  bad = bad || (!empty && (page < 0 || page >= p.c.num_pages));
  if (bad && threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (15 << 8));

  constexpr bool F32 = sizeof(T) == 4;
  auto scaled = [](float4 v, float f, float4 g) { return make_float4(v.x * f * g.x, v.y * f * g.y, v.z * f * g.z, v.w * f * g.w); };
  auto cut = [](float4 v, int left) {                   // padding is zero whatever the linear left there
    return make_float4(left > 0 ? v.x : 0.f, left > 1 ? v.y : 0.f, left > 2 ? v.z : 0.f, left > 3 ? v.w : 0.f);
  };
#pragma unroll 4
  for (int i = threadIdx.x * 4; i < p.q_rank; i += THREADS * 4)
    store4_any(p.cq, F32, static_cast<long long>(tok) * p.ldq + i,
               scaled(cut(*reinterpret_cast<const float4*>(row + i), p.true_q_rank - i), fq, __ldg(reinterpret_cast<const float4*>(p.q_gain + i))));
  const int dk = p.d.rank + p.d.rot;
  const long long rec = (static_cast<long long>(page) * ps + pos % ps) * dk;
  const bool keep = !bad && !empty;
  auto put = [&](int i, float4 v) {
    if (keep) store4_any(p.c.data, F32, rec + i, v);
    if (p.lat) store4_any(p.lat, F32, static_cast<long long>(tok) * dk + i, v);
  };
#pragma unroll 2
  for (int i = threadIdx.x * 4; i < p.d.rank; i += THREADS * 4)
    put(i, scaled(cut(*reinterpret_cast<const float4*>(lat_in + i), p.d.true_rank - i), fc, __ldg(reinterpret_cast<const float4*>(p.c_gain + i))));
  // the last threads take the rotated part: they had the least to do
  const int np = p.d.true_rot / 2, at = bad ? 0 : pos;
  for (int i = (THREADS - 1 - threadIdx.x) * 4; i < p.d.rot; i += THREADS * 4) {
    const float4 x = *reinterpret_cast<const float4*>(rot_in + i);
    const size_t t = static_cast<size_t>(at) * np + i / 2;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i / 2 < np) { const float c = p.cos_tab[t], s = p.sin_tab[t]; o.x = x.x * c - x.y * s; o.y = x.y * c + x.x * s; }
    if (i / 2 + 1 < np) { const float c = p.cos_tab[t + 1], s = p.sin_tab[t + 1]; o.z = x.z * c - x.w * s; o.w = x.w * c + x.z * s; }
    put(p.d.rank + i, o);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) rotary_heads_kernel(T* q, long long ld, int heads, int head_ld, int offset, int np, const int* positions,
                                                           const float* cos_tab, const float* sin_tab, int max_pos, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int tok = blockIdx.x, pos = positions[tok];
  if (pos < 0 || pos >= max_pos) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (16 << 8));
    return;
  }
  const float* ct = cos_tab + static_cast<size_t>(pos) * np;
  const float* st = sin_tab + static_cast<size_t>(pos) * np;
  T* row = q + static_cast<size_t>(tok) * ld + offset;
  for (int i = threadIdx.x; i < heads * np; i += blockDim.x) {
    const int h = i / np, j = i - h * np;
    T* x = row + static_cast<size_t>(h) * head_ld + 2 * j;
    const float u = la_f(x[0]), v = la_f(x[1]), c = ct[j], s = st[j];
    x[0] = static_cast<T>(u * c - v * s);
    x[1] = static_cast<T>(v * c + u * s);
  }
}

// grid (16-token pages, sequences); copies in 16-byte pieces
__global__ void __launch_bounds__(128) latent_gather_kernel(b200_paged_cache c, int elem, const int* ctx, const int* seqs, uint8_t* out, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, seq = seqs[b], n = ctx[b + 1] - ctx[b], t0 = blockIdx.x * c.page_size;
  if (t0 >= n) return;
  const bool known = seq >= 0 && seq < c.num_seqs && static_cast<int>(blockIdx.x) < c.max_pages;
  const int page = known ? c.page_table[static_cast<size_t>(seq) * c.max_pages + blockIdx.x] : -1;
  if (page < 0 || page >= c.num_pages) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (17 << 8));
    return;
  }
  const size_t row = static_cast<size_t>(c.dk) * elem;
  const uint4* src = reinterpret_cast<const uint4*>(static_cast<const uint8_t*>(c.data) + static_cast<size_t>(page) * c.page_size * row);
  uint4* dst = reinterpret_cast<uint4*>(out + (static_cast<size_t>(ctx[b]) + t0) * row);
  const int pieces = static_cast<int>(min(c.page_size, n - t0) * row / 16);
  for (int i = threadIdx.x; i < pieces; i += blockDim.x) dst[i] = src[i];
}

bool latent_cache_ok(const b200_paged_cache* c, const b200_latent_dims* d) {
  return c && d && c->data && c->page_table && c->kv_heads == 1 && c->dv == 0 && c->page_size > 0 && c->num_pages > 0 && d->heads > 0 &&
         d->rank > 0 && d->rot >= 0 && d->rank % 8 == 0 && d->rot % 8 == 0 && c->dk == d->rank + d->rot && d->true_rank > 0 &&
         d->true_rank <= d->rank && d->true_rot <= d->rot && d->true_rot % 2 == 0 && (reinterpret_cast<uintptr_t>(c->data) & 15) == 0;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_append(const float* in, long long ld, int M, int q_rank, int true_q_rank, const float* q_gain, const float* c_gain,
                                  float eps, const b200_latent_dims* dims, const int* positions, const int* seq_ids, const int* seq_lens,
                                  const float* cos_tab, const float* sin_tab, int max_pos, const b200_paged_cache* cache, void* cq,
                                  long long ldq, void* lat, int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!latent_cache_ok(cache, dims)) return -1;
  if (!in || !cq || !q_gain || !c_gain || !positions || q_rank <= 0 || true_q_rank <= 0 || true_q_rank > q_rank || ldq < q_rank) return -2;
  auto al16 = [](const void* a) { return (reinterpret_cast<uintptr_t>(a) & 15) == 0; };
  if (q_rank % 8 || ld % 4 || ldq % 8 || !al16(in) || !al16(cq) || !al16(q_gain) || !al16(c_gain) || !al16(lat)) return -4;
  if (ld < q_rank + cache->dk || max_pos <= 0 || (dims->true_rot > 0 && (!cos_tab || !sin_tab))) return -3;
  LatentAppendParams p;
  p.in = in; p.ld = ld; p.q_rank = q_rank; p.true_q_rank = true_q_rank; p.q_gain = q_gain; p.c_gain = c_gain; p.eps = eps; p.d = *dims;
  p.positions = positions; p.seq_ids = seq_ids; p.seq_lens = seq_lens; p.cos_tab = cos_tab; p.sin_tab = sin_tab; p.max_pos = max_pos;
  p.c = *cache; p.cq = cq; p.ldq = ldq; p.lat = lat; p.status = status;
  // few tokens: as much of a row at once as possible
  if (cache->f32) launch_ex(latent_append_kernel<float, 128>, dim3(M), dim3(128), 0, stream, 0, p);
  else if (M <= 256) launch_ex(latent_append_kernel<__nv_bfloat16, 256>, dim3(M), dim3(256), 0, stream, 0, p);
  else launch_ex(latent_append_kernel<__nv_bfloat16, 128>, dim3(M), dim3(128), 0, stream, 0, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

extern "C" int b200_rotary_heads(void* q, long long ld, int f32, int M, int heads, int head_ld, int offset, int true_rot, const int* positions,
                                 const float* cos_tab, const float* sin_tab, int max_pos, int* status, cudaStream_t stream) {
  if (M <= 0 || true_rot <= 0) return 0;
  if (!q || !positions || !cos_tab || !sin_tab || heads <= 0 || true_rot % 2 || offset < 0 || offset + true_rot > head_ld || ld < static_cast<long long>(heads) * head_ld || max_pos <= 0) return -1;
  if (f32) launch_ex(rotary_heads_kernel<float>, dim3(M), dim3(128), 0, stream, 0, static_cast<float*>(q), ld, heads, head_ld, offset, true_rot / 2, positions, cos_tab, sin_tab, max_pos, status);
  else launch_ex(rotary_heads_kernel<__nv_bfloat16>, dim3(M), dim3(128), 0, stream, 0, static_cast<__nv_bfloat16*>(q), ld, heads, head_ld, offset, true_rot / 2, positions, cos_tab, sin_tab, max_pos, status);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

extern "C" int b200_latent_gather(const b200_paged_cache* cache, const int* ctx, const int* seqs, int B, int max_ctx, void* lat, int* status,
                                  cudaStream_t stream) {
  if (B <= 0 || max_ctx <= 0) return 0;
  if (!cache || !cache->data || !cache->page_table || cache->kv_heads != 1 || cache->dv != 0 || cache->dk % 8 || cache->page_size <= 0 || !ctx || !seqs || !lat || B > 65535) return -1;
  if ((reinterpret_cast<uintptr_t>(lat) & 15) || (reinterpret_cast<uintptr_t>(cache->data) & 15)) return -2;
  launch_ex(latent_gather_kernel, dim3((max_ctx + cache->page_size - 1) / cache->page_size, B), dim3(128), 0, stream, 0, *cache, cache->f32 ? 4 : 2, ctx, seqs, static_cast<uint8_t*>(lat), status);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
