// Token-wise pieces around attention over a paged cache whose heads may have any size, in bf16 or fp32:
//
//   rotary_paged   rotary embedding of the first 2 * pairs dimensions of q (in place) and k, either pairing
//                  (interleaved: 2i with 2i+1; halves: i with i + pairs); k and v go to the cache
//   embed_norm     token ids -> scaled fp32 embedding row (the residual stream, and a second copy when the model adds it
//                  again later) and the first layer's element-wise norm of it
//
// Cache layout of a layer: one record per page, [kv_heads][page_size][dk] keys, then [kv_heads][page_size][dv] values.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "dense_epilogue.cuh"

namespace b200 {

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

struct RotaryPagedParams {
  void* qkv; long long ld;
  const int* positions; const int* seq_ids;
  const float* cos_tab; const float* sin_tab;
  int pairs, interleaved, max_pos;
  b200_paged_cache c;
  int hq, M;
  int* status;
};

// one CTA per token: q pairs, then k (rotated or copied), then v
template <typename T>
__global__ void __launch_bounds__(128) rotary_paged_kernel(const __grid_constant__ RotaryPagedParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int tok = blockIdx.x;
  const int pos = p.positions[tok], seq = p.seq_ids ? p.seq_ids[tok] : tok;
  // a position outside the tables or the sequence's pages must not become a stray write: skipped and reported
  bool bad = pos < 0 || pos >= p.max_pos || seq < 0 || seq >= p.c.num_seqs || pos / p.c.page_size >= p.c.max_pages;
  int page = 0;
  if (!bad) {
    page = p.c.page_table[static_cast<size_t>(seq) * p.c.max_pages + pos / p.c.page_size];
    bad = page < 0 || page >= p.c.num_pages;
  }
  if (bad) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, static_cast<int>(ST_BAD_ARGUMENT) | (12 << 8));
    return;
  }
  const int dk = p.c.dk, dv = p.c.dv, G = p.c.kv_heads, ps = p.c.page_size, slot = pos % ps;
  T* row = static_cast<T*>(p.qkv) + static_cast<size_t>(tok) * p.ld;
  T* rec = static_cast<T*>(p.c.data) + static_cast<size_t>(page) * G * ps * (dk + dv);
  const float* ct = p.cos_tab + static_cast<size_t>(pos) * p.pairs;
  const float* st = p.sin_tab + static_cast<size_t>(pos) * p.pairs;
  const int np = p.pairs, st_u = p.interleaved ? 2 : 1, off_v = p.interleaved ? 1 : np;
  for (int i = threadIdx.x; i < (p.hq + G) * np; i += blockDim.x) {
    const int h = i / np, j = i - h * np;
    T* x = row + static_cast<size_t>(h) * dk + j * st_u;          // k heads follow the q heads
    const float u = to_f(x[0]), v = to_f(x[off_v]), c = ct[j], s = st[j];
    const T ru = from_f<T>(u * c - v * s), rv = from_f<T>(v * c + u * s);
    if (h < p.hq) { x[0] = ru; x[off_v] = rv; }
    else {
      T* kd = rec + (static_cast<size_t>(h - p.hq) * ps + slot) * dk + j * st_u;
      kd[0] = ru; kd[off_v] = rv;
    }
  }
  const T* krow = row + static_cast<size_t>(p.hq) * dk;
  const int rest = dk - 2 * np;
  for (int i = threadIdx.x; i < G * rest; i += blockDim.x) {
    const int h = i / rest, d = 2 * np + i - h * rest;
    rec[(static_cast<size_t>(h) * ps + slot) * dk + d] = krow[static_cast<size_t>(h) * dk + d];
  }
  const T* vrow = krow + static_cast<size_t>(G) * dk;
  T* vrec = rec + static_cast<size_t>(G) * ps * dk;
  constexpr int VEC = 16 / sizeof(T);
  for (int i = threadIdx.x; i < G * dv / VEC; i += blockDim.x) {      // dv is a multiple of eight
    const int h = i * VEC / dv, d = i * VEC - h * dv;
    *reinterpret_cast<uint4*>(vrec + (static_cast<size_t>(h) * ps + slot) * dv + d) = *reinterpret_cast<const uint4*>(vrow + i * VEC);
  }
}

// one CTA per token; d4 = width rounded up to four (the table's padding columns are zero)
template <typename T>
__global__ void __launch_bounds__(256)
embed_norm_kernel(const long long* ids, const T* table, long long ldt, int vocab, float scale, int d4, float* x, float* copy,
                  const __grid_constant__ b200_dense_epilogue e) {
  pdl_launch_dependents();
  pdl_wait();
  const long long m = blockIdx.x;
  long long id = ids[m];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  for (int n = threadIdx.x * 4; n < d4; n += blockDim.x * 4) {
    float4 v;
    v.x = to_f(__ldg(table + id * ldt + n)) * scale; v.y = to_f(__ldg(table + id * ldt + n + 1)) * scale;
    v.z = to_f(__ldg(table + id * ldt + n + 2)) * scale; v.w = to_f(__ldg(table + id * ldt + n + 3)) * scale;
    *reinterpret_cast<float4*>(x + m * e.ldx + n) = v;
    if (copy) *reinterpret_cast<float4*>(copy + m * e.ldx + n) = v;
    if (e.y) store4_any(e.y, e.out_f32 != 0, m * e.ldy + n, epi_norm4(e, epi_norm_columns(e, n), v, e.exact != 0));
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_rotary_paged(void* qkv, long long ld, int hq, int M, const int* positions, const int* seq_ids,
                                 const float* cos_tab, const float* sin_tab, int pairs, int interleaved, int max_pos,
                                 const b200_paged_cache* cache, int* status, cudaStream_t stream) {
  if (M <= 0) return 0;
  if (!qkv || !positions || !cache || !cache->data || !cache->page_table || hq <= 0 || pairs < 0 || 2 * pairs > cache->dk || max_pos <= 0) return -1;
  if (pairs > 0 && (!cos_tab || !sin_tab)) return -1;
  if (cache->dk % 8 || cache->dv % 8 || ld % 8 || (reinterpret_cast<uintptr_t>(qkv) & 15) || (reinterpret_cast<uintptr_t>(cache->data) & 15)) return -2;
  RotaryPagedParams p;
  p.qkv = qkv; p.ld = ld; p.positions = positions; p.seq_ids = seq_ids; p.cos_tab = cos_tab; p.sin_tab = sin_tab;
  p.pairs = pairs; p.interleaved = interleaved; p.max_pos = max_pos; p.c = *cache; p.hq = hq; p.M = M; p.status = status;
  if (cache->f32) launch_ex(rotary_paged_kernel<float>, dim3(M), dim3(128), 0, stream, 0, p);
  else launch_ex(rotary_paged_kernel<__nv_bfloat16>, dim3(M), dim3(128), 0, stream, 0, p);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}

// norm: only y, ldy, out_f32, exact, norm_* and ldx of the epilogue description are used; x and copy share ldx
extern "C" int b200_embed_norm(const long long* ids, const void* table, long long ldt, int vocab, int table_f32, float scale,
                               int M, int d, float* x, float* copy, const b200_dense_epilogue* norm, cudaStream_t stream) {
  if (M <= 0) return 0;
  const int d4 = (d + 3) & ~3;
  if (!ids || !table || !x || !norm || vocab <= 0 || d <= 0 || ldt < d4 || norm->ldx < d4 || norm->ldx % 4) return -1;
  if (norm->y && (norm->ldy < d4 || norm->ldy % 8)) return -2;
  if (table_f32) launch_ex(embed_norm_kernel<float>, dim3(M), dim3(256), 0, stream, 0, ids, static_cast<const float*>(table), ldt, vocab, scale, d4, x, copy, *norm);
  else launch_ex(embed_norm_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, stream, 0, ids, static_cast<const __nv_bfloat16*>(table), ldt, vocab, scale, d4, x, copy, *norm);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
