// Rows of the fp32 residual stream between two sub-layers, for designs whose norm needs a whole row: what the sub-layer
// before left to add, the norm, and the token shift, in one pass.
//
//   x' = embedding row | stream row  (+ sum of the row's expert results, + rows that experts hand through)  (+ one vector)
//   h  = x' / sqrt(mean(x'^2) + eps) * gain
//   with a token shift: h += (h of the previous token - h) * shift, the previous h of a portion's first token from the state
//
// A CTA walks a run of consecutive rows and keeps the row in registers (thread <-> the same columns of every row), so the
// shift needs the row before its first one once more: it is recomputed, which is why x' goes to another buffer than x.
// The CTA of a portion's first rows also writes the state (after it has read it): it recomputes the last row if that is not
// one of its own.
#include "ptx.cuh"
#include "api.h"
#include "launch.cuh"
#include "dense_epilogue.cuh"

namespace b200 {

template <typename T> __device__ __forceinline__ float4 sr_load4(const void* p, long long off);
template <> __device__ __forceinline__ float4 sr_load4<float>(const void* p, long long off) {
  return *reinterpret_cast<const float4*>(static_cast<const float*>(p) + off);
}
template <> __device__ __forceinline__ float4 sr_load4<__nv_bfloat16>(const void* p, long long off) {
  const uint2 r = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + off);
  return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16), __uint_as_float(r.y & 0xffff0000u));
}
__device__ __forceinline__ void sr_fma4(float4& a, float w, float4 v) { a.x += w * v.x; a.y += w * v.y; a.z += w * v.z; a.w += w * v.w; }

struct StreamRowsParams { b200_stream_rows r; int M, d, run; };

template <typename T, int NV, int THREADS>
__global__ void __launch_bounds__(THREADS) stream_rows_kernel(const __grid_constant__ StreamRowsParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const b200_stream_rows& r = p.r;
  __shared__ float red[2][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int turn = 0;

  // rows of this CTA: first .. first + count - 1, part of the portion row0 .. row0 + len - 1
  int row0 = 0, len = p.M;
  if (r.shift) {
    row0 = r.cu ? r.cu[blockIdx.y] : blockIdx.y;
    len = r.cu ? r.cu[blockIdx.y + 1] - row0 : 1;
  }
  const int first = blockIdx.x * p.run, count = min(p.run, len - first);
  if (count <= 0) return;

  auto load_row = [&](long long m, float4 (&v)[NV], bool keep) {
    const long long src = r.index ? r.index[m] : m;
    long long id = 0;
    if (r.ids) { id = r.ids[src]; id = id < 0 ? 0 : (id >= r.vocab ? r.vocab - 1 : id); }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int n = (i * THREADS + threadIdx.x) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (n < p.d) {
        if (r.ids) {
          const float4 e = r.table_f32 ? sr_load4<float>(r.table, id * r.ldt + n) : sr_load4<__nv_bfloat16>(r.table, id * r.ldt + n);
          sr_fma4(v[i], r.scale, e);
        } else {
          v[i] = *reinterpret_cast<const float4*>(r.x + src * r.ldx + n);
        }
      }
    }
    if (r.y) {
      for (int k = 0; k < r.top; ++k) {
        const long long at = src * r.top + k;
        const int s = r.slot[at];
        const float w = r.weight[at];
        const bool own = s >= 0;
        if (!own && r.chosen[at] < r.experts) continue;
        const void* base = own ? r.y : r.through;
        const long long off = own ? s * r.ldy : src * r.ldt2;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int n = (i * THREADS + threadIdx.x) * 4;
          if (n < p.d) sr_fma4(v[i], w, sr_load4<T>(base, off + n));
        }
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int n = (i * THREADS + threadIdx.x) * 4;
      if (n < p.d) {
        if (r.add) {
          const float4 a = __ldg(reinterpret_cast<const float4*>(r.add + n));
          v[i].x += a.x; v[i].y += a.y; v[i].z += a.z; v[i].w += a.w;
        }
        // the last group of four may reach beyond the row: nothing of it may enter the norm
        if (n + 1 >= p.d) v[i].y = 0.f;
        if (n + 2 >= p.d) v[i].z = 0.f;
        if (n + 3 >= p.d) v[i].w = 0.f;
        if (keep && r.x_out) *reinterpret_cast<float4*>(r.x_out + m * r.ldx + n) = v[i];
      }
    }
  };
  // v becomes the normalised row
  auto norm_row = [&](float4 (&v)[NV]) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) red[turn][warp] = s;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) t += red[turn][w];
    turn ^= 1;                                   // the other half: nobody is still reading it when it is written next
    const float f = r.gain / sqrtf(t / static_cast<float>(p.d) + r.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) { v[i].x *= f; v[i].y *= f; v[i].z *= f; v[i].w *= f; }
  };

  float4 prev[NV];
  int seq = 0;
  bool keep_state = false;
  if (r.shift) {
    seq = r.seq_ids ? r.seq_ids[row0] : row0;
    const bool known = seq >= 0 && seq < r.num_seqs;
    keep_state = first == 0 && known && (!r.active || r.active[seq] != 0);
    if (first > 0) {
      load_row(row0 + first - 1, prev, false);
      norm_row(prev);
    } else {
      const bool fresh = r.positions[row0] <= 0 || !known;       // a sequence starts from zeros, whatever the slot held
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int n = (i * THREADS + threadIdx.x) * 4;
        prev[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && n < p.d) prev[i] = *reinterpret_cast<const float4*>(r.state + seq * r.state_ld + n);
      }
    }
  }
  for (int j = 0; j < count; ++j) {
    const long long m = row0 + first + j;
    float4 v[NV];
    load_row(m, v, true);
    norm_row(v);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int n = (i * THREADS + threadIdx.x) * 4;
      if (n < p.d) {
        float4 o = v[i];
        if (r.shift) {
          const float4 t = __ldg(reinterpret_cast<const float4*>(r.shift + n));
          o.x += (prev[i].x - o.x) * t.x; o.y += (prev[i].y - o.y) * t.y; o.z += (prev[i].z - o.z) * t.z; o.w += (prev[i].w - o.w) * t.w;
          prev[i] = v[i];
        }
        if (r.h) store4_any(r.h, r.f32 != 0, m * r.ldh + n, o);
      }
    }
  }
  if (keep_state) {
    if (first + count < len) {
      load_row(row0 + len - 1, prev, false);
      norm_row(prev);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int n = (i * THREADS + threadIdx.x) * 4;
      if (n < p.d) *reinterpret_cast<float4*>(r.state + seq * r.state_ld + n) = prev[i];
    }
  }
}

template <typename T>
static void launch_stream_rows(const StreamRowsParams& p, dim3 grid, cudaStream_t stream) {
  const int d4 = (p.d + 3) / 4;
  if (d4 <= 64) launch_ex(stream_rows_kernel<T, 1, 64>, grid, dim3(64), 0, stream, 0, p);
  else if (d4 <= 256) launch_ex(stream_rows_kernel<T, 1, 256>, grid, dim3(256), 0, stream, 0, p);
  else if (d4 <= 512) launch_ex(stream_rows_kernel<T, 2, 256>, grid, dim3(256), 0, stream, 0, p);
  else if (d4 <= 1024) launch_ex(stream_rows_kernel<T, 4, 256>, grid, dim3(256), 0, stream, 0, p);
  else if (d4 <= 2048) launch_ex(stream_rows_kernel<T, 4, 512>, grid, dim3(512), 0, stream, 0, p);
  else launch_ex(stream_rows_kernel<T, 8, 1024>, grid, dim3(1024), 0, stream, 0, p);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_stream_rows_launch(const b200_stream_rows* r, int M, int d, int num_sms, cudaStream_t stream) {
  if (M <= 0) return 0;
  const int d4 = (d + 3) & ~3;
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (!r || d <= 0 || d4 > 32768 || (!r->ids && !r->x) || (r->ids && (!r->table || r->ldt < d4 || r->ldt % 4 || r->vocab <= 0))) return -1;
  if (r->ldx < d4 || r->ldx % 4 || !al16(r->x) || !al16(r->x_out) || (r->x_out && r->x_out == r->x) || !al16(r->add) || !al16(r->table)) return -2;
  if (r->h && (r->ldh < d4 || r->ldh % 8 || !al16(r->h))) return -3;
  if (r->y && (!r->slot || !r->chosen || !r->weight || !r->through || r->top <= 0 || r->ldy < d4 || r->ldy % 8 || r->ldt2 < d4 || r->ldt2 % 8 || !al16(r->y) || !al16(r->through))) return -4;
  if (r->shift && (!r->state || !r->positions || !al16(r->shift) || !al16(r->state) || r->state_ld < d4 || r->state_ld % 4 || r->index || r->num_seqs <= 0)) return -5;
  if (r->cu && (r->portions <= 0 || r->max_len <= 0)) return -6;
  StreamRowsParams p;
  p.r = *r; p.M = M; p.d = d;
  // short runs while the GPU is not full, then longer ones: a run costs one extra row
  const int len = r->shift ? (r->cu ? r->max_len : 1) : M;
  int run = M / (8 * num_sms);
  run = run < 1 ? 1 : (run > 8 ? 8 : run);
  p.run = run;
  const dim3 grid((len + run - 1) / run, r->shift ? (r->cu ? r->portions : M) : 1);
  if (grid.y > 65535) return -7;
  if (r->f32) launch_stream_rows<float>(p, grid, stream);
  else launch_stream_rows<__nv_bfloat16>(p, grid, stream);
  cudaError_t e = cudaGetLastError();
  return e == cudaSuccess ? 0 : -2000 - static_cast<int>(e);
}
