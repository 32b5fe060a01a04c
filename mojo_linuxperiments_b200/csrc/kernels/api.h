// C ABI of the sm_100a kernel library (loaded from Python with ctypes; usable from any C/C++ host).
// Conventions: every function returns 0 on success and a negative value on a rejected argument or a
// launch error; nothing here synchronises the stream; pointers are device pointers unless noted.
#pragma once
#include <cuda_runtime.h>
#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

// ---- W8A8 linear -----------------------------------------------------------------------------------
// Scratch bytes the stream-K path of b200_w8a8_gemm wants for an [M,N] problem (int32 partial sums).
size_t b200_w8a8_gemm_ws_bytes(int M, int N, int K, int num_sms);
// y[m,n] = (sum_k xq[m,k]*wq[n,k]) * sx[m] * sw[n] (+ residual[m,n]); y is bf16 (or fp32 when out_fp32).
// counters must be zero on entry and are left zero on exit (ws needs no initialisation); force_mode: -1 auto, 0 whole tiles, 1 stream-K.
int b200_w8a8_gemm(const void* xq, const float* sx, const void* wq, const float* sw, void* y,
                   const void* residual, int M, int N, int K, int ldy, int out_fp32,
                   void* ws, size_t ws_bytes, void* counters, int counters_len, int* status,
                   int num_sms, int force_mode, cudaStream_t stream);

// Decode form (M <= 64): split-K thread-block clusters reduced through distributed shared memory; no scratch.
// force_splits: 0 auto, else 1/2/4/8 CTAs per cluster along K.
int b200_w8a8_gemm_decode(const void* xq, const float* sx, const void* wq, const float* sw, void* y,
                          const void* residual, int M, int N, int K, int ldy, int out_fp32, int* status,
                          int num_sms, int force_splits, cudaStream_t stream);

int b200_w8a8_gemm_decode_resident_clusters(int m, int splits);

// Activation prologue carried inside a decode GEMM launch (quantiser CTAs of the same grid, see quant_row.cuh).
// mode: 1 rotate + quantise x [M][K]; 2 RMSNorm(gamma, eps) first; 3 residual += x (bf16, in place) then RMSNorm of the
// residual; 4 x is [M][2K] = gate | up and silu(gate) * up is quantised.  q [M][K] int8 and scale [M] are written by the
// launch (and are what its GEMM CTAs consume); flags: M uint32 words; step: a device uint32 that the caller changes
// between two replays of a captured launch (within one step every launch tags the flags with its own number).
typedef struct b200_quant_prolog {
  int mode;
  const void* x; long long ldx;
  void* residual; long long ldr;
  const void* gamma; float eps;
  void* q; float* scale;
  void* flags; const void* step;
  void* residual_out; long long ldro;   // mode 3: where residual + x is written (NULL: in place, which rules out the
                                        // inline form)
  int allow_inline;                     // up to four tokens: let the GEMM CTAs quantise their own operand (no quantiser
                                        // CTAs, row statistics exchanged inside the split-K cluster) when the shape allows
} b200_quant_prolog;
int b200_w8a8_gemm_decode_p(const b200_quant_prolog* prolog, const void* wq, const float* sw, void* y,
                            const void* residual, int M, int N, int K, int ldy, int out_fp32, int* status, int num_sms,
                            cudaStream_t stream);
int b200_w8a8_gemm_decode_ar_p(const b200_quant_prolog* prolog, const void* wq, const float* sw, void* y,
                               const void* residual, int M, int N, int K, int ldy, int* status, int num_sms,
                               void* const* peer_data, void* const* peer_flags, void* mc_base, int world, int rank,
                               size_t part_off0, size_t part_off1, void* words, int limit_ms, int ll,
                               size_t recv_off0, size_t recv_off1, size_t recv_bytes, int two_hop, size_t recv2_off0,
                               size_t recv2_off1, size_t recv2_bytes, cudaStream_t stream);

// Same, fused with the tensor-parallel all-reduce over peer memory (one launch).  -20: grid not co-resident, use
// b200_w8a8_gemm_decode followed by b200_peer_allreduce instead.  ll: low-latency {payload, epoch} words; two_hop
// (with ll): partials go only to the rank owning the column slice, which sums and broadcasts them through a second
// receive area of M * N/2 words per slot (recv2_off0/1) - less NVLink traffic at more than a few tokens.
int b200_w8a8_gemm_decode_ar(const void* xq, const float* sx, const void* wq, const float* sw, void* y,
                             const void* residual, int M, int N, int K, int ldy, int* status, int num_sms,
                             void* const* peer_data, void* const* peer_flags, void* mc_base, int world, int rank,
                             size_t part_off0, size_t part_off1, void* words, int limit_ms, int ll,
                             size_t recv_off0, size_t recv_off1, size_t recv_bytes, int two_hop, size_t recv2_off0,
                             size_t recv2_off1, size_t recv2_bytes, cudaStream_t stream);

// Mixture-of-experts grouped forms (device-side offsets / tile tables, no host sync).
int b200_w8a8_gemm_decode_grouped(const void* xq, const float* sx, const void* wq, const float* sw, void* y,
                                  int max_tokens, int x_rows, int N, int K, int ldy, int groups,
                                  const int* grp_offsets, const int* grp_counts, int* status, int num_sms,
                                  cudaStream_t stream);
int b200_w8a8_gemm_grouped(const void* xq, const float* sx, const void* wq, const float* sw, void* y, int x_rows,
                           int N, int K, int ldy, int groups, const void* tiles, const int* num_tiles,
                           int max_tiles, int* status, int num_sms, cudaStream_t stream);
int b200_router_topk(const float* logits, long long ld, int M, int E, int k, int renorm, int* ids, float* wts,
                     cudaStream_t stream);
int b200_moe_align(const int* ids, int M, int k, int e0, int n_local, int* counts, int* offsets, int* slot_token,
                   int* inv, void* tiles, int* meta, cudaStream_t stream);
int b200_moe_gather(const void* xq, const float* sx, int d, const int* slot_token, const int* meta, int max_slots,
                    void* xq_perm, float* sx_perm, cudaStream_t stream);
int b200_moe_combine(const void* y, long long ldy, const int* inv, const float* wts, int M, int k, int d, void* out,
                     long long ldo, cudaStream_t stream);

// ---- activation prologue ---------------------------------------------------------------------------
int b200_act_quant(const void* x, long long ldx, void* residual, long long ldr, const void* gamma, float eps,
                   void* q, long long ldq, float* scale, void* xn_out, long long ldn, int M, int K, int mode,
                   cudaStream_t stream);

// ---- attention and token-wise glue ---------------------------------------------------------------------
// max_pos: rows of cos_tab / sin_tab; num_pages: pages of the cache.  A token whose position is outside the tables,
// outside the max_pages pages of its sequence, or whose page id is not a page of the cache is skipped and
// ST_BAD_ARGUMENT is recorded in *status (optional) - never a stray write.
int b200_rope_kv_write(const void* qkv, long long ld_qkv, const int* positions, const int* seq_ids,
                       const float* cos_tab, const float* sin_tab, const void* q_norm_w, const void* k_norm_w,
                       float eps, void* q_out, void* k_out, void* v_out, void* cache, const int* page_table,
                       int max_pages, int page_size, int hq, int hkv, int M, int max_pos, int num_pages, int* status,
                       cudaStream_t stream);
int b200_embed_gather(const long long* ids, const void* table, void* out, int M, int d, int vocab, cudaStream_t stream);
int b200_argmax_rows(const void* logits, long long ld, int rows, int n, int index_offset, int chunks, float* out_val,
                     long long* out_idx, cudaStream_t stream);
int b200_argmax_rows_f32(const float* logits, long long ld, int rows, int n, int index_offset, int chunks, float* out_val,
                         long long* out_idx, cudaStream_t stream);
int b200_argmax_merge(const float* cand_val, const long long* cand_idx, int world, int rows, long long* out_idx,
                      cudaStream_t stream);
size_t b200_attn_decode_scratch_floats(int B, int hq, int splits);
// seq_lens[b] > max_pages * page_size is clamped to that and ST_BAD_ARGUMENT is recorded in *status (optional).
int b200_attn_decode(const void* q, const void* cache, const int* page_table, const int* seq_lens, void* out,
                     float* scratch, unsigned* counters, int B, int hq, int hkv, int page_size, int max_pages,
                     int splits, float scale, int* status, cudaStream_t stream);
int b200_attn_decode_tma(const void* q, const void* cache, int num_pages, const int* page_table, const int* seq_lens,
                         void* out, float* scratch, unsigned* counters, int B, int hq, int hkv, int page_size,
                         int max_pages, int splits, float scale, int* status, cudaStream_t stream);
// Tensor-core form of the same (tcgen05 MMAs, scores in TMEM); needs splits >= b200_attn_decode_tc_min_splits(longest sequence).
int b200_attn_decode_tc_min_splits(int max_len);
int b200_attn_decode_tc(const void* q, const void* cache, int num_pages, const int* page_table, const int* seq_lens,
                        void* out, float* scratch, unsigned* counters, int B, int hq, int hkv, int page_size,
                        int max_pages, int splits, float scale, int* status, cudaStream_t stream);
// The same kernel with its neighbours folded in: raw q | k | v of the new token in, (optional per-head RMSNorm,) rotary
// embedding, KV append, attention over the cache plus the new token, and (xq given) Hadamard rotation + per-token int8
// of the output out.  seq_lens[b] counts the new token; positions[b] is where it goes.  See attn_decode_tc.cu.
int b200_attn_decode_fused(const void* qkv, long long ld_qkv, const int* positions, const float* cos_tab,
                           const float* sin_tab, int max_pos, const void* q_norm_w, const void* k_norm_w, float eps,
                           void* cache, int num_pages, const int* page_table, const int* seq_lens, void* out, void* xq,
                           long long ldq, float* sx, float* scratch, unsigned* counters, float* rot_scratch,
                           float* blk_amax, unsigned* seq_counters, int B, int hq, int hkv, int page_size, int max_pages,
                           int splits, float scale, int* status, const void* next_weights,
                           unsigned long long next_weights_bytes, cudaStream_t stream);
// Persistent form: two CTAs per SM walk the (kv head, sequence, split) items, loads of the next item overlap the
// softmax / output phase of the current one.
int b200_attn_decode_tcp(const void* q, const void* cache, int num_pages, const int* page_table, const int* seq_lens,
                         void* out, float* scratch, unsigned* counters, int B, int hq, int hkv, int page_size,
                         int max_pages, int splits, float scale, int* status, int num_sms, cudaStream_t stream);
int b200_attn_prefill(const void* q, long long ld_q, const void* k, long long ld_k, const void* v, long long ld_v,
                      void* out, const int* cu_seqlens, int B, int total_tokens, int max_len, int hq, int hkv,
                      float scale, int* status, cudaStream_t stream);

// Split-KV form of b200_attn_prefill: every `chunk` KV tiles (of 128 tokens) of a query tile are one CTA; partial rows go
// through `scratch` (b200_attn_prefill_split_scratch_floats floats) and a merge kernel.
size_t b200_attn_prefill_split_scratch_floats(int B, int hq, int max_len, int chunk);
int b200_attn_prefill_split(const void* q, long long ld_q, const void* k, long long ld_k, const void* v, long long ld_v,
                            void* out, const int* cu_seqlens, int B, int total_tokens, int max_len, int hq, int hkv,
                            float scale, int chunk, float* scratch, int* status, cudaStream_t stream);

// ---- in-kernel time stamps (trace.cuh; only in the library variant built with -DB200RT_TRACE) -----------------------
int b200_debug_compiled(void);
int b200_debug_set_heap_extent(size_t bytes);
int b200_trace_compiled(void);
int b200_trace_set(void* ring, unsigned capacity);

// ---- locality query: every CTA writes {sm id, number of sm ids, rank_tag, cta index} (int32 [ctas][4]) -------------
int b200_where_am_i(int* out, int ctas, int rank_tag, cudaStream_t stream);

// ---- config-1 workload: counter-RNG fill + sum ------------------------------------------------------------
int b200_fill_uniform_reduce(float* out, unsigned long long begin, unsigned long long end, unsigned long long seed,
                             double* partials, int max_ctas, unsigned* counter, double* result, cudaStream_t stream);

// ---- collectives over peer-mapped memory ---------------------------------------------------------------
// peer_data / peer_flags: host arrays [world] of device pointers (rank r's heap base / flag block as mapped here).
// algo: 0 one-shot peer loads, 1 one-shot NVLS, 2 two-shot NVLS (in place), 3 chain to rank 0, 4 butterfly,
// 5 low-latency push of {payload, epoch} words (bf16, receive area of 2 * world * n * 4 bytes at scratch_off).
int b200_peer_allreduce(void* const* peer_data, void* const* peer_flags, void* mc_base, int world, int rank,
                        size_t in_off, size_t scratch_off, void* out, const void* residual, size_t n, int dtype,
                        int algo, void* epoch_words, int* status, int limit_ms, int trailing_barrier, int max_ctas,
                        cudaStream_t stream);

int b200_peer_argmax(void* const* peer_data, void* const* peer_flags, int world, int rank, size_t recv_off,
                     const float* cand_val, const long long* cand_idx, int ncand, int rows, long long* out_idx,
                     void* epoch_words, int* status, int limit_ms, cudaStream_t stream);

// ---- tensor-parallel prefill linears fused with their collective (token-sharded layout between blocks) ----------
// All offsets are byte offsets into every rank's symmetric heap (peer_data[r] = rank r's heap as mapped here).
// Rank r owns token rows [r*rows_per_rank, (r+1)*rows_per_rank) of the M rows.  phase: 7 in production (1 tiles,
// 2 scatter tail, 4 gather push; subsets only for single-device tests that run virtual ranks as consecutive launches).
//
// All-gather -> GEMM: y[M,N] = gathered(xq_local)[M,K] * wq[N,K]^T, scaled.  Gather buffers (two, by epoch parity):
// int8 [m_cap][K] at q_off*, fp32 [m_cap] at s_off*; flags uint32 [world][blk_cap] at flag_off; done words uint32
// [world] at done_off; words: 2 local uint32 (epoch, exit counter), row_ctr: blk_cap local uint32, all zero at first.
// finish != 0 acknowledges the epoch at exit; with 0 the gather buffer stays valid until b200_ag_sync(finish=1).
int b200_w8a8_gemm_ag(const void* xq_local, const float* sx_local, const void* wq, const float* sw, void* y,
                      int M, int N, int K, int ldy, int rows_per_rank, void* const* peer_data, void* mc_base,
                      int world, int rank, size_t q_off0, size_t q_off1, size_t s_off0, size_t s_off1,
                      size_t flag_off, size_t done_off, int blk_cap, int m_cap, void* words, void* row_ctr,
                      int finish, int phase, int* status, int limit_ms, int num_sms, cudaStream_t stream);
// GEMM -> reduce-scatter: out[my rows, N] = sum over ranks of (xq[M,K_shard] * wq^T) (+ residual[my rows]).
// Receive slots (two, by parity): bf16 [world][r_cap][N] at recv_off*; arrival counters uint32 [2] at ctr_off (zero at
// first); words: 2 local uint32.
int b200_w8a8_gemm_rs(const void* xq, const float* sx, const void* wq, const float* sw, void* out,
                      const void* residual, int M, int N, int K, int ldo, int ldr, int rows_per_rank,
                      void* const* peer_data, int world, int rank, size_t recv_off0, size_t recv_off1,
                      size_t ctr_off, int r_cap, void* words, int phase, int* status, int limit_ms, int num_sms,
                      cudaStream_t stream);
int b200_ag_sync(void* const* peer_data, int world, int rank, size_t flag_off, size_t done_off, int blk_cap,
                 int rows_per_rank, int M, void* words, int wait, int finish, int* status, int limit_ms,
                 cudaStream_t stream);

// ---- expert-parallel dispatch / combine for token-sharded prefill (buffers of the all-gather / reduce-scatter links) ----
// dispatch: this rank's rows go (int8 + scale) to the ranks owning one of their top-k experts, the routing lists
// (ids / weights padded to 8 per token at ids_off* / wts_off*) to every rank; flags as in b200_w8a8_gemm_ag.
int b200_ep_dispatch(const void* xq_local, const float* sx_local, const int* ids_local, const float* wts_local,
                     int M, int K, int k, int experts_per_rank, int rows_per_rank, void* const* peer_data,
                     int world, int rank, size_t q_off0, size_t q_off1, size_t s_off0, size_t s_off1,
                     size_t ids_off0, size_t ids_off1, size_t wts_off0, size_t wts_off1, size_t flag_off,
                     size_t done_off, int blk_cap, void* words, void* row_ctr, int* status, int limit_ms,
                     cudaStream_t stream);
// wait for all sources, then copy the routing lists of all M tokens to ids_out / wts_out [M][k]
int b200_ep_wait(void* const* peer_data, int world, int rank, size_t ids_off0, size_t ids_off1, size_t wts_off0,
                 size_t wts_off1, size_t flag_off, int blk_cap, int rows_per_rank, int M, int k, void* words,
                 int* ids_out, float* wts_out, int* status, int limit_ms, cudaStream_t stream);
// b200_moe_gather over the gather buffer of the current epoch (heap_base: this rank's heap)
int b200_ep_gather(const void* heap_base, size_t q_off0, size_t q_off1, size_t s_off0, size_t s_off1,
                   const void* words, int d, const int* slot_token, const int* meta, int max_slots,
                   void* xq_perm, float* sx_perm, cudaStream_t stream);
// combine: weighted local expert outputs of each token -> receive slot of the token's owner; blk_ctr: world*blk_cap
// local uint32, zero at first.  reduce: the owner sums the slots of the ranks its own routing names -> out[my rows][d].
int b200_ep_combine_scatter(const void* y, long long ldy, const int* inv, const float* wts, int M, int k, int d,
                            int rows_per_rank, void* const* peer_data, int world, int rank, size_t recv_off0,
                            size_t recv_off1, size_t ctr_off, int r_cap, void* words, void* blk_ctr, int blk_cap,
                            int* status, int limit_ms, cudaStream_t stream);
int b200_ep_combine_reduce(const int* ids_local, int M, int k, int d, int experts_per_rank, int rows_per_rank,
                           void* const* peer_data, int world, int rank, size_t recv_off0, size_t recv_off1,
                           size_t ctr_off, int r_cap, void* words, void* out, long long ldo, int* status,
                           int limit_ms, int num_sms, cudaStream_t stream);

// ---- dense (unquantised) linears with a fused epilogue, dense_epilogue.cuh ---------------------------------------------
enum { B200_EPI_STORE = 0, B200_EPI_RESIDUAL = 1, B200_EPI_GLU = 2 };
enum { B200_ACT_NONE = 0, B200_ACT_RELU2 = 1 };                     // store: activation of the result (square of relu)
typedef struct b200_dense_epilogue {
  int mode;
  int out_f32;                          // element type of y: 0 bf16, 1 fp32
  int exact;                            // library tanh / exp instead of the approximate hardware functions
  void* y; long long ldy;               // store: result; glu: [M][N/2]; residual: normalised rows, or NULL
  float* x; long long ldx;              // residual: the fp32 stream, updated in place
  const float* add;                     // residual: second addend with the pitch of x, or NULL
  float mult;                           // residual: factor on the linear's result
  const float* norm_w; const float* norm_b; float norm_alpha;     // dynamic tanh: tanh(alpha x) w + b
  float limit;                          // glu: bound of both branches
  int act;                              // store: B200_ACT_*
  const float* gate; long long ldg;     // store: gate logits [M][groups]: the result times their sigmoid, or NULL
  long long y_group;                    // store: columns of y between groups
} b200_dense_epilogue;
// Several linears in one launch.  Their weights are stacked ([groups * N][K]); a group takes either all rows of x, at
// columns g * x_group (heads), or the rows offsets[g] .. + counts[g] of x and y (experts).
typedef struct b200_gemm_groups {
  int groups;
  long long x_group;
  const int* offsets; const int* counts;               // NULL: every group takes all M rows
  const void* tiles; const int* num_tiles; int max_tiles;      // int4 {group, first row, rows, 0} per 128 rows (prefill form)
  int expected;                                        // about how many groups have rows (K split of the decode form); 0: all
} b200_gemm_groups;
// x [M][K] and w [N][K] with row pitches in elements (multiples of 8 for bf16, 16-byte aligned); force_bn 0 or 64 / 128 / 256.
int b200_bf16_gemm(const void* x, long long ldx, const void* w, long long ldw, int M, int N, int K,
                   const b200_dense_epilogue* epi, int* status, int num_sms, int force_bn, cudaStream_t stream);
int b200_bf16_gemm_decode(const void* x, long long ldx, const void* w, long long ldw, int M, int N, int K,
                          const b200_dense_epilogue* epi, int* status, int num_sms, int splits, cudaStream_t stream);
int b200_f32_gemm(const float* x, long long ldx, const float* w, long long ldw, int M, int N, int K,
                  const b200_dense_epilogue* epi, cudaStream_t stream);

// Grouped forms.  decode: M = most rows of a group, rows_total = rows of x.  prefill: row lists only.
int b200_bf16_gemm_grouped(const void* x, long long ldx, const void* w, long long ldw, int rows_total, int N, int K,
                           const b200_dense_epilogue* epi, const b200_gemm_groups* g, int* status, int num_sms, int force_bn,
                           cudaStream_t stream);
int b200_bf16_gemm_decode_grouped(const void* x, long long ldx, const void* w, long long ldw, int M, int rows_total, int N, int K,
                                  const b200_dense_epilogue* epi, const b200_gemm_groups* g, int* status, int num_sms, int splits,
                                  cudaStream_t stream);
int b200_f32_gemm_grouped(const float* x, long long ldx, const float* w, long long ldw, int M, int N, int K,
                          const b200_dense_epilogue* epi, const b200_gemm_groups* g, cudaStream_t stream);

// ---- rows of the fp32 residual stream between two sub-layers whose norm needs the whole row (stream_rows.cu) ---------------
// x' = source (+ mixture of experts) (+ add);  h = x' / rms(x') * gain;  with a token shift: h += (h of the previous token - h) * shift
typedef struct b200_stream_rows {
  const long long* ids; const void* table; long long ldt; int vocab, table_f32; float scale;    // source: embedding rows, or
  const float* x; long long ldx; const long long* index;          // rows of the stream (row m is row index[m] if given)
  const void* y; long long ldy; const int* slot; const int* chosen; const float* weight; int top, experts;   // expert results
  const void* through; long long ldt2;                            // rows that experts numbered >= experts hand through
  const float* add;                                               // [d], or NULL
  float* x_out;                                                   // x' (pitch ldx, never x itself), or NULL
  float gain, eps; void* h; long long ldh; int f32;               // element type of h, y and through
  const float* shift; float* state; long long state_ld; int num_seqs;      // state: fp32 [num_seqs][state_ld], previous h
  const int* positions; const int* seq_ids; const int* active;    // seq_ids NULL: row m is sequence m; active NULL: all
  const int* cu; int portions, max_len;                           // shift: consecutive tokens; cu NULL: one token per portion
} b200_stream_rows;
int b200_stream_rows_launch(const b200_stream_rows* r, int M, int d, int num_sms, cudaStream_t stream);

// ---- routing with a correction, expert groups and identity experts (moe_route.cu) ------------------------------------------
int b200_route_grouped(const float* logits, long long ld, const float* correction, int M, int E, int top, int groups, int keep,
                       float scale, int* ids, float* weights, cudaStream_t stream);
int b200_moe_gather_rows(const void* x, long long row_bytes, const int* slot_token, const int* meta, int max_slots, void* out,
                         cudaStream_t stream);

// ---- gated linear recurrence over time (mingru.cu) ---------------------------------------------------------------------------
// zxg fp32 [M][3 * width] (row pitch ld): S = (1 - sigmoid(z + zb)) S + sigmoid(z + zb) cand(x + xb); out = S silu(g).
int b200_mingru_scratch_floats(int portions, int max_len, int width);
int b200_mingru(const float* zxg, long long ld, const float* zb, const float* xb, int M, int width, float* state, long long state_ld,
                int num_seqs, const int* positions, const int* seq_ids, const int* active, const int* cu, int portions, int max_len,
                float* scratch, void* out, long long ldo, int f32, cudaStream_t stream);

// ---- attention over a paged cache with free head sizes, optional chunk mask, sink and output gate ------------------------
typedef struct b200_paged_cache {
  void* data; int f32;                  // records of kv_heads * page_size * (dk + dv) elements (bf16 or fp32)
  int kv_heads, page_size, dk, dv;      // dk, dv multiples of 8
  int num_pages;
  const int* page_table; int num_seqs, max_pages;      // [num_seqs][max_pages]
} b200_paged_cache;
typedef struct b200_attn_spec {
  float scale;
  int chunk;                            // > 0: a position sees only its own block of `chunk` positions; 0: all earlier ones
  const float* sink;                    // [hq] extra exponent in the denominator, or NULL
  const void* gate; long long ldg;      // [M][hq] gate logits (element type of q): head outputs times sigmoid, or NULL
} b200_attn_spec;
int b200_rotary_paged(void* qkv, long long ld, int hq, int M, const int* positions, const int* seq_ids,
                      const float* cos_tab, const float* sin_tab, int pairs, int interleaved, int max_pos,
                      const b200_paged_cache* cache, int* status, cudaStream_t stream);
int b200_embed_norm(const long long* ids, const void* table, long long ldt, int vocab, int table_f32, float scale,
                    int M, int d, float* x, float* copy, const b200_dense_epilogue* norm, cudaStream_t stream);
// General form (any head size up to 512, bf16 or fp32): one warp per (token, head).  q [M][hq][dk] with row pitch ldq;
// out [M][hq][dv] with row pitch ldo.  seq_ids NULL: token i belongs to sequence i; positions < 0 are skipped.
int b200_attn_paged(const void* q, long long ldq, void* out, long long ldo, int hq, int M, const int* positions,
                    const int* seq_ids, const int* seq_lens, const b200_paged_cache* cache, const b200_attn_spec* spec,
                    int* status, cudaStream_t stream);
// Prefill portions on the tensor cores (bf16, dk and dv up to 128, page size 16): rows [cu[b], cu[b+1]) are consecutive
// positions of one sequence whose keys up to there are in the cache already.
int b200_attn_prefill_paged(const void* q, long long ldq, void* out, long long ldo, int hq, int M, int B, int max_len,
                            const int* cu_seqlens, const int* positions, const int* seq_ids,
                            const b200_paged_cache* cache, const b200_attn_spec* spec, int* status, cudaStream_t stream);
// One new token per sequence (row b of qkv = sequence b; bf16, dk and dv up to 256, page size 16): rotary embedding, cache
// append, attention, sink and gate in one launch.  seq_lens[b] counts the new token; 0: empty slot, zero output.
int b200_attn_decode_paged(const void* qkv, long long ld, void* out, long long ldo, int hq, int B, const int* positions,
                           const int* seq_lens, const float* cos_tab, const float* sin_tab, int pairs, int interleaved,
                           int max_pos, const b200_paged_cache* cache, const b200_attn_spec* spec, int splits,
                           int* status, cudaStream_t stream);

// ---- latent attention: the cache holds one normalised latent (rank) and one rotated key part (rot) per token ------------------
// Cache descriptor: kv_heads 1, dk = rank + rot (each padded to 8), dv 0.
typedef struct b200_latent_dims {
  int heads, rank, rot;                 // padded to multiples of 8
  int true_rank, true_rot;              // what the norm averages over, what turns
} b200_latent_dims;
// in fp32 [M][q_rank | rank | rot | ...]: norms of the query latent (-> cq) and of the latent, rotation of the key part;
// the latter two go to the cache and, if given, to lat [M][rank + rot].
int b200_latent_append(const float* in, long long ld, int M, int q_rank, int true_q_rank, const float* q_gain, const float* c_gain,
                       float eps, const b200_latent_dims* dims, const int* positions, const int* seq_ids, const int* seq_lens,
                       const float* cos_tab, const float* sin_tab, int max_pos, const b200_paged_cache* cache, void* cq,
                       long long ldq, void* lat, int* status, cudaStream_t stream);
// q [M][heads][head_ld]: pairs (2i, 2i+1) of the `true_rot` elements at `offset` of every head, in place
int b200_rotary_heads(void* q, long long ld, int f32, int M, int heads, int head_ld, int offset, int true_rot, const int* positions,
                      const float* cos_tab, const float* sin_tab, int max_pos, int* status, cudaStream_t stream);
// cached rows 0 .. ctx[b+1] - ctx[b] of sequence seq_ids[b] -> lat [ctx[B]][dk]
int b200_latent_gather(const b200_paged_cache* cache, const int* ctx, const int* seqs, int B, int max_ctx, void* lat, int* status,
                       cudaStream_t stream);
// General form, bf16 or fp32: q [M][heads][rank] against latents, q_rot [M][heads][rot] (already turned) against the key part;
// out [M][heads][rank] = weighted latents.
int b200_attn_latent_any(const void* q, long long ldq, const void* q_rot, long long ldr, int head_ld_rot, void* out, long long ldo,
                         int M, const b200_latent_dims* dims, float scale, const int* positions, const int* seq_ids,
                         const int* seq_lens, const b200_paged_cache* cache, int* status, cudaStream_t stream);
// bf16, page size 16, rank up to 512: q [M][heads][rank] (moved into the latent space), q_rot: first element of head 0's second
// part, not yet turned, heads head_ld_rot apart.  Rows cu[b] .. cu[b+1] are consecutive positions of one sequence; cu NULL: one
// token per sequence, seq_lens[b] = 0 marks an empty slot (zero output).  splits: CTAs (a cluster) that share the keys of a row tile.
int b200_attn_latent_fits(int rank, int rot);
int b200_attn_latent(const void* q, long long ldq, const void* q_rot, long long ldr, int head_ld_rot, void* out, long long ldo,
                     int M, const b200_latent_dims* dims, float scale, const int* cu, int portions, int max_len, const int* positions,
                     const int* seq_ids, const int* seq_lens, const float* cos_tab, const float* sin_tab, int max_pos,
                     const b200_paged_cache* cache, int splits, int* status, cudaStream_t stream);
// Long portions: q [M][heads][dn + dr] (turned) against expanded rows kv [rows][heads][dn] ++ [heads][dv] and the shared key part
// k_rot [rows][dr]; rows ctx[b] .. ctx[b+1] are positions 0 .. of portion b's sequence.  gate: fp32 logits [M][heads] or NULL.
int b200_attn_prefill_latent_fits(int dn, int dr, int dv);
int b200_attn_prefill_latent(const void* q, long long ldq, int heads, int dn, int dr, int dv, const void* kv, long long ldkv,
                             const void* k_rot, long long ldkr, int rows_kv, void* out, long long ldo, int M, int B, int max_len,
                             float scale, const int* cu, const int* ctx, const int* positions, const float* gate, long long ldg,
                             int* status, cudaStream_t stream);

#ifdef __cplusplus
}
#endif
