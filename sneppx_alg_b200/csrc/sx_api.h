// C ABI of the sm_100a kernel library. Every entry point takes raw device pointers and a stream,
// returns 0 on success (negative: argument / launch error) and never allocates device memory
// unless its comment says so. Kernels that can wait (mbarrier pipelines, peer signals) take a
// `status` word in device memory: 0 = ok, otherwise one of the sx::ST_* codes.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

// ------------------------------------------------------------------ G1 / G2 GEMM
typedef struct SxGemmArgs {
  const void* A;      // a_mn == 0: [M, K] row-major (lda);  a_mn == 1: [K, M] row-major (lda)
  const void* B;      // b_mn == 0: [N, K] row-major (ldb);  b_mn == 1: [K, N] row-major (ldb)
  void* D;            // [M, N] row-major (ldd), bf16 or fp32
  const void* C;      // optional addend, same indexing as D (ldc), bf16 or fp32
  const float* bias;  // optional [N]
  int M, N, K, batch;
  long long lda, ldb, ldd, ldc;
  long long strideA, strideB, strideD, strideC;  // batch strides in elements (0: operand shared)
  int a_mn, b_mn;
  int out_fp32, c_fp32;
  int act;  // 0 none, 1 gelu(tanh), 2 silu, 3 relu, 4 xIELU with coefficients act_a (z > 0) and act_b (z <= 0),
            // 5 squared relu, 6 act_a * tanh(z * act_b)
  float alpha, beta;
  const int* tile_group;  // grouped GEMM: per 128-row block of A, index of the B matrix (-1 skips the block)
  int num_groups;         // number of B matrices when tile_group is set
  const int* k_ranges;    // per batch [k_begin, k_end) rows of the MN-major operands to reduce over
  int k_total;            // total rows of the MN-major operands when k_ranges is set
  int* status;
  int sm_limit;  // cap on CTAs (0: one per SM)
  int force_bn;  // 0 auto, 128 or 256
  int flags;     // bit 0: B is not written by any kernel launched before this one on the stream (a weight at
                 // inference time), so a kernel may start fetching it before its predecessor has finished
  float act_a, act_b;
} SxGemmArgs;
int sx_gemm_bf16(const SxGemmArgs* args, cudaStream_t stream);

// ------------------------------------------------------------------ A1 / A2 flash attention
// Q [B, Sq, Hq, D], K [B, Skv, Hk, D], V [B, Skv, Hk / v_head_div, D], O [B, Sq, Hq, D]; bf16; each given as a
// base pointer plus token (row) and batch strides in elements, so slices of a fused QKV buffer work in place.
typedef struct SxAttnArgs {
  const void* Q; const void* K; const void* V; void* O;
  float* lse;              // [B, Hq, Sq] natural-log LSE (forward: out; backward: in)
  const void* dO;          // backward only
  void* dQ; void* dK; void* dV;  // backward outputs (bf16), same strides as Q / K / V
  float* dq_accum;         // backward scratch: [B, Sq, Hq, D] fp32, zero-filled by the call
  float* delta;            // backward scratch: [B, Hq, Sq] fp32
  long long q_row_stride, k_row_stride, v_row_stride, o_row_stride;
  long long q_batch_stride, k_batch_stride, v_batch_stride;
  long long do_row_stride, dq_row_stride, dk_row_stride, dv_row_stride;
  long long dq_batch_stride, dk_batch_stride, dv_batch_stride;
  int B, Sq, Skv, Hq, Hk, D;
  int v_head_div;          // 1; 2 for differential attention (two score heads share a V head)
  int causal, window;
  float scale;
  int* status;
  // forward only: optional byte per 128 x 128 score tile, [B or 1][Hq or 1][ceil(Sq/128)][ceil(Skv/128)]; a zero
  // byte removes the tile. Strides in bytes (0 = shared over the batch / the heads).
  const void* block_mask;
  long long bm_batch_stride, bm_head_stride;
} SxAttnArgs;
int sx_attn_fwd(const SxAttnArgs* args, cudaStream_t stream);
int sx_attn_bwd(const SxAttnArgs* args, cudaStream_t stream);

// ------------------------------------------------------------------ fused collectives over symmetric memory
// Peer tables hold, for every rank of the group, the peer-mapped address of the same symmetric allocation.
// `pad` is the group's signal pad (uint32 words, zero-initialised once). Every wait inside these kernels is
// bounded by timeout_ns and reports through `status`.
typedef struct SxPeers {
  void* buf[8];
  void* pad[8];
  int rank, world;
  unsigned long long timeout_ns;
} SxPeers;

// Barrier across the group on `channel` (epoch must increase by one per call on that channel).
int sx_peer_barrier(const SxPeers* peers, int channel, unsigned epoch, int* status, cudaStream_t stream);

// F1, ZeRO gradient reduce-scatter fused with the partitioned optimizer.
//   peers->buf[r]  : rank r's flat bf16 gradient buffer (all ranks hold the full bucket)
//   elem_offset/n  : this rank's shard of the bucket, in elements (n % 8 == 0, offset % 8 == 0)
//   mode 1 (reduce): reduced = (sum_r grad_r) / world -> `reduced` (fp32, local, indexed from 0), per-CTA
//                    sum-of-squares partials -> sumsq_partials[0..grid) ; waits for every rank's `ready_epoch`
//                    on channel `ready_channel` first (peers signal it when their bucket is complete).
//   mode 2 (update): exchanges this rank's total sum of squares with all peers (channel norm_channel), derives the
//                    clip coefficient from the global norm, runs AdamW on (p32, m, v) with `reduced` and writes
//                    the bf16 shard to p16_out; ends with a barrier on channel done_channel.
//   mode 3 (fused) : no clipping: reduce + AdamW in one pass, nothing stored in between; same start / end barriers.
typedef struct SxZeroArgs {
  SxPeers peers;
  long long elem_offset, n;
  float* reduced;            // fp32 [n] (modes 1, 2)
  float* sumsq_partials;     // fp32 [num_partials] (mode 1 writes `grid` entries at partial_offset; mode 2 reads all)
  int partial_offset, num_partials;
  float* p32; float* m; float* v; void* p16_out;
  float lr, beta1, beta2, eps, wd; int step;
  float max_norm;            // <= 0: no clipping
  float* norm_out;           // [3] {sum of squares, norm, coefficient}
  int ready_channel; unsigned ready_epoch;
  int norm_channel; unsigned norm_epoch;
  int done_channel; unsigned done_epoch;
  int mode;
  int grid;                  // CTAs to use (0: default)
  int* status;
  const void* mc_buf;        // optional: NVLS multicast mapping of the gradient buffer (same layout as peers.buf[r]).
                             // When set, modes 1 and 3 read each 16 bytes with ONE multimem.ld_reduce (the switch sums
                             // the ranks' values in fp32 and returns bf16) instead of `world` peer loads.
} SxZeroArgs;
int sx_zero_grid_default(void);
int sx_zero_step(const SxZeroArgs* args, cudaStream_t stream);
// Tell all peers that this rank's bucket is complete (one tiny launch on the stream that produced the gradients).
int sx_signal_peers(const SxPeers* peers, int channel, unsigned epoch, cudaStream_t stream);

// F2 (copy form): pull every rank's shard [n elements of `elem_bytes`] into dst[r * n ...] over NVLink.
// Waits for `epoch` on `channel` from every rank first when channel >= 0.
int sx_allgather_pull(const SxPeers* peers, void* dst, long long shard_bytes, long long src_offset_bytes, int channel,
                      unsigned epoch, int grid, int* status, cudaStream_t stream);

// One-shot all-reduce of bf16 activations (tensor-parallel decode / short prefill): out = sum over ranks of their
// staging buffers (peers->buf[r], n values each, n % 8 == 0). The epoch lives in device memory (epoch_ctr, advanced
// by the launch), so the launch can be captured in a CUDA graph. Channels `channel`, `channel + 1`.
int sx_allreduce_bf16(const SxPeers* peers, void* out, long long n, int channel, void* epoch_ctr, void* cta_counter,
                      int grid, int* status, cudaStream_t stream);

// F2 (push form, NVLS): every rank stores its shard ONCE to the multicast mapping of the full-size symmetric buffer
// (multimem.st: the switch delivers it to all ranks), then the grid's last CTA signals `channel` = `epoch` to every rank
// and waits for every rank's signal, so when the kernel ends on a rank, all shards have landed in its copy.
// mc_dst: multicast address of this rank's slot in the full buffer. Callers must make sure no rank still reads the old
// contents of the buffer when any rank starts pushing (the ZeRO engine's optimizer kernel ends with such a barrier).
int sx_allgather_mc(const SxPeers* peers, const void* src_shard, void* mc_dst, long long shard_bytes, int channel,
                    unsigned epoch, int grid, int* status, cudaStream_t stream);
// Link micro-benchmark kernels: move / reduce `bytes` through peer loads, peer stores, multimem.ld_reduce or multimem.st.
//   kind 0: pull   dst_local <- peers.buf[peer]          kind 1: push   peers.buf[peer] <- src_local
//   kind 2: NVLS ld_reduce over mc (bf16 sum) -> dst_local  kind 3: NVLS multimem.st  mc <- src_local
int sx_link_probe(const SxPeers* peers, int kind, int peer, const void* mc, void* local, long long bytes, int grid,
                  cudaStream_t stream);

// F2 / F3 / F4: GEMM with a collective fused into the same kernel.
//   mode 1  all-gather A rows -> GEMM   (TP column-parallel / sequence-parallel input; F3)
//   mode 2  all-gather B rows -> GEMM   (ZeRO-3 weight shards pulled by the consuming GEMM; F2)
//   mode 3  GEMM -> reduce-scatter of output rows (TP row-parallel output; F4)
// Modes 1/2: peers.buf[r] is rank r's copy of the full-size symmetric operand buffer, whose chunk r (chunk_rows rows)
// rank r has filled before the launch; the local copy is the GEMM operand (args->A or args->B must be
// peers.buf[rank]). flags: local uint32 [world * chunk_rows / sub_rows], zeroed once; epoch increases per call.
// Mode 3: peers.buf[r] is rank r's staging buffer, bf16 [world][chunk_rows][N]; rs_out [chunk_rows, N] (ld rs_ldd) gets
// the sum over ranks (+ rs_residual); counter_word: first of chunk_rows/128 words of the signal pad used as counters.
// The grid never exceeds the SM count: all CTAs of a launch are resident together, which the in-kernel waits rely on.
typedef struct SxGemmCommArgs {
  SxPeers peers;
  int mode;
  void* flags;
  unsigned epoch;
  int n_copy;
  int chunk_rows, sub_rows;
  int sig_channel, done_channel, counter_word;
  unsigned rs_expected;  // mode 3: counter value that marks a row block complete (previous value + 4 * ceil(N/BN) * world)
  void* rs_out; const void* rs_residual; long long rs_ldd;
  void* cta_counter;   // local uint32 word, zeroed once
  // mode 4 (F5): expert all-to-all dispatch fused with the grouped GEMM (args->tile_group must be set; args->A is
  // peers.buf[rank], the local expert-sorted row buffer that every rank pushes into). Entry e = (token e / ep_k,
  // choice e % ep_k) goes to row ep_dest_row[e] of rank ep_dest_rank[e] (-1: dropped), scaled by ep_row_scale[e]
  // when given. ep_arrive[r]: rank r's arrival counters (one uint32 per 128-row tile, symmetric memory);
  // ep_tile_expected: local cumulative arrival targets per tile.
  const void* ep_x; const int* ep_dest_rank; const int* ep_dest_row; const float* ep_row_scale;
  int ep_entries, ep_k, ep_d;
  void* ep_arrive[8];
  const void* ep_tile_expected;
} SxGemmCommArgs;
int sx_gemm_bf16_comm(const SxGemmArgs* args, const SxGemmCommArgs* comm, cudaStream_t stream);

// AR1: small all-reduce (sum) of fp32 values through the peers' buffers; n <= 4096. In place on peers->buf[rank].
int sx_allreduce_small(const SxPeers* peers, int n, int channel, unsigned epoch, int* status, cudaStream_t stream);

// ------------------------------------------------------------------ RNG, dropout, LayerNorm backward, FM / ARC steps
// Philox4x32-10 keyed by `seed`; element i of stream `offset` is the same whatever the launch geometry.
// mode 0 uniform [a, b), 1 normal(mean a, std b), 2 bernoulli(p = a) as 0 / 1. `out` 16-byte aligned.
int sx_rng_fill(float* out, long long n, int mode, float a, float b, unsigned long long seed, unsigned long long offset, cudaStream_t stream);
// bf16, n % 8 == 0: y = x * keep / (1 - p). Backward is the same call on dy with the same (seed, offset).
int sx_dropout(const void* x, void* y, long long n, float p, unsigned long long seed, unsigned long long offset, cudaStream_t stream);
// LayerNorm backward: x, dy, dx bf16 [rows, cols]; gamma fp32; mean / rstd fp32 [rows] from sx_layernorm_fwd;
// partials fp32 [sx_layernorm_bwd_blocks(rows), 2, cols] scratch; dgamma_dbeta fp32 [2, cols]. cols % 8 == 0, <= 8192.
int sx_layernorm_bwd_blocks(long long rows);
int sx_layernorm_bwd(const void* x, const void* dy, const float* gamma, const float* mean, const float* rstd, void* dx,
                     float* partials, float* dgamma_dbeta, long long rows, int cols, cudaStream_t stream);
// Gradient compression (fp32): int8 with one scale per 256 values (n % 256 == 0); top-2 of every 32 values with the
// dropped part in `residual` (optional; n % 32 == 0); weighted sum of up to 16 equally sized buffers (n % 4 == 0).
int sx_fm_quant_int8(const float* x, void* q, float* scales, long long n, cudaStream_t stream);
int sx_fm_dequant_int8(const void* q, const float* scales, float* y, long long n, cudaStream_t stream);
int sx_fm_block_top2(const float* x, float* kept, float* residual, long long n, cudaStream_t stream);
int sx_fm_weighted_avg(const float* const* inputs, const float* weights, int count, float* out, long long n, cudaStream_t stream);
// Adversarial steps (fp32, n % 4 == 0). mode 0 FGSM, 1 PGD step with projection onto the eps-ball around x0,
// 2 sine obfuscation x + eps * sin(100 x), 3 Gaussian smoothing sample x + eps * N(0, 1).
int sx_arc_step(const float* x, const float* g, const float* x0, float* out, long long n, int mode, float eps, float alpha,
                float lo, float hi, unsigned long long seed, unsigned long long offset, cudaStream_t stream);

// conv2d backward: x [N,C,H,W], w [K,C,R,S], dy [N,K,OH,OW] (fp32, or bf16 with is_bf16), contiguous; fp32 gradients
// dx / dw / db, any of which may be null to skip it.
int sx_conv2d_bwd(const void* x, const void* w, const void* dy, float* dx, float* dw, float* db, int N, int C, int H, int W,
                  int K, int R, int S, int stride, int pad, int is_bf16, cudaStream_t stream);

// NPE bytecode interpreter: instruction table [n, 8] int32 (op, dest, a, b, immediate, rows, cols, bias register);
// program memory and x / out fp32. The planner returns 0, -1 malformed, -2 shapes do not fit, -3 unsupported opcode.
int sx_npe_plan_program(const int* prog8, int n, long long mem_size, int in_w, int* maxw, int* out_w);
int sx_npe_run(const int* prog_host, const int* prog_dev, int n, const float* mem, long long mem_size, const float* x, long long rows,
               int in_w, float* out, int out_w_expected, cudaStream_t stream);

// Block-scaled fp8 (e4m3) GEMM, y = (xq * sx) (wq * sw)^T: xq [M, K] with fp32 scales sx [M, K/128] (1 x 128 blocks),
// wq [N, K] with sw [ceil(N/128), K/128] (128 x 128 blocks), bf16 out. `work`: sx_gemm_fp8_workspace bytes (or null).
long long sx_gemm_fp8_workspace(int M, int N, int K);
int sx_gemm_fp8(const void* xq, long long ldx, const float* sx, const void* wq, long long ldw, const float* sw,
                const float* bias, void* out, long long ldd, float* work, int M, int N, int K, int* status,
                cudaStream_t stream);
// Grouped form for SER experts: expert-sorted token rows (segments padded to 128 rows) times the stacked expert
// weights [E * N, K] (N % 128 == 0, scales [E * N/128, K/128]); tile_group[t] is the expert of token tile t
// (-1: unused tile, its output rows are zero).
int sx_gemm_fp8_grouped(const void* xq, long long ldx, const float* sx, const void* wq, long long ldw, const float* sw,
                        const int* tile_group, int num_experts, void* out, long long ldd, int rows, int N, int K,
                        int* status, cudaStream_t stream);

// ------------------------------------------------------------------ hybrid decoders (ragged batches, fp32 residual)
// Rows of several sequences, one portion each, packed one after another. Device int32 arrays.
typedef struct SxRagged {
  const int* cu;        // [n + 1] first row of each portion
  const int* pos0;      // [n] position of that row in its sequence; 0 starts from an empty state
  const int* slot;      // [n] state slot (-1: padding row of a captured launch)
  const int* tok_seq;   // [T] portion of each row
  const int* tok_pos;   // [T] position of each row
  int n;
} SxRagged;
// The portions of a batch cut into chunks of 16 rows. Device int32 arrays.
typedef struct SxChunks {
  const int* seq;       // [n] portion of each chunk
  const int* start;     // [n] first row of the chunk within its portion
  const int* first;     // [portions + 1] first chunk of each portion
  int n;
} SxChunks;
// f32: 1 for 32-bit activations, 0 for bf16. Norm weights, convolution weights and biases are fp32.
int sx_embed_f32(const void* table, const int* ids, float* x, int T, int width, float scale, int f32, cudaStream_t stream);
int sx_rmsnorm_f32(const float* x, const float* w, const int* rows, void* y, int T, int width, float eps, int f32, cudaStream_t stream);
int sx_layernorm_f32(const float* x, const float* w, const float* b, const int* rows, void* y, int T, int width, float eps, int f32,
                     cudaStream_t stream);
// RMSNorm of `parts` equal parts of every activation row, in place: y [T, width], row pitch ld, w [width].
int sx_part_rmsnorm(void* y, long long ld, const float* w, int T, int width, int parts, float eps, int f32, cudaStream_t stream);
int sx_head_norm_gate(const float* o, const float* w, const void* gate, long long gate_ld, float mul, void* y, long long y_ld,
                      int T, int H, int dv, float eps, int f32, cudaStream_t stream);
// Stores the last min(length, taps - 1) projected rows of every portion: ring [slots, taps, C], position p in entry p % taps.
int sx_conv_ring(const void* u, long long u_ld, void* ring, const SxRagged* r, int C, int taps, int f32, cudaStream_t stream);
// Attention operands from projected rows u = q [H d] | k [G d] | v [G dv]: causal convolution over time, RMSNorm of the query
// and key heads, interleaved rotation of their first `rot` entries, cache append.
typedef struct SxQkvArgs {
  const void* u; long long u_ld;
  const float* wconv;             // [taps, C], C = H d + G d + G dv
  void* ring;
  const float* qn; const float* kn;
  const double* inv_freq;         // [rot / 2]
  const float* talk;              // [H, H], with qmix_out
  float* q_out;                   // [T, H, d] or null
  void* qmix_out;                 // [T, H, qmix_ld] queries with the head mix folded in (zeros past G d), or null
  int qmix_ld;
  void* k_out; void* v_out;       // packed keys / values, or null; value head j at column j * dvp
  long long k_ld, v_ld;
  const int* kv_row;              // [T] packed row (null: row index)
  void* k_cache; void* v_cache;   // [entries, G, d] / [entries, G, dv]
  const int* cache_entry;         // [T], -1: not stored
  SxRagged ragged;
  SxChunks chunks;                // n == 0: one row per portion (decoding); the row then also goes to its ring entry
  int T, H, G, d, dv, dvp, taps, rot, f32;
  float eps;
} SxQkvArgs;
int sx_qkv_prep(const SxQkvArgs* args, cudaStream_t stream);
int sx_kv_gather(const void* cache, const int* entry, const int* row, int n, void* out, long long out_ld, int G, int w, int wp,
                 int f32, cudaStream_t stream);
// Delta-rule operands from projected rows u = q [G d] | k [G d] | v [H dv].
typedef struct SxDeltaArgs {
  const void* u; long long u_ld;
  const float* wconv; void* ring;
  const void* b; long long b_ld;
  const void* a; long long a_ld;
  const float* a_log; const float* dt_bias;
  void* v;                        // [T, H dv] convolved values (prompt form)
  SxRagged ragged;
  int T, H, G, d, dv, taps, f32;
} SxDeltaArgs;
// Prompt form of the recurrences: a preparation kernel writes one record of `sx_recur_record` floats per (chunk, head), then
// the scan walks each portion from its slot's state (empty at position 0), stores the state back and writes the read-outs.
typedef struct SxGateArgs {
  const void* q; const void* f; long long ld;     // projected rows [T, H d] each
  const float* bias; const float* lower;          // [H d]
  float* rec;
  SxRagged ragged;
  SxChunks chunks;
  int H, d, f32;
} SxGateArgs;
int sx_recur_record(int d, int delta);
int sx_gate_chunks(const SxGateArgs* args, cudaStream_t stream);
int sx_delta_chunks(const SxDeltaArgs* args, const SxChunks* chunks, float* rec, cudaStream_t stream);
typedef struct SxScanArgs {
  const float* rec;
  const void* v; long long v_ld;
  float* state; float* o;         // [slots, H, d, dv], [T, H, dv]
  SxRagged ragged;
  SxChunks chunks;
  int* status;
  int H, d, dv, delta, f32;
} SxScanArgs;
int sx_recur_scan(const SxScanArgs* args, cudaStream_t stream);
// One token per sequence, from the projected rows to the normed and gated output row.
typedef struct SxStepArgs {
  SxDeltaArgs in;
  const void* qr; const void* fr; const void* vr; long long ld;
  const float* fbias; const float* lower;
  float* state; const float* norm;
  const void* gate; long long gate_ld;
  void* y; long long y_ld;
  SxRagged ragged;
  float mul, eps;
  int H, Hq, d, dv, delta, f32;
} SxStepArgs;
int sx_recur_step(const SxStepArgs* args, cudaStream_t stream);
// Attention whose scores are mixed over the heads before the softmax (score_h <- sum_g talk[h, g] score_g), restricted to
// the chunk floor(position / size) of each query. SIMT form for any head size: q fp32 [T, H, d]. Keys either packed rows
// (kv_base[seq] + position) or cache entries through a block table. Output y = o * sigmoid(gate) * mul.
typedef struct SxTalkArgs {
  const float* q;
  const void* k; const void* v;
  long long k_ld, v_ld; int dvp;
  const int* kv_base;             // packed form: [n] row of position 0 of each sequence (may be negative)
  const int* block_table; const int* block_base; int table_ld, block_size;   // paged form (block_table non-null)
  const float* talk;              // [H, H]
  const void* gate; long long gate_ld;
  void* y; long long y_ld;
  SxRagged ragged;
  float scale, mul;
  int T, H, G, d, dv, size, f32;
  float* part; int splits;        // decode: partial results of key splits [n, splits, H, dv + 2]
} SxTalkArgs;
int sx_talk_attn(const SxTalkArgs* args, cudaStream_t stream);
int sx_talk_merge(const SxTalkArgs* args, cudaStream_t stream);
// Tensor-core decode form over the block pool (bf16): queries with the head mix folded in, [n, H, q_ld].
int sx_talk_decode_ok(int H, int G, int d, int dv);
int sx_talk_decode(const SxTalkArgs* args, const void* qmix, int q_ld, cudaStream_t stream);
// Tensor-core prompt form (bf16, value heads up to 128): queries with the head mix folded in, [T, H, nq * 64] with
// nq = ceil(G d / 64) and zeros past G d; packed keys [kv_rows, k_ld] and values (head j at column j * dvp).
typedef struct SxTalkTcArgs {
  const void* qmix; const void* k; const void* v;
  long long k_ld, v_ld, kv_rows;
  const int* kv_base;
  const int* tiles;               // [n_tiles, 2]: portion, first of up to 128 rows of it
  const void* gate; long long gate_ld;
  void* y; long long y_ld;
  SxRagged ragged;
  float scale, mul;
  int T, n_tiles, H, G, d, dv, dvp, size;
  int* status;
} SxTalkTcArgs;
int sx_talk_attn_tc_ok(int H, int G, int d, int dv);
int sx_talk_attn_tc(const SxTalkTcArgs* args, cudaStream_t stream);
// SSD (Mamba-2) recurrence with an fp32 state [slots, H, N, P] per head: S <- a S + dt B x^T, y = (S^T C + D x) silu(z), from
// projected rows u = z [H P] | x [H P] | B [G N] | C [G N] | dt [H]. x, B and C pass a causal convolution with bias and silu.
typedef struct SxSsdArgs {
  const void* u; long long u_ld;
  const float* wconv; const float* bconv; void* ring;   // [taps, C], [C], [slots, taps, C], C = H P + 2 G N
  const float* dt_bias; const float* a_log; const float* D;   // [H]
  void* x; void* b; void* c;      // operands of the prompt forms: [T, H, xp], [T, G, np] (zeros past P and N)
  float* dt; float* la;           // [T, H] step size and logarithm of the decay
  float* state;
  void* y; long long y_ld;        // [T, H P]
  SxRagged ragged;
  SxChunks chunks;
  // tensor-core prompt form with few sequences: portions cut into segments of seg_rows rows (a multiple of 64), or n_seg 0
  const int* seg_seq; const int* seg_first;   // [n_seg] portion, [n + 1] first segment of each portion
  float* seg_state; float* seg_la;            // scratch: [n_seg, H, N, P], [n_seg, H]
  int n_seg, seg_rows;
  int T, H, P, N, G, taps, xp, np, f32;
} SxSsdArgs;
int sx_ssd_operands(const SxSsdArgs* args, cudaStream_t stream);   // u -> x, b, c, dt, la
int sx_ssd_chunks(const SxSsdArgs* args, float* rec, cudaStream_t stream);   // records for sx_recur_scan (d = N, dv = P)
int sx_ssd_gate(const SxSsdArgs* args, const float* o, cudaStream_t stream); // y from the read-outs o [T, H, P] of the scan
int sx_ssd_step(const SxSsdArgs* args, cudaStream_t stream);       // one token per sequence, from u to y
int sx_ssd_scan_ok(int P, int N);
int sx_ssd_scan(const SxSsdArgs* args, cudaStream_t stream);       // prompt form on tensor cores (bf16): operands -> state, y
// Operands of window attention over tokens and averaged blocks, from projected rows u = q [H d] | k [G d] | v [G dv]: bias,
// rotation of the first `rot` entries of query and key heads, rotation of whole value heads, cache append.
typedef struct SxWinPrepArgs {
  const void* u; long long u_ld;
  const float* bias;                                     // [H d + G d + G dv] or null
  const double* freq; const double* vfreq;               // [rot / 2], [dv / 2] angle per position
  const float* temp;                                     // [H] factor on the queries, or null
  float* q32; void* q; int q_ld;                         // [T, H, d] fp32 or [T, H, q_ld] activations (zeros past d)
  void* k_out; void* v_out; long long k_ld, v_ld; int dp, dvp;   // packed rows, head j at column j dp / j dvp; or null
  const int* kv_row;
  void* k_cache; void* v_cache; const int* cache_entry;  // [entries, G, d], [entries, G, dv]; -1: not stored
  float* turn;                                           // [T, dv / 2, 2] cos and sin of the value angles
  SxRagged ragged;
  // decoding: average of the block of `pool` positions that this token completes (entry -1: none)
  const int* pool_entry; const int* block_table; const int* block_base; int table_ld, block_size, pool;
  int T, H, G, d, dv, rot, interleaved, f32;
  float rot_mul;                                         // factor on cos and sin of the query / key rotation
} SxWinPrepArgs;
int sx_win_prep(const SxWinPrepArgs* args, cudaStream_t stream);
// Averages of the blocks completed by a prompt batch: `pool` packed rows from src[i] on -> packed row row[i], cache entry[i].
int sx_pool_blocks(void* rows, long long ld, int wp, void* cache, int G, int w, const int* src, const int* row, const int* entry, int n,
                   int pool, int f32, cudaStream_t stream);
// Attention of each query to the last `size` positions and to the averages of whole earlier blocks of `pool` positions in one
// softmax whose denominator also holds exp(sink[h]). Output: values turned back by the position's angles, times
// sigmoid(gate). Queries carry the temperature. Keys are packed rows (pool_base / kv_base) or cache entries (tables).
typedef struct SxWinAttnArgs {
  const float* q32; const void* q; int q_ld;
  const void* k; const void* v; long long k_ld, v_ld, kv_rows; int dp, dvp;
  const int* kv_base; const int* pool_base;              // packed: row of position 0, row of block 0 of each sequence
  const int* tiles; int n_tiles;
  const int* block_table; const int* block_base; const int* pool_table; int table_ld, pool_ld, block_size;   // paged
  const float* sink; const float* turn;
  const void* gate; long long gate_ld;                   // [T, H dv]
  void* y; long long y_ld;
  SxRagged ragged;
  float scale;
  int T, H, G, d, dv, size, pool, interleaved, f32;
  float* part; int splits;                               // [T, splits, H, dv + 2]
  int* status;
} SxWinAttnArgs;
int sx_win_attn(const SxWinAttnArgs* args, cudaStream_t stream);          // any sizes; q32
int sx_win_attn_tc_ok(int H, int G, int d, int dv);
int sx_win_attn_tc(const SxWinAttnArgs* args, cudaStream_t stream);       // prompts on tensor cores (bf16)
int sx_win_decode_ok(int H, int G, int d, int dv);
int sx_win_decode(const SxWinAttnArgs* args, cudaStream_t stream);        // decoding on tensor cores (bf16)
int sx_win_merge(const SxWinAttnArgs* args, cudaStream_t stream);         // key slices -> y

#ifdef __cplusplus
}
#endif
