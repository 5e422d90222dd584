/*
 * lri_b200.h - C ABI of the B200 (sm_100a) kernels behind the tensor-parallel decode/prefill step.
 *
 * The reference project is pure Python (its kernels are library calls and one Triton kernel),
 * so it has no FFI of its own; each entry point below names the reference code it replaces
 * (paths relative to the reference repository root).  A Python binding (ctypes) passes
 * `tensor.data_ptr()` values and the raw handle of the current CUDA stream.
 *
 * Conventions
 *   - Plain pointers and sizes only.  Every pointer is a DEVICE pointer unless it says "host".
 *   - The caller owns all memory.  No entry point allocates device memory or synchronises the
 *     device unless its comment says so; work is enqueued on `stream`.
 *   - `dtype` is LRI_BF16 or LRI_FP16 (activations, weights and caches share it); all
 *     accumulation is fp32 and results are rounded once to `dtype` where the reference's
 *     nn.Linear / elementwise op would round.
 *   - Matrices are row-major.  Weights have the nn.Linear layout [out_features, in_features].
 *   - Positions are read on the device from `input_pos` (int32 when pos_is_i64 == 0, int64
 *     otherwise), never from a host scalar, so a captured CUDA graph stays valid when the caller
 *     advances the position tensor in place (benchmark.py:209-217).
 *   - Return value: LRI_OK or a negative lri_status; lri_last_error() gives the message of the
 *     calling thread's last failure.  The reference's convention is a Python assert/exception
 *     (gpt_fast/utils.py:52, 155-162); the binding raises RuntimeError on a negative status.
 */
#ifndef LRI_B200_H_
#define LRI_B200_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef void* lri_stream_t; /* a cudaStream_t */

/* LRI_FP32 is taken by the entry points that say so (every product and sum a true 32-bit operation). */
enum lri_dtype { LRI_BF16 = 0, LRI_FP16 = 1, LRI_FP32 = 2 };

enum lri_status {
  LRI_OK = 0,
  LRI_ERR_ARG = -1,         /* null pointer, non-positive extent, inconsistent sizes */
  LRI_ERR_ALIGN = -2,       /* pointer or row pitch not aligned as the kernel needs */
  LRI_ERR_UNSUPPORTED = -3, /* shape or dtype outside what the kernels are built for */
  LRI_ERR_CUDA = -4,        /* a CUDA runtime/driver call failed (message has the CUDA text) */
  LRI_ERR_WORKSPACE = -5,   /* workspace missing or too small */
  LRI_ERR_TIMEOUT = -6,     /* a bounded device-side wait gave up (peer flag, mbarrier) */
  LRI_ERR_NO_DEVICE = -7    /* no usable sm_100 device */
};

/* GEMM back end for M > 8 rows.  AUTO picks tcgen05 when the shape allows it. */
enum lri_gemm_backend { LRI_GEMM_AUTO = 0, LRI_GEMM_TCGEN05 = 1, LRI_GEMM_SIMT = 2 };

const char* lri_last_error(void);
int lri_version(void);
/* Selects the GEMM back end used by the linear-layer entry points (process-wide). */
int lri_set_gemm_backend(int backend);
/* Tuning options: one table per process, each entry initialised from an LRI_* environment variable
 * at first use and changeable at run time; a change applies from the next launch on.  Names (initial
 * value from): stream_rows (LRI_STREAM_ROWS, 1..16, token rows up to which the weight-streaming
 * kernels run), gemv_simt (LRI_GEMV_SMALL=simt), gemv_rows_per_cta (LRI_GEMV_R: 0, 2, 4, 8),
 * gemv_depth (LRI_GEMV_U: 0, 2), gemv_mma_tiles (LRI_GEMV_MT: 0, 1, 2, 4), gemm_group
 * (LRI_GEMM_GROUP), fused_prefill (LRI_FUSED_PREFILL: 0, 1), pdl (LRI_PDL: 0, 1), attn_cluster
 * (LRI_ATTN_CLUSTER: 0, 1), attn_mma (LRI_ATTN_MMA: -1 choose, 0, 1), decode_splits
 * (LRI_DECODE_SPLITS: 0 choose, 1..64), attn_prefill_tc (LRI_ATTN_PREFILL_TC: 0 mma.sync kernel, 1 tcgen05
 * kernel), gemm_reserve_sms (LRI_GEMM_RESERVE_SMS: SMs
 * the persistent prefill GEMM leaves free for a collective running beside it, 0..64), attn_head_tile
 * (LRI_ATTN_HEAD_TILE: query heads of a KV group per CTA of the cluster decode attention, 0 choose, 1, 2, 4),
 * moe_stream_pairs (LRI_MOE_STREAM_PAIRS: (token, expert) pairs up to which experts run as streaming projections),
 * window_tc (LRI_WINDOW_TC: 0 keeps sliding-window attention on the plain kernel), hgrn2_blocks
 * (LRI_HGRN2_BLOCKS: 0 keeps the HGRN2 recurrence token by token), scan_columns (LRI_SCAN_COLUMNS: state columns per
 * lane of the matrix-state recurrences, 0 choose, 1, 2, 4), scan_warps (LRI_SCAN_WARPS: their warps per CTA, 0 choose, 1, 2, 4),
 * scan_lanes (LRI_SCAN_LANES: lanes per state column, 0 choose, 8, 16).  Unknown
 * names and values an option does not take return LRI_ERR_ARG.  No counterpart in the reference
 * (its only switches are benchmark.py's command-line flags). */
int lri_set_option(const char* name, int value);
int lri_get_option(const char* name, int* value_out);
/* Number of kernels this library has launched from the calling process so far. */
int64_t lri_launch_count(void);
/* The tcgen05 GEMM bounds every mbarrier wait; a wait that gives up records its site in a
 * device status word.  Reads and clears it (synchronous copy): LRI_OK or LRI_ERR_TIMEOUT. */
int lri_gemm_status(void);

/* ---- F1: residual add + RMSNorm -------------------------------------------------------
 * residual_out = round(round(residual * residual_scale) + add1) [+ add2, rounded again];
 * normed_out   = round(residual_out * rsqrt(mean(residual_out^2) + eps)) * weight.
 * add1, add2 may be NULL (no add); weight/normed_out may be NULL (add only); residual_out may
 * be NULL (norm only) or alias residual.  residual_scale != 1 is the desync block's x / tp.
 * Replaces: the Triton add kernel gpt_fast/gpt_ladder_TP.py:364-377 (launched :331, :348),
 * the final three-way add gpt_ladder_TP.py:280, RMSNorm.forward gpt_fast/utils.py:62-78 and
 * the `y + x / tp_world_size` of gpt_fast/gpt_desync_TP.py:366-382. */
int lri_add_rmsnorm(int dtype, const void* residual, const void* add1, const void* add2,
                    float residual_scale, const void* weight, float eps, void* residual_out,
                    void* normed_out, int64_t rows, int dim, lri_stream_t stream);

/* ---- embedding gather ------------------------------------------------------------------
 * out[i, :] = table[idx[i], :].  idx is int64 when idx_is_i64 != 0, else int32.
 * Replaces: self.tok_embeddings(idx), gpt_fast/gpt_ladder_TP.py:256. */
int lri_embedding(int dtype, const void* table, const void* idx, int idx_is_i64, void* out,
                  int64_t n_tokens, int dim, int64_t vocab, lri_stream_t stream);

/* ---- F5 / F7: linear layer y = x W^T (+ addend) ------------------------------------------
 * x [M, K], w [N, K], y [M, N].  addend (may be NULL) is added after y's own rounding and the
 * sum rounded again (the parallel block's `w2(...) + y`, gpt_fast/utils.py:385).  M <= 8 runs
 * the weight-streaming kernels (SIMT for one row, mma.sync for 2..8); larger M the tcgen05 GEMM.
 * For 8 < M <= 64 a workspace of lri_linear_workspace_bytes(M, N) bytes (16-byte aligned) selects
 * the tcgen05 stream-K kernel: all SMs stream equal shares of the weight, fp32 partial tiles go
 * to the workspace and the CTA that completes a tile sums them and applies the addend.  With
 * NULL or a smaller workspace the plain GEMM runs.  Two calls that may run at the same time on
 * different streams need different workspaces; at most 16 stream-K kernels (this entry point,
 * lri_qkv_rope_kvcache, lri_gateup_swiglu) may be in flight at once.  Replaces: self.wo / self.w2 / self.output nn.Linear calls, gpt_fast/utils.py:148,
 * 258, 384-385 and gpt_fast/gpt_ladder_TP.py:283. */
size_t lri_linear_workspace_bytes(int64_t M, int N);
/* How the stream-K kernel would cut a projection with N outputs (for lri_gateup_swiglu: N = I) and
 * depth K at 1 <= M <= 64 token rows: 128-output tiles, 64-element K tiles, the number of
 * persistent CTAs, the most segments one tile may be cut into (the workspace holds that many
 * fp32 partial tiles of token_tile x 128 per tile) and the token tile 16 / 32 / 64.  Host
 * arithmetic only, usable without a GPU.  No counterpart in the reference. */
int lri_streamk_plan(int64_t M, int N, int K, int* tiles, int* k_tiles, int* max_segments, int* ctas,
                     int* token_tile);
int lri_linear(int dtype, const void* x, const void* w, const void* addend, void* y, int64_t M,
               int N, int K, void* workspace, size_t workspace_bytes, lri_stream_t stream);
/* y = x W^T with y in fp32, no rounding: projections that feed fp32 arithmetic (norms, gates, recurrences,
 * routers).  Kernels and workspace as lri_linear.  Both entry points also take LRI_FP32 (then y is fp32 in
 * either) and any K; those run a plain SIMT kernel.  No counterpart in the reference. */
size_t lri_linear_f32_workspace_bytes(int64_t M, int N);
int lri_linear_f32(int dtype, const void* x, const void* w, float* y, int64_t M, int N, int K,
                   void* workspace, size_t workspace_bytes, lri_stream_t stream);

/* ---- F2: QKV projection + RoPE + KV-cache write ----------------------------------------
 * x [B*S, K]; wqkv [(n_head + 2 n_kv) * head_dim, K] with rows [q heads | k heads | v heads];
 * rope_table [table_rows, head_dim/2, 2] = (cos, sin) in `dtype`; input_pos [S].  The table row
 * of token s is input_pos[s], or s itself when table_gathered != 0 (the caller already indexed
 * the table by position, as the reference's forward does: freqs_cis[input_pos]).
 * q_out [B, S, n_head, head_dim] receives the rotated queries; rotated keys and the values are
 * written to k_cache / v_cache [B_max, n_kv, smax, head_dim] at [b, h, input_pos[s], :].
 * Rotation is over adjacent pairs in fp32 from the rounded projection, as the reference does.
 * A position outside [0, min(smax, table_rows)) is skipped (nothing is written for it).
 * M = B*S > 8 needs workspace of lri_qkv_workspace_bytes(M, n_head, n_kv, head_dim) bytes.
 * Replaces: gpt_fast/utils.py:187-198 (wqkv, split, apply_rotary_emb) and KVCache.update
 * utils.py:50-59, 249-250. */
size_t lri_qkv_workspace_bytes(int64_t M, int n_head, int n_kv, int head_dim);
int lri_qkv_rope_kvcache(int dtype, const void* x, const void* wqkv, const void* rope_table,
                         const void* input_pos, int pos_is_i64, void* q_out, void* k_cache,
                         void* v_cache, int B, int S, int K, int n_head, int n_kv, int head_dim,
                         int64_t smax, int64_t table_rows, int table_gathered, void* workspace,
                         size_t workspace_bytes, lri_stream_t stream);

/* ---- F6: gate/up projection + SwiGLU -----------------------------------------------------
 * w1 [2*I, K] with rows [up (I rows) | gate (I rows)]; h[m, j] = round(silu(gate_j)) * up_j.
 * M > 8 needs workspace of lri_gateup_workspace_bytes(M, I) bytes.
 * Replaces: FeedForward.forward's w1 / chunk / silu*mul, gpt_fast/utils.py:145-148 (and the
 * u, g part of FuseAttentionMLP, utils.py:311-313, 385). */
size_t lri_gateup_workspace_bytes(int64_t M, int I);
int lri_gateup_swiglu(int dtype, const void* x, const void* w1, void* h, int64_t M, int I, int K,
                      void* workspace, size_t workspace_bytes, lri_stream_t stream);

/* ---- F3: GQA decode attention, split over the sequence --------------------------------------
 * One query token per sequence.  q [B, n_head, head_dim]; caches [B_max, n_kv, smax, head_dim];
 * context = positions 0..input_pos[0] inclusive (the new key is already in the cache); query
 * head h reads kv head h / (n_head / n_kv); scale 1/sqrt(head_dim); out [B, n_head*head_dim].
 * The sequence is cut into num_splits ranges handled by different CTAs and merged by the last
 * CTA to finish, so the grid does not depend on the position.  scratch: at least
 * lri_attn_decode_scratch_bytes(B, n_head, n_kv, head_dim, num_splits) bytes, 16-byte aligned;
 * its first 32768 bytes are arrival counters that must be zero before the first call
 * (each call leaves them zero).  Calls sharing one scratch must not overlap on the device.
 * Three kernels serve this entry point: with 1, 2, 4, 8 or 16 ranges and fewer than 128 (sequence,
 * KV head) pairs the ranges are the CTAs of one thread-block cluster and merge through
 * distributed shared memory (scratch untouched); from 128 pairs on (and n_head / n_kv <= 16) a
 * tensor-core kernel takes the query heads of a KV head as the rows of mma tiles and merges the
 * ranges through the scratch; other range counts use the SIMT scratch kernel.
 * Replaces: the decode case of gpt_fast/utils.py:252-255 (repeat_interleave + SDPA over the
 * whole cache under mask = causal_mask[input_pos]). */
size_t lri_attn_decode_scratch_bytes(int B, int n_head, int n_kv, int head_dim, int num_splits);
/* The num_splits the library recommends for a cache geometry (host arithmetic on the SM count of the
 * current device, 148 without one; honours the decode_splits and attn_mma options): fixed per
 * geometry so that a captured graph stays valid as the position grows. */
int lri_attn_decode_plan(int B, int n_head, int n_kv, int head_dim, int64_t smax, int* num_splits);
int lri_attn_decode(int dtype, const void* q, const void* k_cache, const void* v_cache,
                    const void* input_pos, int pos_is_i64, void* out, int B, int n_head, int n_kv,
                    int head_dim, int64_t smax, int num_splits, void* scratch,
                    size_t scratch_bytes, lri_stream_t stream);

/* lri_attn_decode_static: the same kernel and arguments as lri_attn_decode, minus the scratch
 * pointer.  (No counterpart in the reference: it exists for callers of THIS library that may not
 * allocate - a plug-in that receives only tensors and a stream from its host framework, or a
 * server whose device memory is fixed before traffic starts and where a cudaMalloc, which
 * synchronises the device, must never happen while requests are in flight.)  The split partials
 * and counters live in an 8 MiB array built into the library
 * (lri_attn_decode_static_scratch_capacity()), held by every GPU that loads it until the process
 * ends.  A configuration needing more (lri_attn_decode_scratch_bytes(...) > capacity) is refused
 * with LRI_ERR_WORKSPACE.  Nothing is allocated or freed, here or in anything it calls.
 * The first call on each device looks up the array's device address (with that device current);
 * make that first call outside any stream capture.  All calls on a device share the one array:
 * two calls that overlap on the GPU (different streams) corrupt each other; calls in one stream
 * are fine, and each call leaves the counters at zero for the next. */
size_t lri_attn_decode_static_scratch_capacity(void);
int lri_attn_decode_static(int dtype, const void* q, const void* k_cache, const void* v_cache,
                           const void* input_pos, int pos_is_i64, void* out, int B, int n_head,
                           int n_kv, int head_dim, int64_t smax, int num_splits,
                           lri_stream_t stream);

/* ---- F4: causal GQA prefill attention --------------------------------------------------------
 * q [B, S, n_head, head_dim]; query s has position input_pos[0] + s (positions must be
 * consecutive, as in the reference's only caller, benchmark.py:138) and attends cache positions
 * 0..input_pos[0]+s.  out [B, S, n_head*head_dim].
 * Replaces: the prefill case of gpt_fast/utils.py:252-257. */
int lri_attn_prefill(int dtype, const void* q, const void* k_cache, const void* v_cache,
                     const void* input_pos, int pos_is_i64, void* out, int B, int S, int n_head,
                     int n_kv, int head_dim, int64_t smax, lri_stream_t stream);

/* ---- F8: all-reduce over peer memory (one process per GPU) -----------------------------------
 * A communicator owns, on every rank, one inbox buffer that all peers can write.  One-shot
 * all-reduce: every rank stores its partial into slot `rank` of each peer's inbox, then raises
 * a per-peer flag; the consumer waits (bounded) for all flags of the current epoch and sums
 * the slots in fp32.  The wait gives up after `timeout_ms` and records LRI_ERR_TIMEOUT
 * in a device status word that lri_comm_status() reads; it never traps and never spins forever.
 *
 * lri_comm_create: allocates the local inbox with cudaMalloc (the one allocation this library
 *   makes; it synchronises) and returns an opaque handle plus a 64-byte IPC handle to send
 *   to the peers.  max_elems = largest message in elements; slots are double buffered.
 * lri_comm_connect: `ipc_handles` = world*64 bytes gathered from all ranks (host memory).
 * lri_allreduce: in-place-capable SUM of `count` elements of `dtype`; out = sum over ranks of
 *   their `in`.  Epochs advance from a device-resident counter, so graph replays stay correct.
 * Replaces: all_reduce_func / dist.all_reduce, gpt_fast/utils.py:390-397. */
typedef struct lri_comm lri_comm;
int lri_comm_create(int rank, int world, int64_t max_elems, lri_comm** comm_out,
                    unsigned char ipc_handle_out[64]);
int lri_comm_connect(lri_comm* comm, const unsigned char* ipc_handles /* host, world*64 */);
int lri_allreduce(lri_comm* comm, int dtype, const void* in, void* out, int64_t count,
                  int timeout_ms, lri_stream_t stream);
/* Split form of the all-reduce for small messages (up to lri_comm_push_max_elems() elements): the
 * producer pushes its partial into the peers' inboxes right after the row-parallel projection
 * (lri_comm_push, channel 1 or 2, each with its own device-resident epoch), and the reduction
 * happens inside the consumer: lri_add_rmsnorm_gather is lri_add_rmsnorm whose addend k is, when
 * channel_k > 0, the SUM over ranks of the message last pushed on that channel (add_k then points
 * to this rank's own partial; rank-order fp32 sum, rounded once, bit-identical on all ranks) and,
 * when channel_k == 0, a plain addend pointer or NULL.  No reduce kernel and no stream fork: an
 * all-reduce costs one small push kernel.  A rank must consume message n of a channel before it
 * pushes message n+1 on it (the consumer advances the channel's epoch; two buffers per channel),
 * which every schedule here does; all ranks push the same sequence.  The consumer's wait is bounded by timeout_ms (status word as above).
 * Replaces: all_reduce_func + the residual add + RMSNorm that follow it,
 * gpt_fast/gpt_ladder_TP.py:323-356, gpt_fast/gpt_dense_TP.py:281-282.
 * lri_linear_push is lri_linear (decode, M <= 8) whose epilogue also pushes: every finished
 * output pair goes to the peers as an 8-byte {2 elements, epoch} half line, so the transfer
 * overlaps the tail of the projection and no push kernel is launched (the fused
 * compute + collective form of the row-parallel projections wo / w2). */
int64_t lri_comm_push_max_elems(void);
int lri_linear_push(lri_comm* comm, int channel, int dtype, const void* x, const void* w,
                    const void* addend, void* y, int64_t M, int N, int K, lri_stream_t stream);
int lri_comm_push(lri_comm* comm, int channel, int dtype, const void* in, int64_t count,
                  lri_stream_t stream);
int lri_add_rmsnorm_gather(lri_comm* comm, int dtype, const void* residual, int channel1,
                           const void* add1, int channel2, const void* add2, float residual_scale,
                           const void* weight, float eps, void* residual_out, void* normed_out,
                           int64_t rows, int dim, int timeout_ms, lri_stream_t stream);
/* lri_add_rmsnorm_allreduce: the whole all-reduce inside the consumer.  Same arguments and result as
 * lri_add_rmsnorm_gather, but nothing is pushed beforehand: every thread of the kernel first stores
 * the elements of this rank's partial(s) it is about to sum into the peers' inboxes and then polls
 * for theirs, so all-reduce + residual add + RMSNorm cost one launch on the consuming stream (no
 * all-reduce kernel, no communication stream, no event hop).  Channels, epochs, message limit and
 * ordering rule are those of the push channels; a channel carries either pushed or self-pushed
 * messages, all ranks alike.
 * Replaces: all_reduce_func + residual add + RMSNorm, gpt_fast/gpt_ladder_TP.py:323-356. */
int lri_add_rmsnorm_allreduce(lri_comm* comm, int dtype, const void* residual, int channel1,
                              const void* add1, int channel2, const void* add2, float residual_scale,
                              const void* weight, float eps, void* residual_out, void* normed_out,
                              int64_t rows, int dim, int timeout_ms, lri_stream_t stream);
/* ---- greedy decoding head: LM-head projection + arg-max over vocabulary rows and ranks ---------
 * token_out[m] (int32) = index of the largest logit of sequence m over the whole vocabulary, lowest
 * index on ties, where this rank holds rows [index_offset, index_offset + N) of the output projection
 * (w [N, K]) and the other ranks of `comm` hold the rest; comm == NULL: one rank.  Logits are compared
 * as the projection would store them (fp32 sums rounded to `dtype`).  M <= 8: the weight-streaming
 * kernel folds its candidates in its epilogue (one 64-bit key per sequence in `scratch`) and writes no
 * logits.  8 < M <= 64: the slice's logits go to logits_ws (M*N elements) through lri_linear (workspace
 * as there) and a small kernel folds them.  In both cases one warp launched behind the producer
 * exchanges one 16-byte line per sequence with every peer over NVLink (bounded wait: timeout_ms, status
 * word read by lri_comm_status) and writes the winner.
 * scratch: lri_lm_head_argmax_scratch_bytes() bytes, 16-byte aligned, zero before the first call;
 * every call leaves it zero.  All ranks must call with the same M; N may be 0 on a rank whose slice
 * is empty.  Every rank writes the same tokens.
 * Replaces: the output projection + sampling at top_k = 1 / arg-max of the logits,
 * gpt_fast/gpt_ladder_TP.py:282-283 with benchmark.py:56-77, 86-92. */
size_t lri_lm_head_argmax_scratch_bytes(void);
int lri_lm_head_argmax(lri_comm* comm, int dtype, const void* x, const void* w, int64_t M, int N, int K,
                       int64_t index_offset, int32_t* token_out, void* scratch, size_t scratch_bytes,
                       void* logits_ws, size_t logits_ws_bytes, void* workspace, size_t workspace_bytes,
                       int timeout_ms, lri_stream_t stream);
/* ==== Layers of designs outside the reference: fp32 residual stream, latent attention, gated recurrence, experts.
 * All of these take LRI_BF16, LRI_FP16 and LRI_FP32; every size is a parameter. ==== */

/* ---- residual stream in fp32 ----------------------------------------------------------------
 * y_r   = sum over the row's slots of y[slot]        (slots NULL: rows r * n_slots ...; y has y_rows rows)
 * t     = sigmoid(gate + gate_bias) * y_r            (gate NULL: t = y_r; gate fp32, row pitch gate_ld)
 * resid_out = resid + RMSNorm(t) * post_weight       (post_weight NULL: resid + t; resid NULL: 0; may alias)
 * normed_out = RMSNorm(resid_out) * next_weight      (weight NULL: resid_out; both NULL: none), rounded to `dtype`
 * RMSNorm(x) = x / sqrt(mean(x^2) + eps), fp32 throughout. */
int lri_gated_norm_add(int dtype, const float* resid, const void* y, const int32_t* slots, int n_slots,
                       int64_t y_rows, const float* gate, int64_t gate_ld, const void* gate_bias,
                       const void* post_weight, float eps, float* resid_out, const void* next_weight,
                       void* normed_out, int64_t rows, int dim, lri_stream_t stream);
/* resid_out = table[idx] in fp32, normed_out = RMSNorm(resid_out) * weight. */
int lri_embed_norm(int dtype, const void* table, const void* idx, int idx_is_i64, int64_t vocab,
                   float* resid_out, const void* weight, float eps, void* normed_out, int64_t rows, int dim,
                   lri_stream_t stream);

/* ---- latent attention --------------------------------------------------------------------------
 * proj [B*S, ld] fp32 holds q (heads of [dim | rot_dim]) at q_off and [latent (rank) | key part (rot_dim)] at
 * kv_off.  Rotates the rot_dim parts by halves (pair i, i + rot_dim/2) with rope_table [table_rows, rot_dim/2, 2]
 * (cos, sin; fp32) at the token's position, normalises the latent, and stores q's two parts (pitches in elements)
 * and the cache row [latent | key part] of cache [B, smax, rank + rot_dim]. */
int lri_latent_prepare(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t kv_off,
                       const void* norm_weight, float eps, const float* rope_table, int64_t table_rows,
                       const void* input_pos, int pos_is_i64, void* qn, int64_t qn_row, int64_t qn_head,
                       void* qr, int64_t qr_row, int64_t qr_head, void* cache, int64_t smax, int B, int S,
                       int heads, int dim, int rot_dim, int rank, lri_stream_t stream);
/* Cache rows of positions input_pos[0] - history .. + rows - 1 of every sequence, split into contiguous
 * latents [B, rows, rank] and rotated keys [B, rows, rot_dim]; positions below 0 give zeros. */
int lri_latent_window(int dtype, const void* cache, int64_t smax, int rank, int rot_dim, const void* input_pos,
                      int pos_is_i64, int B, int history, int rows, void* latent_out, void* k_rot_out,
                      lri_stream_t stream);
/* y[row, head] = W[head] x[row, head], W [heads, out, in], or [heads, in, out] when transposed. */
int lri_head_linear(int dtype, const void* x, int64_t x_row, int64_t x_head, const void* w, int transposed,
                    void* y, int64_t y_row, int64_t y_head, int64_t rows, int heads, int in, int out,
                    lri_stream_t stream);
/* Softmax attention of query (row, head) = [d1 | d2] over the key rows j = [k (d1) | k2 (d2, shared by the heads)]
 * at positions input_pos[0] - history + j (history < 0: position j) with 0 <= position of the query - position of the key < window_size.
 * Row j of v has dv elements.  Pitches in elements; a head pitch of 0 shares a row among the heads.
 * 16-bit types: prompt portions (16 tokens on, dim and vdim up to 128, rot_dim up to 64, multiples of 8) run on tcgen05;
 * single tokens over shared rows (k == v, k2 right behind k, d1 = dv up to 512, multiples of 16) on mma.sync, with
 * scratch for the results of splits (keys = most keys a query sees); everything else on a plain kernel. */
size_t lri_window_attention_scratch_bytes(int B, int heads, int dv, int64_t keys);
int lri_window_attention(int dtype, const void* q, int64_t q_row, int64_t q_head, const void* k, int64_t k_batch,
                         int64_t k_row, int64_t k_head, const void* k2, int64_t k2_batch, int64_t k2_row,
                         const void* v, int64_t v_batch, int64_t v_row, int64_t v_head, void* out,
                         const void* input_pos, int pos_is_i64, int history, int64_t k_rows,
                         int64_t window_size, float scale, int B, int S, int heads, int d1, int d2, int dv,
                         void* scratch, size_t scratch_bytes, lri_stream_t stream);

/* ---- HGRN2 recurrence -----------------------------------------------------------------------------
 * proj [B*S, ld] fp32 holds q, f, v at the given offsets.  f = lower + (1 - lower) sigmoid(f + f_bias), q = silu(q);
 * state[c, e] <- f[c] state[c, e] + (1 - f[c]) v[e], o[e] = sum_c q[c] state[c, e] per head, out = RMSNorm over e.
 * state [B, heads, dim, vdim] fp32 is read and written; a call that starts at position 0 starts from zero. */
size_t lri_hgrn2_workspace_bytes(int dtype, int B, int S, int heads, int dim, int vdim);
int lri_hgrn2(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t f_off, int64_t v_off,
              const void* f_bias, const void* lower, const void* norm_weight, float eps, float* state,
              const void* input_pos, int pos_is_i64, void* out, int B, int S, int heads, int dim, int vdim,
              void* workspace, size_t workspace_bytes, lri_stream_t stream);

/* ---- mixture of experts ------------------------------------------------------------------------------
 * lri_moe_packs: whether a call of this size runs on rows packed by expert (1) or pair by pair (0);
 * lri_moe_max_tiles: most 128-row tiles the packed form can need. */
int lri_moe_packs(int dtype, int64_t rows, int top, int dim, int ff);
int64_t lri_moe_max_tiles(int64_t rows, int top, int experts);
/* ids, scores [rows, top]: the `top` largest logistic scores of logits [rows, ld] (lowest index on ties).  For the
 * packed form counts [experts] (zero before the call) and rank [rows * top] are filled too. */
int lri_moe_route(const float* logits, int64_t ld, int experts, int top, int64_t rows, int32_t* ids,
                  float* scores, int32_t* counts, int32_t* rank, lri_stream_t stream);
/* Packs the rows of x by expert into tiles of 128: tiles = {count, expert of each}, packed rows and their scores,
 * slots [rows * top] = packed row of each pair; the buffers hold max_tiles tiles.  Leaves counts at zero. */
int lri_moe_pack(int dtype, const void* x, int64_t rows, int dim, int top, int experts, const int32_t* ids,
                 const float* scores, const int32_t* rank, int32_t* counts, int32_t* first_row, int32_t* tiles,
                 int64_t max_tiles, void* packed, float* row_scale, int32_t* slots, lri_stream_t stream);
/* hidden = g sigmoid(alpha g) (u + offset), g = min(s gate, limit), u = clamp(s up, -limit, limit) with the score s
 * of the pair and gate, up the two products with w1 [experts, 2 ff, dim] = [up | gate].  tiles == NULL: x [rows, dim],
 * hidden [pairs, ff]; else x and hidden are packed rows. */
int lri_moe_gateup(int dtype, const void* x, const void* w1, void* hidden, const int32_t* ids,
                   const float* scores, int64_t pairs, int top, const int32_t* tiles, const float* row_scale,
                   int64_t max_tiles, int experts, int ff, int dim, float alpha, float limit, float offset,
                   lri_stream_t stream);
/* y = w2 hidden per pair (or packed row), w2 [experts, dim, ff]; the sum over a token's choices is taken by
 * lri_gated_norm_add. */
int lri_moe_down(int dtype, const void* hidden, const void* w2, void* y, const int32_t* ids, int64_t pairs,
                 const int32_t* tiles, int64_t max_tiles, int experts, int dim, int ff, lri_stream_t stream);

/* ---- residual held as several streams (hyper-connections) ---------------------------------------------
 * x [rows, streams, dim] fp32.  x_out_t = sum_s mix[s, t] x_s + out[t] y (all from the old streams; x_out may alias x, NULL:
 * not stored), u = sum_s in_next[s] x_out_s (in_next NULL: plain sum), normed = RMSNorm(u) * weight rounded to `dtype`.
 * mix [streams, streams] ([from, to]), out and in_next [streams], weight [dim] in `dtype`; up to 16 streams. */
int lri_join_streams(int dtype, const float* x, const void* y, const void* mix, const void* out, float* x_out,
                     const void* in_next, const void* weight, float eps, void* normed, int64_t rows, int streams, int dim,
                     lri_stream_t stream);
/* Starts the streams: every x_out_s = scale * table[idx], then u and normed as above. */
int lri_embed_streams(int dtype, const void* table, const void* idx, int idx_is_i64, int64_t vocab, float scale,
                      float* x_out, const void* in_next, const void* weight, float eps, void* normed, int64_t rows,
                      int streams, int dim, lri_stream_t stream);

/* ---- gate/up projection + clamped unit --------------------------------------------------------------------
 * w1 [2 I, K] = [up | gate]; h = g sigmoid(alpha g) (u + offset), g = min(gate, limit), u = clamp(up, -limit, limit), from
 * fp32 sums.  Kernels as lri_gateup_swiglu; LRI_FP32 and any K run the plain kernels. */
size_t lri_gateup_glu_workspace_bytes(int dtype, int64_t M, int I, int K);
int lri_gateup_glu(int dtype, const void* x, const void* w1, void* h, int64_t M, int I, int K, float alpha, float limit,
                   float offset, void* workspace, size_t workspace_bytes, lri_stream_t stream);

/* ---- grouped-query attention with whole-projection norms, windows, chunks and sinks --------------------------
 * proj [B*S, ld] fp32 holds q (n_head heads of dim), k (n_kv of dim) and v (n_kv of vdim) at the offsets.  q and k are
 * RMS-normed over all their elements (weights q_norm, k_norm; sums of squares over q_width, k_width elements are taken
 * here or, sums != NULL, read from [rows, 2]), the first rot_dims of each head rotated by halves with rope_table
 * [table_rows, rot_dims/2, 2] (fp32) at the token's position; q goes to [rows, n_head, dim], k and v to the caches
 * [B, n_kv, smax, dim] and [B, n_kv, smax, vdim]. */
int lri_grouped_prepare(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off,
                        const void* q_norm, const void* k_norm, const float* sums, int q_width, int k_width, float eps,
                        const float* rope_table, int64_t table_rows, int rot_dims, const void* input_pos, int pos_is_i64,
                        void* q, void* k_cache, void* v_cache, int64_t smax, int B, int S, int n_head, int n_kv, int dim,
                        int vdim, lri_stream_t stream);
/* sums[row] = sums of squares of x[row, off1 .. off1 + n1) and x[row, off2 .. off2 + n2). */
int lri_row_squares(const float* x, int64_t ld, int64_t off1, int n1, int64_t off2, int n2, float* sums, int64_t rows,
                    lri_stream_t stream);
/* Attention of the query at position p over cache positions j <= p with p - j < window (0: no window) and, chunk > 0,
 * j / chunk == p / chunk.  sink [n_head] (NULL: none): exp(sink) joins the denominator.  out row = out_scale times the
 * heads' results, pitch out_ld.  16-bit types: prompt portions of 16 tokens on (dim, vdim up to 128, multiples of 8) on
 * tcgen05, single tokens on thread-block clusters; everything else on a plain kernel. */
int lri_grouped_attention(int dtype, const void* q, const void* k_cache, const void* v_cache, const void* sink, void* out,
                          int64_t out_ld, float out_scale, const void* input_pos, int pos_is_i64, int64_t smax,
                          int64_t window, int64_t chunk, float scale, int B, int S, int n_head, int n_kv, int dim,
                          int vdim, lri_stream_t stream);

/* ---- matrix-state recurrences with a decay per key channel ----------------------------------------------------
 * Per sequence and head, token by token: S <- g * S (g per row of S [dim, vdim]); u = v (gated linear attention) or
 * u = beta (v - S^T k) (gated delta rule); S <- S + k u^T; o = S^T q.  All fp32.  Several tokens run in blocks of four:
 * lri_delta_blocks / lri_gla_blocks prepare a call's block vectors, lri_state_scan runs it.
 * lri_state_blocks: blocks of a sequence of S tokens; the arrays hold B times as many, blocks [.., heads, dim] for decay and
 * [.., heads, 32] for coef, four rows [heads, dim] a block for qd, kd and ku. */
int64_t lri_state_blocks(int64_t S);
/* proj [B*S, ld] holds q, k (kv_heads of dim), v (heads of vdim) and b (heads).  q, k, v pass a causal convolution over time
 * per channel (conv_* [channels, taps], last column = current token) and silu; q and k become unit vectors
 * x / sqrt(sum x^2 + 1e-6), q also times dim^(-1/2); beta = sigmoid(b); g = exp(-exp(a_log) softplus(z + dt_bias)),
 * z [B*S, heads, dim].  ring [B, taps, 2 kv_heads dim + heads vdim] keeps the last inputs of each channel (position p in slot
 * p % taps); it is read for tokens before the call and updated.  v [B*S, heads, vdim] receives the values. */
int lri_delta_blocks(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int64_t b_off,
                     const void* conv_q, const void* conv_k, const void* conv_v, int taps, float* ring, const float* z,
                     const void* a_log, const void* dt_bias, const void* input_pos, int pos_is_i64, float* qd, float* kd,
                     float* ku, float* decay, float* coef, float* v, int B, int S, int heads, int kv_heads, int dim,
                     int vdim, lri_stream_t stream);
/* q (times dim^(-1/2)) and k from proj, g = sigmoid(z + bias)^(1 / tau). */
int lri_gla_blocks(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, const float* z, const void* bias,
                   float tau, float* qd, float* ku, float* decay, float* coef, int B, int S, int heads, int dim,
                   lri_stream_t stream);
/* The recurrence over a call's tokens; kd NULL: gated linear attention.  v [.., heads, vdim] with row pitch v_row; o [B*S,
 * heads, vdim]; state [B, heads, dim, vdim] is read and written, a call that starts at position 0 starts from zero. */
int lri_state_scan(const float* qd, const float* kd, const float* ku, const float* decay, const float* coef, const float* v,
                   int64_t v_row, float* state, const void* input_pos, int pos_is_i64, float* o, int B, int S, int heads,
                   int dim, int vdim, lri_stream_t stream);
/* One token per sequence, everything between the input projections and the output projection's rows in one kernel; inputs
 * as above, the low-rank second projections included: a2 [heads dim, a_rank] and g2 [heads vdim, g_rank] in `dtype` multiply
 * the columns at a_off and g_off rounded to `dtype` (ranks multiples of 8, zero padded).  out (pitch out_ld) = factor *
 * RMSNorm over vdim * norm_weight * gate; gate = sigmoid(g2 ..) or, gla, silu of the columns at g_off. */
int lri_state_step_supports(int dim, int vdim, int decay_rank, int gate_rank);
int lri_delta_step(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int64_t a_off,
                   int64_t g_off, int64_t b_off, const void* conv_q, const void* conv_k, const void* conv_v, int taps,
                   float* ring, const void* a2, int a_rank, const void* g2, int g_rank, const void* a_log,
                   const void* dt_bias, const void* norm_weight, float eps, float factor, float* state,
                   const void* input_pos, int pos_is_i64, void* out, int64_t out_ld, int B, int heads, int kv_heads,
                   int dim, int vdim, lri_stream_t stream);
int lri_gla_step(int dtype, const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, int64_t a_off,
                 int64_t g_off, const void* a2, int a_rank, const void* bias, float tau, const void* norm_weight, float eps,
                 float factor, float* state, const void* input_pos, int pos_is_i64, void* out, int64_t out_ld, int B,
                 int heads, int dim, int vdim, lri_stream_t stream);
/* out[row, head] = scale * RMSNorm(o[row, head]) * norm_weight * act(gate[row, head]), gate fp32 with row pitch gate_ld. */
enum lri_gate { LRI_GATE_SIGMOID = 0, LRI_GATE_SILU = 1 };
int lri_head_norm_gate(int dtype, const float* o, const void* norm_weight, float eps, const float* gate, int64_t gate_ld,
                       int activation, float scale, void* out, int64_t out_ld, int64_t rows, int heads, int vdim,
                       lri_stream_t stream);
/* y [rows, n] = x[row, off .. off + n) rounded to `dtype`. */
int lri_round_columns(int dtype, const float* x, int64_t ld, int64_t off, int n, void* y, int64_t rows, lri_stream_t stream);

/* Reads (and clears) the device status word: LRI_OK or LRI_ERR_TIMEOUT.  Synchronises `stream`. */
int lri_comm_status(lri_comm* comm, lri_stream_t stream);
int lri_comm_destroy(lri_comm* comm);

#ifdef __cplusplus
}
#endif
#endif /* LRI_B200_H_ */
