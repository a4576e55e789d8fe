/* dlti_b200 — C ABI of the native sm_100a kernel library (libdlti_b200.so).
 *
 * Every entry point:
 *   - takes raw device pointers plus a cudaStream_t and is asynchronous on that stream;
 *   - returns 0 on success, a positive cudaError_t, or a negative DLTI_ERR_* code
 *     (dlti_error_string() / dlti_last_error() describe it);
 *   - allocates no device memory unless its comment says so (workspaces are passed in).
 *
 * dtype codes: 0 = bf16, 1 = fp16, 2 = fp32.
 *
 * The reference repository (rokulkarni15/distributed-llm-training-inference) has no native
 * code; each declaration cites the library call it replaces in the reference's stack
 * (SURVEY.md section 2.4 / 2.7 numbering).
 */
#ifndef DLTI_B200_H_
#define DLTI_B200_H_

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef struct CUstream_st* dlti_stream_t;

#define DLTI_BF16 0
#define DLTI_FP16 1
#define DLTI_FP32 2

/* ---- runtime ---------------------------------------------------------------------------- */
int dlti_version(void);
int dlti_sm_count(void);
/* Programmatic dependent launch on the decode path (skinny GEMM, dlti_acc_*, paged decode). Level 1 (default):
 * those kernels start while their predecessor in the stream drains and order all global accesses behind a
 * dependency wait. Level 2: dlti_gemm_skinny additionally requests its first weight tiles before that wait —
 * only for weights that no kernel still in flight writes (the serving engine sets this). Level 0 = plain stream
 * ordering. Environment: DLTI_PDL=0|1|2. */
void dlti_set_pdl(int level);
int dlti_get_pdl(void);
long long dlti_launch_count(void);      /* kernels launched by this library since reset */
void dlti_reset_launch_count(void);
const char* dlti_last_error(void);
const char* dlti_error_string(int code);

/* ---- K2/K3: tcgen05 GEMM with K-extension (fused LoRA) ------------------------------------
 * C[M,N] = alpha * ( op(A)·op(B) + A2·op(B2) ) + R          (out bf16/fp16, optional residual R)
 * C[M,N] (+)= alpha * ( ... )                               (out fp32, accumulate = 0/1)
 *   a_mn = 0: A is [M,K] row-major (pitch lda).   a_mn = 1: A is stored [K,M] row-major.
 *   b_mn = 0: B is [N,K] row-major (x·W^T).       b_mn = 1: B is stored [K,N] row-major.
 *   A2/B2 (optional, K2 % 64 == 0) use the same majorness as A/B and are accumulated into the
 *   same tensor-memory tile after the main K loop (LoRA: A2 = dropout(x)·A^T, B2 = (alpha/r)·B).
 *   split_k > 1 requires fp32 output with accumulate = 1 (atomic adds).
 *   block_n: 0 = auto, or 64/128/256. max_ctas: 0 = all SMs.
 * Replaces cuBLAS GEMM under torch.nn.functional.linear + PEFT lora.Linear
 * (reference training/train_baseline.py:122-140). */
int dlti_gemm(const void* A, const void* B, void* C, const void* R, int M, int N, int K,
              long long lda, long long ldb, long long ldc, long long ldr, int a_mn, int b_mn,
              const void* A2, const void* B2, int K2, long long lda2, long long ldb2,
              int in_dtype, int out_dtype, float alpha, int accumulate, int split_k, int block_n,
              int max_ctas, dlti_stream_t stream);

/* ---- K4: RMSNorm ---------------------------------------------------------------------------
 * fwd: y = w * T(x * rsqrt(mean(x^2) + eps)); optional residual_inout (+= x, then normalised: the
 * serving path's fused add+norm), optional ydrop = dropout(y) (LoRA-branch input, Philox mask
 * keyed by (seed, stream_id, element index)), rstd (fp32 per row) for the backward.
 * bwd: dx (norm weights are frozen: no dw); dres (optional) is added to dx.
 * Replaces HF LlamaRMSNorm's ~5 ATen kernels / vLLM rms_norm + fused_add_rms_norm. */
int dlti_rmsnorm_fwd(const void* x, void* residual_inout, const void* w, void* y, void* ydrop,
                     float* rstd, long long rows, int d, float eps, float drop_p,
                     unsigned long long seed, unsigned long long stream_id, int dtype,
                     dlti_stream_t stream);
int dlti_rmsnorm_bwd(const void* dy, const void* x, const void* w, const float* rstd,
                     const void* dres, void* dx, long long rows, int d, int dtype,
                     dlti_stream_t stream);

/* ---- K5: RoPE (rotate-half), in place on the first n_rot_heads heads of each [tokens, row_stride]
 * row (merged qkv: q heads then k heads). cos/sin: fp32 [max_pos, hd/2]. backward = inverse
 * rotation. Replaces HF apply_rotary_pos_emb / vLLM rotary_embedding. */
int dlti_rope(void* buf, const int* pos, const float* cos_t, const float* sin_t, long long tokens,
              int n_rot_heads, int hd, long long row_stride, int backward, int dtype,
              dlti_stream_t stream);

/* ---- K7: SwiGLU on gu = [tokens, 2*ff] (gate | up). Replaces silu + mul / vLLM silu_and_mul
 * (SURVEY O7, S8). */
int dlti_swiglu_fwd(const void* gu, void* h, long long tokens, int ff, long long gu_stride,
                    long long h_stride, int dtype, dlti_stream_t stream);
int dlti_swiglu_bwd(const void* dh, const void* gu, void* dgu, long long tokens, int ff,
                    long long dh_stride, long long gu_stride, int dtype, dlti_stream_t stream);

/* ---- dropout / a + dropout(b): counter-based masks (mask index = row*cols + col), reproducible in
 * layer recompute. Replaces torch.nn.Dropout inside PEFT lora.Linear (lora_dropout = 0.05). */
int dlti_dropout(const void* x, void* y, long long rows, int cols, long long x_stride,
                 long long y_stride, float p, unsigned long long seed, unsigned long long stream_id,
                 int dtype, dlti_stream_t stream);
int dlti_add_dropout(const void* a, const void* b, void* y, long long rows, int cols, float p,
                     unsigned long long seed, unsigned long long stream_id, int dtype,
                     dlti_stream_t stream);

/* ---- K15: embedding gather; ids outside [vocab_start, vocab_start + vocab_rows) give zero rows
 * (vocab-parallel shard contribution). Replaces ATen embedding. */
int dlti_embedding(const long long* ids, const void* table, void* out, long long tokens, int d,
                   long long vocab_start, long long vocab_rows, int dtype, dlti_stream_t stream);

/* ---- K8 (loss): softmax cross-entropy over 16-bit logits, fp32 math. loss_rows[t] = lse - logit
 * [label] (0 when label == ignore_index); dlogits (may alias logits) = (softmax - onehot) * *gscale.
 * Replaces ATen log_softmax + nll_loss (+ backward). */
int dlti_cross_entropy(const void* logits, void* dlogits, const long long* labels, float* loss_rows,
                       const float* gscale, long long rows, int V, long long ld, long long ldd,
                       long long ignore_index, int dtype, dlti_stream_t stream);

/* ---- K9 (single-GPU part): out[0] (+)= sum(g^2) over a flat fp32 vector (gradient norm; a
 * non-finite element makes it non-finite = fp16 overflow). `partials` is caller-provided SCRATCH of
 * dlti_sumsq_scratch_floats() floats. Replaces clip_grad_norm_ + GradScaler's finite check
 * (SURVEY N7, O12, C6, C7). */
int dlti_sumsq_scratch_floats(void);
int dlti_sumsq(const float* g, long long n, float* partials, float* out, int accumulate,
               dlti_stream_t stream);

/* Same reduction as dlti_sumsq for callers that cannot hand the library a device workspace: a
 * process whose own pool (e.g. a KV-cache arena) already holds all free HBM, a loop that must not
 * pay the device-wide synchronisation of cudaMalloc/cudaFree, or a plain C host with no tensor
 * allocator. The partial sums live in a 32 KB array built into the library (one copy per GPU that
 * loads it, until exit), so n is limited to dlti_sumsq_noalloc_max_elems() = 134,217,728 floats;
 * larger n returns DLTI_ERR_TOO_LARGE (-4) with a message in dlti_last_error(). The first call on
 * each device looks up the array's device address (cudaGetSymbolAddress) — make it before any
 * stream capture. Calls share the array: calls whose kernels overlap on the GPU race; keep them
 * ordered. No cudaMalloc/cudaFree is made. This entry point has no counterpart in the reference. */
long long dlti_sumsq_noalloc_max_elems(void);
int dlti_sumsq_noalloc(const float* g, long long n, float* out, int accumulate,
                       dlti_stream_t stream);

/* Fused unscale + global-norm clip + AdamW (decoupled weight decay) on a flat fp32 partition with
 * optional 16-bit copy-out; skipped (and *skipped_out = 1) when *gnorm_sq is not finite.
 * Replaces torch.optim.AdamW / DeepSpeed FusedAdam multi_tensor_adam.cu. */
int dlti_adamw(float* p, float* m, float* v, float* g, void* p16, int p16_dtype, long long n,
               float lr, float b1, float b2, float eps, float wd, int step, const float* gnorm_sq,
               float inv_scale, float max_norm, int* skipped_out, int zero_grad,
               dlti_stream_t stream);

/* Batched 2-D fp32 -> 16-bit casts with per-job scale; jobs_dev = device array of 48-byte records
 * {src*, dst*, rows, cols, src_pitch, dst_pitch, scale, pad}. Refreshes the packed LoRA buffers. */
int dlti_cast_job_bytes(void);
int dlti_multi_cast(const void* jobs_dev, int njobs, int dst_dtype, dlti_stream_t stream);

/* ---- K6: causal varlen flash attention, head_dim 128, GQA. qkv = [T, (H+2KV)*128] (q|k|v per
 * token row, RoPE applied); out = [T, H*128]; lse = [H, T] fp32 (NULL allowed for inference).
 * Backward writes dqkv = [T, (H+2KV)*128]; D_scratch = [H, T] fp32 workspace.
 * Replaces PyTorch SDPA / flash-attn. */
int dlti_attn_fwd(const void* qkv, void* out, float* lse, const int* cu_seqlens, int batch,
                  int max_seqlen, long long T_total, int H, int KV, int hd, float scale, int dtype,
                  dlti_stream_t stream);
int dlti_attn_bwd(const void* dout, const void* qkv, const void* out, const float* lse,
                  float* D_scratch, void* dqkv, const int* cu_seqlens, int batch, int max_seqlen,
                  long long T_total, int H, int KV, int hd, float scale, int dtype,
                  dlti_stream_t stream);

/* ---- K2 (CTA-pair form): same contract as dlti_gemm with A K-major and no split-K, computed by
 * tcgen05 cta_group::2 pairs (256x256 tile per pair, each CTA stages half of the B tile). A ragged
 * last wave is removed by stream-K: the last waves' tiles are cut into equal (tile, k-block) ranges and
 * the owner of a split tile adds its helper's fp32 partial from a per-stream workspace. */
int dlti_gemm_2cta(const void* A, const void* B, void* C, const void* R, int M, int N, int K,
                   long long lda, long long ldb, long long ldc, long long ldr, int b_mn, const void* A2,
                   const void* B2, int K2, long long lda2, long long ldb2, int in_dtype, int out_dtype,
                   float alpha, int accumulate, int stream_k /* -1 auto, 0 off, 1 force */,
                   dlti_stream_t stream);

/* K1 on the CTA-pair kernel (ZeRO-3 all-gather fused into the GEMM; replaces the reference's DeepSpeed
 * stage-3 parameter all-gather, /root/reference/configs/ds_config_zero3.json:16-37). Attaches to the NEXT
 * dlti_gemm_2cta / _rope_2cta / _swiglu_2cta / _swiglu_bwd_2cta launch made from this host thread:
 *  - a gather job (j_count > 0): one extra warp per CTA pulls the 64-row units (rot_unit + j) % n_units,
 *    j in [j_begin, j_begin + j_count), of a row-sharded matrix [world * rows_per_rank, row_bytes] from their
 *    owner ranks (peer loads; own rows locally) into `staging` and publish per-unit counters: unit u is
 *    complete once counters[u] >= epoch * 16. The job may feed this launch's own B operand or, normally, a
 *    matrix that a later launch consumes (the next layer's weights ride on this layer's GEMMs);
 *  - a wait spec (wait_counters != NULL): the launch's B operand is such a staging buffer; the TMA producer
 *    acquires the counters of the units each tile needs (fast path when everything has landed already).
 * dlti_gather_job_run executes an attached job as a kernel of its own. */
int dlti_gemm2_attach(const void* const* peer_shards, void* staging, unsigned int* counters, long long row_bytes,
                      int rows_per_rank, int world, int rot_unit, int j_begin, int j_count, unsigned int epoch,
                      const unsigned int* wait_counters, int wait_units, unsigned int wait_epoch, int* err_flag);
int dlti_gather_job_run(int ctas, dlti_stream_t stream);
/* K11 (all-gather -> column-parallel GEMM; the reference's surface is vLLM tensor parallelism,
 * /root/reference/README.md:10): after dlti_gemm2_attach, declare that the job / wait spec concern the A operand
 * (activation rows pulled from their owner ranks by the launch's gather warp; the A producer waits per 64-row
 * unit) and that the M blocks are visited starting at block m_rot (this rank's own rows, which land first). */
int dlti_gemm2_attach_a_side(int m_rot);
/* K10 for prefill-sized steps (row-parallel GEMM -> reduce-scatter): the next CTA-pair launch stores output row r
 * into the receive slot of rank r / rows_per_owner (peer stores from the epilogue, tile by tile); the owner then
 * sums its slots in rank order (dlti_tp_own_reduce_norm). */
int dlti_gemm2_attach_scatter(const void* const* slot_peers, int world, int rank, int rows_per_owner);

/* Llama gate_up projection + SwiGLU in one kernel: h[M, ff] = silu(A·Wg^T) * (A·Wu^T), W = [gate; up]
 * stored [2*ff, K]. CTA rank 0 of a pair stages gate rows, rank 1 the matching up rows; the [M, 2*ff]
 * intermediate is never written. Rounding points match dlti_swiglu_fwd on a stored gate|up tensor. */
int dlti_gemm_swiglu_2cta(const void* A, const void* W, void* Hout, int M, int ff, int K, long long lda,
                          long long ldw, long long ldh, int dtype, dlti_stream_t stream);

/* Fused QKV projection (+ LoRA K-extension) with the rotary embedding applied in the epilogue to the first
 * rope_cols output columns (heads of 128, rotate-half; cos/sin fp32 [max_pos, 64]; pos[M] int32). */
int dlti_gemm_rope_2cta(const void* A, const void* B, void* C, int M, int N, int K, long long lda,
                        long long ldb, long long ldc, const void* A2, const void* B2, int K2, long long lda2,
                        long long ldb2, int dtype, float alpha, const int* pos, const float* cos_t,
                        const float* sin_t, int rope_cols, dlti_stream_t stream);

/* Input-gradient GEMM of the down projection with the SwiGLU backward in its epilogue:
 * dGU[M, 2*ff] = swiglu_bwd(dY[M, K] · Wdown[K, ff], GU[M, 2*ff]); dh is never written. */
int dlti_gemm_swiglu_bwd_2cta(const void* dY, const void* Wdown, const void* GU, void* dGU, int M, int ff, int K,
                              long long ldy, long long ldw, long long ldgu, long long lddgu, int dtype,
                              dlti_stream_t stream);

/* ---- Decode-sized GEMM (M <= 256): swap-AB (the weight is the 128-row tensor-core operand), K split
 * over CTAs, fp32 partials reduced with atomics into acc32[M,N] (must be zero on entry);
 * dlti_skinny_finish converts acc32 -> out and re-zeroes it. split_k: 0 = stream-K (the (tile, K block)
 * space cut into equal ranges per CTA; default), n > 0 = n tile-major splits, < 0 = automatic tile-major
 * split. Replaces the cuBLAS GEMV/GEMM calls of the vLLM decode path. */
int dlti_gemm_skinny(const void* X, const void* W, float* acc32, int M, int N, int K, long long ldx,
                     long long ldw, int in_dtype, int split_k, dlti_stream_t stream);
int dlti_skinny_finish(float* acc32, void* out, long long rows, int cols, long long out_stride, int dtype,
                       dlti_stream_t stream);

/* Consumers of acc32 that replace dlti_skinny_finish + the next elementwise op of a decode step (each value
 * is rounded to `dtype` first, so results equal finish -> op bit for bit; acc32 is zero on return):
 *   residual += acc ; y = RMSNorm(residual) * w          (o_proj / down_proj; vLLM fused_add_rms_norm, S7/S9)
 *   h = silu(acc[:, :ff]) * acc[:, ff:]                  (gate_up; vLLM silu_and_mul, S8)
 *   qkv = rope(acc) + k/v rows into the paged cache      (qkv_proj; vLLM rotary_embedding + reshape_and_cache, S4) */
int dlti_acc_add_rmsnorm(float* acc32, void* residual_inout, const void* w, void* y, long long rows, int d,
                         float eps, int dtype, dlti_stream_t stream);
int dlti_acc_swiglu(float* acc32, void* h, long long rows, int ff, long long h_stride, int dtype,
                    dlti_stream_t stream);
int dlti_acc_rope_cache(float* acc32, void* qkv, const int* pos, const float* cos_t, const float* sin_t,
                        const long long* slot_mapping, void* k_cache, void* v_cache, long long tokens, int H,
                        int KV, int hd, long long row_stride, int dtype, dlti_stream_t stream);

/* ---- Peer memory plumbing (symmetric arena fallbacks): CUDA IPC handle export/open/close and the
 * base/size of the allocation that contains a pointer. */
int dlti_ipc_get_handle(const void* dev_ptr, void* handle_out_64);
int dlti_ipc_open(const void* handle_64, void** out_ptr);
int dlti_ipc_close(void* ptr);
int dlti_mem_base(const void* dev_ptr, void** base_out, unsigned long long* size_out);

/* ---- K1/K9/K10/K11: fused compute + collective kernels over NVLink peer memory. All pointer tables
 * are DEVICE arrays of `world` peer pointers (index = rank); `err_flag` receives a non-zero code when a
 * bounded wait expires (the kernels never spin forever). Replace NCCL all-gather / reduce-scatter /
 * all-reduce in DeepSpeed ZeRO and vLLM TP. */
int dlti_comm_max_ranks(void);
/* all ranks arrive on `channel` with a host-chosen epoch (eager) or a device-side counter (graph-safe) */
int dlti_peer_barrier(const void* const* signal_pads, int rank, int world, int channel,
                      unsigned int epoch, int* err_flag, dlti_stream_t stream);
int dlti_peer_barrier_auto(const void* const* signal_pads, int rank, int world, int channel,
                           unsigned int* device_counter, int* err_flag, dlti_stream_t stream);
/* K9, overlapped form (replaces DeepSpeed's bucketed gradient reduce-scatter with overlap_comm, the global-norm
 * all-reduce, the partitioned optimizer step and the parameter all-gather:
 * /root/reference/configs/ds_config_zero3.json:29-31, ds_config_zero1.json:38-40).
 * dlti_grad_ready_signal: "my gradients of range `slot` are final for step `epoch`" to every rank.
 * dlti_rs_wait_accumulate: once all ranks have signalled, part[plo..] += sum_r grads[r][glo..] (fixed rank order).
 * dlti_k9_step: exchange of {sum of squares, loss sum}, unscale/clip/AdamW on [lo, lo+n) with the new fp32 values
 * stored into every rank's master, then a completion flag to every peer; dlti_peer_wait waits for those flags. */
int dlti_grad_ready_signal(const void* const* flags, int rank, int world, int slot, unsigned int epoch,
                           dlti_stream_t stream);
int dlti_rs_wait_accumulate(const void* const* grads, const unsigned int* my_flags, float* part, long long glo,
                            long long plo, long long n, int world, int slot, unsigned int epoch, int ctas,
                            int* err_flag, dlti_stream_t stream);
int dlti_k9_step(const void* const* masters, const void* const* boards, const void* const* signal_pads, float* m,
                 float* v, float* g, long long lo, long long n, int rank, int world, float lr, float b1, float b2,
                 float eps, float wd, int step, const float* local2, float* out2, float inv_scale, float max_norm,
                 int* skipped_out, unsigned int* done_scratch, int ch_norm, int ch_push, unsigned int epoch,
                 int* err_flag, dlti_stream_t stream);
int dlti_peer_wait(const unsigned int* my_pads, int world, int channel, unsigned int epoch, int* err_flag,
                   dlti_stream_t stream);

/* Owner side of K10 for prefill-sized steps: sum this rank's receive slots [world * per, d] in rank order, add the
 * (row-sharded) residual, RMSNorm, write the normalised rows to this rank's symmetric [per, d] buffer. */
int dlti_tp_own_reduce_norm(const void* slots, int world, long long per, long long row_lo, long long rows,
                            void* residual, const void* w, void* xn_own, int d, float eps, int dtype,
                            dlti_stream_t stream);

/* K15: embedding lookup over a vocabulary-sharded table in peer memory: out[t] = row ids[t] fetched from its
 * owner rank (ids outside [0, vocab) give zero rows). Replaces all-gather + lookup of the reference's ZeRO-3
 * embedding (HF LlamaModel.embed_tokens under DeepSpeed stage 3). */
int dlti_embedding_peer(const long long* ids, const void* const* shards, void* out, long long tokens, int d,
                        long long rows_per_rank, long long vocab, int world, int dtype, dlti_stream_t stream);
/* pull-based all-gather of equally sized row shards into `out` (K1 stand-alone form) */
int dlti_allgather_rows(const void* const* shards, void* out, long long shard_bytes, int rank, int world,
                        int blocks_per_peer, dlti_stream_t stream);
/* K1: C = A · op(gathered B): B is row-sharded over `world` ranks; gather warps inside the GEMM pull
 * the shards into B_staging (own rows are read in place) and publish per-unit counters (= epoch*16)
 * that the TMA producer waits on, so the transfer overlaps the math tile by tile. */
int dlti_gemm_gather(const void* A, void* B_staging, void* C, const void* R, int M, int N, int K,
                     long long lda, long long ldb, long long ldc, long long ldr, int b_mn, const void* A2,
                     const void* B2, int K2, long long lda2, long long ldb2, int in_dtype, int out_dtype,
                     float alpha, int block_n, int max_ctas, const void* const* peer_shards,
                     unsigned int* counters, unsigned int epoch, int rank, int world, int rows_per_rank,
                     int* err_flag, dlti_stream_t stream);
/* K10: row-parallel GEMM whose epilogue stores the partial tile into slot `rank` of every peer's
 * receive buffer [world, slot_stride] (followed by a barrier and dlti_tp_reduce_add_norm). */
int dlti_gemm_push(const void* A, const void* B, int M, int N, int K, long long lda, long long ldb,
                   long long ldc, int in_dtype, int block_n, const void* const* recv_peers, int rank,
                   int world, long long slot_stride, dlti_stream_t stream);
/* K11: residual += sum over ranks (fixed order) of the received partials; y = rmsnorm(residual) * w */
int dlti_tp_reduce_add_norm(const void* recv, long long slot_stride, int world, void* residual,
                            const void* w, void* y, long long rows, int d, float eps, int dtype,
                            dlti_stream_t stream);
/* K11 with the rank barrier inside the kernel (CTA 0 signals the peers, every CTA waits for all of them; the
 * epoch is a device counter bumped by the last CTA, so the launch replays from a CUDA graph): replaces
 * dlti_peer_barrier_auto + dlti_tp_reduce_add_norm on the decode path. done_scratch: zero-initialised u32. */
int dlti_tp_barrier_reduce_add_norm(const void* recv, long long slot_stride, int world, void* residual,
                                    const void* w, void* y, long long rows, int d, float eps, int dtype,
                                    const void* const* signal_pads, int rank, int channel,
                                    unsigned int* device_counter, unsigned int* done_scratch, int* err_flag,
                                    dlti_stream_t stream);
/* Prefill-sized K10/K11: reduce-scatter + all-gather over peer memory. Each rank's partial [T, d] sits in its own
 * symmetric buffer; this call handles rows [row_lo, row_lo + rows) (the caller's share): pull the rows of all
 * ranks' partials (rank order), add the residual rows (row-sharded on this path), RMSNorm, push the normalised
 * rows into every rank's activation buffer. Needs a rank barrier before (partials complete) and after. */
int dlti_tp_pull_reduce_norm_push(const void* const* partial_peers, const void* const* xn_peers, int world,
                                  long long row_lo, long long rows, void* residual, const void* w, int d, float eps,
                                  int dtype, dlti_stream_t stream);
/* K9: reduce-scatter by pull: part[0:n] += sum over ranks of grads[r][lo:lo+n] (fixed rank order) */
int dlti_rs_accumulate(const void* const* grads, float* part, long long lo, long long n, int world,
                       dlti_stream_t stream);
/* K9: all-reduce of one fp32 scalar (the grad-norm partial) through per-rank boards + signal pads */
int dlti_sumsq_exchange(const float* local, const void* const* boards, const void* const* signal_pads,
                        int rank, int world, int channel, unsigned int epoch, float* out, int* err_flag,
                        dlti_stream_t stream);
/* K9: AdamW on this rank's fp32 partition whose updated values are pushed into every rank's fp32
 * master copy (the all-gather of ZeRO-1/2 folded into the optimizer kernel). */
int dlti_adamw_push(const void* const* masters, float* m, float* v, float* g, long long lo, long long n,
                    int rank, int world, float lr, float b1, float b2, float eps, float wd, int step,
                    const float* gnorm_sq, float inv_scale, float max_norm, int* skipped_out,
                    dlti_stream_t stream);

/* ---- Serving kernels (replace vLLM's rotary_embedding + reshape_and_cache,
 * paged_attention_v2 and the sampler). */
/* RoPE on q,k in place + write of the rotated k and v rows into the paged cache slots (one kernel) */
int dlti_rope_cache(void* qkv, const int* pos, const float* cos_t, const float* sin_t,
                    const long long* slot_mapping, void* k_cache, void* v_cache, long long tokens, int H,
                    int KV, int hd, long long row_stride, int dtype, dlti_stream_t stream);
/* split-KV paged decode attention; workspace holds per-split (m, l, acc) in fp32 */
int dlti_paged_decode_workspace_floats(int batch, int H, int splits);
int dlti_paged_decode(const void* q, long long q_stride, const void* k_cache, const void* v_cache,
                      const int* block_tables, int max_blocks, const int* ctx_lens, int batch,
                      int block_size, int H, int KV, int hd, float scale, int splits, float* workspace,
                      void* out, long long out_stride, int dtype, dlti_stream_t stream);
/* temperature / top-k / top-p / greedy sampling, one CTA per sequence, counter-based RNG keyed by
 * (seeds[b], step); out_logprob may be NULL */
int dlti_sample(const void* logits, long long ld, int batch, int V, const float* temperature,
                const int* top_k, const float* top_p, const unsigned long long* seeds,
                unsigned long long step, long long* out, float* out_logprob, int dtype,
                dlti_stream_t stream);

/* ---- Layer-stack models (models/stack.py): csrc/stack.cu, streams.cu, recurrent.cu, attention_paged.cu, latent.cu, dyt.cu, prenorm.cu,
 * conv_qkv.cu, moe.cu, delta.cu, gemm_f32.cu. Row pitches (*_ld) in
 * elements. Sequences of a step: the first nd are single rows, sequence nd + i has rows nd + cu[i] ... nd + cu[i+1]; ctx[s] = tokens
 * of sequence s after the step, rseq[t] = sequence of row t, sslot[s] = its state slot (-1 = none). */
/* C[M,N] = A[M,K] * B[N,K]^T in true fp32 (no TF32) */
int dlti_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, long long lda, long long ldb, long
    long ldc, dlti_stream_t stream);
/* x[t] = table[ids[t]] as fp32; xa (16-bit, may be NULL) = the same rows */
int dlti_embed_rows(const long long* ids, const void* table, float* x, void* xa, long long xa_ld, long long tokens, int
    d, long long vocab, int dtype, dlti_stream_t stream);
/* out = scale * acc, cap > 0: cap * tanh(scale * acc / cap) (fp32 logits); clear: acc = 0, else out may be acc */
int dlti_take_rows(float* acc, float* out, float scale, float cap, int clear, long long rows, int cols, dlti_stream_t stream);
/* x += RMSnorm(y) * w (1 + w with one_plus), fp32 residual x [rows,d]; xa (may be NULL) = x in dtype.
 * acc: y is the fp32 accumulator of dlti_gemm_skinny, zero on return (also below) */
int dlti_post_norm_add(const void* y, long long y_ld, float* x, const float* w, void* xa, long long xa_ld, long long
    rows, int d, float eps, int one_plus, int acc, int dtype, dlti_stream_t stream);
/* out[i] = RMSnorm(x[idx[i]]) * w; idx NULL = all rows */
int dlti_rms_rows(const float* x, const long long* idx, const float* w, void* out, long long out_ld, long long rows,
    int d, float eps, int one_plus, int dtype, dlti_stream_t stream);
/* h = relu(x W^T)^2 in the epilogue of the CTA-pair GEMM (16-bit) */
int dlti_gemm_relu2_2cta(const void* X, const void* W, void* Hout, int M, int N, int K, long long ldx, long long ldw,
    long long ldh, int dtype, dlti_stream_t stream);
/* h = relu(u)^2 over the first ff columns */
int dlti_relu2(const void* u, long long u_ld, void* h, long long h_ld, long long rows, int ff, int acc, int dtype,
    dlti_stream_t stream);
/* norm over `groups` parts of a row. mode 0: norm(y) * w * sigmoid(gate), 1: norm(y * silu(gate)) * w, 2: norm(y) * w * silu(gate) */
int dlti_gated_norm(const void* y, long long y_ld, const void* gate, long long g_ld, const float* w, void* out, long
    long o_ld, long long rows, int n, int groups, float eps, int mode, int acc, int dtype, dlti_stream_t stream);
/* projection rows (sections at columns oq/ok/ov/og; ok, og < 0 = absent) -> normed and rotated q, k and v into the paged
 * cache at slots[t] (-1 = skip), sigmoid of the head gates. kp/vp: also packed k, v rows; dst: packed row of row t >= nd */
int dlti_qk_norm_rope_cache(const void* proj, long long ld, int oq, int ok, int ov, int og, const float* qn, const
    float* kn, float eps, const int* pos, const float* cos_t, const float* sin_t, int rot, int interleaved, const long
    long* slots, void* kc, void* vc, int kd, int vd, void* q, long long q_ld, int q_hd, void* kp, void* vp, const int*
    dst, int nd, float* gate, long long tokens, int H, int G, int dim, int vdim, int acc, int dtype, dlti_stream_t
    stream);
/* whole projection rows + bias -> q and k normed over all their heads, v mixed with `first` (share[0] of it); own = v before mixing. Null:
 * bias, qn and kn, first and share, own; kp, vp, dst as above */
int dlti_qkv_rows(const void* proj, long long ld, int oq, int ok, int ov, const float* bias, const float* qn, const float* kn, float eps,
    const void* first, long long f_ld, const float* share, void* own, long long own_ld, const long long* slots, void* kc, void* vc, int kd,
    int vd, void* q, long long q_ld, int q_hd, void* kp, void* vp, const int* dst, int nd, long long tokens, int H, int G, int dim, int vdim,
    int acc, int dtype, dlti_stream_t stream);
/* packed rows[i] <- zero queries, cached keys and values of slots[i] (portions that continue a chunk or a window) */
int dlti_prefix_rows(void* packed, long long ld, int hd, const int* rows, const int* slots, const void* kc, const void*
    vc, int kd, int vd, int H, int G, long long n, dlti_stream_t stream);
/* silu(causal convolution) of channels [col, col+C) of the rows of every sequence; inputs before the step come from state. acc: raw = the
 * accumulator's columns in dtype, from tail0 on (tail not null) in fp32 to tail */
int dlti_short_conv(const void* src, long long ld, int col, int C, int taps, const float* w, const float* b, int w_ld,
    const void* state, const int* sslot, const int* rseq, const int* ctx, const int* cu, int nd, void* out, long long
    o_ld, void* raw, long long raw_ld, int raw_n, float* tail, long long tail_ld, int tail0, long long rows, int acc, int dtype,
    dlti_stream_t stream);
/* S <- a S + k (s v)^T, o = S^T q + D v token by token over sequences [seq0, seq0+nseq); a constant (decay) or from raw step
 * sizes (dt, dt_bias, A_log); state [slots, heads, N, P] fp32; tail job: new convolution state from conv_src */
int dlti_linear_scan(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, int
    rep, int silu, const float* decay, const void* dt, long long dt_ld, const float* dt_bias, const float* A_log, const
    float* D, float* state, const int* sslot, const int* ctx, const int* cu, int nd, int seq0, int nseq, int heads, int
    N, int P, void* out, long long o_ld, const void* conv_src, long long conv_ld, int conv_col, int conv_rows, int
    conv_C, void* conv_state, int dtype, dlti_stream_t stream);
/* the same for prompt sequences, 64 tokens at a time on the tensor cores (bf16) */
int dlti_linear_scan_chunked(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long
    v_ld, int rep, const float* decay, const void* dt, long long dt_ld, const float* dt_bias, const float* A_log, const
    float* D, float* state, const int* sslot, const int* ctx, const int* cu, int nd, int seq0, int nseq, int heads, int
    N, int P, void* out, long long o_ld, const void* conv_src, long long conv_ld, int conv_col, int conv_rows, int
    conv_C, void* conv_state, dlti_stream_t stream);
/* x = silu(x) in place */
int dlti_silu_rows(void* x, long long ld, long long rows, int n, int dtype, dlti_stream_t stream);
/* paged attention, one warp per (row, head), fp32 arithmetic; chunk > 0: a position sees its own chunk only; window > 0: itself and the
 * window - 1 positions before it; cap > 0: scores become cap tanh(score / cap). sink [H] (may be NULL): one more term exp(sink) in a head's
 * softmax denominator; bias [H, span] (may be NULL): added to the scores at the distances below span; ogate [rows, H * vdim] (may be NULL):
 * outputs are multiplied by its sigmoid (all also below) */
int dlti_attn_rows(const void* q, long long q_ld, int q_hd, const void* kc, const void* vc, int kd, int vd, const int*
    tables, int max_blocks, int bs, const int* ctx, const int* rseq, const int* pos, int H, int G, int dim, int vdim,
    int chunk, int window, float scale, float cap, const float* gate, const float* sink, const float* bias, int span, const void* ogate,
    long long og_ld, void* out, long long o_ld, long long rows, int dtype,
    dlti_stream_t stream);
/* paged attention of prompt portions (bf16, heads <= 256) */
int dlti_attn_paged_prefill(const void* q, long long q_ld, int q_hd, const void* kc, const void* vc, int kd, int vd,
    const int* tables, int max_blocks, int bs, const int* ctx, const int* cu, int nd, int nseq, int max_rows, int H,
    int G, int dim, int vdim, int chunk, int window, float scale, float cap, const float* gate, const float* sink, const float* bias, int span,
    const void* ogate, long long og_ld, void* out, long long o_ld, dlti_stream_t stream);
/* paged attention of decode rows (bf16, grouped heads, split over CTAs); ws: batch * H * splits * (vdim + 2) floats */
int dlti_attn_paged_decode(const void* q, long long q_ld, int q_hd, const void* kc, const void* vc, int kd, int vd,
    const int* tables, int max_blocks, int bs, const int* ctx, int batch, int H, int G, int dim, int vdim, int chunk,
    int window, float scale, float cap, const float* gate, const float* sink, const float* bias, int span, const void* ogate, long long
    og_ld, int splits, float* ws, void* out, long long o_ld, dlti_stream_t stream);
/* varlen causal attention with the softmax weights as two bf16 terms; see attention.cu */
int dlti_attn_fwd_split(const void* qkv, void* out, long long ldo, const float* gate, const float* sink, const int* cu_seqlens, const int*
    seq_q0, const int* seq_out0, int batch, int max_seqlen, long long T_total, int H, int KV, int vdim, int window,
    float scale, float cap, const float* bias, int span, const void* ogate, long long og_ld, dlti_stream_t stream);

/* mLSTM: the recurrence above with exponential gates, a running maximum and a normaliser; see recurrent.cu. gates [rows, >= 2 heads]
 * raw fp32 (input, forget), vec [slots, heads, ceil(P / 32), N + 1] */
int dlti_mlstm_scan(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, const float* gates,
    long long g_ld, const float* gate_b, float cap, float q_scale, float* state, float* vec, const int* sslot, const int* ctx, const
    int* cu, int nd, int seq0, int nseq, int heads, int N, int P, void* out, long long o_ld, int chunked, int dtype, dlti_stream_t stream);
/* streams.cu. Hyper-connections between two sublayers: x_t <- sum_s mix[s,t] x_s + out[t] y on x [rows, S, d] (y may be NULL), then
 * h = layer_norm(sum_s in[s] x_s) * w (w may be NULL), then (cw, one token per sequence) plus its causal convolution */
int dlti_hyper(float* x, int S, int d, const void* y, long long y_ld, const float* mix, const float* out, const float* in, const float*
    w, float eps, const float* cw, int cw_ld, int taps, void* cstate, const int* sslot, const int* ctx, void* h, long long h_ld, const
    long long* idx, long long rows, int acc, int dtype, dlti_stream_t stream);
/* x[t, s] = table[ids[t]] * scale */
int dlti_embed_streams(const long long* ids, const void* table, float* x, long long tokens, int S, int d, long long vocab, float scale,
    int dtype, dlti_stream_t stream);
/* out = h + causal convolution of h; state [slots, taps - 1, d] is read and renewed */
int dlti_canon(const void* h, long long h_ld, int d, int taps, const float* w, int w_ld, void* state, const int* sslot, const int* ctx,
    const int* cu, int nd, int seq0, int nseq, int max_rows, void* out, long long o_ld, int dtype, dlti_stream_t stream);
/* out = a N(z) + b N(z^2) + c N(z^3) + e, N(y) = y / rms(y); coef = {a, b, c, e} */
int dlti_poly_norm(const void* z, long long z_ld, const float* coef, void* out, long long o_ld, long long rows, int n, float eps, int
    acc, int dtype, dlti_stream_t stream);
/* accumulator columns [0, split) as dtype, the rest as fp32; the accumulator becomes zero */
int dlti_split_rows(float* acc, void* out, long long o_ld, float* tail, long long t_ld, long long rows, int n, int split, int dtype,
    dlti_stream_t stream);
/* latent.cu: latent attention. A cache row is [c, zeros, k_rot, zeros], rot_at = round16(rank), pitch = rot_at + round16(rot) + 8 */
int dlti_latent_prep(const void* proj, long long ld, int oq, int od, int og, int H, int dim, int rot, int rank, int rd, int interleaved,
    const float* cos_t, const float* sin_t, const int* pos, const float* kvw, float eps, const long long* slots, void* cache, int
    pitch, int rot_at, int nabs, void* qn, int qn_hd, void* ql, void* qp, long long qp_ld, int qp_hd, void* lat, const int* qdst, const int* dst,
    float* gate, long long tokens, int acc, int dtype, dlti_stream_t stream);
/* lat[rows[i]] = cache[slots[i]] */
int dlti_latent_rows(void* lat, const void* cache, int pitch, const int* rows, const int* slots, long long n, dlti_stream_t stream);
/* out[t, h] = a[t, h] B_h, B_h = K rows of b [H*K, N] (kn) or the transpose of N rows of b [H*N, K] */
int dlti_head_gemm(const void* a, long long a_ld, int a_hd, const void* b, long long b_ld, void* out, long long o_ld, int o_hd, long long
    rows, int H, int K, int N, int kn, int dtype, dlti_stream_t stream);
/* absorbed latent attention (bf16): q [rows, H, pitch] against the cached rows, values = their first rank columns */
int dlti_latent_decode(const void* q, const void* cache, int pitch, int rank, const int* tables, int max_blocks, int bs, const int* ctx,
    const int* rseq, const int* pos, long long rows, int H, float scale, const float* sink, const float* gate, int heads_per_cta, int
    splits, float* ws, void* out, int o_hd, dlti_stream_t stream);

/* dyt.cu: dynamic tanh norms n(x) = tanh(alpha x) * w + b around sublayers. x = table[ids] * scale (fp32), h = n(x) */
int dlti_tanh_embed(const long long* ids, const void* table, long long vocab, float scale, const float* alpha, const float* w, const float*
    b, float* x, void* h, long long h_ld, long long tokens, int d, int dtype, dlti_stream_t stream);
/* x += n1(y + sum_k weights[t, k] rows[t * top + k]), h = n2(x); y, rows (weights, counts), w2 (h) may be NULL; counts are cleared */
int dlti_tanh_between(float* x, const void* y, long long y_ld, const void* rows, long long r_ld, const float* weights, int top, int* counts,
    int ncounts, const float* alpha1, const float* w1, const float* b1, const float* alpha2, const float* w2, const float* b2, void* h,
    long long h_ld, long long tokens, int d, int acc, int dtype, dlti_stream_t stream);
/* h[i] = n(x[idx[i]]); idx NULL = all rows */
int dlti_tanh_rows(const float* x, const long long* idx, const float* alpha, const float* w, const float* b, void* h, long long h_ld, long
    long rows, int d, int dtype, dlti_stream_t stream);
/* prenorm.cu: x (zero if fresh) += mult * (y * share[t] + sum_k weights[t, k] rows[t * top + k]), with post: mult * RMSnorm(that) * post; x +=
 * scale * table[ids[t]]; h = RMSnorm(x) * pre (pre NULL: x). All but x may be NULL; counts are cleared */
int dlti_prenorm_between(float* x, const void* y, long long y_ld, const void* rows, long long r_ld, const float* weights, int top, const float*
    share, int* counts, int ncounts, float mult, const float* post, const long long* ids, const void* table, long long vocab, float scale, int
    fresh, const float* pre, void* h, long long h_ld, long long tokens, int d, float eps, int acc, int dtype, dlti_stream_t stream);
/* h[t, c] = gelu_tanh(u[t, c]) * table[ids[t], col + c], c < n */
int dlti_token_gate(const void* u, long long u_ld, const long long* ids, const void* table, long long t_ld, long long vocab, int col, int n,
    void* h, long long h_ld, long long tokens, int acc, int dtype, dlti_stream_t stream);
/* conv_qkv.cu: projection rows -> causal convolution (w tap-major by column, NULL: none; state [slots, taps - 1, C] is read and renewed), per-head
 * RMS norms of q and k, q times factors[pos[t]]; k and v into the paged cache at slots[t]; kp, vp, dst as in dlti_qk_norm_rope_cache. acc: also
 * gate = columns from og on */
int dlti_conv_qkv(const void* proj, long long ld, int oq, int ok, int ov, int og, const float* w, int taps, int w_ld, void* state, int C, const
    int* sslot, const int* rseq, const int* ctx, const int* cu, int nd, int nseq, const float* qn, const float* kn, float eps, const float* factors,
    const int* pos, const long long* slots, void* kc, void* vc, int kd, int vd, void* q, long long q_ld, int q_hd, void* kp, void* vp, const int*
    dst, void* gate, long long g_ld, long long tokens, int H, int G, int dim, int vdim, int acc, int dtype, dlti_stream_t stream);
/* moe.cu: routing of the logits z (E > 0): sigmoid scores, groups, the top experts by score + corr, their scores made to sum to scale
 * (softmax: the top experts by logit + corr, scale times their softmax); share (sg >= 0) = sigmoid of column sg;
 * wgt [T, top] and, per expert, the list of its pairs token * top + choice (lists [E, T], counts [E] zero on entry); and / or (ff > 0)
 * the gated activation of projection columns og (gate) and ou (up): silu(g) u, with a limit g sigmoid(1.702 g) (u + 1) of clipped values;
 * og < 0: square of relu(u) */
int dlti_moe_route(const float* z, long long z_ld, int col, const float* corr, int E, int top, int groups, int keep, float scale, int softmax,
    float* wgt, int* lists, int* counts, int sg, float* share, const void* p, long long p_ld, int og, int ou, int ff, float limit, void* h, long long h_ld, long long T, int acc,
    int dtype, dlti_stream_t stream);
/* grouped GEMM over the lists. up: rows X[pair / div] times W_e, out = activation, one list after the other (1: of gate / up rows 2 r, 2 r + 1,
 * 2: square of relu of row r); else rows of X in that order times W_e, out[pair]. W_e = rows e * wrows ... of W */
int dlti_moe_gemm(const void* X, long long x_ld, long long x_rows, int div, const void* W, long long w_ld, int wrows, int E, const int* lists,
    const int* counts, int cap, int rows, int up, int K, float limit, void* out, long long o_ld, int o_rows, int dtype, dlti_stream_t stream);
/* delta.cu: gated delta rule S <- g S, u = b (v - S^T k), S <- S + k u^T, o = S^T q over sequences [seq0, seq0+nseq); gates [rows, >= 2
 * heads] raw fp32 (decay, step). ws NULL: token by token; else prompts in chunks of 64 tokens (bf16) with dlti_delta_workspace bytes */
int dlti_delta_scan(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, const float* gates, long
    long g_ld, const float* A_log, const float* dt_bias, float* state, const int* sslot, const int* ctx, const int* cu, int nd, int seq0, int
    nseq, int heads, int groups, int N, int P, void* out, long long o_ld, const void* conv_src, long long conv_ld, int conv_col, int
    conv_rows, int conv_C, void* conv_state, void* ws, int longest, int dtype, dlti_stream_t stream);
long long dlti_delta_workspace(long long rows, int nseq, int heads);

#ifdef DLTI_ATTN_TRACE
/* Developer builds only (-DDLTI_ATTN_TRACE): clock64() timeline of CTA (0,0,0) of the last backward
 * kernels, [dQ | dK/dV][role: softmax, mma, producer][iteration < 64][event < 4]. */
int dlti_attn_trace_read(long long* host_out);
#endif

/* ---- libdlti_cpu.so: shared-memory control ring for the tensor-parallel workers of one node (no
 * counterpart in the reference, which ships no serving code; vLLM's shm_broadcast queue plays this role there).
 * One writer (reader < 0 creates the ring), up to 16 readers, every reader sees every message in order. */
void* dlti_shm_ring_open(const char* name, int reader, int n_readers, int n_slots, int slot_bytes);
int dlti_shm_ring_write(void* ring, const void* data, long long nbytes, int timeout_ms);
long long dlti_shm_ring_read(void* ring, void* out, long long capacity, int timeout_ms);
void dlti_shm_ring_close(void* ring);

#ifdef __cplusplus
}
#endif
#endif /* DLTI_B200_H_ */
