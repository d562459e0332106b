/*
 * energon_b200 — C ABI of the B200 (sm_100a) implementation of EnergonAI's tensor-parallel
 * transformer layer forward.
 *
 * Conventions (all entry points):
 *   - plain pointers and sizes only; every tensor is allocated by the caller and must be
 *     device memory of the current CUDA device, contiguous in the stated layout;
 *   - `dtype` is one of EB_F32 / EB_F16 / EB_BF16;
 *   - `stream` is a cudaStream_t passed as void* (NULL = the legacy default stream); all work
 *     is enqueued on it, nothing synchronises the device;
 *   - the return value is EB_OK or a negative EB_E* code; on failure eb_last_error() returns
 *     a thread-local human-readable message.  Nothing throws, exits or prints.
 *
 * Each declaration cites the reference interface it replaces (path inside the EnergonAI
 * repository : line).
 */
#ifndef ENERGON_B200_H
#define ENERGON_B200_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#if defined(__GNUC__)
#define EB_API __attribute__((visibility("default")))
#else
#define EB_API
#endif

#define EB_OK 0
#define EB_EINVAL (-1)       /* bad argument (null pointer, size, alignment, dtype)          */
#define EB_ECUDA (-2)        /* the CUDA runtime / driver reported an error at launch        */
#define EB_EUNSUPPORTED (-3) /* valid request outside what the kernels implement            */
#define EB_ETIMEDOUT (-4)    /* a bounded device-side wait expired (see eb_device_status)    */
#define EB_ELIMIT (-5)       /* request exceeds a documented fixed capacity                 */

#define EB_F32 0
#define EB_F16 1
#define EB_BF16 2

/* activation codes for eb_gemm */
#define EB_ACT_NONE 0
#define EB_ACT_RELU 1
#define EB_ACT_GELU_TANH 2 /* energonai/model/model_factory.py:32-35 (gelu_impl)            */
#define EB_ACT_GELU_ERF 3  /* torch.nn.functional.gelu                                      */
#define EB_ACT_XIELU 4     /* eb_gemm_parts, eb_gemm_f32                                    */

/* units of a feed-forward, fp32 on the accumulators.  The gated ones read columns in blocks of 8 gates g
 * and their 8 ups u and give half as many:
 *   CLAMPED  g' sigmoid(alpha g') (u' + 1), g' = min(g, limit), u' = clamp(u, -limit, limit)
 *   GEGLU    gelu_tanh(g) u
 *   GELU     gelu(x) of every column, the erf form (no gate) */
#define EB_UNIT_NONE 0
#define EB_UNIT_CLAMPED 1
#define EB_UNIT_GEGLU 2
#define EB_UNIT_GELU 3

/* flags for eb_gemm */
#define EB_GEMM_STATIC_W 1 /* W is constant (model weights): the kernel may start reading it while
                              earlier work of the stream is still running */

/* flags for eb_scale_mask_softmax */
#define EB_SM_CAUSAL 1  /* keys j > query i are masked to exactly 0 (reference behaviour)    */
#define EB_SM_KEYLEN 2  /* keys j >= real_seq_len[b] are masked to exactly 0                 */
#define EB_SM_ALLROWS 4 /* also rewrite query rows i >= real_seq_len[b] (reference skips them) */

EB_API int eb_version(void);
EB_API const char *eb_last_error(void);

/* ---- padding offsets and (un)padding copies ------------------------------------------ */

/* Replaces ft_build_padding_offsets_wrapper
 * (energonai/kernel/cuda_native/csrc/transpose_pad_fusion_wrapper.cpp:93-104, kernel
 * transpose_pad_fusion_kernel.cu:112-131).  seq_lens[batch] (each 0..max_seq_len);
 * valid_word_num[0] = sum of lengths; tmp_mask_offset[k], k < sum, = number of padding slots
 * before valid token k in the [batch, max_seq_len] layout.  tmp_mask_offset must hold at
 * least sum(seq_lens) entries (batch*max_seq_len always suffices).  Entries beyond the sum
 * are not written. */
EB_API int eb_build_padding_offsets(const int32_t *seq_lens, int batch, int max_seq_len, int32_t *valid_word_num,
                             int32_t *tmp_mask_offset, void *stream);

/* Replaces ft_remove_padding_wrapper (transpose_pad_fusion_wrapper.cpp:113-140, kernel
 * transpose_pad_fusion_kernel.cu:142-155): tgt[k,:] = src[k + off[k],:] for k < valid, and
 * mask_offset[k] = tmp_mask_offset[k].  src [batch*max_seq_len, n], tgt [valid, n]. */
EB_API int eb_remove_padding(const void *src, void *tgt, const int32_t *tmp_mask_offset, int32_t *mask_offset, int valid,
                      int n, int dtype, void *stream);

/* Replaces ft_rebuild_padding_wrapper (transpose_pad_fusion_wrapper.cpp:147-172, kernel
 * transpose_pad_fusion_kernel.cu:178-190): tgt[k + off[k],:] = src[k,:].  The reference
 * scatters into a freshly zeroed tensor; here the same kernel writes the zero rows
 * (zero_fill != 0), so tgt [batch*max_seq_len, n] may be uninitialised memory. */
EB_API int eb_rebuild_padding(const void *src, void *tgt, const int32_t *mask_offset, int valid, int n, int batch,
                       int max_seq_len, int dtype, int zero_fill, void *stream);

/* Replaces ft_transpose_rebuild_padding_wrapper (transpose_pad_fusion_wrapper.cpp:181-209,
 * kernel transpose_pad_fusion_kernel.cu:213-236): packed Q,K,V [valid, head_num,
 * size_per_head] -> q_buf,k_buf,v_buf [batch, head_num, seq_len, size_per_head].  With
 * zero_fill == 0 rows of padding tokens are left untouched, as in the reference (whose
 * callers pre-zero the buffers); with zero_fill != 0 they are written as zeros. */
EB_API int eb_transpose_rebuild_padding(const void *Q, const void *K, const void *V, void *q_buf, void *k_buf, void *v_buf,
                                 int batch, int seq_len, int head_num, int size_per_head, int valid,
                                 const int32_t *mask_offset, int dtype, int zero_fill, void *stream);

/* Replaces ft_transpose_remove_padding_wrapper (transpose_pad_fusion_wrapper.cpp:218-244,
 * kernel transpose_pad_fusion_kernel.cu:268-289): src [batch, head_num, seq_len,
 * size_per_head] -> dst [valid, head_num*size_per_head]. */
EB_API int eb_transpose_remove_padding(const void *src, void *dst, int valid, int batch, int seq_len, int head_num,
                                int size_per_head, const int32_t *mask_offset, int dtype, void *stream);

/* Replaces transpose_pad_wrapper (transpose_pad_fusion_wrapper.cpp:33-57, kernel
 * transpose_pad_fusion_kernel.cu:58-84): packed src [sum_len, head_num, size_per_head] ->
 * dst [batch, head_num, max_seq_len, size_per_head], zeros where position >= seq_lens[b]. */
EB_API int eb_transpose_pad(const void *src, void *dst, int batch, int max_seq_len, const int32_t *seq_lens, int head_num,
                     int size_per_head, int dtype, void *stream);

/* Replaces transpose_depad_wrapper (transpose_pad_fusion_wrapper.cpp:59-83, kernel
 * transpose_pad_fusion_kernel.cu:8-35): src [batch, head_num, max_seq_len, size_per_head] ->
 * dst [sum_seq, head_num, size_per_head]; rows of dst beyond sum(seq_lens) are zeroed. */
EB_API int eb_transpose_depad(const void *src, void *dst, int batch, int sum_seq, int max_seq_len, const int32_t *seq_lens,
                       int head_num, int size_per_head, int dtype, void *stream);

/* ---- scale-mask-softmax ----------------------------------------------------------------- */

/* Replaces scale_mask_softmax_wrapper (csrc/scale_mask_softmax_wrapper.cpp:25-44, kernel
 * scale_mask_softmax_kernel.cu:12-42).  In place over scores [batch, head_num, seq_len,
 * seq_len].  Reference behaviour = flags EB_SM_CAUSAL, scale 1.0f: rows i < real_seq_len[b]
 * become softmax over keys j <= i with keys j > i set to 0, other rows are untouched.  The
 * scores are multiplied by `scale` before the softmax.  No limit on seq_len (the reference
 * stops at 1024).  dtype F32, F16 or BF16. */
EB_API int eb_scale_mask_softmax(void *scores, const int32_t *real_seq_len, int batch, int seq_len, int head_num, int dtype,
                          int flags, float scale, void *stream);

/* ---- LayerNorm forward -------------------------------------------------------------------- */

/* Replaces forward_affine (csrc/layer_norm_cuda.cpp:82-103, kernel
 * layer_norm_cuda_kernel.cu:243-279) and the LayerNorm1D modules of the block
 * (energonai/model/endecoder.py:28,39).  Rows n1, row length n2.
 *   t   = x (+ residual) (+ bias[n2])            (optional operands may be NULL)
 *   with residual or bias, t is rounded to in_dtype first (what a residual stream stores);
 *   sum_out = t (in in_dtype), if sum_out != NULL
 *   y   = gamma * (t - mean) * invvar + beta     (gamma/beta NULL: no affine)
 *   mean[n1], invvar[n1] fp32, if non-NULL.
 * Statistics in fp32 over a register-resident row (one pass over the row shifted by its first
 * element), biased variance. */
EB_API int eb_layer_norm_fwd(void *y, float *mean, float *invvar, const void *x, const void *residual, const void *bias,
                      void *sum_out, const void *gamma, const void *beta, int64_t n1, int n2, double eps, int in_dtype,
                      int out_dtype, void *stream);

/* ---- tensor-parallel exchange context --------------------------------------------------------
 *
 * One eb_comm per rank of a tensor-parallel group (one process per GPU).  It takes the place of
 * what the reference obtains from colossalai.launch (energonai/worker.py:27-28: the NCCL
 * process groups) and of its unbuilt NCCL-id helper
 * (energonai/kernel/cuda_native/csrc/get_ncclid.cpp:104-127), for the exchanges this library
 * performs itself: the all-reduce of the row-parallel layers (colossalai's Linear1D_Row,
 * constructed at energonai/model/attention.py:37 and energonai/model/mlp.py:22).
 *
 * Each rank owns a receive area its peers write into over NVLink with plain stores.  Set-up:
 *   eb_comm_create(rank, world, line_bytes, bulk_bytes, NULL, &c)   allocates and zeroes the local area
 *   eb_comm_export_handle(c, blob, n)                        n = eb_comm_handle_bytes()
 *   ... the caller gathers every rank's blob with its own process group, in rank order ...
 *   eb_comm_connect(c, all_blobs, world * n)                 maps the peers' areas (CUDA IPC)
 *   ... a barrier of the caller's: nobody exchanges before everybody is connected ...
 * A caller that maps peer memory itself (one process driving several GPUs, or another symmetric
 * allocator) passes its own area (eb_comm_area_bytes(line_bytes, bulk_bytes) bytes, zero-filled)
 * as recv_local and the peers' addresses to eb_comm_connect_pointers instead.  An area has two
 * regions.  The flagged-line region (line_bytes) carries generation-step exchanges:
 * eb_comm_exchange_bytes(world, rows, cols) bytes per HALF of it for a [rows, cols] 16-bit
 * matrix (data travels with a sequence number beside every 4 bytes, so it takes twice its size).
 * The bulk region (bulk_bytes, may be 0) carries prompt-sized tensors as plain data: the staging
 * and gather areas of eb_gemm_reduce_scatter / eb_reduce_broadcast, at offsets the caller
 * chooses; eb_comm_local_area returns its local address so that results can be read in place.
 * All ranks must issue the same exchanges in the same order.  A wait on a peer that lasts longer
 * than the budget (5 s unless changed) is abandoned: the kernel records EB_ETIMEDOUT in the
 * context (eb_comm_status) or in the device status word (eb_device_status), its result is then
 * unspecified and the ranks' sequence numbers no longer agree: tear the group down.  One host
 * thread at a time per context; exchanges sharing a context must not overlap on the device. */
typedef struct eb_comm eb_comm;
EB_API size_t eb_comm_handle_bytes(void);
EB_API size_t eb_comm_exchange_bytes(int world, int rows, int cols);
EB_API int eb_comm_create(int rank, int world, size_t line_bytes, size_t bulk_bytes, void *recv_local, eb_comm **out);
EB_API size_t eb_comm_area_bytes(size_t line_bytes, size_t bulk_bytes);
EB_API int eb_comm_local_area(eb_comm *comm, void **bulk_ptr, size_t *bulk_bytes);
EB_API int eb_comm_export_handle(const eb_comm *comm, void *blob, size_t blob_bytes);
EB_API int eb_comm_connect(eb_comm *comm, const void *all_blobs, size_t all_blobs_bytes);
EB_API int eb_comm_connect_pointers(eb_comm *comm, void *const *peer_recv);
EB_API int eb_comm_set_wait_budget(eb_comm *comm, double seconds);
EB_API int eb_comm_status(eb_comm *comm, int *out4, int clear);
EB_API int eb_comm_destroy(eb_comm *comm);

/* All-reduce of a prompt-sized row-parallel product in two launches, replacing "F.linear, then
 * dist.all_reduce, then + bias" of colossalai's Linear1D_Row for M > 128 rows (the layers
 * constructed at energonai/model/attention.py:37 and energonai/model/mlp.py:22, called with the
 * whole prompt at attention.py:127-128 and mlp.py:35).
 *   eb_gemm_reduce_scatter: A [M,K] . W [N,K]^T (this rank's column shard of the weight) on the
 *     tensor cores; every finished 128-row tile is stored, in the operand type, straight into
 *     the staging area of the rank that owns those rows (bulk region + stage_offset of that
 *     rank, over NVLink, 128-byte row segments), so the reduce-scatter half of the all-reduce
 *     travels while the product is still being computed.  Rows are dealt out in `world`
 *     contiguous blocks of whole 128-row tiles.
 *   eb_reduce_broadcast: after a barrier over the ranks, each rank adds the `world` partials of
 *     its own rows in fp32, in rank order, + bias + residual (rows ldr apart, may be NULL),
 *     rounds to the operand type and stores the finished rows into the gather area (bulk region
 *     + gather_offset, [M][N]) of every rank; a second barrier ends the kernel, after which
 *     every rank reads the complete [M, N] sum at its own eb_comm_local_area + gather_offset.
 * The staging area takes eb_reduce_broadcast_stage_bytes(world, M, N) bytes, the gather area
 * M*N*2; offsets are multiples of 256 and the two must not overlap, nor be reused while a peer
 * may still read them (alternate two gather areas between consecutive calls).  Waits are
 * bounded (eb_comm_status).  N a multiple of 8, fp16 / bf16. */
EB_API int eb_gemm_reduce_scatter(const void *A, long long lda, const void *W, long long ldw, int M, int N, int K, int dtype,
                           int flags, eb_comm *comm, size_t stage_offset, void *stream);
EB_API int eb_reduce_broadcast(eb_comm *comm, long long M, int N, int dtype, size_t stage_offset, size_t gather_offset,
                        const void *bias, const void *residual, long long ldr, void *stream);
EB_API size_t eb_reduce_broadcast_stage_bytes(int world, long long M, int N);

/* In-place SUM of buf[count] (dtype fp32 / fp16 / bf16, sums formed in fp32 in rank order, so
 * every rank holds the bit-identical result) over the ranks of `comm`: each rank stores its
 * buffer into every rank's receive area and adds up what it received ("one-shot": one NVLink
 * crossing, meant for the kilobyte-to-megabyte messages of generation steps; NCCL remains the
 * tool for prompt-sized tensors).  buf 8-byte aligned, count * size a multiple of 8 bytes,
 * world * count * size * 2 <= line_bytes / 2.  Replaces dist.all_reduce inside Linear1D_Row. */
EB_API int eb_allreduce(eb_comm *comm, void *buf, size_t count, int dtype, void *stream);

/* ---- dense layers (tcgen05 tensor-core GEMM) --------------------------------------------- */

/* C = act(A . W^T + bias) + residual, fp32 accumulation in tensor memory.
 * Replaces the F.linear inside the column-parallel and row-parallel layers the reference
 * builds from colossalai (Linear1D_Col / Linear1D_Row, constructed at
 * energonai/model/attention.py:29-37 and energonai/model/mlp.py:20-22) and mlp_gemm
 * (energonai/kernel/cuda_native/csrc/linear_wrapper.cpp:82-111).
 *   A [M,K] rows lda apart, W [N,K] rows ldw apart (both fp16 or both bf16, `dtype`);
 *   C [M,N] in `out_dtype` (= dtype, or EB_F32); bias [N] (dtype) or NULL; residual [M,N]
 *   rows ldr apart (dtype) or NULL; act one of EB_ACT_*.
 *   Row m of C starts at element m*ldc, or, when c_rows_per_batch > 0, at
 *   (m / c_rows_per_batch)*c_batch_stride + (m % c_rows_per_batch)*ldc  (this lets a
 *   projection write straight into a [batch, max_len, width] cache at a position offset).
 *   c_row_offset_device, if non-NULL, is a device int32 read by the kernel: that many further
 *   rows (of ldc elements) are added to every row's offset, so a captured launch can append
 *   at a position that advances between replays.  c_row_offset_limit > 0 bounds it: a device
 *   value outside [0, limit) stores nothing and records EB_ELIMIT in the device status word
 *   (the caller's buffer was not sized for that position).
 *   K must be a multiple of 8 and pointers 16-byte aligned; for M > 128 also N, all leading
 *   dimensions and c_batch_stride (for M <= 128 the output is written element by element).
 * The kernel is launched so that it may begin before the preceding kernel of the stream has
 * finished; it reads A, bias and residual only after that kernel completed, and W too unless
 * flags has EB_GEMM_STATIC_W.
 * For M <= 32 (generation steps; up to 128 where the output's strides are not multiples of 8) the
 * kernel streams W exactly once, split evenly over all SMs
 * (stream-K over 128-row tiles; a K of at most 1280 is not cut, one CTA per tile), and combines
 * the partial sums of tiles shared by several CTAs
 * through `workspace`: at least eb_gemm_workspace_bytes(M,N,K) bytes, 16-byte aligned,
 * zero-filled once before first use (the kernel leaves it reusable; summation order is fixed,
 * results are deterministic).  Calls that share a workspace must not overlap on the device.
 * workspace may be NULL for M > 128. */
EB_API int eb_gemm(const void *A, long long lda, const void *W, long long ldw, void *C, long long ldc, const void *bias,
            const void *residual, long long ldr, int M, int N, int K, int dtype, int out_dtype, int act,
            int c_rows_per_batch, long long c_batch_stride, const int32_t *c_row_offset_device,
            int c_row_offset_limit, int flags, void *workspace, size_t workspace_bytes, void *stream);
EB_API size_t eb_gemm_workspace_bytes(int M, int N, int K);

/* eb_gemm (no residual, plain rows) for several things at once that read the same A, their weights
 * stacked in W.  act_params (or NULL): xIELU on the columns below act_cols, a multiple of 8; device floats
 * (softplus(p), 1/2 + softplus(q)) of
 *   z > 0: softplus(p) z^2 + z/2;   z <= 0: (1/2 + softplus(q)) (exp(z) - 1 - z) + z/2.
 * tail (or NULL): the columns from tail_col on, a multiple of 8, go there in fp32, rows ld_tail apart;
 * C then holds the tail_col columns before them.  bias [N] or NULL. */
EB_API int eb_gemm_parts(const void *A, long long lda, const void *W, long long ldw, void *C, long long ldc, const void *bias,
                  int M, int N, int K, int act_cols, const float *act_params, int tail_col, float *tail, long long ld_tail,
                  int dtype, int flags, void *workspace, size_t workspace_bytes, void *stream);

/* Row-parallel GEMM with the tensor-parallel all-reduce fused into its epilogue, for the
 * generation orientation (M <= 128).  Replaces "F.linear, then dist.all_reduce, then + bias" of
 * colossalai's Linear1D_Row (the row-parallel layers constructed at
 * energonai/model/attention.py:37 and energonai/model/mlp.py:22).  Arguments as eb_gemm, plus the
 * exchange context.  The thread that completes the batch values of an output column stores them
 * (rounded to the operand type, as an all-reduce of the product would see them) into every
 * rank's receive area over NVLink, then adds up what all ranks sent it, in rank order, so every
 * rank obtains the bit-identical result; bias, activation and residual are applied after the
 * sum on every rank.  One launch = one exchange of the context (see eb_comm above):
 * eb_comm_exchange_bytes(world, M rounded up to 16 / 32 / 64 / 128, N) must fit half of the
 * receive area, N must be a multiple of 4.  A context of one rank exchanges with itself (same result
 * as eb_gemm up to the rounding of the product to the operand type). */
EB_API int eb_gemm_allreduce(const void *A, long long lda, const void *W, long long ldw, void *C, long long ldc,
                      const void *bias, const void *residual, long long ldr, int M, int N, int K, int dtype,
                      int out_dtype, int act, int c_rows_per_batch, long long c_batch_stride,
                      const int32_t *c_row_offset_device, int c_row_offset_limit, int flags, void *workspace,
                      size_t workspace_bytes, eb_comm *comm, void *stream);

/* eb_gemm for M <= 32 rows with a LayerNorm folded in (generation steps): A holds the
 * UN-normalised rows x [M, K] and W the weights already multiplied by the LayerNorm scale,
 * W'[n][k] = W[n][k] * gamma[k], rounded to the operand type.  The kernel computes each row's
 * mean and 1/sqrt(var + eps) over the K columns (fp32, as eb_layer_norm_fwd does) and evaluates
 *   C[m][n] = act( rstd[m] * (sum_k x[m][k] W'[n][k] - mean[m] * ln_colsum[n]) + ln_bias[n] ) + residual[m][n]
 * with ln_colsum[n] = sum_k W'[n][k] and ln_bias[n] = bias[n] + sum_k W[n][k] * beta[k], both fp32
 * device vectors prepared once by the caller.  This is LayerNorm (energonai/model/endecoder.py:52,
 * 63) followed by the column-parallel projection (attention.py:73-80, mlp.py:38) in one launch,
 * without rounding the normalised activations to the operand type in between; K must be the
 * whole normalised width.  Other arguments, workspace and errors as eb_gemm. */
EB_API int eb_gemm_ln(const void *A, long long lda, const void *W, long long ldw, void *C, long long ldc,
               const float *ln_colsum, const float *ln_bias, double eps, const void *residual, long long ldr,
               int M, int N, int K, int dtype, int out_dtype, int act, int c_rows_per_batch,
               long long c_batch_stride, const int32_t *c_row_offset_device, int c_row_offset_limit, int flags,
               void *workspace, size_t workspace_bytes, void *stream);

/* ---- a chain of generation-step operations in one launch ----------------------------------- */

#define EB_OP_GEMM 0
#define EB_OP_LAYERNORM 1
#define EB_OP_REDUCE_LAYERNORM 2

/* One operation of eb_decode_chain.
 * EB_OP_GEMM: C = act(A . W^T + bias) + residual with the fields of eb_gemm (A [M,K], W [N,K],
 *   static weights).  With `exchange` != 0 the product is this rank's part of a row-parallel
 *   layer: it is not stored but sent to every rank of the chain's context (bias, residual and
 *   act must be unset, C is unused), and the next operation must be EB_OP_REDUCE_LAYERNORM.
 * EB_OP_LAYERNORM: y = gamma * norm(x) + beta over M rows of n2 elements (x, y, gamma, beta in
 *   the chain's dtype).
 * EB_OP_REDUCE_LAYERNORM: t = (sum over ranks of the preceding exchanged product) + bias +
 *   residual, rounded to the chain's dtype and written to C (rows ldc apart); then
 *   y = gamma * norm(t) + beta (gamma NULL: no normalisation).  This is the all-reduce, bias and
 *   skip connection of Linear1D_Row followed by the LayerNorm of the next sub-layer
 *   (energonai/model/endecoder.py:56-63).  n2 = the product's N. */
typedef struct eb_chain_op {
  int type;
  const void *A; long long lda; const void *W; long long ldw; void *C; long long ldc;
  const void *bias; const void *residual; long long ldr;
  int N, K, out_dtype, act, c_rows_per_batch;
  long long c_batch_stride;
  const int32_t *c_row_offset_device;
  int c_row_offset_limit;
  int exchange;
  const void *x; void *y; const void *gamma; const void *beta;
  int n2;
  double eps;
} eb_chain_op;

/* Runs up to 8 dependent operations (each consumes the previous one's complete output) of a
 * generation step, M <= 128 rows, as ONE persistent kernel: e.g. the tail of a decoder layer
 * (energonai/model/endecoder.py:48-70) out-proj -> norm2 -> FC1 -> FC2 -> next layer's norm1 ->
 * next layer's QKV projection.  Between operations the grid synchronises through arrival
 * counters in `workspace`, while the weights of the following GEMM keep streaming into shared
 * memory (weights must be static: nobody may be writing them).  Results are identical to
 * running eb_gemm / eb_layer_norm_fwd one after the other.  Buffers written by an operation
 * must not alias anything an earlier operation of the same chain reads.  `workspace`:
 * eb_decode_chain_workspace_bytes(...) bytes, 16-byte aligned, zero-filled once before first
 * use; launches sharing it must not overlap on the device.  All grid-wide waits are bounded
 * (1 s, eb_device_status).  The kernel needs every SM to host one of its CTAs at the same time:
 * do not run it concurrently with other work that pins shared memory on the device.
 * `comm` (NULL unless an operation exchanges): the tensor-parallel context; a launch performs
 * as many exchanges of it as it has exchanged products, and while the grid waits for the other
 * ranks' parts the weights of the following GEMM keep arriving, so the NVLink flight and the
 * ranks' skew hide under the weight stream. */
EB_API int eb_decode_chain(const eb_chain_op *ops, int n_ops, int M, int dtype, void *workspace,
                    size_t workspace_bytes, eb_comm *comm, void *stream);
EB_API size_t eb_decode_chain_workspace_bytes(const eb_chain_op *ops, int n_ops, int M);

/* ---- products of a mixture of experts, 32-bit products ---------------------------------------- */

/* The prompt-orientation GEMM with several groups of weights: row tile i of A (128 rows) is
 * multiplied by the weights of group tile_group[i].  W holds the groups' [N, K] matrices one below
 * the other ([groups * N, K], rows ldw apart); only the first *live_tiles row tiles are processed
 * (both device memory, read at run time).  M, a multiple of 128, is the room A and C have.
 * unit: EB_UNIT_* (a gated one: C is [M, N/2]).  fp16 / bf16. */
EB_API int eb_gemm_grouped(const void *A, long long lda, const void *W, long long ldw, void *C, long long ldc, int M, int N, int K,
                    int groups, const int32_t *tile_group, const int32_t *live_tiles, int unit, float limit, float alpha,
                    int dtype, void *stream);

/* C = gated unit of (A . W^T), W [N, K] in blocks of 8 gate rows and their 8 up rows, C [M, N/2]: eb_gemm with a
 * gated unit, in both orientations (workspace as eb_gemm). */
EB_API int eb_gemm_gated(const void *A, long long lda, const void *W, long long ldw, void *C, long long ldc, int M, int N, int K, int unit,
                  float limit, float alpha, int dtype, int flags, void *workspace, size_t workspace_bytes, void *stream);

/* The same kind of product for a handful of rows per group (generation steps), as one pass over
 * the weights of the groups that have rows.  idx != NULL: entry i of the list (rows entries)
 * belongs to group idx[i] (negative: none), reads row i / a_div of A and writes row i of C.  idx
 * NULL: every group takes all rows, with group strides on A and C (heads of an absorbed attention
 * projection).  Strides in elements; unit as above. */
EB_API int eb_grouped_skinny(const void *A, long long lda, long long a_group_stride, int a_div, const void *W,
                      long long w_group_stride, long long ldw, void *C, long long ldc, long long c_group_stride,
                      const int32_t *idx, int rows, int groups, int N, int K, int unit, float limit, float alpha, int dtype,
                      void *stream);

/* C = A . W^T in true 32-bit.  Strided groups, or row tiles with their group (one of the two).  A single
 * product may add bias [N] and apply xIELU to the columns below act_cols (act_params as
 * eb_gemm_parts; either NULL: left out). */
EB_API int eb_gemm_f32(const float *A, long long lda, long long a_group_stride, const float *W, long long ldw,
                long long w_group_stride, float *C, long long ldc, long long c_group_stride, int M, int N, int K, int groups,
                const int32_t *tile_group, const int32_t *live_tiles, const float *bias, int act_cols, const float *act_params,
                void *stream);

/* A unit alone: x [n1, n2] or, gated, [n1, 2*n2] in the 8 + 8 column order -> y [n1, n2].
 * eb_gated_act: the clamped one. */
EB_API int eb_unit_act(const void *x, long long ldx, void *y, long long ldy, int n1, int n2, int unit, float limit, float alpha,
                int dtype, void *stream);
EB_API int eb_gated_act(const void *x, long long ldx, void *y, long long ldy, int n1, int half, float limit, float alpha,
                 int dtype, void *stream);

/* Router of a mixture: idx[t][k], weights[t][k] = the `top` largest softmax scores over all experts
 * of logits[t] (fp32, not renormalised; the lowest index among equals).  first (or NULL): rows
 * t with t mod rows_per_batch < first[t / rows_per_batch] are padding and get idx -1.  With counts
 * (one int every 32, EB_MOE_COUNT_STRIDE; zero on entry), ranks[t][k] = the choice's place among its
 * expert's rows. */
#define EB_MOE_COUNT_STRIDE 32
EB_API int eb_moe_route(const float *logits, long long ld, int tokens, int experts, int top, const int32_t *first,
                 int rows_per_batch, int32_t *idx, float *weights, int32_t *counts, int32_t *ranks, void *stream);

/* Router with a rule.  Scores are the softmax over all `choices` logits, of which the first `experts` are experts
 * and the others stand for the input itself (they take no ticket: rank -1).  Choice scores are score +
 * correction (or NULL).  The choices form `groups` equal groups of neighbours; only the `keep` groups with
 * the largest choice score in them are open.  The `top` largest choice scores of the open groups are
 * chosen; the weights are their scores, divided by their sum (+ 1e-20).  shared_gate (or NULL)[t] =
 * sigmoid of the logit behind the choices (0 for padding).  Otherwise as eb_moe_route. */
EB_API int eb_moe_route_rule(const float *logits, long long ld, int tokens, int choices, int experts, int top, const float *correction,
                      int groups, int keep, const int32_t *first, int rows_per_batch, int32_t *idx, float *weights, int32_t *counts,
                      int32_t *ranks, float *shared_gate, void *stream);

/* Row layout in which every expert owns whole 128-row tiles: offsets[e], tile_group[] (at most
 * max_tiles), *live_tiles; counts are zeroed for the next batch. */
EB_API int eb_moe_plan(int32_t *counts, int experts, int32_t *offsets, int32_t *tile_group, int max_tiles, int32_t *live_tiles,
                void *stream);

/* rows[t][k] = offsets[idx] + rank (or -1: no index or no rank) and out[rows[t][k]] = x[t]. */
EB_API int eb_moe_permute(const void *x, long long ldx, int n2, int dtype, int tokens, int top, const int32_t *idx,
                   const int32_t *ranks, const int32_t *offsets, int32_t *rows, void *out, long long ldo, int max_rows,
                   void *stream);

/* ---- RMS norm ---------------------------------------------------------------------------------- */

/* y = x / sqrt(sum(x^2) / count + eps) * (w_offset + w) over n1 rows of n2 elements (count < n2: the
 * row is zero-padded).  x is fp32 or of the output type, w of the output type; fp32 inside.  ring
 * (or NULL): the rows also go to a ring cache, row (b, s) of n1 = batch * rows_per_batch to row
 * (pos0 + s) mod ring_rows of sequence b, pos0 read from pos_device (NULL: 0); of a longer prompt
 * only the last ring_rows positions are kept. */
EB_API int eb_rms_norm(const void *x, long long ldx, int in_dtype, const void *w, float w_offset, float eps, void *y,
                long long ldy, int out_dtype, int n1, int n2, int count, void *ring, long long ring_batch_stride,
                long long ring_ld, int ring_rows, int rows_per_batch, const int32_t *pos_device, void *stream);

/* x += norm(y) with the residual stream x in fp32, in place; xt (or NULL) receives the new rows in
 * `dtype`.  idx != NULL: y is the output of a mixture, the row of token t being
 * sum_k weights[t][k] * y[rows ? rows[t][k] : t*top + k] over the k with idx[t][k] >= 0.
 * router (or NULL, [experts][n2]): the router of the mixture that follows is evaluated on the new
 * row as rounded to `dtype` (as eb_moe_route). */
EB_API int eb_rms_residual(const void *y, long long ldy, int dtype, const int32_t *idx, const int32_t *rows,
                    const float *weights, int top, const void *w, float w_offset, float eps, float *x, long long ldx, void *xt,
                    long long ldt, int n1, int n2, int count, const void *router, int experts, int router_top,
                    int32_t *router_idx, float *router_weights, void *stream);

/* The residual step of blocks with a norm in front of and behind every sublayer, per row of n2 elements
 * (means over the first `count`; norm(z) = z / sqrt(mean(z^2) + eps)):
 *   x = src_scale * src          if src (the embedding rows, `dtype`), else x as it is (fp32)
 *   x += norm(y * sigmoid(gate)) * w_out        if y  (gate NULL: 1; w_out fp32)
 *   h = norm(x) * w_next                        if w_next; h in `dtype` */
EB_API int eb_stream_update(const void *src, long long lds, float src_scale, const void *y, long long ldy, const void *gate,
                     long long ldg, const float *w_out, float *x, long long ldx, const void *w_next, void *h, long long ldh,
                     float eps, int n1, int n2, int count, int dtype, void *stream);

/* The residual step of blocks with a norm in front of every sublayer only, per row of n2 elements (means over
 * the first `count`):
 *   x = src + src2               if src (embedding rows, `dtype`; src2 or NULL), else x as it is (fp32)
 *   x += scale * Y               Y = y;  with y2: norm(y) * w + norm(y2) * w2 (w, w2 fp32);  with idx, the output of
 *                                a mixture: sum_k weights[t][k] * (idx[t][k] < experts ? y[rows ? rows[t][k] :
 *                                t*top + k] : ident[t]) over the k with idx >= 0, + gate[t] * shared[t]
 *   h = norm(x) * w_next * next_scale          if w_next; h in `dtype`
 * router (or NULL, [choices (+ 1 with r_gate)][n2]): the router of the mixture that follows is evaluated on
 * h, by the rule of eb_moe_route_rule (r_gate: its shared_gate). */
EB_API int eb_stream_add(const void *src, long long lds, const void *src2, long long lds2, const void *y, long long ldy, const float *w,
                  const void *y2, long long ldy2, const float *w2, const int32_t *idx, const int32_t *rows, const float *weights,
                  int top, int experts, const void *ident, long long ldi, const void *shared, long long ldsh, const float *gate,
                  float scale, float *x, long long ldx, const void *w_next, float next_scale, void *h, long long ldh, float eps,
                  int n1, int n2, int count, const void *router, int choices, int r_experts, int r_top, const float *r_correction,
                  int r_groups, int r_keep, int32_t *r_idx, float *r_weights, float *r_gate, int dtype, void *stream);

/* The residual step of blocks whose two sublayers read the same stream, each through a norm and a causal
 * convolution of the normed rows over time, per row of n2 elements (means over the first `count`):
 *   x_out = (src, else x_in) + y (or NULL);  u = x_out / sqrt(mean(x_out^2) + eps)
 *   h1_t = sum_j k1[j] u_(t - taps + 1 + j),  h2_t likewise with k2 (h2 NULL: one sublayer)
 * k1, k2 fp32 [taps][n2] (norm weight times tap, one more for the current token's; taps 2, 3, 4, 8 or 16), rows in front
 * of first[b] count as zero.  Rows b*seq + s; the last ring_rows rows u also go to the ring, position p in row
 * p mod ring_rows.  x_out must not be x_in.  With pos_device: one token per sequence at that position (seq 1; in place
 * allowed), earlier rows come from the ring. */
EB_API int eb_stream_conv(const void *src, long long lds, const float *x_in, long long ldx, const void *y, long long ldy, float *x_out,
                   const float *k1, const float *k2, int taps, void *h1, void *h2, long long ldh, void *ring,
                   long long ring_batch_stride, long long ring_ld, int ring_rows, int batch, int seq, int n2, int count, float eps,
                   const int32_t *first, const int32_t *pos_device, int dtype, void *stream);

/* Queries, keys and values of a projected row [q: heads*dk | k: kv_heads*dk | v: kv_heads*dv] made ready
 * for attention.  q and k are divided by the root mean square over ALL their rows (counts q_count and
 * k_count: heads may be zero-padded) and multiplied by q_norm / k_norm; q also by
 *   1 + temp_coef * ln(floor((p + 1) / temp_every) + 1)      at position p (temp_every 0: 1);
 * with vmix (device scalar) v becomes (1 - vmix) v + vmix v_first, v_first the cached value row of the
 * same token in another layer's cache.  q goes to q_out, k and v to cache row col = pos0 + s of
 * sequence b (row b*rows_per_batch + s of n1; pos0 from pos_device, NULL: 0); nothing is stored for
 * col >= cache_rows.  p = col - first[b]. */
EB_API int eb_attention_inputs(const void *proj, long long ldp, int heads, int kv_heads, int dk, int dv, const void *q_norm,
                        int q_count, const void *k_norm, int k_count, float eps, float temp_coef, int temp_every,
                        const float *vmix, const void *v_first, long long vf_batch_stride, long long vf_row_stride,
                        void *q_out, long long ldq, void *k_cache, long long k_batch_stride, long long k_row_stride,
                        void *v_cache, long long v_batch_stride, long long v_row_stride, int cache_rows, int n1,
                        int rows_per_batch, const int32_t *pos_device, const int32_t *first, int dtype, void *stream);

/* Queries and keys of a projected row [q: heads*dk | k: kv_heads*dk], every head by itself:
 *   z = q_h / sqrt(mean over dk_count + eps) * q_norm  (k_norm for keys), then for i < pairs
 *   (z_2i, z_2i+1) turned by the angle p * freq[i],     p = pos0 + s - first[b]
 * q goes to q_out; the key to k_out (or NULL) and, with the value, which is the key as projected, to the
 * ring caches: row b*rows_per_batch + s of n1 to row (pos0 + s) mod ring_rows of sequence b (of a longer
 * prompt only the last ring_rows positions).  pos0 from pos_device (NULL: 0). */
EB_API int eb_attention_rotary(const void *proj, long long ldp, int heads, int kv_heads, int dk, int dk_count, const void *q_norm,
                        const void *k_norm, float eps, const float *freq, int pairs, void *q_out, long long ldq, void *k_out,
                        long long ldk, void *k_cache, long long k_batch_stride, long long k_row_stride, void *v_cache,
                        long long v_batch_stride, long long v_row_stride, int ring_rows, int n1, int rows_per_batch,
                        const int32_t *pos_device, const int32_t *first, int dtype, void *stream);

/* Every value head is divided by its root mean square (over dv_count columns), in place, and key and value go to a
 * cache of `keep` rows for the first positions of a sequence followed by a ring of ring_rows rows: position col =
 * pos0 + s of row b*rows_per_batch + s to ring row col mod ring_rows (of a longer prompt only the last ring_rows
 * positions) and, while col - first[b] < keep, to that row in front.  k and v are column ranges of rows ld apart. */
EB_API int eb_attention_values(const void *k, void *v, long long ld, int kv_heads, int dk, int dv, int dv_count, float eps, void *k_cache,
                        long long k_batch_stride, long long k_row_stride, void *v_cache, long long v_batch_stride, long long v_row_stride,
                        int keep, int ring_rows, int n1, int rows_per_batch, const int32_t *pos_device, const int32_t *first, int dtype,
                        void *stream);

/* out = y * sigmoid(g), rows of n2 columns. */
EB_API int eb_sigmoid_gate(const void *y, long long ldy, const void *g, long long ldg, void *out, long long ldo, int n1, int n2, int dtype,
                    void *stream);

/* Rows [query latent: q_cols | c | rotated key part] of a projection, the latter two row_cols together, the rotated part
 * from rot_col on (row_cols and q_cols multiples of 8, zero-padded):
 *   q_out = norm(query latent) * q_norm                     norm(z) = z / sqrt(sum(z^2) / count + eps)
 *   row   = [norm(c) * c_norm | (u, v) turned by p freq[i] and times factor, for its first `pairs` neighbouring pairs | 0]
 * at position p = pos0 + s - first[b].  The row goes to ring row (pos0 + s) mod ring_rows (as eb_attention_rotary) and to
 * rows_out (or NULL).  ring NULL: only the query latent. */
EB_API int eb_latent_inputs(const void *proj, long long ldp, int q_cols, int q_count, const void *q_norm, void *q_out, long long ldq,
                     int row_cols, int rot_col, int c_count, const void *c_norm, int pairs, const float *freq, float factor, float eps,
                     void *rows_out, long long ldr, void *ring, long long ring_batch_stride, long long ring_ld, int ring_rows, int n1,
                     int rows_per_batch, const int32_t *pos_device, const int32_t *first, int dtype, void *stream);

/* The pairs from column `col` of every head (head_cols columns) of rows x, turned in place as above. */
EB_API int eb_rotate_heads(void *x, long long ldx, int heads, int head_cols, int col, int pairs, const float *freq, float factor, int n1,
                    int rows_per_batch, const int32_t *pos_device, const int32_t *first, int dtype, void *stream);

/* ---- decaying memories --------------------------------------------------------------------------- */

/* Recurrent layers whose fp32 state per head is a matrix S [dk][dv] that decays.  Everything between the
 * projections and S is fp32; head sizes are multiples of 8 (zero-padded); rows in front of first[b] are
 * padding: they add nothing and forget nothing.
 *
 * State space:  dt' = softplus(dt + dt_bias[h]);  S' = exp(-exp(a_log[h]) dt') S + dt' B x^T;  y = S'^T C + skip[h] x,
 * B and C shared by heads / groups heads.  xbc rows: [x: heads*dv | B: groups*dk | C: groups*dk].
 * Gated linear:  S' = diag(sigmoid(z)^(1/tau)) S + k v^T;  o = S'^T (q scale).  z [row][heads*dk]. */

/* Causal convolution per channel and SiLU of a prompt: out[t] = silu(b + sum_j w[j] x[t - (taps-1) + j]), w [taps]
 * [channels], inputs in front of first[b] zero.  The last ring_rows inputs also go to the ring, position p
 * in row p mod ring_rows. */
EB_API int eb_short_conv(const void *x, long long ldx, const void *w, const void *b, void *out, long long ldo, int batch, int seq,
                  int channels, int taps, const int32_t *first, void *ring, long long ring_batch_stride, long long ring_ld,
                  int ring_rows, int dtype, void *stream);

/* A whole prompt from an empty state, token by token on the CUDA cores, any sizes; xbc behind the convolution. */
EB_API int eb_ssm_scan(const void *xbc, long long ldx, const float *dt, long long ldt, const float *dt_bias, const float *a_log,
                const float *skip, const int32_t *first, void *y, long long ldy, float *S, int batch, int seq, int heads,
                int groups, int dk, int dv, int dtype, void *stream);
EB_API int eb_gla_scan(const void *q, const void *k, const void *v, long long ldp, const float *z, long long ldz, float tau,
                float scale, const int32_t *first, void *o, long long ldo, float *S, int batch, int seq, int heads, int dk,
                int dv, int dtype, void *stream);

/* The same on the tensor cores, 128 tokens at a time: bf16, dk 64 or 128 (heads zero-padded to it), the state and all
 * gates fp32, what enters the state as an operand split into two bf16 parts.  Waits are bounded ("where"
 * codes 400 and up).  eb_gla_chunks: two launches, workspace of eb_gla_chunks_workspace_bytes. */
EB_API int eb_ssm_chunks(const void *xbc, long long ldx, const float *dt, long long ldt, const float *dt_bias, const float *a_log,
                  const float *skip, const int32_t *first, void *y, long long ldy, float *S, int batch, int seq, int heads,
                  int groups, int dk, int dv, int dtype, void *stream);
EB_API int eb_gla_chunks(const void *q, const void *k, const void *v, long long ldp, const float *z, long long ldz, float tau,
                  float scale, const int32_t *first, void *o, long long ldo, float *S, int batch, int seq, int heads, int dk,
                  int dv, int dtype, void *workspace, size_t workspace_bytes, void *stream);
EB_API size_t eb_gla_chunks_workspace_bytes(int batch, int seq, int heads, int dk);

/* One token per sequence; xbc in front of the convolution, whose earlier inputs are read from the ring (and
 * this one's put there). */
EB_API int eb_ssm_step(const void *xbc, long long ldx, const void *conv_w, const void *conv_b, int taps, void *ring,
                long long ring_batch_stride, long long ring_ld, int ring_rows, const int32_t *pos_device, const int32_t *first,
                const float *dt, long long ldt, const float *dt_bias, const float *a_log, const float *skip, void *y,
                long long ldy, float *S, int batch, int heads, int groups, int dk, int dv, int dtype, void *stream);

/* One token per sequence: z = w2 low + b2 (w2 [heads*dk][rank]), the state goes on, and
 * out[h] = unit(o_h) * norm * silu(g), unit(o) = o / sqrt(mean over dv_count of o^2 + eps). */
EB_API int eb_gla_step(const void *q, const void *k, const void *v, const void *g, const void *low, long long ldp, const void *w2,
                const void *b2, int rank, float tau, float scale, const void *norm, int dv_count, float eps, void *out,
                long long ldo, float *S, int batch, int heads, int dk, int dv, int dtype, void *stream);

/* out = unit(y * silu(z)) * norm, unit over `parts` equal parts of the heads*dv real columns (heads of dv
 * columns padded to dv_padded; padding columns of out are not written). */
EB_API int eb_gate_group_norm(const void *y, long long ldy, const void *z, long long ldz, const void *norm, float eps, void *out,
                       long long ldo, int rows, int heads, int dv, int dv_padded, int parts, int dtype, void *stream);

/* ---- selective state space (a state per channel) ----------------------------------------------------- */

/* Channel c of `inner`, state n of `states` (multiples of 8 and 4, zero-padded):
 *   dt = softplus(z_c + bias[c]);  S[c][n] = exp(-exp(a_log[c][n]) dt) S[c][n] + dt x_c B_n;  y_c = sum_n S[c][n] C_n + skip[c] x_c
 *   out_c = y_c silu(gate_c)
 * x is behind the convolution (eb_short_conv), bc rows are [B: states | C: states] and, like z and the state
 * S [batch][inner][states], fp32.
 *
 * eb_selective_scan: a whole prompt from an empty state, rows b*seq + s; rows in front of first[b] add nothing and
 * forget nothing. */
EB_API int eb_selective_scan(const void *x, long long ldx, const void *gate, long long ldg, const float *z, long long ldz, const float *bc,
                      long long ldbc, const float *bias, const float *a_log, const float *skip, const int32_t *first, void *out,
                      long long ldo, float *S, int batch, int seq, int inner, int states, int dtype, void *stream);

/* One token per sequence, the state goes on; z = w low, w [inner][rank] (rank a multiple of 8, zero-padded). */
EB_API int eb_selective_step(const void *x, long long ldx, const void *gate, long long ldg, const void *low, long long ldl, const void *w,
                      int rank, const float *bc, long long ldbc, const float *bias, const float *a_log, const float *skip, void *out,
                      long long ldo, float *S, int batch, int inner, int states, int dtype, void *stream);

/* eb_short_conv of one token per sequence: earlier inputs come from the ring, this one goes there. */
EB_API int eb_short_conv_step(const void *x, long long ldx, const void *w, const void *b, void *out, long long ldo, int batch, int channels,
                       int taps, const int32_t *pos_device, const int32_t *first, void *ring, long long ring_batch_stride,
                       long long ring_ld, int ring_rows, int dtype, void *stream);

/* ---- matrix memory ------------------------------------------------------------------------------ */

/* A recurrent layer whose state per head is a matrix S [dk][dv], a vector n [dk] and a scalar m.  With
 *   i = cap tanh((a_i + bias_i) / cap),  f = logsigmoid(cap tanh((a_f + bias_f) / cap)):
 *   m' = max(f + m, i);  S' = exp(f + m - m') S + exp(i - m') k v^T;  n' likewise with k alone;
 *   o = S'^T (q scale) / (max(|n' . q scale|, exp(-m')) + 1e-6)
 * all in fp32.  gates: fp32 rows ldg apart, a_i of head h at column h, a_f at column heads + h.
 * q, k (heads*dk), v (heads*dv) and o are column ranges of rows ldp / ldo apart.  The state is
 * S [batch][heads][dk][dv], n [batch][heads][dk], m [batch][heads], fp32.
 *
 * eb_memory_scan: a whole prompt, rows b*seq + s, from an empty state; rows s < first[b] are padding
 * and leave it empty; CUDA cores, any sizes, token by token. */
EB_API int eb_memory_scan(const void *q, const void *k, const void *v, long long ldp, const float *gates, long long ldg,
                   const float *bias_i, const float *bias_f, float cap, float scale, const int32_t *first, void *o,
                   long long ldo, float *S, float *n, float *m, int batch, int seq, int heads, int dk, int dv, int dtype,
                   void *stream);

/* eb_memory_scan on the tensor cores, 128 tokens at a time: bf16, dk 64 or 128 (heads zero-padded to it).
 * State and gates are fp32; what enters or leaves the state as an operand is split into two bf16
 * parts, a weighted score is rounded to one.  Waits are bounded ("where" codes 300 and up). */
EB_API int eb_memory_chunks(const void *q, const void *k, const void *v, long long ldp, const float *gates, long long ldg,
                     const float *bias_i, const float *bias_f, float cap, float scale, const int32_t *first, void *o,
                     long long ldo, float *S, float *n, float *m, int batch, int seq, int heads, int dk, int dv, int dtype,
                     void *stream);

/* One token per sequence: the state goes on by one step, and
 *   out[h] = unit(o_h) * norm * sigmoid(g), unit(o) = o / sqrt(mean over dv_count of o^2 + eps). */
EB_API int eb_memory_step(const void *q, const void *k, const void *v, const void *g, long long ldp, const float *gates,
                   long long ldg, const float *bias_i, const float *bias_f, float cap, float scale, const void *norm,
                   int dv_count, float eps, void *out, long long ldo, float *S, float *n, float *m, int batch, int heads,
                   int dk, int dv, int dtype, void *stream);

/* The same tail for the rows of a prompt: out[h] = unit(o_h) * norm * sigmoid(g) per head of dv elements
 * (dv_count of them real). */
EB_API int eb_head_norm_gate(const void *o, long long ldo, const void *g, long long ldg, const void *norm, float eps, void *out,
                      long long ld_out, int rows, int heads, int dv, int dv_count, int dtype, void *stream);
/* silu != 0: the gate is g * sigmoid(g). */
EB_API int eb_head_norm_gate_act(const void *o, long long ldo, const void *g, long long ldg, const void *norm, float eps, void *out,
                          long long ld_out, int rows, int heads, int dv, int dv_count, int silu, int dtype, void *stream);

/* ---- the tail of a greedy generation step ----------------------------------------------------- */

/* Replaces, per step, the arg-max / concatenate / embed sequence of the reference's generation
 * loop (energonai/model/model_factory.py:124-131, energonai/model/embedding.py:44-57) by one launch:
 *   token[b]   = argmax_v logits[b][v]                      (lowest index among equal maxima)
 *   tok[b]     = token[b]  (if tok != NULL);  out_ids[b][kv_state[1]] = token[b]  (if that column < out_cols)
 *   hidden_out[b][:] = word_emb[token[b] - vocab_start][:] (zero if the token belongs to another
 *                      rank's slice of the vocabulary) + pos_emb[kv_state[0] + 1][:] (if add_pos)
 *   kv_state[0] += 1; kv_state[1] += 1                      (after every sequence has read them)
 * kv_state = {position of the token the step just processed, column of out_ids for the new token},
 * device int32[2]; counter: one device int32, zero between launches.  `dtype` is the logits' type,
 * `emb_dtype` that of the embedding tables and of hidden_out; word_emb == NULL skips the embedding.  With the vocabulary split over a
 * tensor-parallel group every rank passes its own slice and exactly one rank passes add_pos = 1;
 * the all-reduce of hidden_out that follows completes the sum. */
EB_API int eb_greedy_step(const void *logits, long long ld_logits, int batch, int vocab, int dtype, int64_t *out_ids,
                   long long ld_out, int out_cols, int64_t *tok, int32_t *kv_state, const void *word_emb,
                   long long vocab_start, int vocab_rows, const void *pos_emb, int pos_rows, int add_pos, int hidden,
                   int emb_dtype, void *hidden_out, long long ld_hidden, int32_t *counter, void *stream);

/* eb_greedy_step with a bigram table: pair_out[b] = pair_emb[(previous token * mul_prev + token * mul_cur) mod pair_rows],
 * the previous token being out_ids[b][kv_state[1] - 1]. */
EB_API int eb_greedy_step_bigram(const void *logits, long long ld_logits, int batch, int vocab, int dtype, int64_t *out_ids,
                   long long ld_out, int out_cols, int64_t *tok, int32_t *kv_state, const void *word_emb,
                   long long vocab_start, int vocab_rows, const void *pos_emb, int pos_rows, int add_pos, int hidden,
                   int emb_dtype, void *hidden_out, long long ld_hidden, int32_t *counter, const void *pair_emb, long long pair_rows,
                   long long mul_prev, long long mul_cur, void *pair_out, long long ld_pair, void *stream);

/* ---- fused attention ----------------------------------------------------------------------- */

/* Replaces the score / mask / softmax / value products of MultiHeadAttention1D.forward
 * (energonai/model/attention.py:105-124) for a whole prompt, without materialising the
 * [batch, heads, q_len, kv_len] score tensor:
 *   out[b,i,h,:] = softmax_j( scale * q[b,i,h,:].k[b,j,h,:] + mask[b,j] ; causal ) . v[b,j,h,:]
 * q, k, v, out are addressed as base + b*batch_stride + row*row_stride + h*head_dim + d
 * (elements), so they may be column slices of one fused projection buffer.  mask is an
 * additive per-key row [batch][kv_len] in the tensor dtype (the reference's 0 / -10000
 * padding mask) or NULL.  causal != 0 hides keys j > i + (kv_len - q_len).  head_dim 64 or
 * 128, dtype fp16 or bf16, strides multiples of 8.  Softmax statistics are fp32. */
EB_API int eb_attention_prefill(const void *q, const void *k, const void *v, void *out, const void *mask,
                         long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                         long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                         long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                         int heads, int q_len, int kv_len, int head_dim, int causal, float scale, int dtype,
                         void *stream);

/* The same product on the 5th-generation tensor cores (tcgen05.mma, accumulators in tensor
 * memory, Q / K / V tiles by TMA): the kernel for prompts.  Same arguments and result as
 * eb_attention_prefill (the probabilities are rounded to the tensor dtype before the value
 * product, as the reference's softmax output is); scale must be positive.  One CTA per 256
 * query rows of a (sequence, head): for q_len well under 128 prefer eb_attention_prefill.  A
 * wait that runs out is reported by eb_device_status ("where" codes 100 and up). */
EB_API int eb_attention_prefill_tc(const void *q, const void *k, const void *v, void *out, const void *mask,
                            long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                            long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                            long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                            int heads, int q_len, int kv_len, int head_dim, int causal, float scale, int dtype,
                            void *stream);

/* eb_attention_prefill_tc with a sliding window: row i sees the keys j with 0 <= i - j < window
 * (window 0: all up to i). */
EB_API int eb_attention_prefill_window_tc(const void *q, const void *k, const void *v, void *out, const void *mask,
                            long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                            long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                            long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                            int heads, int q_len, int kv_len, int head_dim, int window, float scale, int dtype,
                            void *stream);

/* eb_attention_prefill_tc of a sequence with itself (len queries and keys) with a chunk mask and a sink: kv_group
 * query heads share a key / value head; row i sees the keys j <= i with floor((i - f) / chunk) =
 * floor((j - f) / chunk), f = first[b] (chunk 0: all from f on; rows in front of f, padding, see only
 * themselves); sinks (or NULL) [heads]: exp(sinks[h]) joins the softmax denominator. */
EB_API int eb_attention_prefill_chunk_tc(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                            long long q_row_stride, long long k_batch_stride, long long k_row_stride, long long v_batch_stride,
                            long long v_row_stride, long long o_batch_stride, long long o_row_stride, int batch, int heads,
                            int kv_group, int len, int head_dim, int chunk, const int32_t *first, const float *sinks,
                            float scale, int dtype, void *stream);

/* table[h][d] = r1[h] log2(1 + r2[h] d), d < len: the distance bias of eb_attention_prefill_biased_tc. */
EB_API int eb_distance_bias(const float *r1, const float *r2, int heads, int len, float *table, void *stream);

/* eb_attention_prefill_window_tc in which kv_group query heads share a key / value head (k and v have
 * heads / kv_group heads), bias_table[h][i - j] * ln 2 is taken off the scaled score, and sink != 0 adds
 * one to the softmax denominator.  bias_table: fp32 [heads][bias_len] from eb_distance_bias, at
 * least kv_len + 256 distances. */
EB_API int eb_attention_prefill_biased_tc(const void *q, const void *k, const void *v, void *out, const void *mask,
                            long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                            long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                            long long o_batch_stride, long long o_row_stride, long long mask_batch_stride, int batch,
                            int heads, int kv_group, int q_len, int kv_len, int head_dim, int window, const float *bias_table,
                            int bias_len, int sink, float scale, int dtype, void *stream);

/* eb_attention_prefill_chunk_tc without chunks, with value heads of v_dim and the output times sigmoid(gate), gate (or
 * NULL) laid out like the output.  k_dim / v_dim: 64 / 64, 128 / 64 or 128, 192 / 64 or 128. */
EB_API int eb_attention_prefill_gated_tc(const void *q, const void *k, const void *v, void *out, const void *gate, long long q_batch_stride,
                            long long q_row_stride, long long k_batch_stride, long long k_row_stride, long long v_batch_stride,
                            long long v_row_stride, long long o_batch_stride, long long o_row_stride, long long g_batch_stride,
                            long long g_row_stride, int batch, int heads, int kv_group, int len, int k_dim, int v_dim,
                            const int32_t *first, const float *sinks, float scale, int dtype, void *stream);

/* The rule of eb_attention_plain_capped for a prompt on the tensor cores, with a gate as above. */
EB_API int eb_attention_prefill_capped_tc(const void *q, const void *k, const void *v, void *out, const void *gate, long long q_batch_stride,
                            long long q_row_stride, long long k_batch_stride, long long k_row_stride, long long v_batch_stride,
                            long long v_row_stride, long long o_batch_stride, long long o_row_stride, long long g_batch_stride,
                            long long g_row_stride, int batch, int heads, int kv_group, int len, int k_dim, int v_dim, int window,
                            int keep, const int32_t *first, const float *slopes, float cap, int sink, float scale, int dtype,
                            void *stream);

/* Generation step for query heads in groups that share a key / value head: q [batch][heads*head_dim], one
 * row per sequence at position pos (device scalar); k / v rows first[b] .. pos of the cache,
 *   s_j = scale q.k_j - r1[h] ln(1 + r2[h] (pos - j));   out = sum_j exp(s_j) v_j / ([sink] + sum_j exp(s_j)).
 * The keys and values of a group are read once for all its heads.  nsplit > 1 splits the positions over
 * that many CTAs; the last to arrive merges them through `scratch`
 * (eb_attention_group_decode_scratch_bytes, zero-filled once; calls sharing it must not overlap). */
EB_API int eb_attention_group_decode(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                              long long k_batch_stride, long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                              long long out_batch_stride, int batch, int heads, int kv_heads, int head_dim, int cache_rows,
                              const int32_t *pos_device, const int32_t *first, const float *bias_r1, const float *bias_r2,
                              int sink, float scale, int dtype, int nsplit, void *scratch, size_t scratch_bytes, void *stream);
/* With a chunk mask and a sink as eb_attention_prefill_chunk_tc, no bias.  chunk > 0: the cache is a ring,
 * position p in row p mod ring_rows, that holds at least what of the chunk has come. */
EB_API int eb_attention_group_decode_chunk(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                              long long k_batch_stride, long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                              long long out_batch_stride, int batch, int heads, int kv_heads, int head_dim, int ring_rows, int chunk,
                              const int32_t *pos_device, const int32_t *first, const float *sinks, float scale, int dtype,
                              int nsplit, void *scratch, size_t scratch_bytes, void *stream);
/* The rule of eb_attention_plain_capped over a cache of `keep` rows for the first positions and a ring of ring_rows rows
 * (eb_attention_values fills it), the output times sigmoid(gate), gate (or NULL) [batch][heads*head_dim]. */
EB_API int eb_attention_group_decode_capped(const void *q, const void *k, const void *v, void *out, const void *gate, long long q_batch_stride,
                              long long k_batch_stride, long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                              long long out_batch_stride, long long gate_batch_stride, int batch, int heads, int kv_heads, int head_dim,
                              int keep, int ring_rows, int window, const int32_t *pos_device, const int32_t *first, const float *slopes,
                              float cap, int sink, float scale, int dtype, int nsplit, void *scratch, size_t scratch_bytes, void *stream);
EB_API size_t eb_attention_group_decode_scratch_bytes(int batch, int heads, int kv_heads, int head_dim, int nsplit);

/* Windowed causal attention for any head sizes and fp32 / fp16 / bf16 on the CUDA cores: query row
 * i holds position pos0 + i (pos0 from pos_device, NULL: 0) and sees the positions
 * max(first[b], its own - window + 1) .. its own; the key / value of position j is row
 * j mod ring_rows.  Head strides may be 0 (keys shared by the heads); kv_group query heads share a
 * key / value head.  bias_r1 / bias_r2 (or NULL): per query head, r1 * ln(1 + r2 * distance) is taken off
 * the scaled score.  sink != 0 adds one to the softmax denominator (a key of score 0 without a value). */
EB_API int eb_attention_plain(const void *q, const void *k, const void *v, void *out, long long q_batch_stride,
                       long long q_row_stride, long long q_head_stride, long long k_batch_stride, long long k_row_stride,
                       long long k_head_stride, long long v_batch_stride, long long v_row_stride, long long v_head_stride,
                       long long o_batch_stride, long long o_row_stride, long long o_head_stride, int batch, int heads,
                       int kv_group, int q_len, int k_dim, int v_dim, int window, int ring_rows, const int32_t *pos_device,
                       const int32_t *first, const float *bias_r1, const float *bias_r2, int sink, float scale, int dtype,
                       void *stream);

/* The same with a chunk mask and a sink per head (as eb_attention_prefill_chunk_tc) instead of window and bias. */
EB_API int eb_attention_plain_chunk(const void *q, const void *k, const void *v, void *out, long long q_batch_stride, long long q_row_stride,
                       long long q_head_stride, long long k_batch_stride, long long k_row_stride, long long k_head_stride,
                       long long v_batch_stride, long long v_row_stride, long long v_head_stride, long long o_batch_stride,
                       long long o_row_stride, long long o_head_stride, int batch, int heads, int kv_group, int q_len, int k_dim,
                       int v_dim, int chunk, int ring_rows, const int32_t *pos_device, const int32_t *first, const float *sinks,
                       float scale, int dtype, void *stream);

/* The same with a window that keeps the first positions of a sequence visible, capped scores and a linear bias:
 * position i sees max(first[b], i - window + 1) .. i and first[b] .. first[b] + keep - 1 (up to itself; window 0: all),
 *   s = cap tanh(scale q.k / cap) - slopes[h] (i - j)            (cap 0: no cap; slopes NULL: no bias)
 * and sink != 0 adds one to the softmax denominator.  kept_rows: cache rows in front of the ring which hold the
 * first `keep` positions of each sequence (keep or 0; 0: position j is always row j mod ring_rows). */
EB_API int eb_attention_plain_capped(const void *q, const void *k, const void *v, void *out, long long q_batch_stride, long long q_row_stride,
                       long long q_head_stride, long long k_batch_stride, long long k_row_stride, long long k_head_stride,
                       long long v_batch_stride, long long v_row_stride, long long v_head_stride, long long o_batch_stride,
                       long long o_row_stride, long long o_head_stride, int batch, int heads, int kv_group, int q_len, int k_dim,
                       int v_dim, int window, int keep, int kept_rows, int ring_rows, const int32_t *pos_device, const int32_t *first,
                       const float *slopes, float cap, int sink, float scale, int dtype, void *stream);

/* Generation step of latent attention with absorbed projections: q [batch][heads * rank] are the
 * queries in latent space, the cached latent row of a position is key and value of every head,
 *   out[b][h] = sum_j softmax_j(scale * q[b][h] . c[b][j]) c[b][j]
 * over the positions max(first[b], pos - window + 1) .. pos (window 0: all), position j in cache row
 * j mod ring_rows.  rank 64, 128, 192, 256, 320, 384, 512 or 576.  Every cache row must hold finite numbers, also
 * those no position has been written to yet (they are multiplied by a weight of exactly 0).
 * nsplit > 1 splits the positions over that many CTAs per (sequence, head tile): 2, 4 or 8 are
 * clusters that merge their parts on chip, any other number merges in a second launch through
 * `scratch` (eb_latent_decode_scratch_bytes).  Waits are bounded ("where" codes 200 and up). */
EB_API int eb_latent_decode(const void *q, long long q_batch_stride, const void *cache, long long cache_batch_stride,
                     long long cache_row_stride, int ring_rows, void *out, long long out_batch_stride, int batch, int heads,
                     int rank, int window, const int32_t *pos_device, const int32_t *first, float scale, int dtype,
                     int nsplit, void *scratch, size_t scratch_bytes, void *stream);
/* sinks (or NULL): exp(sinks[h]) joins the softmax denominator. */
EB_API int eb_latent_decode_sink(const void *q, long long q_batch_stride, const void *cache, long long cache_batch_stride,
                     long long cache_row_stride, int ring_rows, void *out, long long out_batch_stride, int batch, int heads,
                     int rank, int window, const int32_t *pos_device, const int32_t *first, const float *sinks, float scale, int dtype,
                     int nsplit, void *scratch, size_t scratch_bytes, void *stream);
EB_API size_t eb_latent_decode_scratch_bytes(int batch, int heads, int rank, int nsplit);

/* The same product for one new query row per sequence against the cached keys/values (the
 * generation step; replaces the torch.cat past_cache reads of attention.py:86-98 followed by
 * attention.py:105-124).  q[b] is the row at base + b*q_batch_stride + (kv_len-1)*q_row_stride +
 * h*head_dim: q_row_stride 0 for a plain [batch, heads*head_dim] tensor, or the cache row
 * stride when the query projection sits in the cache row of the new token.  All kv_len cached
 * keys are visible.  kv_len_device, if non-NULL, is a device int32 that overrides
 * kv_len at run time (so a captured launch can be replayed while the cache grows); kv_len, when
 * positive, is then the capacity the device value is clamped to.  The key
 * range is split over `nsplit` CTAs per (sequence, head); for nsplit > 1 `scratch` must hold
 * eb_attention_decode_scratch_bytes(...) bytes, 16-byte aligned, zero-filled once before
 * first use.  Calls sharing a scratch must not overlap on the device. */
EB_API int eb_attention_decode(const void *q, const void *k, const void *v, void *out, const void *mask,
                        long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                        long long k_row_stride, long long v_batch_stride, long long v_row_stride, long long o_batch_stride,
                        long long mask_batch_stride, int batch, int heads, int kv_len, const int32_t *kv_len_device,
                        int head_dim, float scale, int dtype, int nsplit, void *scratch, size_t scratch_bytes,
                        void *stream);
EB_API size_t eb_attention_decode_scratch_bytes(int batch, int heads, int head_dim, int nsplit);

/* The same computation as eb_attention_decode for callers that cannot allocate device memory
 * (a serving worker whose pool was carved up at start-up, code running while the allocator is
 * locked, a host that only receives raw pointers): the split-KV scratch is an 8 MiB array built
 * into the library, resident on every GPU that loads it until the process exits.  The caller
 * passes inputs and outputs only.  Requests whose scratch (see
 * eb_attention_decode_scratch_bytes) exceeds 8 MiB are refused with EB_ELIMIT.  The first call on
 * each device looks the array's address up and clears its counters on `stream`; make that
 * first call outside any stream capture.  All calls on a device share the one array and it
 * keeps the previous call's contents, so calls that overlap on the GPU (two streams, two
 * threads) race: serialise them, the first call per device included (the address look-up is
 * guarded against concurrent host threads, but the clearing of the counters is ordered only
 * on the stream of the call that does it).  A request with nsplit 1 uses no scratch and skips
 * all of this.  Nothing is allocated or freed.  No counterpart in the reference. */
EB_API int eb_attention_decode_noalloc(const void *q, const void *k, const void *v, void *out, const void *mask,
                                long long q_batch_stride, long long q_row_stride, long long k_batch_stride,
                                long long k_row_stride, long long v_batch_stride, long long v_row_stride,
                                long long o_batch_stride, long long mask_batch_stride, int batch, int heads,
                                int kv_len, const int32_t *kv_len_device, int head_dim, float scale, int dtype,
                                int nsplit, void *stream);

/* Device-side waits are bounded; when one expires the kernel records it and returns.  This
 * reads (synchronously) the status word of the current device: out4[0] = 0 or EB_ETIMEDOUT,
 * out4[1] = which wait, out4[2] = block, out4[3] = detail.  clear != 0 resets it.  No
 * counterpart in the reference, whose kernels have no waits. */
EB_API int eb_device_status(int *out4, int clear);

#ifdef __cplusplus
}
#endif
#endif /* ENERGON_B200_H */
