/* tangq.h — C ABI of libtangq, the sm_100a implementation of tang-infer's quantised decode path.
 *
 * Every entry point takes plain pointers and sizes, returns a tq_status, never unwinds, and is
 * what a Rust `extern "C"` block in tang-compute / tang-infer would bind.  Each declaration names
 * the reference interface it stands in for (paths relative to the ecto/tang repository root).
 *
 * Conventions
 *   - "dev" pointers are CUDA device pointers valid on the context's GPU; "host" pointers are
 *     ordinary host memory.  Matrices are row-major.
 *   - All work is issued on the context's stream and is asynchronous unless the name ends in
 *     _host or the comment says it synchronises.
 *   - The library has no CPU fallback: without a usable CUDA device tq_ctx_create fails.
 */
#ifndef TANGQ_H_
#define TANGQ_H_

#include <stddef.h>
#include <stdint.h>

#if defined(__GNUC__)
#define TQ_API __attribute__((visibility("default")))
#else
#define TQ_API
#endif

#ifdef __cplusplus
extern "C" {
#endif

typedef struct tq_ctx tq_ctx;         /* one per (host thread, GPU): stream, workspace, error state */
typedef struct tq_qweight tq_qweight; /* a quantised weight matrix resident in HBM */

typedef enum tq_status {
  TQ_OK = 0,
  TQ_EINVAL = 1,       /* bad argument (the reference panics via assert!, e.g. quantize.rs:228-231) */
  TQ_ECUDA = 2,        /* a CUDA runtime call failed; see tq_last_error */
  TQ_ENCCL = 3,        /* a NCCL call failed */
  TQ_ETIMEOUT = 4,     /* a kernel gave up a bounded wait and recorded a device error code */
  TQ_ENOMEM = 5,
  TQ_EUNSUPPORTED = 6
} tq_status;

typedef enum tq_dtype { TQ_F32 = 0, TQ_BF16 = 1, TQ_F16 = 2, TQ_I8 = 3, TQ_U8 = 4, TQ_I32 = 5, TQ_F64 = 6 } tq_dtype;

/* Weight formats.  Q4/Q8 blocks are tang-infer's: 32 weights along K share one scale; a Q4 byte
 * holds k=2i in its low nibble and k=2i+1 in its high nibble, each stored as q+8
 * (crates/tang-infer/src/quantize.rs:11-31,110-111). */
typedef enum tq_qkind {
  TQ_Q4_F32 = 0, /* Q4Block: f32 scale per block (quantize.rs:25-31) */
  TQ_Q4_F16 = 1, /* same blocks, scale narrowed to IEEE half */
  TQ_Q8_F32 = 2, /* Q8Block: f32 scale + 32 x i8 (quantize.rs:15-20) */
  TQ_I8_ROW = 3  /* int8 [rows, cols] with one f32 scale per output row */
} tq_qkind;

/* ---- context --------------------------------------------------------------------------------
 * Stands in for CudaComputeDevice::new (crates/tang-compute/src/cuda.rs:151-179): one device,
 * one stream.  `stream` is a cudaStream_t to adopt, or NULL to create a private non-blocking one. */
TQ_API int tq_ctx_create(int device, void* stream, tq_ctx** out);
TQ_API int tq_ctx_destroy(tq_ctx* ctx);
/* Text of the last failure on this context (never NULL). */
TQ_API const char* tq_last_error(const tq_ctx* ctx);
/* ComputeDevice::sync (crates/tang-compute/src/device.rs:367): waits for the stream, then reports
 * any error code a kernel recorded (TQ_ETIMEOUT) and clears it. */
TQ_API int tq_sync(tq_ctx* ctx);
TQ_API void* tq_ctx_stream(tq_ctx* ctx);
TQ_API int tq_version(void);

/* ---- raw buffers ----------------------------------------------------------------------------
 * ComputeDevice::alloc / upload / download (device.rs:33-60; cuda.rs:1078-1133).  upload and
 * download synchronise, like the reference's. */
TQ_API int tq_buf_alloc(tq_ctx* ctx, size_t bytes, void** dev_out);
TQ_API int tq_buf_free(tq_ctx* ctx, void* dev);
TQ_API int tq_upload(tq_ctx* ctx, void* dst_dev, const void* src_host, size_t bytes);
TQ_API int tq_download(tq_ctx* ctx, void* dst_host, const void* src_dev, size_t bytes);
TQ_API int tq_memset(tq_ctx* ctx, void* dst_dev, int byte, size_t bytes);
/* dtype conversion on device: f32 <-> bf16 with the reference's round-to-nearest-even
 * (crates/tang-compute/src/kernels/util_cuda.rs:7-40; cuda.rs:22-31). */
TQ_API int tq_convert(tq_ctx* ctx, const void* src_dev, int src_dtype, void* dst_dev, int dst_dtype, size_t n);

/* ---- quantised weights ----------------------------------------------------------------------
 * Upload of a QuantizedQ4 / QuantizedQ8 (quantize.rs:34-44), shape [rows, cols], blocks in
 * row-major order, ceil(cols/32) per row (quantize.rs:193-220).
 *
 * tq_qweight_from_blocks takes the array-of-structs wire form: per block a little-endian f32
 * scale followed by the 16 (Q4) or 32 (Q8) payload bytes — 20 / 36 bytes per block, no padding.
 * kind must be TQ_Q4_F32 or TQ_Q8_F32. */
TQ_API int tq_qweight_from_blocks(tq_ctx* ctx, int kind, const void* blocks_host, size_t rows, size_t cols,
                           tq_qweight** out);
/* Structure-of-arrays host form: payload [rows][ceil(cols/32)*16] (Q4) or [rows][ceil(cols/32)*32]
 * (Q8) or [rows][cols] (TQ_I8_ROW); scales [rows][ceil(cols/32)] as f32 or f16 bits, or [rows]
 * f32 for TQ_I8_ROW. */
TQ_API int tq_qweight_from_arrays(tq_ctx* ctx, int kind, const void* payload_host, const void* scales_host, size_t rows,
                           size_t cols, tq_qweight** out);
/* The same structure-of-arrays form, but already in HBM (payload 8-byte, scales 4-byte aligned).
 * The arrays are read once and can be freed after the next tq_sync.
 *
 * All three constructors regroup the numbers into the library's device layout (16-row x 128-k
 * fragment tiles, see csrc/qlayout.cuh); integer codes and scale bits are copied unchanged. */
TQ_API int tq_qweight_from_device_arrays(tq_ctx* ctx, int kind, const void* payload_dev, const void* scales_dev,
                                         size_t rows, size_t cols, tq_qweight** out);
/* quantize_matrix_q4 / quantize_matrix_q8 (crates/tang-infer/src/quantize.rs:193-220, with quantize_q4/q8 :47-118)
 * on the device: `src` is the [rows, cols] matrix as it comes out of a checkpoint (f32, bf16 or f16, widened to
 * f32 exactly, crates/tang-safetensors/src/lib.rs:262-297; ld = row stride in elements, 0 = dense), `kind` is
 * TQ_Q4_F32 or TQ_Q8_F32.  Scales and integer codes are the reference's bit for bit (scale = amax/7 or amax/127,
 * 1.0 for a zero block, round half away from zero, clamp, ragged tail padded with zeros). */
TQ_API int tq_quantize_matrix(tq_ctx* ctx, const void* src_dev, int src_dtype, size_t ld, size_t rows, size_t cols, int kind,
                              tq_qweight** out);
TQ_API int tq_qweight_free(tq_ctx* ctx, tq_qweight* w);
TQ_API int tq_qweight_shape(const tq_qweight* w, size_t* rows, size_t* cols, int* kind);
TQ_API size_t tq_qweight_bytes(const tq_qweight* w); /* payload + scale bytes one matvec has to stream */

/* dequantize_q4 / dequantize_q8 (quantize.rs:73-81,121-132): out_dev f32 [rows, cols] =
 * (integer as f32) * scale.  With ints_dev != NULL also writes the signed integers (i8
 * [rows, cols]) so the unpack can be checked bit for bit. */
TQ_API int tq_dequantize(tq_ctx* ctx, const tq_qweight* w, float* out_dev, int8_t* ints_dev);

/* ---- quantised linear -----------------------------------------------------------------------
 * y[m, rows] = x[m, cols] . W^T for m activation rows.  This is q4_matvec / q8_matvec
 * (quantize.rs:227-289) at m = 1 and Linear::forward_2d -> matmul_b_transposed (crates/
 * tang-compute/src/modules.rs:56-70, device.rs:407-419) for a quantised W at m > 1.
 *   x_dtype: TQ_BF16 or TQ_F32 (f32 activations are used exactly, as three bf16 terms).
 *   y_dtype: TQ_F32 or TQ_BF16.   ldx / ldy: row strides in elements (0 = dense).
 *   residual_dev: optional f32 [m, rows] (stride ldy) added to the result; may equal y_dev when
 *   y is f32.  Products are exact; accumulation is f32. */
TQ_API int tq_qlinear(tq_ctx* ctx, const tq_qweight* w, const void* x_dev, int x_dtype, size_t ldx, size_t m, void* y_dev,
               int y_dtype, size_t ldy, const float* residual_dev);

/* The reference call itself: q4_matvec(&QuantizedQ4, &[f64]) -> Vec<f64> (quantize.rs:256) and
 * q8_matvec (quantize.rs:227), with HOST vectors.  x_host [m, cols], y_host [m, rows]; dtype is
 * TQ_F64 (the reference's), TQ_F32 or TQ_BF16 (bit patterns) for both.  f64 input is narrowed to
 * f32 (on the device, after upload).  Synchronises. */
TQ_API int tq_q_matvec_host(tq_ctx* ctx, const tq_qweight* w, const void* x_host, void* y_host, int dtype, size_t m);

/* The same call without the final wait, for a caller with several matvecs to run (a list of layers, a batch of
 * independent requests): the upload, the kernel and the read-back are queued on the context's stream in call
 * order, and ONE tq_sync after the last call makes every y_host valid (and reports a device-side failure).  Both
 * vectors must stay alive and untouched until that tq_sync; pageable vectors make the copies themselves block, so
 * pinned ones (cudaHostAlloc / cudaHostRegister) are what this form is for -- a pinned y_host is written by the
 * kernel directly, and pinned bf16 / f32 x_host of up to eight rows are read by a small staging kernel through their
 * device alias instead of being copied.  The reference has no asynchronous form: this replaces a loop of
 * quantize.rs:256 calls.
 * With pinned vectors the call may be recorded between tq_graph_begin and tq_graph_end (after one eager call has set
 * the staging ring up): every tq_graph_launch then reads the vectors' current contents and writes the results again,
 * so a step of many matvecs costs the host one launch and one tq_sync. */
TQ_API int tq_q_matvec_host_async(tq_ctx* ctx, const tq_qweight* w, const void* x_host, void* y_host, int dtype, size_t m);

/* Row-wise concatenation of weights already on the device (same kind and column count; every part
 * but the last with a multiple of 16 rows): builds the fused [q;k;v] and [gate;up] projections
 * from the reference's separate matrices (weight order [wq, wk, wv, wo, gate, up, down],
 * crates/tang-mesh/src/inference.rs:1306-1413). */
TQ_API int tq_qweight_concat_rows(tq_ctx* ctx, const tq_qweight* const* parts, size_t n_parts, tq_qweight** out);

/* A fused [gate; up] projection (gate rows, then the same number of up rows) regrouped so that every 16-row block
 * holds eight gate rows and the eight up rows of the same outputs.  In that order the decode step applies
 * swiglu_fused_buf (crates/tang-compute/src/device.rs:727-736) inside the projection kernel and the 2 x ffn f32
 * intermediate never reaches HBM; tq_llama_set_layer accepts either order.  tq_qlinear on the result yields the
 * outputs in the regrouped order.  Integer codes and scale bits are copied unchanged; the source can be freed
 * after the next tq_sync. */
TQ_API int tq_qweight_interleave_gate_up(tq_ctx* ctx, const tq_qweight* w_gate_up, tq_qweight** out);

/* ---- small operators of the decode step ------------------------------------------------------
 * dtypes are TQ_F32 or TQ_BF16 throughout. */

/* ComputeDevice::rms_norm (crates/tang-compute/src/device.rs:121-128; cpu.rs:126-149) and, with
 * residual_dev != NULL, rms_norm_residual (device.rs:546-575): v = x + residual,
 * out = v / sqrt(mean(v^2) + eps) * weight, and v itself to sum_out_dev (f32, may alias
 * residual_dev) when that is non-NULL.  dim <= 8192. */
TQ_API int tq_rms_norm(tq_ctx* ctx, const void* x_dev, int x_dtype, const float* residual_dev, const void* weight_dev,
                       int w_dtype, size_t n_groups, size_t dim, float eps, void* out_dev, int out_dtype,
                       float* sum_out_dev);
/* InterleavedRoPE::new (crates/tang-compute/src/modules.rs:495-510): cos/sin tables
 * [max_seq_len, head_dim/2], computed in f64 on the host and stored as f32 on the device. */
TQ_API int tq_rope_tables(tq_ctx* ctx, size_t head_dim, size_t max_seq_len, double base, float* cos_dev, float* sin_dev);
/* ComputeDevice::rope_forward (device.rs:582-610): x [seq_len, n_heads, head_dim], pairs (2i, 2i+1)
 * rotated by the table row of position start_pos + s — or positions_dev[s] when that is non-NULL
 * (one decode token per sequence, each at its own position). */
TQ_API int tq_rope_forward(tq_ctx* ctx, const void* x_dev, int x_dtype, const float* cos_dev, const float* sin_dev,
                           const int* positions_dev, size_t seq_len, size_t n_heads, size_t head_dim, size_t start_pos,
                           void* out_dev, int out_dtype);
/* ComputeDevice::swiglu_fused_buf (device.rs:727-736): out[r, i] = silu(gate[r*ld + i]) * up[r*ld + i]
 * (ld = 0: dense).  gate and up may be the two halves of one fused projection. */
TQ_API int tq_swiglu(tq_ctx* ctx, const void* gate_dev, const void* up_dev, int in_dtype, size_t ld, size_t rows, size_t n,
                     void* out_dev, int out_dtype);
/* ComputeDevice::embedding (device.rs:131-138; cpu.rs:151-167): out[i, :] = weight[ids[i], :];
 * ids are int32 (the reference smuggles u32 bit patterns through an f32 buffer, cpu.rs:51-56). */
TQ_API int tq_embedding(tq_ctx* ctx, const void* weight_dev, int w_dtype, const int* ids_dev, size_t seq_len, size_t dim,
                        size_t vocab, void* out_dev, int out_dtype);
/* The greedy branch of Sampler::sample (crates/tang-infer/src/sampling.rs:108-111,183-194): the index of the
 * FIRST maximum of each row (strict '>' scan; NaN is never chosen).  x is f32 [slices][rows][cols] -- a
 * vocabulary gathered rank-major from `slices` tensor-parallel ranks, slices = 1 for a plain matrix -- and the
 * index written is slice * cols + column. */
TQ_API int tq_argmax_rows(tq_ctx* ctx, const float* x_dev, size_t slices, size_t rows, size_t cols, int* idx_out_dev);
/* Sampler::sample (crates/tang-infer/src/sampling.rs:86-158) for `rows` sequences at once, on the device:
 * repetition penalty (once per occurrence in the sequence's past tokens: positive logits divided, the others
 * multiplied), temperature (0 = greedy: first maximum), exp(l - max), top-k (entries equal to the k-th largest
 * survive; 0 = off), normalisation, top-p (descending probability, equal probabilities in index order, cut after
 * the first rank whose running sum reaches p; 1 = off), re-normalisation, and one step of the reference's LCG
 * (sampling.rs:72-79) per sequence for the categorical draw.  logits f32 [slices][rows][cols] as for
 * tq_argmax_rows.  rng_states [rows] are read and advanced (unused when temperature = 0).  past_tokens
 * [rows][past_ld] / past_lens [rows] may be null (no penalty).  While at most 1024 probabilities survive the
 * top-k filter, every sum whose order matters is formed in the reference's order. */
typedef struct tq_sampler_config {
  double temperature;
  uint64_t top_k;
  double top_p;
  double repetition_penalty;
} tq_sampler_config;
TQ_API int tq_sample(tq_ctx* ctx, const float* logits_dev, size_t slices, size_t rows, size_t cols, const tq_sampler_config* cfg,
                     unsigned long long* rng_states_dev, const int* past_tokens_dev_or_null, const int* past_lens_dev_or_null,
                     size_t past_ld, int* tokens_out_dev);
/* The bookkeeping of `generate` (sampling.rs:229-256) between two decode steps, on the device: stores the chosen
 * tokens in out_tokens[row][*step], makes them the next step's input, adds one to every position, to *step and
 * (when given) to every entry of lens_io -- the per-sequence count of past tokens that tq_sample's repetition
 * penalty reads when out_tokens is the sequences' whole history and *step starts at the prompt length.
 * step_io = NULL: row i is stored at column lens_io[i] instead (prompts of different lengths).
 * With the decode step and tq_argmax_rows / tq_sample in front of it, one captured graph generates a token per
 * replay and no logits leave the device.  rows <= 1024. */
TQ_API int tq_generate_advance(tq_ctx* ctx, const int* chosen_dev, size_t rows, int* tokens_io_dev, int* positions_io_dev,
                               int* out_tokens_dev, size_t out_ld, int* step_io_dev_or_null, int* lens_io_dev_or_null);

/* ---- attention -------------------------------------------------------------------------------
 * ComputeDevice::kv_attention (device.rs:161-180; cpu.rs:257-315) on f32 buffers, exactly the
 * reference's signature: q [q_len, n_heads*head_dim], caches [cache_start + q_len, n_kv_heads*
 * head_dim], query i attends positions 0..cache_start+i.  Any q_len; head_dim <= 256. */
TQ_API int tq_kv_attention(tq_ctx* ctx, const float* q_dev, const float* k_cache_dev, const float* v_cache_dev,
                           size_t cache_start, size_t q_len, size_t n_heads, size_t n_kv_heads, size_t head_dim,
                           float* out_dev);
/* The decode hot path: the same attention for ONE new token of each of `batch` sequences, bf16
 * q [batch, n_heads*128] and bf16 caches [batch][position][n_kv_heads*128] (sequence b starts at
 * element b*seq_stride; tang-infer's KVCache layout, crates/tang-infer/src/kv_cache.rs:12-24).
 * Sequence b attends positions 0..lens_dev[b]-1; max_len >= every length.  head_dim = 128,
 * n_heads/n_kv_heads <= 8.  out [batch, n_heads*128] bf16 or f32. */
TQ_API int tq_gqa_decode(tq_ctx* ctx, const void* q_dev, const void* k_cache_dev, const void* v_cache_dev,
                         const int* lens_dev, size_t batch, size_t n_heads, size_t n_kv_heads, size_t head_dim,
                         size_t seq_stride, size_t max_len, void* out_dev, int out_dtype);

/* No counterpart in the reference.  tq_gqa_decode for callers that may not allocate device memory
 * (a serving loop that froze its allocator after start-up, a callback that only owns a stream):
 * same arguments and results, but the per-split partial results live in a fixed 3 MiB array inside
 * the library instead of the context's growable workspace, and the call never reaches cudaMalloc
 * or cudaFree.  It fails with TQ_EINVAL when batch x heads x splits needs more than that.  The
 * first call on a device looks the array's address up and sets a kernel attribute: make it before
 * any stream capture.  All calls on a device share the array — keep them ordered; two that overlap
 * on the GPU corrupt each other's partials. */
TQ_API int tq_gqa_decode_noalloc(tq_ctx* ctx, const void* q_dev, const void* k_cache_dev, const void* v_cache_dev,
                                 const int* lens_dev, size_t batch, size_t n_heads, size_t n_kv_heads,
                                 size_t head_dim, size_t seq_stride, size_t max_len, void* out_dev, int out_dtype);
/* The same attention for a chunk of q_len new positions per sequence (prefill; kv_attention with q_len > 1,
 * device.rs:161-180): q bf16 [batch][q_len][n_heads*128]; query i of sequence b attends cache positions
 * 0 .. cache_start[b] + i, the chunk's own K/V rows being in the cache already; out [batch][q_len][n_heads*128]
 * bf16 or f32.  Probabilities enter the tensor core as bf16 (results to the bf16 bar).  n_heads/n_kv_heads in
 * {1, 2, 4, 8}. */
TQ_API int tq_gqa_prefill(tq_ctx* ctx, const void* q_dev, const void* k_cache_dev, const void* v_cache_dev,
                          const int* cache_start_dev, size_t batch, size_t q_len, size_t n_heads, size_t n_kv_heads,
                          size_t head_dim, size_t seq_stride, void* out_dev, int out_dtype);

/* ---- collectives -----------------------------------------------------------------------------
 * NCCL over NVLink at the shard boundaries (the reference's only collective is a star sum over
 * QUIC, crates/tang-mesh/src/allreduce.rs:43-70).  One communicator per context; calls are
 * issued on the context's stream.  tq_comm_unique_id fills 128 bytes that rank 0 shares with the
 * other ranks by any host-side means. */
typedef struct tq_comm tq_comm;
TQ_API int tq_comm_unique_id(void* id_out128);
TQ_API int tq_comm_create(tq_ctx* ctx, const void* id128, int rank, int world, tq_comm** out);
TQ_API int tq_comm_destroy(tq_ctx* ctx, tq_comm* comm);
/* Tears the communicator down from the host without waiting for peers (ncclCommAbort); later
 * collective calls on it fail with TQ_EINVAL. */
TQ_API int tq_comm_abort(tq_comm* comm);
TQ_API int tq_comm_rank(const tq_comm* comm);
TQ_API int tq_comm_world(const tq_comm* comm);
/* Sum of buf_dev [n] f32 over the ranks, in place (the coordinator's sum of crates/tang-mesh/src/allreduce.rs:43-70,
 * with every rank ending up with the result).  NCCL, unless the communicator has the peer-memory path below and
 * n fits it: then one kernel per rank stores its partial into every rank's buffer, waits (bounded) for the others'
 * flags and adds the partials in rank order -- every rank gets the same bits.  A peer that never arrives turns
 * into TQ_ETIMEOUT at the next tq_sync, with buf_dev left as this rank's own partial. */
TQ_API int tq_all_reduce_f32(tq_ctx* ctx, tq_comm* comm, float* buf_dev, size_t n);
/* Gives the communicator the peer-memory path for sums of up to max_elems floats (a multiple of 4): allocates
 * this rank's buffer, exchanges CUDA IPC handles through the communicator and maps every peer's buffer.  Collective:
 * every rank calls it with the same max_elems.  Ranks must be separate processes on GPUs with peer access (NVLink).
 * With world = 1 or more than 8 ranks it does nothing.  No reference counterpart (tang-mesh sums over QUIC). */
TQ_API int tq_comm_enable_peer(tq_ctx* ctx, tq_comm* comm, size_t max_elems);
/* The same path over buffers the caller has already made visible to this GPU (its own symmetric-memory
 * allocator, or a test): peer_bufs_dev[r] is rank r's buffer as addressed from this device, each of
 * tq_comm_peer_bytes(world, max_elems) bytes, zeroed before the first sum.  The communicator only supports
 * tq_all_reduce_f32 of at most max_elems floats. */
TQ_API int tq_comm_peer_local(tq_ctx* ctx, int rank, int world, void* const* peer_bufs_dev, size_t max_elems, tq_comm** out);
TQ_API size_t tq_comm_peer_bytes(int world, size_t max_elems);
/* How many times the peer path looks at a peer's flag before it gives up (default 4 Mi looks, a few seconds). */
TQ_API int tq_comm_set_wait_limit(tq_comm* comm, unsigned polls);
TQ_API int tq_all_gather(tq_ctx* ctx, tq_comm* comm, const void* send_dev, void* recv_dev, size_t bytes_per_rank);
TQ_API int tq_all_to_all(tq_ctx* ctx, tq_comm* comm, const void* send_dev, void* recv_dev, size_t bytes_per_peer);

/* ---- Llama-shaped decode step ----------------------------------------------------------------
 * The reference's decode loop (crates/tang-train/examples/smollm.rs:215-296) for `batch`
 * sequences at once, one new token each, KV cache resident in HBM.  Dimensions in the config are
 * the WHOLE model's; with a communicator of size n each rank holds n_heads/n, n_kv_heads/n,
 * ffn/n and vocab/n and is given weights of those shard shapes:
 *   wqkv [ (n_heads + 2 n_kv_heads)/n * head_dim, d_model ]   rows = this rank's q heads, k heads, v heads
 *   wo   [ d_model, n_heads/n * head_dim ]                    columns = this rank's heads
 *   wgate_up [ 2 ffn/n, d_model ] (gate rows then up rows)    wdown [ d_model, ffn/n ]
 *   lm_head [ vocab/n, d_model ]
 * Norm gains and the embedding table are bf16 and replicated.  Weight handles are borrowed. */
typedef struct tq_llama tq_llama;
typedef struct tq_llama_config {
  uint32_t n_layers, d_model, n_heads, n_kv_heads, head_dim, ffn, vocab;
  uint32_t max_seq;   /* cache positions per sequence */
  uint32_t max_batch; /* sequences (<= 64) */
  float eps;          /* RMSNorm epsilon (1e-5 in smollm.rs:29) */
  double rope_base;   /* RoPE theta */
} tq_llama_config;
TQ_API int tq_llama_create(tq_ctx* ctx, const tq_llama_config* cfg, tq_comm* comm_or_null, tq_llama** out);
TQ_API int tq_llama_destroy(tq_llama* model);
TQ_API int tq_llama_set_layer(tq_llama* model, size_t layer, const tq_qweight* wqkv, const tq_qweight* wo,
                              const tq_qweight* wgate_up, const tq_qweight* wdown, const void* attn_norm_bf16_dev,
                              const void* ffn_norm_bf16_dev);
TQ_API int tq_llama_set_head(tq_llama* model, const void* embed_bf16_dev, const void* final_norm_bf16_dev,
                             const tq_qweight* lm_head);
/* This rank's bf16 caches of one layer, [max_batch][max_seq][n_kv_heads/n * head_dim], so a caller
 * can prefill them; seq_stride_elems = elements between sequences. */
TQ_API int tq_llama_kv_cache(tq_llama* model, size_t layer, void** k_cache_dev, void** v_cache_dev,
                             size_t* seq_stride_elems);
/* KVCache::trim_to (crates/tang-infer/src/kv_cache.rs:138-149), for every layer and for each of `batch` sequences
 * at once: seq_lens_io_dev[b] is the number of positions sequence b holds (its next position); a sequence that
 * holds more than `keep` drops its OLDEST positions -- rows [len - keep, len) of its K and V caches move to
 * [0, keep) -- and its length becomes `keep`; shorter sequences are untouched.  The K rows keep the rotation of
 * the positions they were appended at, exactly as the reference's trimmed cache does.  Asynchronous. */
TQ_API int tq_llama_kv_trim(tq_llama* model, int* seq_lens_io_dev, size_t batch, size_t keep);
/* The f32 residual stream [max_batch, d_model] after the last tq_llama_decode (the input of the final norm). */
TQ_API int tq_llama_hidden(tq_llama* model, float** hidden_dev);
/* One decode step: sequence b consumes token_ids_dev[b] at position positions_dev[b] (its k, v are
 * appended there) and attends positions 0..positions_dev[b].  max_len > every position.
 * logits_dev: f32 [batch, vocab] for one rank; with n ranks [n][batch][vocab/n] (rank-major
 * vocabulary slices).  Asynchronous; capturable once run eagerly. */
TQ_API int tq_llama_decode(tq_llama* model, const int* token_ids_dev, const int* positions_dev, size_t batch,
                           size_t max_len, float* logits_dev);
/* The same step for caches that have been trimmed (tq_llama_kv_trim): sequence b's K/V are appended at cache row
 * positions_dev[b] and positions 0..positions_dev[b] are attended, but the rotation of its q and k uses
 * rope_positions_dev[b], the caller's running position count (model.forward(&[tok], cache, pos) with a cache whose
 * seq_len is no longer pos, smollm.rs:535 + kv_cache.rs:138-149).  Both stay below max_seq.  NULL rope positions =
 * tq_llama_decode. */
TQ_API int tq_llama_decode_at(tq_llama* model, const int* token_ids_dev, const int* positions_dev, const int* rope_positions_dev,
                              size_t batch, size_t max_len, float* logits_dev);
/* The same step for a chunk of q_len new tokens per sequence (prompt processing): token_ids [batch][q_len],
 * sequence b's chunk starts at position cache_start[b] (its earlier positions are in the cache already).
 * Appends the chunk's K/V rows, runs causal attention over cache + chunk (tq_gqa_prefill) and the linear layers
 * on all batch*q_len rows at once; logits [batch, vocab] (gathered as for tq_llama_decode) are those of each
 * sequence's LAST chunk position.  Workspaces grow on first use: not inside a graph capture. */
TQ_API int tq_llama_prefill(tq_llama* model, const int* token_ids_dev, const int* cache_start_dev, size_t batch, size_t q_len,
                            float* logits_dev);

/* ---- mixture-of-experts FFN -------------------------------------------------------------------
 * No counterpart in the reference (it has no MoE); composed from its primitives.  Router: logits =
 * h . Wg^T in f64 (ascending k), top_k experts by (logit descending, index ascending), weights =
 * softmax over ALL experts (optionally renormalised over the chosen ones).  Expert: down(bf16(
 * silu(gate h) * (up h))) with int4/int8 block weights.  out = sum_chosen w_e expert_e(h) + sum
 * shared experts. */
TQ_API int tq_moe_router(tq_ctx* ctx, const void* h_bf16_dev, const void* wg_bf16_dev, size_t n_tokens, size_t d_model,
                         size_t n_experts, size_t top_k, int renormalize, int* idx_out_dev, float* weight_out_dev,
                         double* logits_out_dev);
typedef struct tq_moe tq_moe;
typedef struct tq_moe_config {
  uint32_t d_model, ffn, n_experts, top_k, n_shared;
  uint32_t renormalize;      /* 1: divide the chosen weights by their sum */
  uint32_t ep_rank, ep_size; /* this rank holds experts [ep_rank, ep_rank+1) * n_experts / ep_size */
} tq_moe_config;
/* Stacked weights: this rank's experts concatenated by rows (tq_qweight_concat_rows): gate|up
 * [n_local * 2*ffn, d_model] (per expert: gate rows then up rows) and down [n_local * d_model, ffn].
 * Shared experts: n_shared pairs of fused gate|up [2*ffn, d_model] and down [d_model, ffn],
 * replicated.  Handles are borrowed. */
TQ_API int tq_moe_create(tq_ctx* ctx, const tq_moe_config* cfg, const void* wg_bf16_dev, const tq_qweight* w_gate_up_stacked,
                         const tq_qweight* w_down_stacked, const tq_qweight* const* shared_gate_up,
                         const tq_qweight* const* shared_down, tq_moe** out);
TQ_API int tq_moe_destroy(tq_moe* moe);
/* h bf16 [n_tokens, d_model] (the same on every rank) -> out f32 [n_tokens, d_model].  With a
 * communicator each rank adds its own experts' terms (and the shared experts for its slice of the
 * tokens) and the result is all-reduced.  idx_out / weight_out (optional): the router's choices,
 * [n_tokens, top_k]. */
TQ_API int tq_moe_ffn(tq_moe* moe, const void* h_bf16_dev, size_t n_tokens, float* out_dev, tq_comm* comm_or_null,
                      int* idx_out_dev, float* weight_out_dev);
/* The same layer with the tokens SHARDED over the expert-parallel ranks: every rank passes its own n_tokens
 * (>= 1, the SAME count on every rank: pad the shorter shards) rows and gets their outputs.  Each (token, choice) row travels to the rank that owns the expert
 * (all-to-all dispatch, padded to the worst case of n_tokens*top_k rows per peer so that the exchange has a
 * fixed size and can be captured in a graph), the owners run their experts on what arrived, and a second
 * all-to-all brings the f32 results back to be weighted and summed where the token lives; shared experts run
 * locally.  The communicator must have the layer's ep_size and ep_rank.  No reference counterpart.
 * From 256 (token, choice) rows per rank on, and when no graph capture is open (on ALL ranks alike), the ranks
 * exchange their per-peer row counts first and the call waits once for the stream to read them; rows, expert ids
 * and results then travel with their true sizes.  Results do not depend on which form ran. */
TQ_API int tq_moe_ffn_dispatch(tq_moe* moe, const void* h_bf16_dev, size_t n_tokens, float* out_dev, tq_comm* comm_or_null,
                               int* idx_out_dev_or_null, float* weight_out_dev_or_null);

/* ---- multi-head latent attention, decode ------------------------------------------------------
 * No counterpart in the reference (it has no MLA).  Absorbed form: the bf16 cache row of position j
 * is [c_j (kv_lora = 512) | r_j (rope = 64)], sequence b starting at element b*seq_stride;
 *   s_j = (q_lat . c_j + q_rope . r_j) * softmax_scale,   o_lat = sum_j softmax(s)_j c_j.
 * q_full [batch, n_heads, 576] bf16 holds q_lat | q_rope per head; o_lat [batch, n_heads, 512] bf16.
 * n_heads (per rank, when heads are sharded) must be a multiple of 16. */
TQ_API int tq_mla_decode(tq_ctx* ctx, const void* q_full_bf16_dev, const void* cache_bf16_dev, const int* lens_dev,
                         size_t batch, size_t n_heads, size_t kv_lora, size_t rope_dim, size_t seq_stride, size_t max_len,
                         float softmax_scale, void* o_lat_bf16_dev);
/* q_lat = W_qk[h] q_nope[h] for every head (int8 per-row weights stacked by rows,
 * [n_heads*512, nope_dim]) written as bf16 into q_full, with q_rope copied behind it.
 * q_nope [batch, n_heads, nope_dim], q_rope [batch, n_heads, 64] bf16; batch <= 64. */
TQ_API int tq_mla_absorb_q(tq_ctx* ctx, const tq_qweight* w_qk_stacked, const void* q_nope_bf16_dev,
                           const void* q_rope_bf16_dev, size_t batch, size_t n_heads, size_t nope_dim,
                           void* q_full_bf16_dev);
/* o[h] = W_uv[h] o_lat[h] (stacked [n_heads*v_dim, 512]); out [batch, n_heads, v_dim] f32 or bf16. */
TQ_API int tq_mla_unabsorb(tq_ctx* ctx, const tq_qweight* w_uv_stacked, const void* o_lat_bf16_dev, size_t batch,
                           size_t n_heads, size_t v_dim, void* out_dev, int out_dtype);

/* One MLA attention layer of a decode step, composed from the calls above (no reference counterpart):
 *   c_q = q_a h                      [q_lora]            (h bf16 [batch, d_model])
 *   c_q = rms_norm(c_q) * gain       when the layer has a gain (eps = norm_eps)
 *   q[h] = q_b[h] c_q                [nope_dim | 64] per head, the 64 rope dimensions rotated (interleaved pairs,
 *                                    device.rs:582-610) by the table row of the query's position lens[b] - 1
 *   o_lat = tq_mla_decode(absorb(q)) over the latent cache (which already holds the current token's row)
 *   out = W_O concat_h(W_uv[h] o_lat[h])  f32 [batch, d_model], summed over the ranks when heads are sharded.
 * All five weights are int8 with one f32 scale per row (any kind tq_qlinear takes works).  n_heads is THIS rank's
 * head count: q_b, W_qk and W_uv hold its heads' rows, W_O [d_model, n_heads * v_dim] its heads' columns; the
 * cache is replicated.  rope tables: tq_rope_tables(head_dim = 64, max_pos, ...).  The layer owns a workspace
 * for max_batch <= 64 rows, so tq_mla_layer_decode allocates nothing and can be captured in a graph. */
typedef struct tq_mla tq_mla;
typedef struct tq_mla_config {
  uint32_t d_model, n_heads, q_lora, kv_lora, nope_dim, rope_dim, v_dim, max_batch, max_pos;
  float norm_eps;
} tq_mla_config;
TQ_API int tq_mla_create(tq_ctx* ctx, const tq_mla_config* cfg, const tq_qweight* q_a, const void* q_a_norm_gain_bf16_dev_or_null,
                         const tq_qweight* q_b, const tq_qweight* w_qk_stacked, const tq_qweight* w_uv_stacked,
                         const tq_qweight* w_o, const float* rope_cos_dev, const float* rope_sin_dev, tq_mla** out);
TQ_API int tq_mla_destroy(tq_mla* layer);
TQ_API int tq_mla_layer_decode(tq_mla* layer, const void* h_bf16_dev, const void* cache_bf16_dev, const int* lens_dev, size_t batch,
                               size_t seq_stride, size_t max_len, tq_comm* comm_or_null, float* out_dev);

/* ---- dense (unquantised) linear layers ---------------------------------------------------------
 * y[m, rows] = x[m, cols] . W^T with W in bf16 (tensor cores, f32 accumulation: a GEMV kernel up to 8 rows, tcgen05
 * above) or in f32 (x and every operation f32, no reduced-precision mode); Linear::forward_2d,
 * crates/tang-compute/src/modules.rs:56-70, on an unquantised weight.  A handle owns its storage, zero when created;
 * tq_dweight_put copies a [rows, cols] block (bf16 or f32, host or device memory) to (row0, col0), so that several
 * projections of one input can share a handle.  interleave = 1 / 2 places the rows as the gate / up halves of 16-row
 * blocks (eight gate rows, then the eight up rows of the same outputs). */
typedef struct tq_dweight tq_dweight;
TQ_API int tq_dweight_create(tq_ctx* ctx, size_t rows, size_t cols, int dtype, tq_dweight** out);
TQ_API int tq_dweight_put(tq_ctx* ctx, tq_dweight* w, const void* src, int src_dtype, size_t rows, size_t cols, size_t row0,
                          size_t col0, int interleave);
TQ_API int tq_dweight_free(tq_ctx* ctx, tq_dweight* w);
/* The stored matrix: [rows_padded][cols_padded] of the handle's dtype. */
TQ_API int tq_dweight_data(const tq_dweight* w, void** dev, size_t* rows_padded, size_t* cols_padded);
/* x has the weight's dtype, 16-byte aligned rows for bf16; y f32 or bf16; ldx / ldy row strides (0 = dense). */
TQ_API int tq_dlinear(tq_ctx* ctx, const tq_dweight* w, const void* x_dev, size_t ldx, size_t m, void* y_dev, int y_dtype, size_t ldy);
/* out = g * sigmoid(alpha g) * (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit); no reference counterpart. */
TQ_API int tq_clamped_glu(tq_ctx* ctx, const void* gate_dev, const void* up_dev, int in_dtype, size_t n, float limit, float alpha,
                          void* out_dev, int out_dtype);

/* Several weights of one shape stacked by rows in one handle: job j (int[4]: group, first row, rows <= chunk, 0; on the device,
 * *n_jobs <= max_jobs of them) multiplies activation rows first .. with rows group * group_rows .. of the weight.  chunk: up to
 * 8 (GEMV), a multiple of 16 up to 256 (tcgen05), or 64 for f32 weights.  x_rows: where activation row i is in x (NULL: row i;
 * not for tcgen05).  row_scale: a factor on every row's products.  glu_alpha = 0: y[row][group_rows] gets the products;
 * otherwise the group's rows are interleaved gate / up halves and y[row][group_rows / 2] gets tq_clamped_glu of them. */
/* The chunk the library takes for `rows` activation rows over n_groups weights of up to `cols` columns. */
TQ_API size_t tq_dense_group_chunk(int dtype, size_t cols, size_t rows, size_t n_groups);
TQ_API int tq_dlinear_grouped(tq_ctx* ctx, const tq_dweight* w, const void* x_dev, size_t ldx, size_t rows, const int* jobs_dev,
                              const int* n_jobs_dev, size_t max_jobs, size_t chunk, size_t group_rows, const int* x_rows_dev_or_null,
                              const float* row_scale_dev_or_null, float glu_limit, float glu_alpha, void* y_dev, int y_dtype, size_t ldy);

/* ---- steps over ragged batches ------------------------------------------------------------------
 * No reference counterpart.  A step's rows are the next tokens of n_seqs sequences, packed: sequence b's are rows
 * seq_rows[b] .. seq_rows[b+1]-1 (seq_rows = NULL: row b), its first one sits at position starts[b], and its cache is
 * slot slots[b] (NULL: b) of max_seq rows.  tq_embedding_pos forms out[m, :] = table[id] + pos_table[position] (f32)
 * and leaves each row's position and cache row (slot * max_seq + position; -1 outside the cache, which tq_sync reports). */
TQ_API int tq_embedding_pos(tq_ctx* ctx, const void* table_dev, const void* pos_table_dev, int dtype, const int* ids_dev,
                            const int* seq_rows_dev_or_null, const int* starts_dev, const int* slots_dev_or_null, size_t n_seqs,
                            size_t rows, size_t dim, size_t vocab, size_t n_pos, size_t max_seq, size_t n_slots, float* out_dev,
                            int* row_pos_dev, int* cache_row_dev);
/* Differential attention: two softmax maps per head over the same values, o = a1 - lambda a2, then
 * o / sqrt(mean(o^2) + eps) * out_scale over the head's vdim values.  The query at position i sees key j when j <= i and
 * (i - j < window or j < keep_first).  q [rows][ldq]: head h's map m at column (2h + m) * dim.  Caches: key row
 * [kv_heads][2][dim rounded up to 8], value row [kv_heads][vdim rounded up to 8], padding zero; the step's own rows are
 * in them already.  out [rows][ldo], head h at column h * vdim.  dtype (TQ_BF16 or TQ_F32) is that of all four.  max_q
 * bounds the rows a sequence brings, max_len every position + 1.  bf16: f32 scores and weights, weights into the tensor
 * core as two bf16 terms. */
typedef struct tq_diff_attn_config {
  uint32_t heads, kv_heads, dim, vdim;
  uint32_t window, keep_first;
  float scale, lambda, out_scale, eps;
} tq_diff_attn_config;
TQ_API int tq_diff_attention(tq_ctx* ctx, const tq_diff_attn_config* cfg, int dtype, const void* q_dev, size_t ldq, const void* k_cache_dev,
                             const void* v_cache_dev, size_t cache_rows, const int* seq_rows_dev_or_null, const int* row_pos_dev,
                             const int* cache_row_dev, size_t n_seqs, size_t rows, size_t max_q, size_t max_len, void* out_dev,
                             size_t ldo);

/* ---- Tofazen ------------------------------------------------------------------------------------
 * No reference counterpart.  A decoder with learned absolute positions and parallel layers,
 *   h = rms_norm(x);  x <- x + residual_mult * (W_o attention(h) + W_down glu(W_gate h, W_up h)),
 * with the differential attention above, layers that read an earlier layer's keys and values (kv_from) and the clamped
 * GLU (sigmoid factor 1.702).  The model owns weights, caches (one per layer with keys of its own, [max_slots][max_seq])
 * and workspaces.  dtype TQ_BF16: bf16 weights, activations and caches, f32 stream, norms and scores; TQ_F32: everything f32. */
typedef struct tq_tofazen tq_tofazen;
typedef struct tq_tofazen_config {
  uint32_t n_layers, width, vocab;
  uint32_t max_positions;  /* rows of the position table */
  uint32_t max_seq;        /* cache rows per slot (<= max_positions) */
  uint32_t max_slots;
  int dtype;
  float eps, residual_mult;
} tq_tofazen_config;
typedef struct tq_tofazen_layer {
  uint32_t heads, kv_heads, dim, vdim;
  uint32_t ff;             /* 0: no feed-forward */
  int kv_from;             /* -1: keys and values of its own */
  uint32_t window, keep_first;
  float scale, lambda, out_scale, limit;
} tq_tofazen_layer;
typedef enum tq_tofazen_tensor {
  TQ_TZ_EMBED = 0, TQ_TZ_POS = 1, TQ_TZ_FINAL_NORM = 2, TQ_TZ_HEAD = 3,
  TQ_TZ_NORM = 4, TQ_TZ_Q = 5, TQ_TZ_K = 6, TQ_TZ_V = 7, TQ_TZ_O = 8, TQ_TZ_GATE = 9, TQ_TZ_UP = 10, TQ_TZ_DOWN = 11
} tq_tofazen_tensor;
TQ_API int tq_tofazen_create(tq_ctx* ctx, const tq_tofazen_config* cfg, const tq_tofazen_layer* layers, tq_tofazen** out);
TQ_API int tq_tofazen_destroy(tq_tofazen* model);
/* Copies one tensor (row-major [rows, cols], bf16 or f32, host or device memory; a vector is [1, n]) into the model. */
TQ_API int tq_tofazen_put(tq_tofazen* model, int tensor, size_t layer, const void* src, int src_dtype, size_t rows, size_t cols);
/* One step over a ragged batch (see tq_embedding_pos): appends the rows' keys and values, attends, and writes f32 logits
 * [n_logits, vocab] of the rows listed in logit_rows (NULL: every row, n_logits = rows); n_logits = 0 skips the head.
 * Decoding (one row per sequence) and prompt portions of any size are the same call.  Asynchronous; capturable once run
 * eagerly with the same sizes. */
TQ_API int tq_tofazen_step(tq_tofazen* model, const int* token_ids_dev, size_t rows, const int* seq_rows_dev_or_null, const int* starts_dev,
                           const int* slots_dev_or_null, size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev_or_null,
                           size_t n_logits, float* logits_dev);
/* The f32 stream [rows, width] after the last step's layers. */
TQ_API int tq_tofazen_hidden(tq_tofazen* model, float** hidden_dev);
/* While set, every step also copies the stream after each layer to streams [n_layers][rows][width] (NULL turns it off). */
TQ_API int tq_tofazen_trace(tq_tofazen* model, float* streams_dev_or_null);

/* ---- row operators, windowed attention, gated linear attention, routing to dense experts --------
 * No reference counterpart.  All take the ragged rows above (row_pos and cache_row of tq_embedding_pos). */
/* Frequencies of a rotary embedding, host arrays: base^(-2i/dims), and with factor > 0 stretched by YaRN (divided by `factor`
 * for pairs with fewer than `slow` turns over `original` positions, kept above `fast`, blended between).  *mult: the factor
 * on cosine and sine, 0.1 ln(factor) + 1 (1 without scaling). */
TQ_API int tq_yarn_frequencies(size_t dims, double base, double factor, double original, double fast, double slow, float* freq_host,
                               float* mult_host);
/* Per row: y = sum of n_y rows of y (y_rows[m * n_y + i], negative: none; y_rows NULL: row m);  x += y / rms(y) * gain_post;
 * out = x / rms(x) * gain_next.  f32 x, y and gains; y NULL: only the second half, gain_next NULL: only the first. */
TQ_API int tq_add_norm(tq_ctx* ctx, float* x_dev, const float* y_dev_or_null, const int* y_rows_dev_or_null, size_t n_y,
                       const float* gain_post_dev_or_null, const float* gain_next_dev_or_null, size_t rows, size_t width, float eps,
                       void* out_dev_or_null, int out_dtype, size_t ld_out);
/* Queries [rows][ldq] and the raw keys of the rows' cache rows [kv_heads][dim rounded up to 8] are divided by their root mean
 * square over the whole projection, multiplied by the gains, and the first rot_dims dimensions of every head rotated
 * (dimension i with i + rot_dims / 2).  Queries in place, keys to the same rows of another cache. */
TQ_API int tq_qk_norm_rope(tq_ctx* ctx, int dtype, size_t heads, size_t kv_heads, size_t dim, void* q_dev, size_t ldq, const void* raw_dev,
                           void* keys_dev, size_t cache_rows, const void* q_gain_dev, const void* k_gain_dev, size_t rot_dims,
                           const float* freq_dev, float rot_mult, float eps, const int* row_pos_dev, const int* cache_row_dev, size_t rows);
/* Per-head norm and rotation.  Queries (head h of row m at q + m * ldq + h * q_head) are divided by the root mean square over
 * their `dim` values and multiplied by q_gain [dim] (NULL: no norm), then rotated in place: pair i of the rot_dims dimensions from
 * rot_first on is (i, i + rot_dims / 2), or with `interleaved` (2i, 2i + 1).  Keys (kv_heads of them, may be 0) as in
 * tq_qk_norm_rope, with k_gain [dim]. */
TQ_API int tq_head_norm_rope(tq_ctx* ctx, int dtype, size_t heads, size_t kv_heads, size_t dim, void* q_dev, size_t ldq, size_t q_head,
                             const void* raw_dev_or_null, void* keys_dev_or_null, size_t cache_rows, const void* q_gain_dev_or_null,
                             const void* k_gain_dev_or_null, size_t rot_first, size_t rot_dims, int interleaved, const float* freq_dev, float rot_mult,
                             float eps, const int* row_pos_dev, const int* cache_row_dev, size_t rows);
/* base^(-2i/dims) with factor > 0 stretched by wavelength: kept below original / high, divided by `factor` above original / low,
 * blended between. */
TQ_API int tq_banded_frequencies(size_t dims, double base, double factor, double low, double high, double original, float* freq_host);
/* Residual streams.  x has `streams` rows of `width` per row of the batch (src_streams 1: one row that stands for all).
 *   x'_t = sum_s mix[s * streams + t] x_s + w_out[t] y             (y NULL: x' = x, nothing is stored)
 *   out  = rms_norm(sum_s w_in[s] x'_s) * gain                     (gain NULL: not formed);   sum = sum_s x'_s (NULL: not stored)
 * y = sum over n_y of weight[m * n_y + i] * row (y_rows[m * n_y + i]) of y, where a negative row stands for `self` row m (of
 * out_dtype, ld_out apart; may be `out` itself), + row m of y_more.  y_rows NULL: row m of y with weight 1. */
TQ_API int tq_stream_mix(tq_ctx* ctx, size_t streams, size_t src_streams, const float* src_dev, float* dst_dev_or_null, const float* y_dev_or_null,
                         const int* y_rows_dev_or_null, const float* y_weight_dev_or_null, size_t n_y, const void* self_dev_or_null,
                         const float* y_more_dev_or_null, const float* mix_dev_or_null, const float* w_out_dev_or_null, const float* w_in_dev_or_null,
                         const float* gain_dev_or_null, size_t rows, size_t width, float eps, void* out_dev_or_null, int out_dtype, size_t ld_out,
                         float* sum_dev_or_null);
/* One stream with what a step of one row per sequence needs beside that: x' = src + w_out y, where row m of y_more is multiplied by
 * sigmoid(y_more_gate[m * ld_gate]); sum = x'; x' += inject row m (NULL: nothing); dst = x'; h = rms_norm(x') * gain, rounded to
 * out_dtype; out = h + conv(h) with conv_w [taps][width] f32 and conv_state [slots][taps - 1][width] of out_dtype, moved on by the row
 * (conv_w NULL: out = h).  mix_one_dev: the value 1. */
TQ_API int tq_stream_step(tq_ctx* ctx, const float* src_dev, float* dst_dev, const float* y_dev, const int* y_rows_dev_or_null,
                          const float* y_weight_dev_or_null, size_t n_y, const float* y_more_dev_or_null, const float* y_more_gate_dev_or_null, size_t ld_gate,
                          const float* inject_dev_or_null, const float* mix_one_dev, const float* w_out_dev, const float* gain_dev, size_t rows, size_t width,
                          float eps, const float* conv_w_dev_or_null, void* conv_state_dev_or_null, size_t taps, size_t max_seq, const int* row_pos_dev,
                          const int* cache_row_dev, void* out_dev, int out_dtype, size_t ld_out, float* sum_dev_or_null);
/* Grouped-query attention: s = (q . k) scale, softcap * tanh(s / softcap) unless softcap is 0; weights
 * exp(s_j) / (exp(sink) + sum exp(s)) (sink -infinity: none); the query at position i sees j when 0 <= i - j < window; the
 * result times sigmoid(gate).  q [rows][ldq], gate (may be NULL) [rows][ldg], caches as in tq_diff_attention with one map. */
typedef struct tq_window_attn_config {
  uint32_t heads, kv_heads, dim, vdim;
  uint32_t window;
  float scale, softcap, sink;
} tq_window_attn_config;
TQ_API int tq_window_attention(tq_ctx* ctx, const tq_window_attn_config* cfg, int dtype, const void* q_dev, size_t ldq,
                               const void* gate_dev_or_null, size_t ldg, const void* k_cache_dev, const void* v_cache_dev, size_t cache_rows,
                               const int* seq_rows_dev_or_null, const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t rows,
                               size_t max_q, size_t max_len, void* out_dev, size_t ldo);
/* The same with a sink per head (sinks [heads] f32; NULL: cfg->sink for all). */
TQ_API int tq_window_attention_sinks(tq_ctx* ctx, const tq_window_attn_config* cfg, const float* sinks_dev_or_null, int dtype, const void* q_dev,
                                     size_t ldq, const void* gate_dev_or_null, size_t ldg, const void* k_cache_dev, const void* v_cache_dev,
                                     size_t cache_rows, const int* seq_rows_dev_or_null, const int* row_pos_dev, const int* cache_row_dev,
                                     size_t n_seqs, size_t rows, size_t max_q, size_t max_len, void* out_dev, size_t ldo);
/* The same with an averaged key and value per block of `pool` older tokens (0: none): once the window of the query at position i has
 * moved past all of block b, b pool + pool - 1 <= i - window, the block is one more term of its softmax.  Pooled rows have the layout of the cache
 * rows; block b of a slot is row slot * pool_rows + b, and a slot has max_seq cache rows.  The result is multiplied by out_scale. */
TQ_API int tq_window_attention_pooled(tq_ctx* ctx, const tq_window_attn_config* cfg, const float* sinks_dev_or_null, int dtype, const void* q_dev,
                                      size_t ldq, const void* gate_dev_or_null, size_t ldg, const void* k_cache_dev, const void* v_cache_dev,
                                      size_t cache_rows, size_t pool, const void* pooled_keys_dev_or_null, const void* pooled_values_dev_or_null,
                                      size_t pool_rows, size_t max_seq, float out_scale, const int* seq_rows_dev_or_null, const int* row_pos_dev,
                                      const int* cache_row_dev, size_t n_seqs, size_t rows, size_t max_q, size_t max_len, void* out_dev, size_t ldo);
/* Short causal convolutions per channel, y_t = sum_j w[j] u_(t - taps + 1 + j), zeros before a sequence's position 0.  w [taps][channels]
 * f32; state [slots][taps - 1][channels] of `dtype` holds a slot's last inputs (slot = cache_row / max_seq) and is moved on by the
 * step's rows.
 * tq_conv_residual: out = x + conv(x), in another buffer. */
TQ_API int tq_conv_residual(tq_ctx* ctx, int dtype, size_t channels, size_t taps, const float* w_dev, void* state_dev, size_t max_seq, size_t cache_rows,
                            const void* x_dev, size_t ldx, const int* seq_rows_dev_or_null, const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs,
                            size_t rows, size_t max_q, size_t max_len, void* out_dev, size_t ldo);
/* tq_conv_heads: rows of raw queries (heads * dim at column 0), keys (kv_heads * dim at k0) and values (kv_heads * vdim at v0).
 * All are convolved (channels: the raw columns; w NULL: not); queries and keys are rotated (first rot_dims dimensions, in halves, freq
 * [rot_dims / 2], cos and sin times rot_mult) and, if norm, rms-normed per head.  Queries go to q, keys and
 * values to the row's cache row ([kv_heads][dim or vdim padded to 8], zero padding).  pool > 0: the means of blocks of `pool` keys and
 * values are left in the pooled rows (as in tq_window_attention_pooled) as soon as a later row can need them. */
typedef struct tq_conv_heads_config {
  uint32_t heads, kv_heads, dim, vdim;
  uint32_t k0, v0, channels, taps;
  uint32_t rot_dims;
  int norm;
  uint32_t pool, pool_rows;
  float rot_mult, eps;
} tq_conv_heads_config;
TQ_API int tq_conv_heads(tq_ctx* ctx, const tq_conv_heads_config* cfg, int dtype, const void* raw_dev, size_t ld, const float* w_dev_or_null,
                         void* state_dev_or_null, const float* freq_dev_or_null, size_t max_seq, size_t cache_rows, const int* seq_rows_dev_or_null,
                         const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t rows, size_t max_q, size_t max_len, void* q_dev,
                         size_t ldq, void* keys_dev, void* values_dev, void* pooled_keys_dev_or_null, void* pooled_values_dev_or_null);
/* minGRU, per channel: z = sigmoid(z_t + z_bias), u = u_t + u_bias, S_t = (1 - z) S_(t-1) + z (u >= 0 ? u + 1/2 : sigmoid(u)),
 * out_t = S_t silu(gate_t) out_scale.  Rows of z, u and gate are `ld` elements apart (even, as ldo); biases and state [slots][width
 * rounded up to 2] are f32; slot = cache_row / max_seq; a sequence's position 0 starts from zero. */
TQ_API int tq_min_gru(tq_ctx* ctx, int dtype, size_t width, const void* z_dev, const void* u_dev, const void* gate_dev, size_t ld, const float* z_bias_dev,
                      const float* u_bias_dev, float out_scale, float* state_dev, size_t max_seq, size_t cache_rows, const int* seq_rows_dev_or_null,
                      const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t rows, size_t max_q, void* out_dev, size_t ldo);
/* Gated linear attention: S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T (q_scale q_t), per head, with
 * alpha_t = sigmoid(a2 a1_t + bias)^(1/tau) per key channel; out = o / sqrt(mean(o^2) + eps) * norm * silu(gate).  Rows of q, k
 * (heads * dim), v, gate (heads * vdim) are `ld` elements apart, a1 [rows][ld_a1] and everything about the state is f32.
 * state [slots][heads][dim][vdim], slot = cache_row / max_seq; a sequence's position 0 starts from zero. */
typedef struct tq_gla_config {
  uint32_t heads, dim, vdim, rank;
  float tau, q_scale, eps;
} tq_gla_config;
TQ_API int tq_gla(tq_ctx* ctx, const tq_gla_config* cfg, int dtype, const void* q_dev, const void* k_dev, const void* v_dev, const void* gate_dev,
                  size_t ld, const float* a1_dev, size_t ld_a1, const float* a2_dev, const float* a2_bias_dev, const float* norm_dev,
                  float* state_dev, size_t max_seq, size_t cache_rows, const int* seq_rows_dev_or_null, const int* row_pos_dev,
                  const int* cache_row_dev, size_t n_seqs, size_t rows, size_t max_q, void* out_dev, size_t ldo);
/* Lightning attention: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head; out = o / sqrt(mean(o^2) + eps) * norm *
 * sigmoid(gate) over the heads' values side by side (norm [heads * vdim] f32).  Rows and states as in tq_gla. */
TQ_API int tq_lightning(tq_ctx* ctx, int dtype, size_t heads, size_t dim, size_t vdim, float eps, const float* decay_dev, const void* q_dev,
                        const void* k_dev, const void* v_dev, const void* gate_dev, size_t ld, const float* norm_dev, float* state_dev, size_t max_seq,
                        size_t cache_rows, const int* seq_rows_dev_or_null, const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs,
                        size_t rows, size_t max_q, void* out_dev, size_t ldo);
/* Latent attention of one bf16 query per sequence over cache rows [latent: rank padded to 16 | rotated part: rot padded to 16] (the
 * padding zero): out[h] = sum_j softmax_j((q_lat[h] . c_j + q_rot[h] . r_j) scale) c_j.  q_lat and out [heads][n_seqs][rank padded
 * to 16], q [heads][n_seqs][ldq] with the rotated part from column dim on; rotate: its first rot_dims are still to be rotated
 * (2i with 2i + 1).  rank at most 512. */
TQ_API int tq_latent_decode(tq_ctx* ctx, size_t heads, size_t dim, size_t rot, size_t rank, float scale, size_t rot_dims, const float* freq_dev,
                            float rot_mult, int rotate, const void* q_lat_dev, const void* q_dev, size_t ldq, const void* cache_dev, size_t cache_rows,
                            const int* row_pos_dev, const int* cache_row_dev, size_t n_seqs, size_t max_len, void* out_dev);
/* The `top` experts with the largest logits [rows][experts] per row (the lower index among equals) with weights sigmoid(z)
 * (score 0) or softmax (score 1), divided by their sum if renorm.  Pair p = row * top + i gets a slot; the slots of an expert are
 * consecutive.  jobs int[.][4]: (expert, first slot, slots <= chunk, 0), at most min(pairs, experts + pairs / chunk). */
TQ_API int tq_route(tq_ctx* ctx, const float* logits_dev, size_t rows, size_t experts, size_t top, int score, int renorm, size_t chunk,
                    int* expert_dev, float* weight_dev, int* slot_dev, int* slot_row_dev, int* jobs_dev, int* n_jobs_dev);
/* The same with a correction [experts] (NULL: none) added to the scores for the choice but not for the weights, and `identity`
 * experts without weights at the end of the list: a pair that chose one of them has slot -1 and is in no job. */
TQ_API int tq_route_rule(tq_ctx* ctx, const float* logits_dev, size_t rows, size_t experts, size_t top, int score, int renorm,
                         const float* correction_dev_or_null, size_t identity, size_t chunk, int* expert_dev, float* weight_dev, int* slot_dev,
                         int* slot_row_dev, int* jobs_dev, int* n_jobs_dev);
/* The same with rows of logits `ld` apart and a bias [experts] (NULL: 0) that is part of the logits. */
TQ_API int tq_route_biased(tq_ctx* ctx, const float* logits_dev, size_t ld, size_t rows, size_t experts, size_t top, int score, int renorm,
                           const float* bias_dev_or_null, const float* correction_dev_or_null, size_t identity, size_t chunk, int* expert_dev,
                           float* weight_dev, int* slot_dev, int* slot_row_dev, int* jobs_dev, int* n_jobs_dev);

/* ---- Numuzen ------------------------------------------------------------------------------------
 * No reference counterpart.  A decoder with a norm before and after every sublayer (weights stored around zero),
 *   x <- x + norm1b(mixer(norm1(x)));  x <- x + norm2b(experts(norm2(x))),
 * whose mixers are windowed attention (whole-projection query/key norm, YaRN rotation, capped scores, a sink of score 0, output
 * gate, the raw keys as values) or gated linear attention, with sigmoid-routed experts whose weight multiplies their input,
 * the clamped GLU (sigmoid factor 1.702) and tied embeddings.  The model owns weights, caches, states (one slot per sequence)
 * and workspaces.  dtype TQ_BF16: bf16 weights, activations and caches; stream, norms, scores, router, recurrences f32; TQ_F32:
 * everything f32. */
typedef struct tq_numuzen tq_numuzen;
typedef struct tq_numuzen_config {
  uint32_t n_layers, width, vocab;
  uint32_t max_seq;        /* positions per slot */
  uint32_t max_slots;
  int dtype;
  float eps;
} tq_numuzen_config;
typedef enum tq_numuzen_mixer { TQ_NZ_ATTENTION = 0, TQ_NZ_GLA = 1 } tq_numuzen_mixer;
typedef struct tq_numuzen_layer {
  uint32_t kind;
  uint32_t heads, kv_heads, dim, vdim;   /* kv_heads: attention only */
  uint32_t window, rot_dims;             /* attention */
  uint32_t rank;                         /* recurrent: rows of a1 */
  uint32_t experts, top, ff;             /* experts = 0: no feed-forward */
  float scale;                           /* attention: of the scores; recurrent: of the queries */
  float softcap, tau, limit;
  double rot_base, rot_factor, rot_original, rot_fast, rot_slow;   /* rot_factor = 0: no scaling */
} tq_numuzen_layer;
typedef enum tq_numuzen_tensor {
  TQ_NZ_EMBED = 0, TQ_NZ_FINAL_NORM = 1, TQ_NZ_NORM1 = 2, TQ_NZ_NORM1B = 3, TQ_NZ_NORM2 = 4, TQ_NZ_NORM2B = 5, TQ_NZ_Q = 6, TQ_NZ_K = 7,
  TQ_NZ_V = 8, TQ_NZ_G = 9, TQ_NZ_O = 10, TQ_NZ_Q_NORM = 11, TQ_NZ_K_NORM = 12, TQ_NZ_O_NORM = 13, TQ_NZ_A1 = 14, TQ_NZ_A2 = 15,
  TQ_NZ_A2_BIAS = 16, TQ_NZ_ROUTER = 17, TQ_NZ_GATE = 18, TQ_NZ_UP = 19, TQ_NZ_DOWN = 20
} tq_numuzen_tensor;
TQ_API int tq_numuzen_create(tq_ctx* ctx, const tq_numuzen_config* cfg, const tq_numuzen_layer* layers, tq_numuzen** out);
TQ_API int tq_numuzen_destroy(tq_numuzen* model);
/* As tq_tofazen_put; `expert` counts for gate, up and down. */
TQ_API int tq_numuzen_put(tq_numuzen* model, int tensor, size_t layer, size_t expert, const void* src, int src_dtype, size_t rows, size_t cols);
/* As tq_tofazen_step; a sequence's recurrent states advance with its rows, and its position 0 starts them from zero. */
TQ_API int tq_numuzen_step(tq_numuzen* model, const int* token_ids_dev, size_t rows, const int* seq_rows_dev_or_null, const int* starts_dev,
                           const int* slots_dev_or_null, size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev_or_null,
                           size_t n_logits, float* logits_dev);
TQ_API int tq_numuzen_hidden(tq_numuzen* model, float** hidden_dev);
TQ_API int tq_numuzen_trace(tq_numuzen* model, float* streams_dev_or_null);

/* ---- Dotanex ------------------------------------------------------------------------------------
 * No reference counterpart.  A decoder with several residual streams (tq_stream_mix) around its mixers -- windowed attention
 * (per-head query/key norm, rotation in halves with banded frequencies, a learned sink per head, the raw keys as values), latent
 * attention (low-rank queries, keys and values from one cached latent and one rotated part per position, interleaved YaRN
 * rotation, output gate) and lightning attention -- and its feed-forwards: gated dense, or softmax-routed experts with a choice
 * correction, identity experts and a shared expert, both of the clamped GLU (sigmoid factor 1.702).  A layer may use another
 * layer's weights (weights_of) with a cache and states of its own.  The model owns weights, caches, states (one slot per sequence)
 * and workspaces.  dtype TQ_BF16: bf16 weights, activations and caches; streams, norms, scores, router, recurrences f32; TQ_F32:
 * everything f32. */
typedef struct tq_dotanex tq_dotanex;
typedef struct tq_dotanex_config {
  uint32_t n_layers, width, vocab;
  uint32_t streams;
  uint32_t max_seq;        /* positions per slot */
  uint32_t max_slots;
  int dtype;
  float eps;
  size_t expand_bytes;     /* latent attention expands keys and values of as many sequences at a time as fit (0: 1 GiB) */
} tq_dotanex_config;
typedef enum tq_dotanex_mixer { TQ_DX_ATTENTION = 0, TQ_DX_LATENT = 1, TQ_DX_LIGHTNING = 2 } tq_dotanex_mixer;
typedef enum tq_dotanex_ff { TQ_DX_NONE = 0, TQ_DX_DENSE = 1, TQ_DX_MOE = 2 } tq_dotanex_ff;
typedef struct tq_dotanex_layer {
  uint32_t kind;
  int weights_of;                        /* -1: tensors of its own; else the rest equals that layer's */
  uint32_t heads, kv_heads, dim, vdim;   /* kv_heads: attention only; dim: without the rotated part of latent attention */
  uint32_t window, rot_dims;             /* window: attention; rot_dims: attention and latent attention */
  uint32_t q_rank, kv_rank, rot_dim;     /* latent attention */
  uint32_t ff_kind, ff;                  /* ff: of the dense feed-forward or of an expert */
  uint32_t experts, identity, top, shared_ff;   /* shared_ff = 0: no shared expert */
  float scale, limit, shared_limit;
  double rot_base, rot_factor, rot_original;    /* rot_factor = 0: no scaling */
  double rot_low, rot_high;              /* attention: banded */
  double rot_fast, rot_slow;             /* latent attention: YaRN */
  const float* decay;                    /* lightning: host [heads], read by tq_dotanex_create */
} tq_dotanex_layer;
typedef enum tq_dotanex_tensor {
  TQ_DX_EMBED = 0, TQ_DX_FINAL_NORM = 1, TQ_DX_HEAD = 2, TQ_DX_NORM1 = 3, TQ_DX_NORM2 = 4, TQ_DX_HC1_IN = 5, TQ_DX_HC1_OUT = 6, TQ_DX_HC1_MIX = 7,
  TQ_DX_HC2_IN = 8, TQ_DX_HC2_OUT = 9, TQ_DX_HC2_MIX = 10, TQ_DX_Q = 11, TQ_DX_K = 12, TQ_DX_V = 13, TQ_DX_G = 14, TQ_DX_O = 15, TQ_DX_Q_NORM = 16,
  TQ_DX_K_NORM = 17, TQ_DX_SINK = 18, TQ_DX_O_NORM = 19, TQ_DX_DQ = 20, TQ_DX_DQ_NORM = 21, TQ_DX_UQ = 22, TQ_DX_DKV = 23, TQ_DX_DKV_NORM = 24,
  TQ_DX_UK = 25, TQ_DX_UV = 26, TQ_DX_ROUTER = 27, TQ_DX_CORRECTION = 28, TQ_DX_GATE = 29, TQ_DX_UP = 30, TQ_DX_DOWN = 31, TQ_DX_SHARED_GATE = 32,
  TQ_DX_SHARED_UP = 33, TQ_DX_SHARED_DOWN = 34
} tq_dotanex_tensor;
TQ_API int tq_dotanex_create(tq_ctx* ctx, const tq_dotanex_config* cfg, const tq_dotanex_layer* layers, tq_dotanex** out);
TQ_API int tq_dotanex_destroy(tq_dotanex* model);
/* As tq_tofazen_put; `expert` counts for gate, up and down of routed experts.  Layers with weights_of take none. */
TQ_API int tq_dotanex_put(tq_dotanex* model, int tensor, size_t layer, size_t expert, const void* src, int src_dtype, size_t rows, size_t cols);
/* As tq_numuzen_step. */
TQ_API int tq_dotanex_step(tq_dotanex* model, const int* token_ids_dev, size_t rows, const int* seq_rows_dev_or_null, const int* starts_dev,
                           const int* slots_dev_or_null, size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev_or_null,
                           size_t n_logits, float* logits_dev);
/* While set, every step also leaves the sum of the streams after each layer in sums [n_layers][rows][width] (NULL turns it off). */
TQ_API int tq_dotanex_trace(tq_dotanex* model, float* sums_dev_or_null);

/* ---- Sakinex ------------------------------------------------------------------------------------
 * No reference counterpart.  A decoder with one residual stream, x <- x + residual_mult * sublayer(h), h = n + conv(n), n = norm(x),
 * whose mixer has two branches on the same h,
 *   mixer = left_scale * attention(h) + right_scale * recurrence(h),
 * attention with short convolutions on queries, keys and values, YaRN rotation in halves, a gainless query/key norm per head behind
 * it, a sliding window and pooled blocks before the window (tq_conv_heads, tq_window_attention_pooled), and a minGRU (tq_min_gru).
 * Its feed-forward has experts routed by biased logits and weighed by a softmax over the chosen ones, and a shared expert behind a
 * sigmoid gate; all of the SiLU form.  An entry of `layers` is a run of a layer: runs that repeat another's weights (weights_of)
 * have caches and states of their own, and add_embedding adds the embedding output to the stream ahead of the run.  The model owns
 * weights, caches, states (one slot per sequence) and workspaces.  dtype TQ_BF16: bf16 weights, activations, caches and convolution
 * inputs; stream, norms, scores, router, recurrence f32; TQ_F32: everything f32. */
typedef struct tq_sakinex tq_sakinex;
typedef struct tq_sakinex_config {
  uint32_t n_layers, width, vocab;
  uint32_t taps;           /* of the convolution on a sublayer's input */
  uint32_t max_seq;        /* positions per slot */
  uint32_t max_slots;
  int dtype;
  float eps, residual_mult;
} tq_sakinex_config;
typedef struct tq_sakinex_layer {
  int weights_of;                        /* -1: tensors of its own; else the rest equals that run's, but for add_embedding */
  int add_embedding;
  uint32_t heads, kv_heads, dim, vdim;   /* attention */
  uint32_t window, pool;                 /* pool = 0: no pooled blocks */
  uint32_t taps, rot_dims;               /* taps = 0: no convolution on queries, keys and values */
  uint32_t state_width;                  /* recurrence */
  uint32_t experts, top, ff, shared_ff;  /* experts = 0: no feed-forward; shared_ff = 0: no shared expert */
  float scale, left_scale, right_scale;
  double rot_base, rot_factor, rot_original, rot_fast, rot_slow;   /* rot_factor = 0: no scaling */
} tq_sakinex_layer;
typedef enum tq_sakinex_tensor {
  TQ_SX_EMBED = 0, TQ_SX_FINAL_NORM = 1, TQ_SX_HEAD = 2, TQ_SX_NORM1 = 3, TQ_SX_NORM2 = 4, TQ_SX_CANON1 = 5, TQ_SX_CANON2 = 6, TQ_SX_Q = 7, TQ_SX_K = 8,
  TQ_SX_V = 9, TQ_SX_Q_CONV = 10, TQ_SX_K_CONV = 11, TQ_SX_V_CONV = 12, TQ_SX_LEFT_O = 13, TQ_SX_Z = 14, TQ_SX_Z_BIAS = 15, TQ_SX_X = 16, TQ_SX_X_BIAS = 17,
  TQ_SX_G = 18, TQ_SX_RIGHT_O = 19, TQ_SX_ROUTER = 20, TQ_SX_ROUTER_BIAS = 21, TQ_SX_GATE = 22, TQ_SX_UP = 23, TQ_SX_DOWN = 24, TQ_SX_SHARED_GATE = 25,
  TQ_SX_SHARED_UP = 26, TQ_SX_SHARED_DOWN = 27, TQ_SX_SHARED_SWITCH = 28
} tq_sakinex_tensor;
TQ_API int tq_sakinex_create(tq_ctx* ctx, const tq_sakinex_config* cfg, const tq_sakinex_layer* layers, tq_sakinex** out);
TQ_API int tq_sakinex_destroy(tq_sakinex* model);
/* As tq_tofazen_put; `expert` counts for gate, up and down of routed experts; convolutions are [channels, taps].  Runs with weights_of
 * take none. */
TQ_API int tq_sakinex_put(tq_sakinex* model, int tensor, size_t layer, size_t expert, const void* src, int src_dtype, size_t rows, size_t cols);
/* As tq_numuzen_step. */
TQ_API int tq_sakinex_step(tq_sakinex* model, const int* token_ids_dev, size_t rows, const int* seq_rows_dev_or_null, const int* starts_dev,
                           const int* slots_dev_or_null, size_t n_seqs, size_t max_q, size_t max_len, const int* logit_rows_dev_or_null,
                           size_t n_logits, float* logits_dev);
/* While set, every step also leaves the stream after each run in streams [n_layers][rows][width] (NULL turns it off). */
TQ_API int tq_sakinex_trace(tq_sakinex* model, float* streams_dev_or_null);

/* ---- CUDA graphs ------------------------------------------------------------------------------
 * CudaComputeDevice::begin_capture / end_capture (crates/tang-compute/src/cuda.rs:344-356): every
 * asynchronous call made on the context between begin and end is recorded instead of run, and
 * replayed by tq_graph_launch.  Calls that allocate or synchronise (uploads, downloads, _host
 * calls, the first tq_qlinear that needs a larger staging buffer) must not be made while
 * capturing: run the sequence once eagerly first.  The recorded kernels hold the addresses of the
 * context's workspaces; when a later call makes one of them grow (it is freed and reallocated),
 * tq_graph_launch of a graph recorded before that fails with TQ_EINVAL: record the graph again. */
typedef struct tq_graph tq_graph;
TQ_API int tq_graph_begin(tq_ctx* ctx);
TQ_API int tq_graph_end(tq_ctx* ctx, tq_graph** out);
TQ_API int tq_graph_launch(tq_ctx* ctx, tq_graph* graph);
TQ_API int tq_graph_free(tq_ctx* ctx, tq_graph* graph);
/* Kernels launched through this context so far (graph replays count their recorded kernels). */
TQ_API unsigned long long tq_launch_count(const tq_ctx* ctx);

#ifdef __cplusplus
}
#endif
#endif /* TANGQ_H_ */
