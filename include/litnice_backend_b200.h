/*
 * liblitnice_backend_b200.so — NVIDIA B200 (sm_100a) backend plugin for litnicelm.
 *
 * Two groups of entry points, all plain C ABI:
 *
 *  1. litnice_backend_get_api(): the `backend.library` plugin contract of
 *     litnicelm (src/model/backend/backend_plugin_api.hpp:7-168). The host
 *     resolves this one symbol after dlopen (device_backend.cpp:182-230) and
 *     then calls through the returned table, so the unchanged `infer`,
 *     `inspect` and `inferloop` commands run on the GPU.
 *
 *  2. litnice_b200_*: a native token loop in which nothing but token ids
 *     crosses the host/device boundary per generated token. It replaces the
 *     host-driven loop of src/model/inference.cpp:265-296 and the per-row
 *     logits read-back of host_tensor_stage.hpp:101-125.
 *
 * Group 1 reports failures as C++ exceptions (the contract of the reference
 * loader: no status codes, main.cpp:37-40). Group 2 never throws: functions
 * return 0 on success and a negative LITNICE_B200_E* code otherwise, with
 * text available from litnice_b200_last_error().
 *
 * There is no CPU fallback anywhere: without a CUDA device every compute entry
 * fails loudly.
 */
#ifndef LITNICE_BACKEND_B200_H
#define LITNICE_BACKEND_B200_H

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* ------------------------------------------------------------------------ */
/* 1. The litnicelm plugin contract (backend_plugin_api.hpp).                 */
/* ------------------------------------------------------------------------ */

#define LITNICE_TENSOR_MAX_RANK 6
#define LITNICE_BACKEND_ABI_VERSION 16u /* backend_plugin_api.hpp:164 */

/* backend_plugin_api.hpp:7-18. Strides are in bytes; rows/cols/stride_r/stride_c
 * repeat dims[0], dims[1] and the strides of the last two axes
 * (device_backend.cpp:154-169). device: 0 CPU, 1 GPU. dtype: 0 f32, 1 i32. */
typedef struct BackendTensorView {
  uint32_t device;
  uint32_t dtype;
  void *data;
  uint32_t rank;
  int64_t rows;
  int64_t cols;
  int64_t stride_r_bytes;
  int64_t stride_c_bytes;
  int64_t dims[LITNICE_TENSOR_MAX_RANK];
  int64_t strides_bytes[LITNICE_TENSOR_MAX_RANK];
} BackendTensorView;

/* backend_plugin_api.hpp:20-24 */
typedef struct BackendMemoryInfo {
  uint32_t available;
  uint64_t free_bytes;
  uint64_t total_bytes;
} BackendMemoryInfo;

typedef const BackendTensorView *LitniceView;

/* backend_plugin_api.hpp:26-162: abi_version followed by 55 entries, in this
 * exact order. Entries marked [inference] are reached by infer / inspect /
 * inferloop; the others belong to training and throw "not implemented" here. */
typedef struct BackendApiV1 {
  uint32_t abi_version;
  void *(*create)(uint32_t device);                                        /* [inference] */
  void (*destroy)(void *backend);                                          /* [inference] */
  uint32_t (*device)(void *backend);                                       /* [inference] */
  void *(*alloc)(void *backend, uint64_t bytes, uint32_t alignment);       /* [inference] */
  void (*free)(void *backend, void *ptr);                                  /* [inference] */
  void (*copy_host2device)(void *backend, void *dst, const void *src, uint64_t bytes); /* [inference] */
  void (*copy_device2host)(void *backend, void *dst, const void *src, uint64_t bytes); /* [inference] */
  void (*copy)(void *backend, LitniceView src, LitniceView dst);           /* [inference] */
  void (*fill)(void *backend, LitniceView t, float v);                     /* [inference] */
  void (*add)(void *backend, LitniceView a, LitniceView b, LitniceView out); /* [inference] */
  void (*add_inplace)(void *backend, LitniceView a, LitniceView b);
  void (*add_bias_rowwise)(void *backend, LitniceView x, LitniceView bias_1xC, LitniceView out); /* [inference] */
  void (*add_bias_relu_rowwise)(void *backend, LitniceView x, LitniceView bias_1xC, LitniceView out); /* [inference] */
  void (*add_bias_relu_rowwise_inplace)(void *backend, LitniceView x, LitniceView bias_1xC); /* [inference] */
  void (*mul_scalar)(void *backend, LitniceView x, float s, LitniceView out); /* [inference] */
  float (*sum_squares_f32)(void *backend, LitniceView x);
  void (*relu)(void *backend, LitniceView x, LitniceView out);             /* [inference] */
  void (*relu_backward)(void *backend, LitniceView preact, LitniceView dout, LitniceView dx);
  void (*relu_backward_inplace)(void *backend, LitniceView preact, LitniceView dout_dx);
  void (*row_sum)(void *backend, LitniceView x, LitniceView out_1xC);
  void (*gemm)(void *backend, LitniceView a, LitniceView b, LitniceView out);
  void (*gemm_ranked_matrix_rhs)(void *backend, LitniceView a, LitniceView b, LitniceView out); /* [inference] */
  void (*gemm_ranked_matrix_rhs_t)(void *backend, LitniceView a, LitniceView b, LitniceView out);
  void (*gemm_ranked_reduce_lhs_t)(void *backend, LitniceView a, LitniceView b, LitniceView out);
  void (*gemm_batched)(void *backend, LitniceView a, LitniceView b, LitniceView out); /* [inference] */
  void (*gemm_batched_lhs_t)(void *backend, LitniceView a, LitniceView b, LitniceView out);
  void (*gemm_batched_rhs_t)(void *backend, LitniceView a, LitniceView b, LitniceView out); /* [inference] */
  void (*transpose)(void *backend, LitniceView x, LitniceView out);
  void (*layernorm_forward)(void *backend, LitniceView x, LitniceView gamma_1xC, LitniceView beta_1xC, LitniceView out); /* [inference] */
  void (*layernorm_backward)(void *backend, LitniceView x, LitniceView gamma_1xC, LitniceView dout, LitniceView dx, LitniceView dgamma_1xC, LitniceView dbeta_1xC);
  void (*embedding_lookup)(void *backend, LitniceView table, LitniceView ids, LitniceView out); /* [inference] */
  void (*accumulate_embedding_grads)(void *backend, LitniceView ids, LitniceView d_cur, LitniceView d_tok, LitniceView d_pos);
  void (*cross_entropy_mean)(void *backend, LitniceView logits, LitniceView targets, LitniceView out_loss);
  void (*cross_entropy_mean_backward_inplace)(void *backend, LitniceView logits, LitniceView targets, LitniceView out_loss);
  float (*read_scalar_f32)(void *backend, LitniceView x);
  void (*backward_from_logits_targets)(void *backend, LitniceView logits, LitniceView targets);
  void (*softmax_rows)(void *backend, LitniceView x, LitniceView out);     /* [inference] */
  void (*softmax_backward_rows)(void *backend, LitniceView softmax, LitniceView dout, LitniceView dx);
  void (*scaled_causal_softmax_rows)(void *backend, LitniceView scores, float scale, LitniceView out); /* [inference] */
  uint32_t (*supports_exec_context_iteration)(void *backend);             /* [inference] */
  void (*start_exec_context_iteration)(void *backend);                     /* [inference] */
  void (*finish_exec_context_iteration)(void *backend);                    /* [inference] */
  void (*start_exec_context_group)(void *backend);                         /* [inference] */
  void (*finish_exec_context_group)(void *backend);                        /* [inference] */
  void (*gemm_batched_exec_context)(void *backend, LitniceView a, LitniceView b, LitniceView out); /* [inference] */
  void (*gemm_batched_lhs_t_exec_context)(void *backend, LitniceView a, LitniceView b, LitniceView out);
  void (*gemm_batched_rhs_t_exec_context)(void *backend, LitniceView a, LitniceView b, LitniceView out); /* [inference] */
  void (*scaled_causal_softmax_rows_exec_context)(void *backend, LitniceView scores, float scale, LitniceView out); /* [inference] */
  void (*softmax_backward_causal_rows_exec_context)(void *backend, LitniceView softmax, LitniceView dout, LitniceView dx);
  void (*softmax_backward_causal_rows)(void *backend, LitniceView softmax, LitniceView dout, LitniceView dx);
  void (*apply_causal_mask_inplace)(void *backend, LitniceView scores, float neg_inf); /* [inference] */
  void (*adamw_step)(void *backend, LitniceView params, LitniceView grads, LitniceView m, LitniceView v, uint64_t step, float learning_rate, float beta1, float beta2, float weight_decay, uint32_t apply_weight_decay);
  uint32_t (*is_file2device_read_supported)(void *backend);
  void (*read_file2device)(void *backend, const char *path, void *dst, uint64_t size, uint64_t file_offset);
  BackendMemoryInfo (*memory_info)(void *backend);
} BackendApiV1;

/* The symbol the litnicelm loader resolves (device_backend.cpp:191-206;
 * the CPU plugin's counterpart is backend_plugin_cpu.cpp:498-500). The table
 * has static storage and abi_version == 16. The GPU is chosen by
 * CUDA_VISIBLE_DEVICES or the LITNICE_B200_DEVICE environment variable: the
 * contract's create(device) carries the CPU/GPU enum, not an ordinal. */
const BackendApiV1 *litnice_backend_get_api(void);

/* ------------------------------------------------------------------------ */
/* 2. Native token loop.                                                      */
/* ------------------------------------------------------------------------ */

#define LITNICE_B200_OK 0
#define LITNICE_B200_EINVAL (-1)   /* bad argument or shape */
#define LITNICE_B200_ECUDA (-2)    /* CUDA runtime error */
#define LITNICE_B200_ENOMEM (-3)   /* device allocation failed */
#define LITNICE_B200_EIO (-4)      /* checkpoint file unreadable or mismatched */
#define LITNICE_B200_EDEVICE (-5)  /* a kernel reported an error (bad token id, wait ran out) */
#define LITNICE_B200_ETOOBIG (-6)  /* litnice_b200_gemv_noalloc: sizes beyond its built-in scratch */

typedef struct litnice_b200_session litnice_b200_session;

/* model.* and memory.alignment_bytes of the YAML (include/types.hpp:134-146). */
typedef struct litnice_b200_dims {
  int32_t n_layers, n_heads, d_model, d_ff, vocab_size, max_seq_len;
  uint64_t alignment_bytes;
} litnice_b200_dims;

/* inference.temp / top_k / top_p (include/types.hpp:112-119). temp <= 0 or
 * top_k == 1 selects greedy, as in inference.cpp:206-208. */
typedef struct litnice_b200_sampling {
  float temp;
  uint32_t top_k;
  float top_p;
} litnice_b200_sampling;

/* Counters of the most recent generate / run call. */
typedef struct litnice_b200_stats {
  double device_ms;          /* CUDA-event time of the token loop on the session's stream */
  int64_t kernel_launches;   /* kernels of this library launched inside that region */
  int64_t tokens;            /* tokens produced over all streams */
  int64_t h2d_bytes, d2h_bytes;
  double gemm_ms;            /* filled only by litnice_b200_profile_step */
  int64_t gemm_launches;
  double gemm_flops;         /* algorithmic flops of those launches */
  double attn_ms;
  int64_t attn_launches;
  /* litnice_b200_profile_step, one step without events: per launch the span from the
   * earliest CTA start to the latest CTA end on the device clock (launches overlap as in
   * the token loop), summed per kernel class, and the span of the whole step. Filled for
   * the tensor-core kernels only. */
  double gemm_span_ms;
  int64_t gemm_span_launches;
  double gemm_span_flops;
  double attn_span_ms;
  int64_t attn_span_launches;
  double step_span_ms;
} litnice_b200_stats;

/* Builds a session on the current CUDA device (or LITNICE_B200_DEVICE) for up
 * to max_streams independent streams decoded in lockstep. Replaces the runtime
 * object of inference.cpp:49-71 and its three arena allocations
 * (inference_memory_manager.cpp:7-33). */
int litnice_b200_session_create(const litnice_b200_dims *dims, int32_t max_streams,
                                litnice_b200_session **out);
/* The same on an explicit CUDA device ordinal (LITNICE_B200_DEVICE is not consulted): what a
 * host that runs one thread per GPU calls, each thread with its own share of the streams
 * (the reference runs one stream per process, inference.cpp:362-405; streams never
 * exchange data, so the shares need no collective). Every call on a session selects the
 * session's device first, so a session may be driven from any one thread at a time. */
int litnice_b200_session_create_on(const litnice_b200_dims *dims, int32_t max_streams, int32_t device,
                                   litnice_b200_session **out);
/* A session on a model folder (config.json + model.safetensors) of one of the registered decoder
 * designs, weights loaded. config.json's "architecture" names the design; the names known are
 * litnice_b200_architectures(), with commas between them. dtype: LITNICE_B200_DTYPE_BF16 (bfloat16
 * weights and matrix products with 32-bit accumulation; norms, attention scores and weights, the
 * residual stream and state in 32-bit) or LITNICE_B200_DTYPE_F32 (everything in 32-bit). device:
 * CUDA ordinal, negative for LITNICE_B200_DEVICE or the current device. Such a session keeps its
 * caches and state in max_streams slots and serves generate / upload_prompts / run /
 * download_tokens, forward, inspect and sample_logits like any other (a step computes the new rows
 * only), and extend / release below. On failure *out may be null; litnice_b200_last_error(NULL)
 * then has the reason. */
#define LITNICE_B200_DTYPE_BF16 0
#define LITNICE_B200_DTYPE_F32 1
int litnice_b200_session_create_model(const char *model_dir, int32_t dtype, int32_t max_streams, int32_t device,
                                      litnice_b200_session **out);
const char *litnice_b200_architectures(void);
/* Sizes of the session's model (n_layers, d_model, vocab_size and max_seq_len for a registered design). */
int litnice_b200_model_dims(const litnice_b200_session *s, litnice_b200_dims *out);
/* Appends n tokens to the sequence in a slot (0 .. max_streams - 1; empty at first) and computes
 * their rows from the cache and state that earlier calls left. want: places 0 .. n-1 among the new
 * tokens whose logits go to out_logits [n_want, vocab] (host), in that order. Portions may be cut
 * anywhere. On failure the slot is empty. Sessions of registered designs only. */
int litnice_b200_extend(litnice_b200_session *s, int32_t slot, const int32_t *tokens, int32_t n, const int32_t *want,
                        int32_t n_want, float *out_logits);
/* Gives a slot back: its next extend starts a new sequence. */
int litnice_b200_release(litnice_b200_session *s, int32_t slot);
void litnice_b200_session_destroy(litnice_b200_session *s);
const char *litnice_b200_last_error(const litnice_b200_session *s);

/* Weights enter as the parameter-arena image (layout of named_layout.cpp:40-161),
 * either from host memory or from a version-6 checkpoint file; mirrors
 * load_checkpoint (checkpoint.cpp:588-652), including its dimension checks. */
int litnice_b200_load_params(litnice_b200_session *s, const void *host_arena, uint64_t bytes);
int litnice_b200_load_checkpoint(litnice_b200_session *s, const char *path);

/* generate_text (inference.cpp:265-296) for n_streams independent streams in
 * lockstep: every step recomputes the whole context (the reference keeps no
 * KV cache), samples on the GPU and appends the token on the GPU. All streams
 * share prompt_len. Stops after max_new tokens or when the context reaches
 * max_seq_len (guard of inference.cpp:278). prompts: [n_streams, prompt_len]
 * host int32; seeds: [n_streams] (inference.seed per stream) or NULL for
 * 12345; out_tokens: [n_streams, max_new] host int32; *out_count receives the
 * tokens produced per stream. Host buffers in, host buffers out. */
int litnice_b200_generate(litnice_b200_session *s, const int32_t *prompts, int32_t n_streams,
                          int32_t prompt_len, int32_t max_new,
                          const litnice_b200_sampling *sampling, const uint32_t *seeds,
                          int32_t *out_tokens, int32_t *out_count);

/* The same loop split in three so that the middle part can be timed with the
 * prompts already resident in HBM: upload, run (returns tokens per stream),
 * download. */
int litnice_b200_upload_prompts(litnice_b200_session *s, const int32_t *prompts,
                                int32_t n_streams, int32_t prompt_len, const uint32_t *seeds);
int litnice_b200_run(litnice_b200_session *s, int32_t max_new,
                     const litnice_b200_sampling *sampling, int32_t *out_count);
int litnice_b200_download_tokens(litnice_b200_session *s, int32_t *out_tokens, int32_t max_new);

/* When enabled, every step of generate/run also keeps its last-row logits
 * ([step][stream][vocab]) for litnice_b200_read_step_logits. Parity runs only. */
int litnice_b200_keep_step_logits(litnice_b200_session *s, int32_t enable);
int litnice_b200_read_step_logits(litnice_b200_session *s, float *out, int64_t max_floats);

/* Transformer::forward (transformer.cpp:70-114) on ids [n_streams, seq_len]:
 * writes logits of every row ([n_streams, seq_len, vocab], all_rows != 0) or of
 * the last row of each stream ([n_streams, vocab]) to host memory. */
int litnice_b200_forward(litnice_b200_session *s, const int32_t *ids, int32_t n_streams,
                         int32_t seq_len, int32_t all_rows, float *out_logits);

/* inspect_distribution (inference.cpp:298-359): next-token probabilities of
 * the last row of each stream, softmax evaluated in double; probs is
 * [n_streams, vocab] host float. */
int litnice_b200_inspect(litnice_b200_session *s, const int32_t *ids, int32_t n_streams,
                         int32_t seq_len, float *probs);

/* select_next_token_sampled (inference.cpp:200-263) alone: one draw per row of
 * host logits [n_rows, vocab] with generator std::mt19937(seeds[row]) advanced
 * `draws` times; out is [n_rows, draws]. Used to check the fused sampler
 * against the host selector on identical logits. */
int litnice_b200_sample_logits(litnice_b200_session *s, const float *logits, int32_t n_rows,
                               const litnice_b200_sampling *sampling, const uint32_t *seeds,
                               int32_t draws, int32_t *out);

int litnice_b200_get_stats(const litnice_b200_session *s, litnice_b200_stats *out);

/* No counterpart in the reference. Few-row product out[m, n] = x[m, k] * W[k, n]
 * (+ bias[n]) for callers that cannot allocate device memory while they run:
 * a host that has already given all device memory to its own arenas, or a
 * loop that cannot afford the device-wide stall of an allocation. It calls no
 * cudaMalloc / cudaFree or any other allocating routine; the split-k partial
 * sums live in a 1.5 MiB array built into the library image (held by every GPU
 * that loads the library until the process exits).
 *   x [m, k], W [k, n] row-major, bias [n] or NULL, out [m, n]: device pointers
 *   owned by the caller; m must be 1, 2, 4 or 8; stream is a cudaStream_t
 *   (NULL = default stream). The call only enqueues work on that stream.
 * Returns 0, LITNICE_B200_EINVAL, LITNICE_B200_ECUDA, or LITNICE_B200_ETOOBIG
 * when m, k, n would need more than the 393216 floats of built-in scratch
 * (a line on stderr says how much was needed). The kernel cuts k into
 * min(ceil(296 / ceil(n / 128)), ceil(k / 64)) ranges when n < 18944 and keeps
 * ranges * m * n partial sums, so in practice only m = 8 is ever refused: with
 * 16385..18816 columns and k > 128 (3 ranges), or 12289..12544 columns and k > 192
 * (4 ranges). Shapes with n >= 18944 or k <= 64 need no scratch at all.
 * The first call on each device looks up the device address of the built-in
 * array (and loads the kernels): make that first call before any stream
 * capture begins. All calls share the one array: it keeps the previous call's
 * partial sums, which is harmless because each call overwrites every entry it
 * later reads, but two calls whose kernels overlap on the GPU (different
 * streams, or different host threads) race on it. */
int litnice_b200_gemv_noalloc(const float *x, int32_t m, const float *w, int32_t k, int32_t n,
                              const float *bias, float *out, void *stream);

/* ------------------------------------------------------------------------ */
/* 3. Diagnostics and measurement aids.                                       */
/*    None of these is part of the token loop and a host binds none of them;  */
/*    the tests, bench.py and the profiling commands call them.               */
/* ------------------------------------------------------------------------ */

/* Runs one step at context length seq_len for n_streams streams with CUDA
 * events around each projection and attention launch, `repeats` times, and
 * fills the gemm_* / attn_* fields of the stats. Measurement aid. */
int litnice_b200_profile_step(litnice_b200_session *s, int32_t n_streams, int32_t seq_len,
                              int32_t repeats);

/* One projection on host buffers: c[m,n] = a[m,k] * w[k,n] (+ bias[n]) (+ residual[m,n])
 * (ReLU when relu != 0), i.e. gemm_ranked_matrix_rhs followed by add_bias_rowwise
 * / add_bias_relu_rowwise / add (device_backend.cpp:1112-1131, 840-908, 752-813).
 * engine 0: fp32 SIMT kernel; engine 1: tcgen05 tensor-core kernel with the
 * three-product TF32 split (needs k % 32 == 0 and n % 64 == 0); engine 2: the
 * same kernel on fp16 pairs with one power-of-two scale per 64 consecutive k of
 * a row (k % 64 == 0), the operand format of the native loop. Allocates and
 * frees its own device buffers; meant for checking the two engines against
 * each other and against the CPU. */
int litnice_b200_projection_host(int32_t engine, const float *a, int32_t m, int32_t k, const float *w, int32_t n,
                                 const float *bias, const float *residual, int32_t relu, float *c);

/* Measurement aid: the same projection (no epilogue terms) launched `repeats`
 * times back to back on one stream; *avg_us receives the mean device time per
 * launch after the first (CUDA events on that stream). */
int litnice_b200_projection_time(int32_t engine, const float *a, int32_t m, int32_t k, const float *w, int32_t n,
                                 float *c, int32_t repeats, double *avg_us);

/* The few-row product out[m, n] = x[m, k] * W[k, n] (+ bias[n]) (+ residual[m, n])
 * (ReLU when relu != 0), m <= 8, on host buffers: the M <= 8 case of
 * gemm_ranked_matrix_rhs (device_backend.cpp:1112-1131) as the output head uses it
 * on the last rows (output_head.cpp:58-70), followed by add_bias_rowwise / add /
 * relu (:840-908, 752-813, 978-1001). With ln_gamma and ln_beta ([k], both or
 * neither) the rows of x pass through layernorm_forward (:1247-1279) first, inside
 * the same kernel; only shapes the streaming kernel takes (EINVAL otherwise).
 * Allocates and frees its own device buffers. */
int litnice_b200_gemv_host(const float *x, int32_t m, const float *w, int32_t k, int32_t n,
                           const float *bias, const float *residual, int32_t relu, const float *ln_gamma,
                           const float *ln_beta, float *out);

/* Device time of that product. cold_l2 = 2: `repeats` calls back to back between one
 * pair of CUDA events, each on the next of a ring of weight copies larger than three
 * times the L2 (every call reads its matrix from HBM); 1: events around each call
 * with a 256 MB buffer written before it; 0: the same matrix every call. force_tn
 * (0, 128, 256) and force_splits (0 = planned; negative: that many k ranges joined through
 * scratch and a second kernel instead of a thread-block cluster) override the tile plan. *avg_us: mean
 * microseconds per call; *launches: kernels per call. */
int litnice_b200_gemv_time(int32_t m, int32_t k, int32_t n, int32_t repeats, int32_t cold_l2,
                           int32_t force_tn, int32_t force_splits, double *avg_us, int32_t *launches);

/* Single operators of the registered designs on host float buffers (rounded to bfloat16 where the
 * operator stores bfloat16); see csrc/model.cuh for what each computes. They allocate and free
 * their own device memory.
 *
 * c[m, n] = a[m, k] w[n, k]^T on bfloat16 operands. engine 0: few-row kernel (m <= 64), 1: tensor-core
 * kernel. Columns below n_half come back rounded to bfloat16 (through the activation: 0 none, 1 GELU with the
 * error function, 2 its tanh form), the others as floats, added to what c holds when accumulate is set. gated:
 * columns 2 j and 2 j + 1 below n_half make one column act(c_2j) * c_2j+1, and c has n - n_half / 2 columns. */
int litnice_b200_bf16_product_host(int32_t engine, const float *a, int32_t m, int32_t k, const float *w, int32_t n,
                                   int32_t n_half, int32_t act, int32_t gated, int32_t accumulate, float *c);
/* x [n, d] += rms(y) * (base + after) (y may be null), h = rms(x) * (base + before) (h may be null); rms(z) =
 * z / sqrt(mean(z^2) + eps) per row. */
int litnice_b200_residual_norm_host(int32_t dtype, float *x, const float *y, const float *after, const float *before,
                                    float base, int32_t n, int32_t d, float eps, float *h);
/* The gated delta rule on projected rows [n_streams, n, q | k | v | gate] (groups * dim twice, heads * vdim twice) and
 * ba [n_streams, n, beta | decay] (heads each), in the given portions with state and history carried between them, from
 * zero: convolution conv [2 groups dim + heads vdim, taps] and SiLU, recurrence, norm and gate. out [n_streams, n,
 * heads * vdim], state [n_streams, heads, dim, vdim]: what the sequences leave behind. */
int litnice_b200_delta_host(int32_t dtype, const float *rows, const float *ba, const float *conv, const float *a_log,
                            const float *dt_bias, const float *norm, float eps, int32_t n_streams, int32_t n, int32_t heads,
                            int32_t groups, int32_t dim, int32_t vdim, int32_t taps, const int32_t *portions,
                            int32_t n_portions, float *out, float *state);
/* Grouped attention of the rows p0 .. p0 + n - 1 of n_streams sequences, rows [n_streams, p0 + n, q | k | v] (heads * dim,
 * groups * dim, groups * vdim): norm over whole rows of q and of k, rotation by p * turns[i] half turns, softmax over the
 * keys of the span (0: the last span_size positions, 1: the query's own chunk of span_size). q_out [n_streams, n,
 * heads * dim] and k_out [n_streams, p0 + n, groups * dim]: rotated; out [n_streams, n, heads * vdim]. engine 0: 32-bit,
 * 1: the same on bfloat16 storage, 2: tensor-core kernel. */
int litnice_b200_grouped_attention_host(int32_t engine, const float *rows, const float *q_weight, const float *k_weight,
                                        float eps, int32_t rot_dims, const double *turns, float amplitude, int32_t n_streams,
                                        int32_t p0, int32_t n, int32_t heads, int32_t groups, int32_t dim, int32_t vdim,
                                        float scale, int32_t span_kind, int32_t span_size, float *q_out, float *k_out,
                                        float *out);
/* h = x / sqrt(mean(x^2) + eps) * gain for the rows of one sequence, out_i = h + conv_i(h) with the causal
 * per-channel convolutions w_i [d, taps] (w2 and out2 both or neither), computed in the given portions
 * with the state carried between them. */
int litnice_b200_rms_canon_host(int32_t dtype, const float *x, int32_t n, int32_t d, float gain, float eps, int32_t taps,
                                const float *w1, const float *w2, const int32_t *portions, int32_t n_portions, float *out1,
                                float *out2);
/* Latent attention of the rows p0 .. p0 + n - 1 of n_streams sequences: q [n_streams, n, heads * dim],
 * dkv [n_streams, p0 + n, rank] (normalised into the cache with latent_gain and eps), w_uk
 * [heads * dim, rank], w_uv [heads * vdim, rank], out [n_streams, n, heads * vdim]. engine 0: any size
 * in 32-bit, 1: the same on bfloat16 storage, 2: few-row kernels, 3: tensor-core kernel. */
int litnice_b200_latent_attention_host(int32_t engine, const float *q, const float *dkv, const float *latent_gain,
                                       float eps, const float *w_uk, const float *w_uv, int32_t n_streams, int32_t p0,
                                       int32_t n, int32_t heads, int32_t dim, int32_t vdim, int32_t rank, float scale,
                                       int32_t window, float *out);

/* Self-test of the bounded waits: a one-CTA kernel waits on a barrier that nothing
 * completes, with a limit of limit_us microseconds (1..1000). It must come back on
 * its own with *code == 2 (a wait ran out), *detail == 99 and *waited_us >= limit_us,
 * and the device must stay usable. */
int litnice_b200_selftest_wait_timeout(int32_t limit_us, int32_t *code, int32_t *detail, double *waited_us);

#ifdef __cplusplus
}
#endif
#endif /* LITNICE_BACKEND_B200_H */
